// Talking-heads attention of prompt portions on tcgen05 tensor cores; definitions in talk_attention.cu, the mix over heads in talk_decode.cu.
//
// One CTA owns 128 consecutive query tokens of one request for one head and up to 256 columns of the cached rows of all key heads, and walks the keys
// in tiles of 128, newest first:
//   S = Q K^T       tcgen05.mma on TMA-loaded tiles (128-byte swizzle) of the head's own key head, two TMEM buffers
//   P = 2^(s - m)   sixteen warps, four threads per query row (32 keys each). The reference m of a row only moves when a score exceeds it by 2^8:
//                   then the row's results in TMEM are rescaled. The distance bias makes the newest keys' scores the largest as a rule, so after
//                   the first tile this is rare. P replaces S in its columns as two bf16 terms, the rounded weight and what rounding took from it.
//   O += P V        operand A from TMEM, V (the same cached rows, 256 columns) as an MN-major operand, accumulated in TMEM
// Key and value tiles share one ring of 16 KB slots (64 columns of 128 keys, or 256 columns of 32 values), filled in the order in which the MMA
// warp uses them. The MMA warp looks after the slots of a product while the product ahead of it runs. O leaves unnormalised in fp32, with m
// and the row's sum beside it.
// Roles: warp 0 TMA producer, warp 1 MMA issue, warps 2-17 softmax and epilogue. Every mbarrier wait is bounded; on expiry the CTA raises the
// status word and tears down. The softmax warps also meet at named barriers, which have no time-out: they pass all of them whatever happened.
#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

constexpr int TQ = 128, TK = 128;
constexpr int kChunk = 128 * 128;          // bytes of one 64-column chunk of a 128-row operand tile
constexpr int kSlots = 10, kSlot = kChunk, kVChunk = 32 * 128, kThreads = 576;   // kVChunk: 64 columns of 32 values
constexpr uint32_t kColS = 0, kColO = 256;
constexpr float kLog2e = 1.4426950408889634f, kSlack = 8.f, kNear = 1.f / 16.f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// two fp32 numbers in a register pair
typedef unsigned long long f2;
__device__ __forceinline__ f2 pair(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpair(f2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f2 add2(f2 a, f2 b) {
  f2 r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// MN-major operand B: 64 columns x 8 keys form a 1024-byte swizzle atom; the next 8 keys are 1024 bytes on, the next 64 columns 32 keys on.
__device__ __forceinline__ uint64_t desc_mn(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)((kVChunk >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

// the 128 threads of a lane quarter (four warps): barrier, and barrier with a vote
__device__ __forceinline__ void quarter_sync(int q) { asm volatile("bar.sync %0, 128;" ::"r"(q + 1) : "memory"); }
__device__ __forceinline__ bool quarter_any(int q, bool x) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred a, b;\n\t"
      "setp.ne.u32 a, %2, 0;\n\t"
      "barrier.cta.red.or.pred b, %1, 128, a;\n\t"
      "selp.u32 %0, 1, 0, b;\n\t}"
      : "=r"(r)
      : "r"(q + 1), "r"((uint32_t)x)
      : "memory");
  return r != 0;
}

template <int NC>
constexpr int smem_bytes() { return NC * kChunk + kSlots * kSlot + 1024 + (16 * 32 + 4 * TQ) * 4; }

// NC: 64-column chunks of a cached row
template <int NC>
__global__ void __launch_bounds__(kThreads, 1)
talk_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const TalkTcParams p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int DP = NC * 64, kEnd = NC * kChunk + kSlots * kSlot;
  uint8_t* sQ = smem;
  uint8_t* ring = smem + NC * kChunk;
  uint64_t* q_full = reinterpret_cast<uint64_t*>(smem + kEnd);   // [1]
  uint64_t* full = q_full + 1;         // [kSlots] the slots of a tile have arrived: the barrier of the first one
  uint64_t* empty = full + kSlots;     // [kSlots]
  uint64_t* s_full = empty + kSlots;   // [2] scores of a tile are complete
  uint64_t* p_ready = s_full + 2;      // [2] weights written over the scores
  // [2] the tile's product is complete. Scores of tile j are there only once the product of tile j - 2 is, so a barrier per buffer is never
  // more than one phase ahead of a thread that waits for it.
  uint64_t* o_done = p_ready + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_req = const_cast<int*>(reinterpret_cast<volatile int*>(tmem_slot + 2));
  float* s_f = reinterpret_cast<float*>(smem + kEnd + 1024);     // [16 warps][32] factors of the keys
  float* s_x = s_f + 16 * 32;                                    // [4 threads of a row][TQ]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, H = p.t.H, G = p.t.G, hk = h / (H / G), bs = p.bs_shift;
  const int chunk0 = blockIdx.z * 4, vchunks = min(4, G * NC - chunk0);   // 64-column chunks of the key heads' rows that this CTA multiplies

  if (threadIdx.x == 0) {
    // which request and which of its 128-token tiles this CTA owns; the last tiles of the launch, which see the most keys, go first
    const int tile = p.tile0 + (int)(gridDim.x - 1 - blockIdx.x);
    int b = tile, found = -1, t0 = 0;
    for (int i = 0; i < p.t.R; ++i) {
      const int ql = p.t.query_start_loc[i + 1] - p.t.query_start_loc[i];
      const int nt = ql >= p.min_len ? (ql + TQ - 1) / TQ : 0;
      if (b < nt) { found = i; t0 = b * TQ; break; }
      b -= nt;
    }
    s_req[0] = found;
    s_req[1] = t0;
    mbar_init(q_full, 1);
    for (int i = 0; i < kSlots; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_ready[i], 16);
      mbar_init(&o_done[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const int r = s_req[0], tq0 = s_req[1];
  int ntiles = 0, qs = 0, qlen = 0, S = 0, ctx0 = 0;
  if (r >= 0) {
    qs = p.t.query_start_loc[r];
    qlen = p.t.query_start_loc[r + 1] - qs;
    S = p.t.seq_lens[r];
    ctx0 = S - qlen;
    ntiles = (min(S, ctx0 + min(tq0 + TQ, qlen)) + TK - 1) / TK;   // up to the last key that the tile's last row sees
  }
  const int* bt = p.t.block_table + (size_t)max(r, 0) * p.t.bt_stride;

  if (warp == 0) {
    // ------------------------------------------------------------------ producer: K(0), then K(j + 1) and the values of j
    if (ntiles > 0) {
      if (lane == 0) {
        mbar_expect_tx(q_full, NC * kChunk);
        // rows past the end of the tensor are zero-filled; rows of the next request are loaded and never stored
#pragma unroll
        for (int c = 0; c < NC; ++c) tma_load_2d(sQ + c * kChunk, &tmQ, h * DP + c * 64, qs + tq0, q_full);
      }
      int at = 0;   // slots handed out so far
      bool ok = true;
      const int sub = lane >> 3, box = lane & 7;   // eight lanes fill a slot with boxes of 16 rows x 64 columns
      auto row_of = [&](int key0, int g) {         // keys past the sequence read the null block
        return key0 < S ? ((bt[key0 >> bs] * G + g) << bs) + (key0 & (p.t.bs - 1)) : g << bs;
      };
      uint64_t* arrived = nullptr;                 // barrier of the tile
      auto take = [&](int slots, int bytes) {      // lane groups 0 .. slots - 1 wait for their slots; returns this lane's
        const int n = at + sub, s = n % kSlots;
        if (ok && sub < slots && box == 0) ok = mbar_wait(&empty[s], ((n / kSlots) & 1) ^ 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        arrived = &full[at % kSlots];
        if (ok && lane == 0) mbar_expect_tx(arrived, slots * bytes);
        __syncwarp();
        at += slots;
        return s;
      };
      auto load_k = [&](int j) {
        const int key0 = (ntiles - 1 - j) * TK + box * 16, s = take(NC, kChunk);
        if (ok && sub < NC) tma_load_2d(ring + s * kSlot + box * 2048, &tmK, sub * 64, row_of(key0, hk), arrived);
      };
      auto load_v = [&](int j) {                   // slot: 32 keys; box: 16 of them and one of the chunks
        const int key0 = (ntiles - 1 - j) * TK + sub * 32 + (box & 1) * 16, s = take(4, vchunks * kVChunk), c = chunk0 + (box >> 1);
        if (ok && (box >> 1) < vchunks)
          tma_load_2d(ring + s * kSlot + (box >> 1) * kVChunk + (box & 1) * 2048, &tmK, (c % NC) * 64, row_of(key0, c / NC), arrived);
      };
      load_k(0);
      for (int j = 0; j < ntiles && ok; ++j) {
        if (j + 1 < ntiles) load_k(j + 1);
        load_v(j);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issue, in the same order
    // The whole warp walks the loop (descriptors stay in uniform registers), one elected lane issues.
    if (ntiles > 0) {
      const bool leader = elect_one();
      const uint32_t idesc_qk = umma_idesc_bf16(TQ, TK), idesc_pv = umma_idesc_bf16(TQ, vchunks * 64) | (1u << 16);   // operand B (V) is MN-major
      // Descriptors are a constant beside the address in 16-byte units, so one thread issues the products with an addition for each.
      const uint64_t dq = umma_desc_sw128(smem_u32(sQ)), dk0 = umma_desc_sw128(smem_u32(ring)), dv0 = desc_mn(smem_u32(ring));
      // Barrier of the tile whose first slot is number n. A slot is the first of a tile in some rounds of the ring only, so its phase is counted apart.
      int at = 0;   // slots used so far
      uint32_t phases = 0;
      auto wait_tile = [&]() {
        const int s = at % kSlots;
        const bool good = mbar_wait(&full[s], (phases >> s) & 1u, abort_flag);
        phases ^= 1u << s;
        return good;
      };
      auto issue_qk = [&](int j) {   // its slots have been waited for
        tc_fence_after();
        const uint32_t d = tmem_base + kColS + (j & 1) * TK;
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          const int s = (at + c) % kSlots;
          const uint64_t dk = dk0 + (uint64_t)(s * (kSlot >> 4)), da = dq + (uint64_t)(c * (kChunk >> 4));
          if (leader) {
#pragma unroll
            for (int i = 0; i < 4; ++i) umma_bf16(d, da + (uint64_t)(i * 2), dk + (uint64_t)(i * 2), idesc_qk, (c | i) ? 1u : 0u);
            umma_commit(&empty[s]);
          }
        }
        if (leader) umma_commit(&s_full[j & 1]);
        __syncwarp();
        at += NC;
      };
      bool ok = mbar_wait(q_full, 0, abort_flag) && wait_tile();
      if (ok) issue_qk(0);
      if (ok && ntiles > 1) ok = wait_tile();
      for (int j = 0; j < ntiles && ok; ++j) {
        if (j + 1 < ntiles) {
          // the buffer holds the weights of tile j - 1: their product must be complete
          if (j > 0) ok = mbar_wait(&o_done[(j - 1) & 1], ((j - 1) >> 1) & 1, abort_flag);
          if (!ok) break;
          issue_qk(j + 1);
        }
        ok = wait_tile() && mbar_wait(&p_ready[j & 1], (j >> 1) & 1, abort_flag);
        if (!ok) break;
        tc_fence_after();
        const uint32_t a = tmem_base + kColS + (j & 1) * TK, d = tmem_base + kColO;
#pragma unroll
        for (int q = 0; q < 4; ++q) {   // 32 keys: 32 TMEM columns of P (16 of first terms, 16 of second ones), one slot of V
          const int s = (at + q) % kSlots;
          const uint64_t dv = dv0 + (uint64_t)(s * (kSlot >> 4));
          if (leader) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
              umma_bf16_ts(d, a + q * 32 + i * 8, dv + (uint64_t)(i * 128), idesc_pv, (q | i) ? 1u : (j ? 1u : 0u));
              umma_bf16_ts(d, a + q * 32 + i * 8 + 16, dv + (uint64_t)(i * 128), idesc_pv, 1u);
            }
            umma_commit(&empty[s]);
          }
        }
        if (leader) umma_commit(&o_done[j & 1]);
        __syncwarp();
        at += 4;
        if (j + 2 < ntiles) ok = wait_tile();
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax + epilogue: four threads per query row
    const int q4 = warp & 3;                 // TMEM lane quarter this warp may touch
    const int part = (warp - 2) >> 2;        // which 32 keys of a tile / which 64 output columns this thread owns
    const int row = q4 * 32 + lane;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(q4 * 32) << 16);
    const int tq = tq0 + row, pos = ctx0 + tq;
    const float r1 = p.t.bias[h], r2 = p.t.bias[H + h];
    float* f = s_f + (warp - 2) * 32;
    // page of this lane's key in the j-th tile from the end, and the key's factor: loaded two tiles and one tile ahead, so that nobody waits
    auto key_of = [&](int j) { return (ntiles - 1 - j) * TK + part * 32 + lane; };
    auto page = [&](int j) { return j < ntiles && key_of(j) < S ? bt[key_of(j) >> bs] : -1; };
    auto factor = [&](int j, int pg) { return pg >= 0 ? p.t.k_scale[((size_t)pg << bs) + (key_of(j) & (p.t.bs - 1))] : 0.f; };
    auto both = [](float x) { return pair(x, x); };
    f2 l = 0ull;
    float m = -INFINITY, fk = factor(0, page(0));
    int pg = page(1);
    bool ok = ntiles > 0;
    for (int j = 0; j < ntiles; ++j) {
      const int k0 = (ntiles - 1 - j) * TK + part * 32;
      const bool all = __all_sync(0xffffffffu, k0 + 31 <= pos), none = __all_sync(0xffffffffu, k0 > pos);
      f[lane] = fk * kLog2e;
      __syncwarp();
      fk = factor(j + 1, pg);
      pg = page(j + 2);
      if (ok) ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      const uint32_t s_addr = lane_addr + kColS + (j & 1) * TK + part * 32;
      uint32_t v[32];
      float top = -INFINITY;
      if (ok && !none) {
        tc_fence_after();
        tmem_ld_32x32(s_addr, v);
        tmem_ld_wait();
        // r1 log2(1 + r2 d) over the 32 keys, d = d0 - i. Away from the row's own position a series around the middle key takes the place of the
        // logarithms: with u = r2 (d - dm) / (1 + r2 dm) it ends at u^4, whose successor is below 2^-22 for |u| <= 1/16.
        const float d0 = (float)(pos - k0), am = fmaf(r2, d0 - 15.5f, 1.f), inv = __fdividef(1.f, am), g = -r2 * inv;
        if (__all_sync(0xffffffffu, fabsf(g) * 15.5f <= kNear && am > 0.f)) {
          const float c = -r1 * kLog2e * g;
          const f2 c0 = both(-r1 * lg2(am)), c1 = both(c), c2 = both(c * g * -0.5f), c3 = both(c * g * g * (1.f / 3.f)), c4 = both(c * g * g * g * -0.25f);
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const ulonglong2 ff = *reinterpret_cast<const ulonglong2*>(f + i);
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
              const f2 x = pair((float)(i + e) - 15.5f, (float)(i + e) - 14.5f);
              const f2 bias = fma2(x, fma2(x, fma2(x, fma2(x, c4, c3), c2), c1), c0);
              const float2 t = unpair(fma2(pair(__uint_as_float(v[i + e]), __uint_as_float(v[i + e + 1])), e ? ff.y : ff.x, bias));
              v[i + e] = __float_as_uint(t.x);
              v[i + e + 1] = __float_as_uint(t.y);
            }
          }
        } else {
          const f2 a0 = both(fmaf(r2, d0, 1.f)), step = both(-r2), factor1 = both(-r1);
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const ulonglong2 ff = *reinterpret_cast<const ulonglong2*>(f + i);
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
              const float2 t = unpair(fma2(step, pair((float)(i + e), (float)(i + e + 1)), a0));
              const float2 y = unpair(fma2(factor1, pair(lg2(t.x), lg2(t.y)), mul2(pair(__uint_as_float(v[i + e]), __uint_as_float(v[i + e + 1])), e ? ff.y : ff.x)));
              v[i + e] = __float_as_uint(y.x);
              v[i + e + 1] = __float_as_uint(y.y);
            }
          }
        }
        if (!all) {
          const int seen = pos - k0;
#pragma unroll
          for (int i = 0; i < 32; ++i) v[i] = i <= seen ? v[i] : 0xff800000u;
        }
        float top2 = -INFINITY;
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          top = fmaxf(top, fmaxf(__uint_as_float(v[i]), __uint_as_float(v[i + 1])));
          top2 = fmaxf(top2, fmaxf(__uint_as_float(v[i + 2]), __uint_as_float(v[i + 3])));
        }
        top = fmaxf(top, top2);
      }
      // does any row of the quarter have to move its reference?
      if (quarter_any(q4, top > m + kSlack)) {
        s_x[part * TQ + row] = top;
        quarter_sync(q4);
        const float nm = fmaxf(fmaxf(fmaxf(s_x[row], s_x[TQ + row]), fmaxf(s_x[2 * TQ + row], s_x[3 * TQ + row])), m);
        const float al = nm == -INFINITY ? 1.f : ex2(m - nm);
        m = nm;
        l = mul2(l, both(al));
        if (j > 0) {
          if (ok) ok = mbar_wait(&o_done[(j - 1) & 1], ((j - 1) >> 1) & 1, abort_flag);   // every earlier product is complete, none is issued before these weights
          ok = __all_sync(0xffffffffu, ok);
          if (ok && __any_sync(0xffffffffu, al != 1.f)) {
            tc_fence_after();
#pragma unroll 1
            for (int c = part * 64; c < min(part * 64 + 64, vchunks * 64); c += 32) {
              uint32_t o[32];
              tmem_ld_32x32(lane_addr + kColO + c, o);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * al);
              tmem_st_32x32(lane_addr + kColO + c, o);
            }
            tmem_st_wait();
          }
        }
      }
      if (ok) {
        uint32_t out[32];   // 16 words of first terms, 16 of second ones
        if (none) {
#pragma unroll
          for (int i = 0; i < 32; ++i) out[i] = 0u;
        } else {
          const f2 base = both(m == -INFINITY ? 0.f : -m), minus = both(-1.f);
          f2 l2 = 0ull;
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const float2 x = unpair(add2(pair(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), base));
            const f2 w = pair(ex2(x.x), ex2(x.y));
            if (i & 2) l2 = add2(l2, w);
            else l = add2(l, w);
            const float2 wf = unpair(w);
            __nv_bfloat162 b = __floats2bfloat162_rn(wf.x, wf.y);
            const uint32_t bits = *reinterpret_cast<uint32_t*>(&b);
            const float2 d = unpair(fma2(pair(__uint_as_float(bits << 16), __uint_as_float(bits & 0xffff0000u)), minus, w));
            __nv_bfloat162 e = __floats2bfloat162_rn(d.x, d.y);
            out[i >> 1] = bits;
            out[16 + (i >> 1)] = *reinterpret_cast<uint32_t*>(&e);
          }
          l = add2(l, l2);
        }
        tmem_st_32x32(s_addr, out);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready[j & 1]);
      }
    }
    quarter_sync(q4);   // s_x has been read
    const float2 lsum = unpair(l);
    s_x[part * TQ + row] = lsum.x + lsum.y;
    quarter_sync(q4);
    if (ok) ok = mbar_wait(&o_done[(ntiles - 1) & 1], ((ntiles - 1) >> 1) & 1, abort_flag);
    ok = __all_sync(0xffffffffu, ok);
    if (ok && !*abort_flag) {
      tc_fence_after();
      const size_t at = ((size_t)(gridDim.x - 1 - blockIdx.x) * TQ + row) * H + h;
      const bool live = tq < qlen;
      if (live && part == 0 && blockIdx.z == 0)
        reinterpret_cast<float2*>(p.ws_ml)[at] = make_float2(m, (s_x[row] + s_x[TQ + row]) + (s_x[2 * TQ + row] + s_x[3 * TQ + row]));
      float* dst = p.ws_o + at * (G * DP) + chunk0 * 64;
#pragma unroll 1
      for (int c = part * 64; c < min(part * 64 + 64, vchunks * 64); c += 32) {
        uint32_t o[32];
        tmem_ld_32x32(lane_addr + kColO + c, o);
        tmem_ld_wait();
        if (live) {
#pragma unroll
          for (int i = 0; i < 32; i += 4) *reinterpret_cast<uint4*>(dst + c + i) = make_uint4(o[i], o[i + 1], o[i + 2], o[i + 3]);
        }
      }
    }
  }

  // ------------------------------------------------------------------ teardown
  tc_fence_before();
  __syncthreads();
  if (*abort_flag && threadIdx.x == 0) {
    // give copies that are still in flight a bounded chance to land before the CTA's shared memory is released
    uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) {}
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                  const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// bf16 [rows][cols], contiguous -> boxes of {64 columns, box_rows rows}, 128-byte swizzle, zero fill
int make_tmap(CUtensorMap* tm, const void* base, uint64_t rows, uint64_t cols, uint32_t box_rows) {
  static EncodeTiledFn enc = nullptr;
  if (!enc) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres);
    enc = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  if (!enc) return -1;
  cuuint64_t dims[2] = {cols, rows}, strides[1] = {cols * 2};
  cuuint32_t box[2] = {64, box_rows}, estr[2] = {1, 1};
  return enc(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : -1;
}

template <int NC>
int go(TalkTcParams p, int tiles, int segment, long long num_blocks, cudaStream_t st) {
  CUtensorMap tmQ, tmK;
  if (make_tmap(&tmQ, p.t.q, (uint64_t)p.t.T, (uint64_t)p.t.H * NC * 64, TQ)) return -2;
  if (make_tmap(&tmK, p.t.pages, (uint64_t)num_blocks * p.t.G * p.t.bs, NC * 64, 16)) return -3;
  constexpr int smem = smem_bytes<NC>() + 1024;
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (cudaFuncSetAttribute(talk_prefill_tc_kernel<NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -4;
    configured = true;
  }
  for (p.tile0 = 0; p.tile0 < tiles; p.tile0 += segment) {
    const int n = tiles - p.tile0 < segment ? tiles - p.tile0 : segment;
    talk_prefill_tc_kernel<NC><<<dim3(n, p.t.H, (p.t.G * NC + 3) / 4), kThreads, smem, st>>>(tmQ, tmK, p);
    if (cudaGetLastError() != cudaSuccess) return -5;
    const int rc = talk_join_launch(p, false, n * TQ, st);
    if (rc) return rc;
  }
  return 0;
}

}  // namespace

int talk_prefill_launch(const TalkTcParams& p_, int tiles, int segment, long long num_blocks, cudaStream_t st) {
  TalkTcParams p = p_;
  if (p.t.T == 0 || tiles <= 0) return 0;
  if (p.t.f32 || talk_tc_row(p.t.H, p.t.G, p.t.dim) != p.t.row || p.t.bs < 16 || (p.t.bs & (p.t.bs - 1)) || segment < 1 || p.ws_ml == nullptr || p.ws_o == nullptr ||
      ((uintptr_t)p.t.q & 15) || ((uintptr_t)p.t.pages & 15)) return -1;
  p.bs_shift = __builtin_ctz((unsigned)p.t.bs);
  return p.t.row == 64 ? go<1>(p, tiles, segment, num_blocks, st) : go<2>(p, tiles, segment, num_blocks, st);
}

unsigned int talk_prefill_read_status(bool clear) { return read_status_tu(clear); }
void talk_prefill_read_status_async(unsigned int* dst, cudaStream_t st) { read_status_tu_async(dst, st); }

}  // namespace oc
