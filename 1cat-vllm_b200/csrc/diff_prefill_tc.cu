// Differential attention prefill on tcgen05 tensor cores, for soft-capped scores (rows of 64 or 128 columns, see AttnParams::maps).
//
// One CTA owns 128 consecutive query tokens of one request for one head, both of its maps, and walks the keys in tiles of 128. A cached key
// row holds both maps side by side, so the tiles' K and V are loaded once:
//   S_m = Q_m K_m^T   tcgen05.mma on TMA-loaded tiles (128-byte swizzle), one TMEM buffer per map
//   P_m = exp(S_m)    sixteen warps, four threads per query row (32 keys each). A soft cap bounds the scores (|s| <= cap), so the weights need
//                     no running maximum: exp(s) and its sums stay far inside fp32's range for caps up to 55, no tile ever rescales what earlier
//                     ones left, and the products of all tiles accumulate in TMEM. P replaces S in its columns as two bf16 terms, the
//                     rounded weight and what rounding took from it.
//   O_m += P_m V      operand A from TMEM, V as an MN-major operand
// While the softmax warps are at one map's tile, the tensor core multiplies the other one's. The epilogue takes (O_1 / l_1 - lam O_2 / l_2), its
// root mean square over the row (the four threads of a row meet in shared memory), scales and stores.
// Chunks: key tiles before the chunk of the tile's first query are not visited; a row's visible keys are a range [lo, hi).
// Roles: warp 0 TMA producer, warp 1 MMA issue, warps 2-17 softmax and epilogue. Every wait is bounded; on expiry the CTA raises the status
// word and tears down (see common.cuh).
#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

constexpr int TQ = 128, TK = 128;
constexpr int kChunkBytes = 128 * 128;   // one 64-column chunk of a 128-row operand tile
constexpr int kStages = 2, kThreads = 576;
constexpr uint32_t kColS = 0, kColO = 256;   // TMEM columns: S of both maps | O of both maps
constexpr float kTanhSmall = 0.4f, kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// two fp32 numbers in a register pair
typedef unsigned long long f2;
__device__ __forceinline__ f2 pack2(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(f2 v) {
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

// V tile as operand B, MN-major: 64 columns x 8 keys form a 1024-byte swizzle atom; the next 8 keys are 1024 bytes on, the next 64 columns
// a chunk on.
__device__ __forceinline__ uint64_t desc_mn(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)((kChunkBytes >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

template <int D>
constexpr int smem_bytes() { return (D / 64) * kChunkBytes * (1 + 2 * kStages) + 1024 + 3 * 4 * TQ * 4; }

template <int D>
__global__ void __launch_bounds__(kThreads, 1)
diff_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmKV, const AttnParams p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int NC = D / 64, kTile = NC * kChunkBytes, kEnd = kTile * (1 + 2 * kStages);
  uint8_t* sQ = smem;
  uint8_t* sKV = smem + kTile;             // stage s: K at s * 2 * kTile, V right after it
  uint64_t* q_full = reinterpret_cast<uint64_t*>(smem + kEnd);   // [1]
  uint64_t* k_full = q_full + 1;           // [kStages]
  uint64_t* v_full = k_full + kStages;
  uint64_t* k_empty = v_full + kStages;
  uint64_t* v_empty = k_empty + kStages;
  uint64_t* s_full = v_empty + kStages;    // [2 maps] scores of a tile are complete
  uint64_t* p_ready = s_full + 2;          // [2] weights written over the scores
  uint64_t* o_done = p_ready + 2;          // [2] the tile's product is complete
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_req = const_cast<int*>(reinterpret_cast<volatile int*>(tmem_slot + 2));
  float* s_xch = reinterpret_cast<float*>(smem + kEnd + 1024);   // [l of map 1, l of map 2, squares][4 threads of a row][TQ]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, H = p.Hq / 2, hkv = h / (H / p.Hkv);

  if (threadIdx.x == 0) {
    // which request and which of its 128-token tiles this CTA owns (short queries belong to the decode kernel)
    int b = blockIdx.x, found = -1, t0 = 0;
    for (int i = 0; i < p.R; ++i) {
      const int ql = p.query_start_loc[i + 1] - p.query_start_loc[i];
      const int nt = (ql > p.short_q_len) ? (ql + TQ - 1) / TQ : 0;
      if (b < nt) { found = i; t0 = b * TQ; break; }
      b -= nt;
    }
    s_req[0] = found;
    s_req[1] = t0;
    mbar_init(q_full, 1);
    for (int i = 0; i < kStages; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_ready[i], 16);
      mbar_init(&o_done[i], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmKV);
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

  int ntiles = 0, first = 0, qs = 0, qlen = 0, S = 0, ctx0 = 0;
  auto first_key = [&](int pos) { return p.chunk > 0 ? pos - pos % p.chunk : 0; };
  if (r >= 0) {
    qs = p.query_start_loc[r];
    qlen = p.query_start_loc[r + 1] - qs;
    S = p.seq_lens[r];
    ctx0 = S - qlen;
    const int kv_end = min(S, ctx0 + min(tq0 + TQ, qlen));  // keys the last row of this tile may see
    first = first_key(ctx0 + tq0) / TK;
    ntiles = (kv_end + TK - 1) / TK - first;
  }

  if (warp == 0) {
    // ------------------------------------------------------------------ producer
    if (ntiles > 0) {
      if (lane == 0) {
        mbar_expect_tx(q_full, kTile);
        // rows past the end of the tensor are zero-filled; rows of the next request are loaded and never stored
#pragma unroll
        for (int c = 0; c < NC; ++c) tma_load_2d(sQ + c * kChunkBytes, &tmQ, h * D + c * 64, qs + tq0, q_full);
      }
      const int* bt = p.block_table + (size_t)r * p.bt_stride;
      // lane -> (K or V, 64-column chunk, 16 keys)
      const int is_v = lane / (8 * NC), col = (lane >> 3) % NC, part = lane & 7;
      Ring st;
      bool ok = true;
      for (int j = 0; j < ntiles && ok; ++j) {
        const int key0 = (first + j) * TK + part * 16;
        int page = 0, off = 0;  // keys past the sequence read the null block
        if (key0 < S) {
          page = bt[key0 >> p.bs_shift];
          off = key0 & (p.bs - 1);
        }
        const int row = ((page * 2 + is_v) * p.Hkv + hkv) * p.bs + off;
        if (lane == 0) {
          ok = mbar_wait(&k_empty[st.idx], st.phase ^ 1, abort_flag);
          if (ok) ok = mbar_wait(&v_empty[st.idx], st.phase ^ 1, abort_flag);
          if (ok) {
            mbar_expect_tx(&k_full[st.idx], kTile);
            mbar_expect_tx(&v_full[st.idx], kTile);
          }
        }
        ok = __shfl_sync(0xffffffffu, (int)ok, 0) != 0;
        if (!ok) break;
        if (lane < 16 * NC)
          tma_load_2d(sKV + (st.idx * 2 + is_v) * kTile + col * kChunkBytes + part * 2048, &tmKV, col * 64, row, is_v ? &v_full[st.idx] : &k_full[st.idx]);
        st.advance(kStages);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issue
    if (lane == 0 && ntiles > 0) {
      const uint32_t idesc_qk = umma_idesc_bf16(TQ, TK);
      const uint32_t idesc_pv = umma_idesc_bf16(TQ, D) | (1u << 16);  // operand B (V) is MN-major
      const uint32_t q_addr = smem_u32(sQ), kv_addr = smem_u32(sKV);
      bool ok = mbar_wait(q_full, 0, abort_flag);
      auto issue_qk = [&](int j, int m) {
        const int s = j % kStages;
        if (m == 0) ok = mbar_wait(&k_full[s], (j / kStages) & 1, abort_flag);
        // the weights of this map's last tile lie in these columns: their product must be complete
        if (ok && j > 0) ok = mbar_wait(&o_done[m], (j - 1) & 1, abort_flag);
        if (!ok) return;
        tc_fence_after();
        const uint32_t k_base = kv_addr + (s * 2) * kTile;
#pragma unroll
        for (int i = 0; i < D / 32; ++i) {   // 16 columns a step; this map's half of the columns
          const int step = m * (D / 32) + i, c = (step >> 2) * kChunkBytes;
          umma_bf16(tmem_base + kColS + m * TK, umma_desc_sw128(q_addr + c) + (uint64_t)((step & 3) * 2),
                    umma_desc_sw128(k_base + c) + (uint64_t)((step & 3) * 2), idesc_qk, i ? 1u : 0u);
        }
        umma_commit(&s_full[m]);
        if (m == 1) umma_commit(&k_empty[s]);
      };
      if (ok) issue_qk(0, 0);
      if (ok) issue_qk(0, 1);
      for (int j = 0; j < ntiles && ok; ++j) {
        const int s = j % kStages;
        ok = mbar_wait(&v_full[s], (j / kStages) & 1, abort_flag);
        for (int m = 0; m < 2 && ok; ++m) {
          ok = mbar_wait(&p_ready[m], j & 1, abort_flag);
          if (!ok) break;
          tc_fence_after();
          const uint32_t v_base = kv_addr + (s * 2 + 1) * kTile;
#pragma unroll
          for (int i = 0; i < TK / 16; ++i) {
            // 16 keys per MMA: 8 TMEM columns of P (32 keys take 32 columns: 16 of first terms, 16 of second ones), 2048 bytes of V
            const uint64_t db = desc_mn(v_base + i * 2048);
            const uint32_t a = tmem_base + kColS + m * TK + (i >> 1) * 32 + (i & 1) * 8;
            umma_bf16_ts(tmem_base + kColO + m * D, a, db, idesc_pv, (i | j) ? 1u : 0u);
            umma_bf16_ts(tmem_base + kColO + m * D, a + 16, db, idesc_pv, 1u);
          }
          umma_commit(&o_done[m]);
          if (m == 1) umma_commit(&v_empty[s]);
          if (j + 1 < ntiles) issue_qk(j + 1, m);
        }
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax + epilogue: four threads per query row
    const int q4 = warp & 3;                 // TMEM lane quarter this warp may touch
    const int part = (warp - 2) >> 2;        // which 32 keys of a tile / which 32 output columns this thread owns
    const int row = q4 * 32 + lane;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(q4 * 32) << 16);
    const int tq = tq0 + row, pos = ctx0 + tq;
    const int lo = first_key(pos), hi = min(S, pos + 1);   // keys [lo, hi) are visible to this row
    // weight = 2^(cap log2e tanh(u)), u = score * scale / cap
    const float a = p.scale / p.softcap, post = p.softcap * kLog2e;
    const f2 a2 = pack2(a, a);
    auto both = [](float v) { return pack2(v, v); };
    const f2 c0 = both(post), c1 = both(post * (-1.f / 3.f)), c2 = both(post * (2.f / 15.f)), c3 = both(post * (-17.f / 315.f)),
             c4 = both(post * (62.f / 2835.f)), c5 = both(post * (-1382.f / 155925.f)), minus = both(-1.f);
    f2 l[2] = {0ull, 0ull};
    bool ok = ntiles > 0;
    for (int j = 0; j < ntiles; ++j) {
      const int k0 = (first + j) * TK + part * 32, hr = hi - k0, lr = lo - k0;
      const uint32_t seen = (hr <= 0 || lr >= 32) ? 0u : ((hr >= 32 ? ~0u : (1u << hr) - 1u) & (lr <= 0 ? ~0u : ~((1u << lr) - 1u)));
      const bool all = __all_sync(0xffffffffu, seen == ~0u), none = __all_sync(0xffffffffu, seen == 0u);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        if (ok) ok = mbar_wait(&s_full[m], j & 1, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        const uint32_t s_addr = lane_addr + kColS + m * TK + part * 32;
        uint32_t out[32];   // 16 words of first terms, 16 of second ones
        if (none) {
#pragma unroll
          for (int i = 0; i < 32; ++i) out[i] = 0u;
        } else {
          uint32_t v[32];
          tmem_ld_32x32(s_addr, v);
          tmem_ld_wait();
          float top = 0.f;
#pragma unroll
          for (int i = 0; i < 32; ++i) top = fmaxf(top, fabsf(__uint_as_float(v[i])));
          const bool small = !__any_sync(0xffffffffu, top * fabsf(a) >= kTanhSmall);
          auto weight = [&](int i, float w0, float w1) {
            __nv_bfloat162 b = __floats2bfloat162_rn(w0, w1);
            const uint32_t bits = *reinterpret_cast<uint32_t*>(&b);
            const f2 w = pack2(w0, w1);
            l[m] = add2(l[m], w);
            const float2 d = unpack2(fma2(pack2(__uint_as_float(bits << 16), __uint_as_float(bits & 0xffff0000u)), minus, w));
            __nv_bfloat162 e = __floats2bfloat162_rn(d.x, d.y);
            out[i >> 1] = bits;
            out[16 + (i >> 1)] = *reinterpret_cast<uint32_t*>(&e);
          };
          // the series of tanh up to u^11 (3e-8 off at 0.4)
          auto series = [&](int i) {
            const f2 u = mul2(pack2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), a2), y = mul2(u, u);
            return unpack2(mul2(u, fma2(y, fma2(y, fma2(y, fma2(y, fma2(y, c5, c4), c3), c2), c1), c0)));
          };
          if (small && all) {
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const float2 s = series(i);
              weight(i, ex2(s.x), ex2(s.y));
            }
          } else {
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              float2 s = series(i);
              if (!small) {   // (1 - e^-2u) / (1 + e^-2u) away from zero
                const float u0 = __uint_as_float(v[i]) * a, u1 = __uint_as_float(v[i + 1]) * a;
                const float e0 = ex2(-2.f * kLog2e * fabsf(u0)), e1 = ex2(-2.f * kLog2e * fabsf(u1));
                if (fabsf(u0) >= kTanhSmall) s.x = copysignf(__fdividef(1.f - e0, 1.f + e0) * post, u0);
                if (fabsf(u1) >= kTanhSmall) s.y = copysignf(__fdividef(1.f - e1, 1.f + e1) * post, u1);
              }
              weight(i, (seen >> i) & 1u ? ex2(s.x) : 0.f, (seen >> (i + 1)) & 1u ? ex2(s.y) : 0.f);
            }
          }
        }
        tmem_st_32x32(s_addr, out);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready[m]);
      }
      if (!ok) break;
    }
    // The four threads of a row (one per group of four warps) meet twice: sums of weights, then squares of the outputs. A named barrier has no
    // time-out, so every softmax thread passes both whatever happened before.
    auto all_rows = [&]() { asm volatile("bar.sync 1, 512;" ::: "memory"); };
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const float2 s = unpack2(l[m]);
      s_xch[(m * 4 + part) * TQ + row] = s.x + s.y;
    }
    all_rows();
    if (ok) ok = mbar_wait(&o_done[0], (ntiles - 1) & 1, abort_flag);
    if (ok) ok = mbar_wait(&o_done[1], (ntiles - 1) & 1, abort_flag);
    ok = __all_sync(0xffffffffu, ok);
    float x[32], ss = 0.f;
    const bool mine = ok && part < D / 32;
    if (mine) {
      tc_fence_after();
      float inv[2];
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) sum += s_xch[(m * 4 + i) * TQ + row];
        inv[m] = sum > 0.f ? 1.f / sum : 0.f;
      }
      const float f = *p.lam * inv[1];
      uint32_t v[32];
      tmem_ld_32x32(lane_addr + kColO + part * 32, v);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) x[i] = __uint_as_float(v[i]) * inv[0];
      tmem_ld_32x32(lane_addr + kColO + D + part * 32, v);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) {   // columns past vdim are zero in the cache
        x[i] -= __uint_as_float(v[i]) * f;
        ss = fmaf(x[i], x[i], ss);
      }
    }
    float* squares = s_xch + 2 * 4 * TQ;
    squares[part * TQ + row] = ss;
    all_rows();
    if (mine && !*abort_flag && tq < qlen) {
      const float total = squares[row] + squares[TQ + row] + squares[2 * TQ + row] + squares[3 * TQ + row];
      const float f = p.out_scale / sqrtf(total / (float)p.vdim + p.eps);
      __nv_bfloat16* dst = p.out + ((size_t)(qs + tq) * H + h) * p.vdim + part * 32;
      const int n = p.vdim - part * 32;
      if (p.vdim % 8 == 0) {
#pragma unroll
        for (int i = 0; i < 32; i += 8)
          if (i < n) {
            __nv_bfloat162 b[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) b[e] = __floats2bfloat162_rn(x[i + 2 * e] * f, x[i + 2 * e + 1] * f);
            *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<uint4*>(b);
          }
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (i < n) dst[i] = __float2bfloat16(x[i] * f);
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

template <int D>
int go(const AttnParams& p, long long num_blocks, cudaStream_t st) {
  CUtensorMap tmQ, tmKV;
  if (make_tmap(&tmQ, p.q, (uint64_t)p.T, (uint64_t)p.Hq * (D / 2), TQ)) return -2;
  if (make_tmap(&tmKV, p.kv_cache, (uint64_t)num_blocks * 2 * p.Hkv * p.bs, D, 16)) return -3;
  constexpr int smem = smem_bytes<D>() + 1024;
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];  // the limit is an attribute of (kernel, device)
  if (!configured) {
    if (cudaFuncSetAttribute(diff_prefill_tc_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -4;
    configured = true;
  }
  diff_prefill_tc_kernel<D><<<dim3(p.num_q_tiles, p.Hq / 2), kThreads, smem, st>>>(tmQ, tmKV, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace

bool diff_prefill_tc_sizes(int D, float softcap) { return (D == 64 || D == 128) && softcap > 0.f && softcap <= 55.f; }

int diff_prefill_tc_launch(const AttnParams& p, long long num_blocks, cudaStream_t st) {
  if (p.maps != 2 || !diff_prefill_tc_sizes(p.D, p.softcap) || p.lam == nullptr || p.vdim < 1 || p.vdim > p.D) return -1;
  if (p.Hq % 2 || (p.Hq / 2) % p.Hkv || p.bs < 16 || (p.bs & (p.bs - 1)) || p.kv_fp8 || p.window > 0 || p.keep > 0 || p.kv_shared || p.bias != nullptr ||
      p.gate != nullptr || p.sinks != nullptr || p.lse != nullptr) return -1;
  if (p.q_sh != p.D / 2 || p.q_st != (long long)p.Hq * (p.D / 2) || ((uintptr_t)p.q & 15) || ((uintptr_t)p.kv_cache & 15) || ((uintptr_t)p.out & 15)) return -1;
  if (p.num_q_tiles <= 0) return 0;
  return p.D == 64 ? go<64>(p, num_blocks, st) : go<128>(p, num_blocks, st);
}

unsigned int diff_prefill_read_status(bool clear) { return read_status_tu(clear); }
void diff_prefill_read_status_async(unsigned int* dst, cudaStream_t st) { read_status_tu_async(dst, st); }

}  // namespace oc
