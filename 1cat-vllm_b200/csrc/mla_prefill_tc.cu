// Latent-attention prefill on tcgen05 tensor cores.
//
// Portions of prompts attend in the expanded form: the cached latents of a request's context are gathered from their pages (with the
// shared key part beside them), one GEMM turns them into per-head keys and values, and the kernel below runs causal attention with query /
// key rows of [unrotated | rotated] and value rows of their own width - per (query, key, head) a third of the products of the absorbed form,
// which is what single tokens use. Sizes are in 64-column chunks: NC unrotated, RC rotated, VC value chunks, zeros in the padding.
//
// One CTA owns 128 consecutive query tokens of one request for one head and walks the keys in tiles of 128:
//   S = Q K^T      tcgen05.mma on TMA-loaded tiles (128-byte swizzle), S in TMEM (fp32, double-buffered)
//   P = softmax    eight warps, two threads per query row; P replaces S in its TMEM columns as bf16 - with FINE as two terms, the rounded
//                  value and what rounding took from it
//   O_tile = P V   operand A from TMEM, V as an MN-major operand; the softmax threads add O_tile into their fp32 row in registers
// Roles: warp 0 TMA producer, warp 1 MMA issue, warps 2-9 softmax and epilogue. Every wait is bounded; on expiry the CTA raises the status
// word and tears down.
#include "common.cuh"
#include "kernels.h"

namespace oc {

namespace {

constexpr int TQ = 128, TK = 128;
constexpr int kChunk = 128 * 128;        // bytes of one 64-column chunk of a 128-row operand tile
constexpr int kStages = 2;
constexpr int kThreads = 320;
constexpr uint32_t kColS = 0, kColO = 256;   // TMEM columns: S0 | S1 | O_tile

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// MN-major operand B: 64 columns x 8 rows form a 1024-byte swizzle atom; the next 8 rows (k) are 1024 bytes on, the next 64 columns a chunk on.
__device__ __forceinline__ uint64_t desc_mn(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFF) >> 4);
  d |= (uint64_t)((kChunk >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

template <int QC, int VC>
constexpr int smem_bytes() { return QC * kChunk + kStages * (QC + VC) * kChunk + 1024 + 2 * 2 * TQ * 4; }

template <int QC, int VC, bool FINE>
__global__ void __launch_bounds__(kThreads, 1)
mla_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmKV, const __grid_constant__ CUtensorMap tmR,
                      const MlaPrefillParams p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int kStage = (QC + VC) * kChunk, kEnd = QC * kChunk + kStages * kStage;
  uint8_t* sQ = smem;
  uint8_t* sKV = smem + QC * kChunk;     // stage: key chunks, value chunks
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + kEnd);
  uint64_t* q_full = bars;               // [1]
  uint64_t* k_full = bars + 1;           // [kStages]
  uint64_t* v_full = k_full + kStages;
  uint64_t* k_empty = v_full + kStages;
  uint64_t* v_empty = k_empty + kStages;
  uint64_t* s_full = v_empty + kStages;  // [2] scores of a tile are complete
  uint64_t* p_ready = s_full + 2;        // [2] probabilities written over the scores
  uint64_t* o_full = p_ready + 2;        // [1] P V of a tile is complete
  uint64_t* o_free = o_full + 1;         // [1] the softmax warps have read O_tile
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_free + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_req = const_cast<int*>(reinterpret_cast<volatile int*>(tmem_slot + 2));
  float* s_xch = reinterpret_cast<float*>(smem + kEnd + 1024);  // [2 tile parities][2 halves][TQ]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y;

  if (threadIdx.x == 0) {
    int b = blockIdx.x, found = -1, t0 = 0;
    for (int i = 0; i < p.num_long; ++i) {
      const int r = p.long_req[i], nt = (p.query_start_loc[r + 1] - p.query_start_loc[r] + TQ - 1) / TQ;
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
      mbar_init(&p_ready[i], 8);
    }
    mbar_init(o_full, 1);
    mbar_init(o_free, 8);
    *abort_flag = 0;
    mbar_fence_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmKV);
    prefetch_tmap(&tmR);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const int li = s_req[0], tq0 = s_req[1];

  int ntiles = 0, qs = 0, qlen = 0, S = 0, ctx0 = 0, base = 0;
  if (li >= 0) {
    const int r = p.long_req[li];
    base = p.long_ctx[li];
    qs = p.query_start_loc[r];
    qlen = p.query_start_loc[r + 1] - qs;
    S = p.seq_lens[r];
    ctx0 = S - qlen;
    const int kv_end = min(S, ctx0 + min(tq0 + TQ, qlen));  // keys the last row of this tile may see
    ntiles = (kv_end + TK - 1) / TK;
  }

  if (warp == 0) {
    // ------------------------------------------------------------------ producer
    if (lane == 0 && ntiles > 0) {
      mbar_expect_tx(q_full, QC * kChunk);
      // rows past the end of a tensor are zero-filled; rows of the next request are loaded and never stored
#pragma unroll
      for (int c = 0; c < QC; ++c) tma_load_2d(sQ + c * kChunk, &tmQ, (h * QC + c) * 64, qs + tq0, q_full);
      const int col = h * (p.NC + VC) * 64;
      bool ok = true;
      for (int j = 0; j < ntiles && ok; ++j) {
        const int s = j % kStages;
        const uint32_t ph = ((j / kStages) & 1) ^ 1;
        ok = mbar_wait(&k_empty[s], ph, abort_flag);
        if (ok) ok = mbar_wait(&v_empty[s], ph, abort_flag);
        if (!ok) break;
        uint8_t* dst = sKV + s * kStage;
        const int row = base + j * TK;   // keys past this request's context are masked
        mbar_expect_tx(&k_full[s], QC * kChunk);
        for (int c = 0; c < QC; ++c) {
          if (c < p.NC) tma_load_2d(dst + c * kChunk, &tmKV, col + c * 64, row, &k_full[s]);
          else tma_load_2d(dst + c * kChunk, &tmR, (c - p.NC) * 64, row, &k_full[s]);
        }
        mbar_expect_tx(&v_full[s], VC * kChunk);
        for (int c = 0; c < VC; ++c) tma_load_2d(dst + (QC + c) * kChunk, &tmKV, col + (p.NC + c) * 64, row, &v_full[s]);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issue
    if (lane == 0 && ntiles > 0) {
      const uint32_t idesc_qk = umma_idesc_bf16(TQ, TK);
      const uint32_t idesc_pv = umma_idesc_bf16(TQ, VC * 64) | (1u << 16);  // operand B (V) is MN-major
      const uint32_t q_addr = smem_u32(sQ), kv_addr = smem_u32(sKV);
      bool ok = mbar_wait(q_full, 0, abort_flag);
      auto issue_qk = [&](int j) {
        const int s = j % kStages;
        ok = mbar_wait(&k_full[s], (j / kStages) & 1, abort_flag);
        // the scores of tile j - 2 share these columns as probabilities: their product must be complete
        if (ok && j >= 2) ok = mbar_wait(o_full, (j - 2) & 1, abort_flag);
        if (!ok) return;
        tc_fence_after();
        const uint32_t d_addr = tmem_base + kColS + (j & 1) * TK, k_base = kv_addr + s * kStage;
#pragma unroll
        for (int c = 0; c < QC; ++c) {
          const uint64_t da = umma_desc_sw128(q_addr + c * kChunk), db = umma_desc_sw128(k_base + c * kChunk);
#pragma unroll
          for (int jj = 0; jj < 4; ++jj) umma_bf16(d_addr, da + (uint64_t)(jj * 2), db + (uint64_t)(jj * 2), idesc_qk, (c | jj) ? 1u : 0u);
        }
        umma_commit(&s_full[j & 1]);
        umma_commit(&k_empty[s]);
      };
      if (ok) issue_qk(0);
      for (int j = 0; j < ntiles && ok; ++j) {
        if (j + 1 < ntiles) issue_qk(j + 1);
        if (!ok) break;
        const int s = j % kStages;
        ok = mbar_wait(&p_ready[j & 1], (j >> 1) & 1, abort_flag);
        if (ok) ok = mbar_wait(&v_full[s], (j / kStages) & 1, abort_flag);
        if (ok && j > 0) ok = mbar_wait(o_free, (j - 1) & 1, abort_flag);
        if (!ok) break;
        tc_fence_after();
        const uint32_t v_base = kv_addr + s * kStage + QC * kChunk;
        const uint32_t pa = tmem_base + kColS + (j & 1) * TK;
#pragma unroll
        for (int jj = 0; jj < TK / 16; ++jj) {
          // 16 keys per MMA: 8 TMEM columns of P (keys 0-63 at column 0, 64-127 at 64; second terms 32 columns on), 2048 bytes of V
          const uint64_t db = desc_mn(v_base + jj * 2048);
          const uint32_t a = pa + (jj >> 2) * 64 + (jj & 3) * 8;
          umma_bf16_ts(tmem_base + kColO, a, db, idesc_pv, jj ? 1u : 0u);
          if (FINE) umma_bf16_ts(tmem_base + kColO, a + 32, db, idesc_pv, 1u);
        }
        umma_commit(o_full);
        umma_commit(&v_empty[s]);
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax + epilogue: two threads per query row
    const int q4 = warp & 3;                 // TMEM lane quarter this warp may touch
    const int half = (warp - 2) >> 2;        // which 64 keys of a tile / which half of the output columns this thread owns
    const int row = q4 * 32 + lane;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(q4 * 32) << 16);
    const float sl2 = p.scale * 1.4426950408889634f;
    const int tq = tq0 + row;                       // query token inside the request
    const int limit = min(S, ctx0 + tq + 1);        // keys [0, limit) are visible to this row
    constexpr int HC = VC * 32, KC = TK / 2;
    float o[HC];
#pragma unroll
    for (int i = 0; i < HC; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    float alpha[2] = {1.f, 1.f};
    bool ok = ntiles > 0;
    auto pair_sync = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(1 + q4) : "memory"); };

    // Both warps of a pair call pair_sync exactly ntiles + 1 times whatever happens (a named barrier has no time-out): a warp whose
    // bounded wait failed keeps walking the tiles without touching TMEM, and its partner learns of it through the abort flag.
    auto softmax_tile = [&](int j) {
      if (ok) ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1, abort_flag);
      tc_fence_after();
      const uint32_t s_addr = lane_addr + kColS + (j & 1) * TK + half * KC;
      const int k0 = j * TK + half * KC;
      const bool masked = k0 + KC > limit;
      float raw = -INFINITY;
      if (ok) {
#pragma unroll
        for (int c = 0; c < KC; c += 32) {
          uint32_t v[32];
          tmem_ld_32x32(s_addr + c, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            float x = __uint_as_float(v[i]);
            if (masked && k0 + c + i >= limit) x = -INFINITY;
            raw = fmaxf(raw, x);
          }
        }
      }
      float* xch = s_xch + (j & 1) * 2 * TQ;
      xch[half * TQ + row] = raw;
      pair_sync();
      if (!ok || *abort_flag) { ok = false; return; }
      // the scale is positive (the launcher checks): it commutes with the maximum
      const float mx = fmaxf(m, fmaxf(raw, xch[(half ^ 1) * TQ + row]) * sl2);
      const float m_use = (mx == -INFINITY) ? 0.f : mx;
      alpha[j & 1] = (m == -INFINITY) ? 0.f : ex2(m - m_use);
      m = mx;
      float sum = 0.f;
      uint32_t pk[32], pl[FINE ? 32 : 1];
#pragma unroll
      for (int c = 0; c < KC; c += 32) {
        uint32_t v[32];
        tmem_ld_32x32(s_addr + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float x0 = __uint_as_float(v[i]) * sl2 - m_use, x1 = __uint_as_float(v[i + 1]) * sl2 - m_use;
          if (masked && k0 + c + i >= limit) x0 = -INFINITY;
          if (masked && k0 + c + i + 1 >= limit) x1 = -INFINITY;
          const float p0 = ex2(x0), p1 = ex2(x1);
          __nv_bfloat162 b = __floats2bfloat162_rn(p0, p1);
          pk[(c + i) >> 1] = *reinterpret_cast<uint32_t*>(&b);
          if (FINE) {
            __nv_bfloat162 d = __floats2bfloat162_rn(p0 - __low2float(b), p1 - __high2float(b));
            pl[FINE ? (c + i) >> 1 : 0] = *reinterpret_cast<uint32_t*>(&d);
            sum += p0 + p1;
          } else {
            sum += __low2float(b) + __high2float(b);   // the sum of what the tensor core will actually multiply
          }
        }
      }
      tmem_st_32x32(s_addr, pk);
      if constexpr (FINE) tmem_st_32x32(s_addr + 32, pl);
      l = l * alpha[j & 1] + sum;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[j & 1]);
    };

    if (ntiles > 0) softmax_tile(0);
    for (int j = 0; j < ntiles; ++j) {
      if (j + 1 < ntiles) softmax_tile(j + 1);
      if (ok) ok = mbar_wait(o_full, j & 1, abort_flag);
      if (!ok) continue;
      tc_fence_after();
      const float a = alpha[j & 1];
#pragma unroll
      for (int c = 0; c < HC; c += 32) {
        uint32_t v[32];
        tmem_ld_32x32(lane_addr + kColO + half * HC + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c + i] = o[c + i] * a + __uint_as_float(v[i]);
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(o_free);
    }
    float* xch = s_xch + (ntiles & 1) * 2 * TQ;   // the row sum is the sum of the two halves' partial sums
    if (ntiles > 0) {
      xch[half * TQ + row] = l;
      pair_sync();
      l += xch[(half ^ 1) * TQ + row];
    }
    if (ok && !*abort_flag && tq < qlen) {
      if (p.sinks != nullptr) l += ex2(p.sinks[h] * 1.4426950408889634f - m);
      float inv = l > 0.f ? 1.f / l : 0.f;
      if (p.gate != nullptr) inv *= 1.f / (1.f + __expf(-__bfloat162float(p.gate[(size_t)(qs + tq) * p.gate_st + h])));
      __nv_bfloat16* dst = p.out + ((size_t)(qs + tq) * p.H + h) * p.vd + half * HC;
      const int n = min(HC, p.vd - half * HC);
      if (p.vd % 8 == 0) {
#pragma unroll
        for (int i = 0; i < HC; i += 8)
          if (i < n) {
            __nv_bfloat162 b[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) b[e] = __floats2bfloat162_rn(o[i + 2 * e] * inv, o[i + 2 * e + 1] * inv);
            *reinterpret_cast<uint4*>(dst + i) = *reinterpret_cast<uint4*>(b);
          }
      } else {
#pragma unroll
        for (int i = 0; i < HC; ++i)
          if (i < n) dst[i] = __float2bfloat16(o[i] * inv);
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

// One warp per context row of the gathered requests: latent and key part out of their page (the key part padded with zeros to RC chunks).
__global__ void __launch_bounds__(256) mla_gather_kernel(const MlaPrefillParams p) {
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= p.rows) return;
  int i = 0;
  while (i + 1 < p.num_long && p.long_ctx[i + 1] <= row) ++i;
  const int key = row - p.long_ctx[i];
  const int page = p.block_table[(size_t)p.long_req[i] * p.bt_stride + key / p.bs];
  const int width = p.lora_pad + p.rope_pad;
  const uint4* src = reinterpret_cast<const uint4*>(p.cache + ((size_t)page * p.bs + key % p.bs) * width);
  uint4* lat = reinterpret_cast<uint4*>(p.lat + (size_t)row * p.lora_pad);
  uint4* rot = reinterpret_cast<uint4*>(p.rot + (size_t)row * p.RC * 64);
  for (int c = lane; c < p.lora_pad / 8; c += 32) lat[c] = src[c];
  for (int c = lane; c < p.RC * 8; c += 32) rot[c] = c < p.rope_pad / 8 ? src[p.lora_pad / 8 + c] : make_uint4(0, 0, 0, 0);
}

// Query rows [unrotated | rotated] in whole chunks: one warp per (token, head), two elements per lane and step.
__global__ void __launch_bounds__(256) mla_query_kernel(const MlaPrefillParams p) {
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= p.T * p.H) return;
  const int t = row / p.H, N = p.NC * 64, QP = N + p.RC * 64, hf = p.rope / 2;
  const __nv_bfloat16* q = p.q + (size_t)t * p.q_st + (size_t)(row - t * p.H) * (p.nope + p.rope);
  const __nv_bfloat16* x = q + p.nope;
  const float* cs = p.cos_sin + (size_t)p.positions[t] * p.rope;
  __nv_bfloat162* dst = reinterpret_cast<__nv_bfloat162*>(p.q_out + (size_t)row * QP);
  const __nv_bfloat16 zero = __float2bfloat16(0.f);
  for (int j = lane; j < N / 2; j += 32) {
    __nv_bfloat162 v;
    v.x = 2 * j < p.nope ? q[2 * j] : zero;
    v.y = 2 * j + 1 < p.nope ? q[2 * j + 1] : zero;
    dst[j] = v;
  }
  for (int j = lane; j < p.RC * 32; j += 32) {
    float v[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = 2 * j + e;
      v[e] = 0.f;
      if (k < p.rope) {
        const int a = p.interleaved ? k >> 1 : (k < hf ? k : k - hf);
        const bool second = p.interleaved ? (k & 1) : k >= hf;
        const float u = __bfloat162float(x[p.interleaved ? 2 * a : a]), w = __bfloat162float(x[p.interleaved ? 2 * a + 1 : a + hf]), cc = cs[a], ss = cs[hf + a];
        v[e] = second ? w * cc + u * ss : u * cc - w * ss;
      }
    }
    dst[N / 2 + j] = __floats2bfloat162_rn(v[0], v[1]);
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledFn get_encode_fn() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres);
    fn = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  return fn;
}

// bf16 [rows][cols] -> boxes of {64 columns, 128 rows}, 128-byte swizzle, zero fill
int make_tmap(CUtensorMap* tm, const void* base, uint64_t rows, uint64_t cols) {
  EncodeTiledFn enc = get_encode_fn();
  if (!enc) return -1;
  cuuint64_t dims[2] = {cols, rows};
  cuuint64_t strides[1] = {cols * 2};
  cuuint32_t box[2] = {64, 128};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = enc(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : (int)r;
}

template <int QC, int VC, bool FINE>
int go(const MlaPrefillParams& p, cudaStream_t st) {
  CUtensorMap tmQ, tmKV, tmR;
  if (make_tmap(&tmQ, p.q_out, (uint64_t)p.T, (uint64_t)p.H * QC * 64)) return -2;
  if (make_tmap(&tmKV, p.kv, (uint64_t)p.rows, (uint64_t)p.H * (p.NC + VC) * 64)) return -3;
  if (make_tmap(&tmR, p.rot, (uint64_t)p.rows, (uint64_t)p.RC * 64)) return -3;
  constexpr int smem = smem_bytes<QC, VC>() + 1024;
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (cudaFuncSetAttribute(mla_prefill_tc_kernel<QC, VC, FINE>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -4;
    configured = true;
  }
  mla_prefill_tc_kernel<QC, VC, FINE><<<dim3(p.num_q_tiles, p.H), kThreads, smem, st>>>(tmQ, tmKV, tmR, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <int QC, int VC>
int go_fine(const MlaPrefillParams& p, cudaStream_t st) { return p.fine ? go<QC, VC, true>(p, st) : go<QC, VC, false>(p, st); }

}  // namespace

bool mla_prefill_sizes(int nope, int rope, int vd) {
  const int QC = (nope + 63) / 64 + (rope + 63) / 64;
  return nope >= 1 && rope >= 2 && vd >= 1 && QC <= 3 && vd <= 128;
}

int mla_prefill_inputs_launch(const MlaPrefillParams& p, cudaStream_t st) {
  if (p.rows <= 0 || p.T <= 0 || p.num_long <= 0) return 0;
  if (p.lora_pad % 8 || p.rope_pad % 8 || ((uintptr_t)p.cache & 15)) return -1;
  mla_gather_kernel<<<(p.rows + 7) / 8, 256, 0, st>>>(p);
  mla_query_kernel<<<(p.T * p.H + 7) / 8, 256, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

int mla_prefill_launch(const MlaPrefillParams& p, cudaStream_t st) {
  if (p.num_q_tiles <= 0 || p.num_long <= 0) return 0;
  if (!mla_prefill_sizes(p.nope, p.rope, p.vd) || p.scale <= 0.f) return -1;
  if (((uintptr_t)p.q_out | (uintptr_t)p.kv | (uintptr_t)p.rot | (uintptr_t)p.out) & 15) return -1;
  const int QC = p.NC + p.RC, VC = (p.vd + 63) / 64;
  if (QC == 2) return VC == 1 ? go_fine<2, 1>(p, st) : go_fine<2, 2>(p, st);
  return VC == 1 ? go_fine<3, 1>(p, st) : go_fine<3, 2>(p, st);
}

unsigned int mla_prefill_read_status(bool clear) { return read_status_tu(clear); }
void mla_prefill_read_status_async(unsigned int* dst, cudaStream_t st) { read_status_tu_async(dst, st); }

}  // namespace oc
