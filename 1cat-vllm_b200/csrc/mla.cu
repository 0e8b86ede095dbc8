// Multi-head latent attention decode (DeepSeek-V2/V3): multi-query attention over the paged latent cache, with W_UK already
// folded into the query ("absorbed" form) and W_UV applied by the caller to the result.
//   scores = [q_nope_abs | q_rope] . [latent | k_rope]^T   (512 + 64 wide for DeepSeek)       out = softmax(scores) . latent   (512 wide)
// All heads of a token share the same keys, so heads are the rows of the tile: a CTA owns 16 (head, query-token) rows of one request
// and one split of its context. Its four warps each score a quarter of a tile's 64 keys, exchange the scores through shared memory and own
// a different quarter of the output columns, so the accumulator stays in registers. The key tile is loaded once into
// shared memory and serves as K (all columns) and as V (the latent ones): the latent is read from HBM exactly once per CTA.
// Split-KV partials are merged by mla_combine_kernel. bf16 mma.sync.m16n8k16, fp32 softmax state in the exp2 domain.
// (reference: csrc/attention/mla/sm100_cutlass_mla_kernel.cu; csrc/cpu/mla_decode.cpp; layers/attention/mla_attention.py forward_mqa)
#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

constexpr int KEYS = 64, ROWS = 16;

__device__ __forceinline__ void cp16(void* smem, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pk(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
// a row holds `pitch` elements, a multiple of 64: XOR the low 3 bits of the 16-byte chunk with the row to spread ldmatrix over the banks
__device__ __forceinline__ uint32_t koff(int row, int chunk, int pitch) { return (uint32_t)(row * pitch * 2 + (((chunk & ~7) | ((chunk ^ row) & 7)) << 4)); }
__device__ __forceinline__ float rounded(float v) { return __bfloat162float(__float2bfloat16(v)); }

__device__ __forceinline__ float ex2(float x) {   // approximate instruction: the softmax of the bf16 kernels
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <typename E> __device__ __forceinline__ float ldf(const E* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename E> __device__ __forceinline__ void stf(E* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// factor of the output gate of (token, head); 1 without a gate
template <typename E>
__device__ __forceinline__ float gate_of(const MlaParams& p, size_t tok, int head) {
  return p.gate != nullptr ? 1.f / (1.f + expf(-ldf<E>(reinterpret_cast<const E*>(p.gate) + tok * p.gate_st + head))) : 1.f;
}

// Element j of a rotated row: pair and half from the layout, (cos | sin) row of the position in the table.
template <typename E>
__device__ __forceinline__ float rotated(const E* x, int j, int n, const float* cs, int interleaved) {
  const int h = n / 2, i = interleaved ? j >> 1 : (j < h ? j : j - h);
  const bool second = interleaved ? (j & 1) : j >= h;
  const float u = ldf<E>(x + (interleaved ? 2 * i : i)), v = ldf<E>(x + (interleaved ? 2 * i + 1 : i + h)), c = cs[i], s = cs[h + i];
  return second ? v * c + u * s : u * c - v * s;
}

// DV: width of the latent (and of the output), a multiple of 64. FINE: the softmax weights enter the value product as two bf16 terms.
template <int DV, bool FINE>
__global__ void __launch_bounds__(128) mla_decode_kernel(const MlaParams p) {
  constexpr int NB = DV / 32;                // output blocks of 8 columns per warp
  __shared__ __align__(16) float sS[ROWS][KEYS + 8];
  extern __shared__ __align__(128) uint8_t smem[];
  const int DK = DV + p.rope_pad, PK = DV + ((p.rope_pad + 63) & ~63), CHK = DK / 8;
  uint8_t* sQ = smem;                        // [16][PK]
  uint8_t* sK = sQ + ROWS * PK * 2;          // [2][64][PK]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g_ = lane >> 2, tg = lane & 3;
  const int r = blockIdx.y, rt = blockIdx.x, split = blockIdx.z;
  const int qs = p.query_start_loc[r], qlen = p.query_start_loc[r + 1] - qs, S = p.seq_lens[r];
  if (qlen <= 0 || S <= 0 || (p.skip_min_len > 0 && qlen >= p.skip_min_len)) return;
  const int total_rows = qlen * p.H;         // row = token * H + head
  const int row0 = rt * ROWS;
  if (row0 >= total_rows) return;
  const int nrows = min(ROWS, total_rows - row0);
  const int ctx0 = S - qlen;
  const int last_tok = (row0 + nrows - 1) / p.H;
  const int kv_end = min(S, ctx0 + last_tok + 1);
  const int ntiles = (kv_end + KEYS - 1) / KEYS;
  int lo = 0, hi = ntiles;
  if (p.splits > 1) {
    const int per = (ntiles + p.splits - 1) / p.splits;
    lo = split * per;
    hi = min(ntiles, lo + per);
  }
  const int* bt = p.block_table + (size_t)r * p.bt_stride;
  const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.cache);
  auto load_tile = [&](int tile, int buf) {
    uint8_t* dk = sK + (size_t)buf * KEYS * PK * 2;
    for (int row = warp; row < KEYS; row += 4) {   // a warp copies whole rows
      const int key = tile * KEYS + row;
      if (key < kv_end) {
        const __nv_bfloat16* src = cache + ((size_t)bt[key >> p.bs_shift] * p.bs + (key & (p.bs - 1))) * DK;
        for (int ch = lane; ch < CHK; ch += 32) cp16(dk + koff(row, ch, PK), src + ch * 8);
      } else {
        for (int ch = lane; ch < CHK; ch += 32) *reinterpret_cast<uint4*>(dk + koff(row, ch, PK)) = make_uint4(0, 0, 0, 0);
      }
    }
  };
  if (lo < hi) load_tile(lo, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  // Q rows: [absorbed query (DV) | rotated part (rope_pad, zeros past rope)]
  for (int idx = threadIdx.x; idx < ROWS * (DV / 8); idx += 128) {
    const int row = idx / (DV / 8), ch = idx % (DV / 8), gr = row0 + row;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row < nrows) v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.q_abs) + ((size_t)(qs + gr / p.H) * p.H + gr % p.H) * DV + ch * 8);
    *reinterpret_cast<uint4*>(sQ + koff(row, ch, PK)) = v;
  }
  for (int idx = threadIdx.x; idx < ROWS * p.rope_pad; idx += 128) {
    const int row = idx / p.rope_pad, j = idx % p.rope_pad, gr = row0 + row;
    float v = 0.f;
    if (row < nrows && j < p.rope) {
      const int tok = gr / p.H;
      const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.q_rope) + (size_t)(qs + tok) * p.qr_st + (size_t)(gr % p.H) * p.qr_sh;
      v = p.cos_sin != nullptr ? rotated(x, j, p.rope, p.cos_sin + (size_t)(ctx0 + tok) * p.rope, p.interleaved) : __bfloat162float(x[j]);
    }
    *reinterpret_cast<__nv_bfloat16*>(sQ + koff(row, DV / 8 + j / 8, PK) + (j & 7) * 2) = __float2bfloat16(v);
  }
  float o[NB][4];  // this warp's quarter of the output columns
#pragma unroll
  for (int i = 0; i < NB; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m2[2] = {-INFINITY, -INFINITY}, l2[2] = {0.f, 0.f};
  const float sc = p.scale * 1.4426950408889634f;
  for (int tile = lo; tile < hi; ++tile) {
    const int buf = (tile - lo) & 1;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (tile + 1 < hi) load_tile(tile + 1, buf ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const uint32_t kb = smem_u32(sK + (size_t)buf * KEYS * PK * 2), qb = smem_u32(sQ);
    {
      // scores of this warp's 16 keys (two accumulator sets, so that products of even and odd steps do not wait for each other)
      float sc4[2][2][4];
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int n = 0; n < 2; ++n) sc4[e][n][0] = sc4[e][n][1] = sc4[e][n][2] = sc4[e][n][3] = 0.f;
      const int steps = DK / 16;
#pragma unroll 2
      for (int kk = 0; kk < steps; kk += 2) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          if (kk + e >= steps) break;
          uint32_t a[4], b[4];
          ldsm4(a, qb + koff(lane & 15, (kk + e) * 2 + (lane >> 4), PK));
          ldsm4(b, kb + koff(warp * 16 + (lane & 7) + ((lane >> 4) << 3), (kk + e) * 2 + ((lane >> 3) & 1), PK));
          mma16816(sc4[e][0], a, b[0], b[1]);
          mma16816(sc4[e][1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h)
          *reinterpret_cast<float2*>(&sS[g_ + h * 8][warp * 16 + n * 8 + tg * 2]) =
              make_float2(sc4[0][n][h * 2] + sc4[1][n][h * 2], sc4[0][n][h * 2 + 1] + sc4[1][n][h * 2 + 1]);
    }
    __syncthreads();   // the tile's scores are complete; every warp takes all of them
    float s[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float2 v = *reinterpret_cast<const float2*>(&sS[g_ + h * 8][n * 8 + tg * 2]);
        s[n][h * 2] = v.x;
        s[n][h * 2 + 1] = v.y;
      }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int gr = row0 + g_ + h * 8;
      const int qpos = ctx0 + gr / p.H;
      float mx = -INFINITY;
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int key = tile * KEYS + n * 8 + tg * 2 + e;
          float v = s[n][h * 2 + e] * sc;
          v = (key <= qpos && key < kv_end) ? v : -INFINITY;
          s[n][h * 2 + e] = v;
          mx = fmaxf(mx, v);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float mn = fmaxf(m2[h], mx), mu = (mn == -INFINITY) ? 0.f : mn;
      const float alpha = ex2(m2[h] - mu);
      float sum = 0.f;
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float pv = ex2(s[n][h * 2 + e] - mu);
          s[n][h * 2 + e] = pv;
          sum += pv;
        }
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      l2[h] = l2[h] * alpha + sum;
      m2[h] = mn;
#pragma unroll
      for (int i = 0; i < NB; ++i) { o[i][h * 2] *= alpha; o[i][h * 2 + 1] *= alpha; }
    }
    // O[:, this warp's quarter] += P . latent[:, that slice]
#pragma unroll
    for (int n2 = 0; n2 < 4; ++n2) {
      uint32_t a[4] = {pk(s[n2 * 2][0], s[n2 * 2][1]), pk(s[n2 * 2][2], s[n2 * 2][3]), pk(s[n2 * 2 + 1][0], s[n2 * 2 + 1][1]), pk(s[n2 * 2 + 1][2], s[n2 * 2 + 1][3])};
      uint32_t al[4];
      if (FINE) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float u = s[n2 * 2 + (e >> 1)][2 * (e & 1)], v = s[n2 * 2 + (e >> 1)][2 * (e & 1) + 1];
          al[e] = pk(u - rounded(u), v - rounded(v));
        }
      }
#pragma unroll
      for (int d2 = 0; d2 < NB / 2; ++d2) {
        uint32_t b[4];
        ldsm4t(b, kb + koff(n2 * 16 + (lane & 15), warp * NB + d2 * 2 + (lane >> 4), PK));
        mma16816(o[d2 * 2], a, b[0], b[1]);
        mma16816(o[d2 * 2 + 1], a, b[2], b[3]);
        if (FINE) {
          mma16816(o[d2 * 2], al, b[0], b[1]);
          mma16816(o[d2 * 2 + 1], al, b[2], b[3]);
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int row = g_ + h * 8;
    if (row >= nrows) continue;
    const int gr = row0 + row, tok = gr / p.H, hd = gr % p.H;
    const size_t orow = (size_t)(qs + tok) * p.H + hd;
    if (p.splits > 1) {
      float* wo = p.ws_o + ((size_t)split * p.T * p.H + orow) * DV + warp * (DV / 4);
#pragma unroll
      for (int i = 0; i < NB; ++i) *reinterpret_cast<float2*>(wo + i * 8 + tg * 2) = make_float2(o[i][h * 2], o[i][h * 2 + 1]);
      if (warp == 0 && tg == 0) {
        float* wm = p.ws_ml + ((size_t)split * p.T * p.H + orow) * 2;
        wm[0] = m2[h];
        wm[1] = l2[h];
      }
    } else {
      const float den = l2[h] + (p.sinks != nullptr ? ex2(p.sinks[hd] * 1.4426950408889634f - m2[h]) : 0.f);
      const float inv = den > 0.f ? gate_of<__nv_bfloat16>(p, qs + tok, hd) / den : 0.f;
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + orow * DV + warp * (DV / 4);
#pragma unroll
      for (int i = 0; i < NB; ++i) *reinterpret_cast<uint32_t*>(dst + i * 8 + tg * 2) = pk(o[i][h * 2] * inv, o[i][h * 2 + 1] * inv);
    }
  }
}

// One warp per (token, head): merge the splits. Rows of padding tokens hold nothing and are skipped by their sum of 0.
__global__ void mla_combine_kernel(const MlaParams p) {
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31, DV = p.kv_lora;
  const int rows = p.T * p.H;
  if (warp >= rows) return;
  float mine = lane < p.splits ? p.ws_ml[((size_t)lane * rows + warp) * 2] : -INFINITY;   // at most 32 splits
  const float M = warp_max(mine);
  const float f_mine = mine == -INFINITY ? 0.f : ex2(mine - M);
  const float L = warp_sum(lane < p.splits ? p.ws_ml[((size_t)lane * rows + warp) * 2 + 1] * f_mine : 0.f);
  const float den = L + (p.sinks != nullptr ? ex2(p.sinks[warp % p.H] * 1.4426950408889634f - M) : 0.f);
  const float inv = L > 0.f ? gate_of<__nv_bfloat16>(p, warp / p.H, warp % p.H) / den : 0.f;
  for (int c = lane * 2; c < DV; c += 64) {
    float x = 0.f, y = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float f = __shfl_sync(0xffffffffu, f_mine, s);
      const float2 v = *reinterpret_cast<const float2*>(p.ws_o + ((size_t)s * rows + warp) * DV + c);
      if (f != 0.f) { x = fmaf(v.x, f, x); y = fmaf(v.y, f, y); }
    }
    *reinterpret_cast<uint32_t*>(reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)warp * DV + c) = pk(x * inv, y * inv);
  }
}

// Any sizes, fp32 arithmetic throughout: the full-precision form (fp32 engines) and the fallback for latents the tensor-core kernel has no
// variant of. A CTA owns 8 (token, head) rows; tiles of 32 keys pass through shared memory: a lane scores one key for its warp's two rows,
// and for the value product a thread owns latent columns tid, tid + 128, ...
template <typename E, int NC>
__global__ void __launch_bounds__(128) mla_plain_kernel(const MlaParams p) {
  constexpr int PR = 8, PKEYS = 32;
  extern __shared__ __align__(128) uint8_t smem[];
  const int W = p.kv_lora + p.rope_pad, pitch = W | 1;
  float* sq = reinterpret_cast<float*>(smem);   // [8][W]
  float* sk = sq + PR * W;                      // [32][pitch]
  __shared__ float sp[PR][PKEYS], sa[PR], sl[PR];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = blockIdx.y, row0 = blockIdx.x * PR;
  const int qs = p.query_start_loc[r], qlen = p.query_start_loc[r + 1] - qs, S = p.seq_lens[r];
  if (qlen <= 0 || S <= 0 || row0 >= qlen * p.H || (p.skip_min_len > 0 && qlen >= p.skip_min_len)) return;
  const int nrows = min(PR, qlen * p.H - row0), ctx0 = S - qlen;
  const int kv_end = min(S, ctx0 + (row0 + nrows - 1) / p.H + 1);
  const int* bt = p.block_table + (size_t)r * p.bt_stride;
  const E* cache = reinterpret_cast<const E*>(p.cache);
  for (int idx = threadIdx.x; idx < PR * W; idx += 128) {
    const int row = idx / W, d = idx - row * W, gr = row0 + row;
    float v = 0.f;
    if (row < nrows) {
      const int tok = gr / p.H, hd = gr % p.H, j = d - p.kv_lora;
      if (j < 0) v = ldf<E>(reinterpret_cast<const E*>(p.q_abs) + ((size_t)(qs + tok) * p.H + hd) * p.kv_lora + d);
      else if (j < p.rope) {
        const E* x = reinterpret_cast<const E*>(p.q_rope) + (size_t)(qs + tok) * p.qr_st + (size_t)hd * p.qr_sh;
        v = p.cos_sin != nullptr ? rotated(x, j, p.rope, p.cos_sin + (size_t)(ctx0 + tok) * p.rope, p.interleaved) : ldf<E>(x + j);
      }
    }
    sq[idx] = v;
  }
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, o[PR][NC];
#pragma unroll
  for (int i = 0; i < PR; ++i)
#pragma unroll
    for (int c = 0; c < NC; ++c) o[i][c] = 0.f;
  for (int k0 = 0; k0 < kv_end; k0 += PKEYS) {
    const int nk = min(PKEYS, kv_end - k0);
    __syncthreads();
    for (int idx = threadIdx.x; idx < nk * W; idx += 128) {
      const int key = idx / W, d = idx - key * W, a = k0 + key;
      sk[key * pitch + d] = ldf<E>(cache + ((size_t)bt[a >> p.bs_shift] * p.bs + (a & (p.bs - 1))) * W + d);
    }
    __syncthreads();
    float s[2] = {0.f, 0.f};
    if (lane < nk)
      for (int d = 0; d < W; ++d) {
        const float k = sk[lane * pitch + d];
        s[0] = fmaf(sq[(warp * 2) * W + d], k, s[0]);
        s[1] = fmaf(sq[(warp * 2 + 1) * W + d], k, s[1]);
      }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = warp * 2 + i;
      const bool seen = row < nrows && lane < nk && k0 + lane <= ctx0 + (row0 + row) / p.H;
      const float v = seen ? s[i] * p.scale : -INFINITY, mn = fmaxf(m[i], warp_max(v)), mu = mn == -INFINITY ? 0.f : mn;
      const float pv = seen ? expf(v - mu) : 0.f, alpha = m[i] == -INFINITY ? 0.f : expf(m[i] - mu);
      l[i] = l[i] * alpha + warp_sum(pv);
      m[i] = mn;
      sp[row][lane] = pv;
      if (lane == 0) sa[row] = alpha;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int col = threadIdx.x + 128 * c;
      if (col < p.kv_lora) {
#pragma unroll
        for (int i = 0; i < PR; ++i) o[i][c] *= sa[i];
        for (int k = 0; k < nk; ++k) {
          const float v = sk[k * pitch + col];
#pragma unroll
          for (int i = 0; i < PR; ++i) o[i][c] = fmaf(sp[i][k], v, o[i][c]);
        }
      }
    }
  }
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {   // the factor of the row's output
      const int gr = row0 + warp * 2 + i, hd = gr % p.H;
      const float den = l[i] + (p.sinks != nullptr ? expf(p.sinks[hd] - m[i]) : 0.f);
      sl[warp * 2 + i] = den > 0.f && warp * 2 + i < nrows ? gate_of<E>(p, qs + gr / p.H, hd) / den : 0.f;
    }
  }
  __syncthreads();
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = threadIdx.x + 128 * c;
    if (col >= p.kv_lora) continue;
#pragma unroll
    for (int i = 0; i < PR; ++i)
      if (i < nrows) {
        const int gr = row0 + i;
        stf<E>(reinterpret_cast<E*>(p.out) + ((size_t)(qs + gr / p.H) * p.H + gr % p.H) * p.kv_lora + col, o[i][c] * sl[i]);
      }
  }
}

// Between the down- and the up-projections: both latent norms, the rotation of the shared key part, the cache insert. One CTA per token.
template <typename E>
__global__ void __launch_bounds__(128) mla_prepare_kernel(const MlaPrepareParams p) {
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int tid = threadIdx.x;
  const E* q = p.q != nullptr ? reinterpret_cast<const E*>(p.q) + t * p.ld_q : nullptr;
  const E* kv = reinterpret_cast<const E*>(p.kv) + t * p.ld_kv;
  float a = 0.f, b = 0.f;
  for (int c = tid; c < p.nq; c += 128) { const float v = ldf<E>(q + c); a = fmaf(v, v, a); }
  for (int c = tid; c < p.lora; c += 128) { const float v = ldf<E>(kv + c); b = fmaf(v, v, b); }
  a = warp_sum(a);
  b = warp_sum(b);
  if ((tid & 31) == 0) { red[tid >> 5] = a; red[4 + (tid >> 5)] = b; }
  __syncthreads();
  a = red[0] + red[1] + red[2] + red[3];
  b = red[4] + red[5] + red[6] + red[7];
  if (q != nullptr) {
    const float inv = 1.f / sqrtf(a / (float)p.nq + p.eps);
    for (int c = tid; c < p.nq; c += 128) stf<E>(reinterpret_cast<E*>(p.q_out) + t * p.nq + c, ldf<E>(q + c) * inv * ldf<E>(reinterpret_cast<const E*>(p.q_w) + c));
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  E* row = reinterpret_cast<E*>(p.cache) + (size_t)slot * p.width;
  const float inv = 1.f / sqrtf(b / (float)p.lora + p.eps);
  for (int c = tid; c < p.lora; c += 128) stf<E>(row + c, ldf<E>(kv + c) * inv * ldf<E>(reinterpret_cast<const E*>(p.kv_w) + c));
  const float* cs = p.cos_sin + (size_t)p.positions[t] * p.rope;
  for (int j = tid; j < p.rope; j += 128) stf<E>(row + p.lora_pad + j, rotated(kv + p.lora, j, p.rope, cs, p.interleaved));
}

template <int DV, bool FINE>
int decode_go(const MlaParams& p, cudaStream_t st) {
  const int PK = DV + ((p.rope_pad + 63) & ~63), smem = (ROWS + 2 * KEYS) * PK * 2;
  if (smem > 220 * 1024) return -1;
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];  // the limit is an attribute of (kernel, device)
  if (!configured) {
    if (cudaFuncSetAttribute(mla_decode_kernel<DV, FINE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return -4;
    configured = true;
  }
  mla_decode_kernel<DV, FINE><<<dim3((p.max_q_len * p.H + ROWS - 1) / ROWS, p.R, p.splits), 128, smem, st>>>(p);
  if (p.splits > 1) mla_combine_kernel<<<(p.T * p.H * 32 + 255) / 256, 256, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <int DV>
int decode_fine(const MlaParams& p, cudaStream_t st) { return p.fine ? decode_go<DV, true>(p, st) : decode_go<DV, false>(p, st); }

template <typename E, int NC>
int plain_go(const MlaParams& p, cudaStream_t st) {
  const int W = p.kv_lora + p.rope_pad, smem = (8 * W + 32 * (W | 1)) * 4;
  if (smem > 220 * 1024) return -1;
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (cudaFuncSetAttribute(mla_plain_kernel<E, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return -4;
    configured = true;
  }
  mla_plain_kernel<E, NC><<<dim3((p.max_q_len * p.H + 7) / 8, p.R), 128, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <typename E>
int plain_e(const MlaParams& p, cudaStream_t st) {
  if (p.kv_lora <= 128) return plain_go<E, 1>(p, st);
  if (p.kv_lora <= 256) return plain_go<E, 2>(p, st);
  if (p.kv_lora <= 512) return plain_go<E, 4>(p, st);
  if (p.kv_lora <= 1024) return plain_go<E, 8>(p, st);
  return -1;
}

}  // namespace

bool mla_tensor_core_sizes(int kv_lora, int rope_pad) {
  const bool dv = kv_lora == 64 || kv_lora == 128 || kv_lora == 192 || kv_lora == 256 || kv_lora == 384 || kv_lora == 512;
  return dv && rope_pad >= 16 && rope_pad % 16 == 0 && (ROWS + 2 * KEYS) * (kv_lora + ((rope_pad + 63) & ~63)) * 2 <= 220 * 1024;
}

int mla_decode_launch(const MlaParams& p, cudaStream_t st) {
  if (p.R == 0 || p.T == 0) return 0;
  if (p.bs < 1 || (p.bs & (p.bs - 1)) || p.splits < 1 || p.splits > 32) return -1;
  if (p.f32) return p.splits == 1 ? plain_e<float>(p, st) : -1;
  if (!mla_tensor_core_sizes(p.kv_lora, p.rope_pad)) return p.splits == 1 ? plain_e<__nv_bfloat16>(p, st) : -1;
  switch (p.kv_lora) {
    case 64: return decode_fine<64>(p, st);
    case 128: return decode_fine<128>(p, st);
    case 192: return decode_fine<192>(p, st);
    case 256: return decode_fine<256>(p, st);
    case 384: return decode_fine<384>(p, st);
    case 512: return decode_fine<512>(p, st);
  }
  return -1;
}

int mla_prepare_launch(const MlaPrepareParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  launch_k(p.f32 ? mla_prepare_kernel<float> : mla_prepare_kernel<__nv_bfloat16>, dim3(p.T), dim3(128), 0, st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

unsigned int mla_read_status(bool clear) { return read_status_tu(clear); }
void mla_read_status_async(unsigned int* dst, cudaStream_t st) { read_status_tu_async(dst, st); }

}  // namespace oc
