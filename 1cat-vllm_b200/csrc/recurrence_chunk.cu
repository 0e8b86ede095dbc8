// Chunked forms of the matrix-state recurrences in recurrence.cu for bf16 portions of at least 64 tokens (chunks of C = 64), on mma.sync.
//
// Channel delta. G_i = sum_{j <= i} log2 g_j inside a chunk, per key channel; every product below pairs decays whose exponents are not positive.
//   A_ij = beta_i sum_d k_id k_jd 2^(G_id - G_jd)  (j < i)        T = (I + A)^-1        P_ij = sum_d q_id k_jd 2^(G_id - G_jd)  (j <= i)
//   W = T (beta 2^G K)     U = T (beta V)     N = U - W S0     O = (2^G Q) S0 + P N     S = 2^(G_C) S0 + (2^(G_C - G) K)^T N
// delta_prepare: everything without S0, one CTA per (chunk, head). Inside blocks of 16 tokens A and P are summed directly with one exponential per
// term; between blocks the decay is split at the first token of the later block, which turns the sums into products of two scaled tiles.
// delta_scan: the chain over chunks, one CTA per (sequence, head, 32 state columns), S in fp32 accumulators.
//
// Mamba-2 (ssd_chunk): scalar decays scale the rows of the results, so B and C stay as they are and nothing needs a workspace; one CTA per
// (sequence, head, 32 columns) does the whole chunk: P_ij = (C_i . B_j) 2^(G_i - G_j) dt_j, O = 2^G (C S0) + P x + D x, S = 2^(G_C) S0 + B^T (2^(G_C - G) dt x).
//
// 32-bit operands (decayed keys and queries, T, P, W, N, S) enter the products as two bf16 planes. Why mma.sync: chains of dependent 64-row products
// with a register-resident state, far too small for the tensor pipe to be the limit.
#include "kernels.h"
#include "mma_sync.cuh"

namespace oc {
namespace {

constexpr int C = 64, VT = 32, THREADS = 256, PREP = 512;   // tokens per chunk, state columns per CTA, threads of a scan and of delta_prepare
constexpr int P64 = 72, PV = 40;          // pitches of [*][64] and [*][32] tiles
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
// 2^x for exponents that are not positive (2 ulp)
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float bf(const __nv_bfloat16 v) { return __bfloat162float(v); }

// two neighbouring outputs, as far as `left` columns go
__device__ __forceinline__ void put2(__nv_bfloat16* dst, float a, float b, int left) {
  if (left >= 2 && ((uintptr_t)dst & 3) == 0) *reinterpret_cast<uint32_t*>(dst) = pack2(a, b);
  else {
    if (left >= 1) dst[0] = __float2bfloat16(a);
    if (left >= 2) dst[1] = __float2bfloat16(b);
  }
}

// rows of `width` bf16 columns (zeros from `cols` on and from row `n` on) into a tile of pitch `pitch`
template <int N>
__device__ __forceinline__ void fetch_rows(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, long long ld, int n, int cols, int width, bool vec) {
  const int segs = width / 8;
  for (int e = threadIdx.x; e < C * segs; e += N) {
    const int row = e / segs, c = e % segs * 8;
    __nv_bfloat16* d = dst + row * pitch + c;
    const int live = row < n ? min(8, cols - c) : 0;
    const __nv_bfloat16* s = src + (size_t)(row < n ? row : 0) * ld + (live > 0 ? c : 0);
    if (vec) cp_async16(smem_u32(d), s, live > 0 ? live * 2 : 0);
    else {
#pragma unroll
      for (int j = 0; j < 8; ++j) d[j] = j < live ? s[j] : __float2bfloat16(0.f);
    }
  }
}

// -------------------------------------------------------------------------------------------------------------- delta_prepare
template <int DP>
struct Ws {   // per (chunk, head), in bf16 elements: W, Qg, Kd (two planes each), P (two planes), then U fp32 [64][Vp] and 2^(G_C) fp32 [DP]
  static constexpr size_t tile = (size_t)C * DP;
  static constexpr size_t w = 0, q = 2 * tile, k = 4 * tile, p = 6 * tile, u = 6 * tile + 2 * C * C;
  static __host__ __device__ size_t elems(int vp) { return u + 2 * (size_t)(C * vp + DP); }
};

template <int DP>
struct PrepSmem {
  static constexpr int PD = DP + 8, PG = DP + 4;
  float G[C][PG];
  __nv_bfloat16 q[C][PD], k[C][PD];
  union {
    struct { __nv_bfloat16 kj[2][48][PD], ki[2][16][PD], qi[2][16][PD]; } f;
    struct { float T[C][C + 1], M[3][16][17]; } t;
    __nv_bfloat16 b[2][C][PD];
  };
  union {
    float A[C][C + 1];
    __nv_bfloat16 tb[2][C][P64];
  };
  float rq[C], rk[C], pd[C], beta[C];   // factors of the unit vectors; diagonal of P; step sizes
};

template <int DP>
__global__ void __launch_bounds__(PREP) delta_prepare_kernel(const DeltaChunkParams p) {
  using SM = PrepSmem<DP>;
  using W_ = Ws<DP>;
  constexpr int PD = SM::PD;
  extern __shared__ __align__(16) uint8_t raw[];
  SM& s = *reinterpret_cast<SM*>(raw);
  pdl_trigger();
  pdl_wait();
  const int ci = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
  const int r = p.chunk_req[ci], tc = p.chunk_t0[ci], n = min(C, p.query_start_loc[r + 1] - tc), D = p.D, hk = h / (p.H / p.Hk);
  fetch_rows<PREP>(&s.q[0][0], PD, p.q + (size_t)tc * p.ld + (size_t)hk * D, p.ld, n, D, DP, p.vec);
  fetch_rows<PREP>(&s.k[0][0], PD, p.k + (size_t)tc * p.ld + (size_t)hk * D, p.ld, n, D, DP, p.vec);
  cp_async_commit();
  const float nega = -expf(p.A_log[h]) * kLog2e;
  {   // all loads of a thread are in flight before the first is used; a thread keeps its channel
    constexpr int N = C * DP / PREP, STEP = PREP / DP;
    const int i0 = tid / DP, d = tid % DP;
    const float* a = p.a + (size_t)tc * p.ld_a + (size_t)h * D + d;
    float x[N];
#pragma unroll
    for (int k = 0; k < N; ++k) x[k] = d < D && i0 + k * STEP < n ? __ldg(a + (size_t)(i0 + k * STEP) * p.ld_a) : 0.f;
    const float bias = d < D ? p.dt_bias[(size_t)h * D + d] : 0.f;
#pragma unroll
    for (int k = 0; k < N; ++k) s.G[i0 + k * STEP][d] = d < D && i0 + k * STEP < n ? nega * softplus(x[k] + bias) : 0.f;
  }
  if (tid < C) s.beta[tid] = tid < n ? 1.f / (1.f + expf(-bf(p.b[(size_t)(tc + tid) * p.ld_b + h]))) : 0.f;
  cp_async_wait<0>();
  __syncthreads();
  constexpr int SEG = PREP / DP < 16 ? PREP / DP : 16, PER = C / SEG;   // a channel's running sum in SEG parts
  if (tid < DP * SEG) {
    const int d = tid % DP, i0 = tid / DP * PER;
    float x[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) x[i] = s.G[i0 + i][d];
#pragma unroll
    for (int i = 1; i < PER; ++i) x[i] += x[i - 1];
#pragma unroll
    for (int i = 0; i < PER; ++i) s.G[i0 + i][d] = x[i];
  }
  for (int i = warp; i < C; i += PREP / 32) {
    float q2 = 0.f, k2 = 0.f, qk = 0.f;
#pragma unroll
    for (int d = lane; d < DP; d += 32) {
      const float a = bf(s.q[i][d]), b = bf(s.k[i][d]);
      q2 = fmaf(a, a, q2);
      k2 = fmaf(b, b, k2);
      qk = fmaf(a, b, qk);
    }
    q2 = warp_sum(q2);
    k2 = warp_sum(k2);
    qk = warp_sum(qk);
    if (lane == 0) {
      const float fq = 1.f / sqrtf(q2 + 1e-6f) * p.scale, fk = 1.f / sqrtf(k2 + 1e-6f);
      s.rq[i] = fq;
      s.rk[i] = fk;
      s.pd[i] = qk * fq * fk;
    }
  }
  __syncthreads();
  if (tid < DP * (SEG - 1)) {   // what the parts ahead add; a part's own last row is left to the end, the others read it
    const int d = tid % DP, part = tid / DP + 1;
    float add = 0.f;
    for (int k = 0; k < part; ++k) add += s.G[(k + 1) * PER - 1][d];
    float x[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) x[i] = s.G[part * PER + i][d] + add;
    asm volatile("bar.sync 1, %0;" ::"n"(DP * (SEG - 1)) : "memory");
#pragma unroll
    for (int i = 0; i < PER; ++i) s.G[part * PER + i][d] = x[i];
  }
  __syncthreads();
  __nv_bfloat16* ws = p.ws + ((size_t)ci * p.H + h) * W_::elems(p.Vp);
  auto put_p = [&](int i, int j, float v) {
    const __nv_bfloat16 hi = __float2bfloat16(v);
    ws[W_::p + (size_t)i * C + j] = hi;
    ws[W_::p + C * C + (size_t)i * C + j] = __float2bfloat16(v - bf(hi));
  };
  // what is not below the diagonal, then A and P inside the diagonal blocks: one thread per pair
  for (int e = tid; e < C * C; e += PREP) {
    const int i = e >> 6, j = e & 63;
    if (j >= i) {
      s.A[i][j] = 0.f;
      put_p(i, j, j == i ? s.pd[i] : 0.f);
    }
  }
  if ((tid & 127) < 120) {   // four warps to a block: lanes read neighbouring rows
    const int blk = tid >> 7, x = tid & 127;   // x = i (i - 1) / 2 + j for 0 <= j < i < 16
    int i = (int)((1.f + sqrtf(8.f * (float)x + 1.f)) * 0.5f);
    if (i * (i + 1) / 2 <= x) ++i;
    if (i * (i - 1) / 2 > x) --i;
    const int j = blk * 16 + x - i * (i - 1) / 2;
    i += blk * 16;
    float kk = 0.f, qk = 0.f;
#pragma unroll 4
    for (int d = 0; d < DP; d += 4) {
      const float4 gi = *reinterpret_cast<const float4*>(&s.G[i][d]), gj = *reinterpret_cast<const float4*>(&s.G[j][d]);
      const uint2 a = *reinterpret_cast<const uint2*>(&s.k[i][d]), b = *reinterpret_cast<const uint2*>(&s.q[i][d]), c = *reinterpret_cast<const uint2*>(&s.k[j][d]);
      auto f2 = [](uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); };
      const float2 a0 = f2(a.x), a1 = f2(a.y), b0 = f2(b.x), b1 = f2(b.y), c0 = f2(c.x), c1 = f2(c.y);
      const float e0 = c0.x * ex2(gi.x - gj.x), e1 = c0.y * ex2(gi.y - gj.y), e2 = c1.x * ex2(gi.z - gj.z), e3 = c1.y * ex2(gi.w - gj.w);
      kk = fmaf(a0.x, e0, fmaf(a0.y, e1, fmaf(a1.x, e2, fmaf(a1.y, e3, kk))));
      qk = fmaf(b0.x, e0, fmaf(b0.y, e1, fmaf(b1.x, e2, fmaf(b1.y, e3, qk))));
    }
    s.A[i][j] = s.beta[i] * s.rk[i] * s.rk[j] * kk;
    put_p(i, j, s.rq[i] * s.rk[j] * qk);
  }
  // between blocks: rows of block I decayed from its first token on, earlier keys decayed up to it
#pragma unroll 1
  for (int I = 1; I < 4; ++I) {
    __syncthreads();
    const float* ref = s.G[16 * I - 1];
    auto planes = [&](__nv_bfloat16* hi, __nv_bfloat16* lo, uint32_t src, float e0, float e1) {
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&src));
      uint32_t a, b;
      split2(v.x * e0, v.y * e1, a, b);
      *reinterpret_cast<uint32_t*>(hi) = a;
      *reinterpret_cast<uint32_t*>(lo) = b;
    };
    for (int e = tid; e < (16 * I + 16) * (DP / 2); e += PREP) {
      const int row = e / (DP / 2), d = e % (DP / 2) * 2;
      if (row < 16 * I) {
        const float2 rf = *reinterpret_cast<const float2*>(ref + d), gr = *reinterpret_cast<const float2*>(&s.G[row][d]);
        const float e0 = ex2(rf.x - gr.x), e1 = ex2(rf.y - gr.y);
        planes(&s.f.kj[0][row][d], &s.f.kj[1][row][d], *reinterpret_cast<const uint32_t*>(&s.k[row][d]), e0, e1);
      } else {
        const int i = row - 16 * I;
        const float2 rf = *reinterpret_cast<const float2*>(ref + d), gr = *reinterpret_cast<const float2*>(&s.G[row][d]);
        const float e0 = ex2(gr.x - rf.x), e1 = ex2(gr.y - rf.y);
        planes(&s.f.ki[0][i][d], &s.f.ki[1][i][d], *reinterpret_cast<const uint32_t*>(&s.k[row][d]), e0, e1);
        planes(&s.f.qi[0][i][d], &s.f.qi[1][i][d], *reinterpret_cast<const uint32_t*>(&s.q[row][d]), e0, e1);
      }
    }
    __syncthreads();
    if (warp < 2 * I) {
      const bool isq = warp & 1;
      const int n0 = (warp >> 1) * 16;
      const uint32_t ah = smem_u32(isq ? &s.f.qi[0][0][0] : &s.f.ki[0][0][0]), al = smem_u32(isq ? &s.f.qi[1][0][0] : &s.f.ki[1][0][0]);
      const uint32_t bh = smem_u32(&s.f.kj[0][0][0]), bl = smem_u32(&s.f.kj[1][0][0]);
      float acc3[3][2][4] = {};   // the three products of the planes, apart: a chain of dependent products each
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t a0[4], a1[4], b0[4], b1[4];
        ldsm_x4(a0, a_addr(ah, PD, 0, ks * 16, lane));
        ldsm_x4(a1, a_addr(al, PD, 0, ks * 16, lane));
        ldsm_x4(b0, bnk_addr(bh, PD, n0, ks * 16, lane));
        ldsm_x4(b1, bnk_addr(bl, PD, n0, ks * 16, lane));
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma16816(acc3[0][t], a0, b0[2 * t], b0[2 * t + 1]);
          mma16816(acc3[1][t], a0, b1[2 * t], b1[2 * t + 1]);
          mma16816(acc3[2][t], a1, b0[2 * t], b0[2 * t + 1]);
        }
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float sum = acc3[0][t][e] + (acc3[1][t][e] + acc3[2][t][e]);
          const int i = 16 * I + g8 + 8 * (e >> 1), j = n0 + 8 * t + 2 * t4 + (e & 1);
          if (isq) put_p(i, j, s.rq[i] * s.rk[j] * sum);
          else s.A[i][j] = s.beta[i] * s.rk[i] * s.rk[j] * sum;
        }
    }
  }
  __syncthreads();
  // decayed queries and keys for the products with the state
  for (int e = tid; e < C * (DP / 2); e += PREP) {
    const int i = e / (DP / 2), d = e % (DP / 2) * 2;
    const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&s.q[i][d])), k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&s.k[i][d]));
    const float2 g = *reinterpret_cast<const float2*>(&s.G[i][d]), end = *reinterpret_cast<const float2*>(&s.G[C - 1][d]);
    uint32_t a, b;
    split2(q.x * s.rq[i] * ex2(g.x), q.y * s.rq[i] * ex2(g.y), a, b);
    *reinterpret_cast<uint32_t*>(ws + W_::q + (size_t)i * DP + d) = a;
    *reinterpret_cast<uint32_t*>(ws + W_::q + W_::tile + (size_t)i * DP + d) = b;
    split2(k.x * s.rk[i] * ex2(end.x - g.x), k.y * s.rk[i] * ex2(end.y - g.y), a, b);
    *reinterpret_cast<uint32_t*>(ws + W_::k + (size_t)i * DP + d) = a;
    *reinterpret_cast<uint32_t*>(ws + W_::k + W_::tile + (size_t)i * DP + d) = b;
  }
  float* wsU = reinterpret_cast<float*>(ws + W_::u);
  if (tid < DP) wsU[(size_t)C * p.Vp + tid] = ex2(s.G[C - 1][tid]);
  // T = (I + A)^-1 in fp32: diagonal blocks by forward substitution, then the block sub-diagonals T_ij = -T_ii sum_{j <= k < i} A_ik T_kj
  {
    float (*T)[C + 1] = s.t.T;
    for (int e = tid; e < C * C; e += PREP) T[e >> 6][e & 63] = 0.f;
    __syncthreads();
    if (tid < C) {
      const int b0 = (tid >> 4) * 16, c = tid & 15;
      float col[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float acc = 0.f;
#pragma unroll
        for (int j = 0; j < 16; ++j)
          if (j < i) acc = fmaf(s.A[b0 + i][b0 + j], col[j], acc);
        col[i] = i < c ? 0.f : (i == c ? 1.f : -acc);
      }
#pragma unroll
      for (int i = 0; i < 16; ++i) T[b0 + i][b0 + c] = col[i];
    }
    __syncthreads();
#pragma unroll 1
    for (int d = 1; d < 4; ++d) {
      for (int o = tid; o < (4 - d) * 256; o += PREP) {
        const int blk = o >> 8, rr = (o >> 4) & 15, c = o & 15, i0 = (blk + d) * 16, j0 = blk * 16;
        float acc = 0.f;
        for (int k = j0; k < i0; ++k) acc = fmaf(s.A[i0 + rr][k], T[k][j0 + c], acc);
        s.t.M[blk][rr][c] = acc;
      }
      __syncthreads();
      for (int o = tid; o < (4 - d) * 256; o += PREP) {
        const int blk = o >> 8, rr = (o >> 4) & 15, c = o & 15, i0 = (blk + d) * 16, j0 = blk * 16;
        float acc = 0.f;
#pragma unroll
        for (int m = 0; m < 16; ++m) acc = fmaf(T[i0 + rr][i0 + m], s.t.M[blk][m][c], acc);
        T[i0 + rr][j0 + c] = -acc;
      }
      __syncthreads();
    }
    for (int e = tid; e < C * C / 2; e += PREP) {   // A is no longer needed
      const int i = e >> 5, j = (e & 31) * 2;
      uint32_t a, b;
      split2(T[i][j], T[i][j + 1], a, b);
      *reinterpret_cast<uint32_t*>(&s.tb[0][i][j]) = a;
      *reinterpret_cast<uint32_t*>(&s.tb[1][i][j]) = b;
    }
  }
  // W = T (beta rk 2^G K), then U = T (beta V) in tiles of DP columns
  const int mt = warp & 3, part = warp >> 2;   // 16 rows; DP / 4 columns
  const uint32_t th = smem_u32(&s.tb[0][0][0]), tl = smem_u32(&s.tb[1][0][0]), bh = smem_u32(&s.b[0][0][0]), bl = smem_u32(&s.b[1][0][0]);
  const int vtiles = (p.Vp + DP - 1) / DP;
#pragma unroll 1
  for (int job = 0; job <= vtiles; ++job) {
    __syncthreads();   // the tile's storage is free
    const int c0 = (job - 1) * DP;
    constexpr int N = C * DP / 2 / PREP, STEP = PREP * 2 / DP;
    const int r0 = tid / (DP / 2), d = tid % (DP / 2) * 2;
    auto put = [&](int i, float x, float y) {
      uint32_t a, b;
      split2(x, y, a, b);
      *reinterpret_cast<uint32_t*>(&s.b[0][i][d]) = a;
      *reinterpret_cast<uint32_t*>(&s.b[1][i][d]) = b;
    };
    if (job == 0) {
#pragma unroll
      for (int e = 0; e < N; ++e) {
        const int i = r0 + e * STEP;
        const float2 k = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&s.k[i][d])), g = *reinterpret_cast<const float2*>(&s.G[i][d]);
        const float f = s.beta[i] * s.rk[i];
        put(i, k.x * f * ex2(g.x), k.y * f * ex2(g.y));
      }
    } else {
      float x[N][2];
#pragma unroll
      for (int e = 0; e < N; ++e) {
        const int i = r0 + e * STEP;
        const __nv_bfloat16* v = p.v + (size_t)(tc + i) * p.ld + (size_t)h * p.V + c0 + d;
        x[e][0] = i < n && c0 + d < p.V ? bf(__ldg(v)) : 0.f;
        x[e][1] = i < n && c0 + d + 1 < p.V ? bf(__ldg(v + 1)) : 0.f;
      }
#pragma unroll
      for (int e = 0; e < N; ++e) put(r0 + e * STEP, s.beta[r0 + e * STEP] * x[e][0], s.beta[r0 + e * STEP] * x[e][1]);
    }
    __syncthreads();
    constexpr int NT = DP / 32;   // tiles of eight columns; DP = 32 has one, loaded with a neighbour that is not used
    float acc[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
    for (int ks = 0; ks <= mt; ++ks) {   // T is lower triangular
      uint32_t a0[4], a1[4];
      ldsm_x4(a0, a_addr(th, P64, mt * 16, ks * 16, lane));
      ldsm_x4(a1, a_addr(tl, P64, mt * 16, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < (NT + 1) / 2; ++np) {
        uint32_t b0[4], b1[4];
        ldsm_x4_t(b0, bkn_addr(bh, PD, ks * 16, part * (DP / 4) + np * 16, lane));
        ldsm_x4_t(b1, bkn_addr(bl, PD, ks * 16, part * (DP / 4) + np * 16, lane));
#pragma unroll
        for (int t = 0; t < (NT < 2 ? 1 : 2); ++t) {
          mma16816(acc[2 * np + t], a0, b0[2 * t], b0[2 * t + 1]);
          mma16816(acc[2 * np + t], a0, b1[2 * t], b1[2 * t + 1]);
          mma16816(acc[2 * np + t], a1, b0[2 * t], b0[2 * t + 1]);
        }
      }
    }
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int i = mt * 16 + g8 + 8 * hh, d = part * (DP / 4) + t * 8 + t4 * 2;
        if (job == 0) {
          uint32_t a, b;
          split2(acc[t][2 * hh], acc[t][2 * hh + 1], a, b);
          *reinterpret_cast<uint32_t*>(ws + W_::w + (size_t)i * DP + d) = a;
          *reinterpret_cast<uint32_t*>(ws + W_::w + W_::tile + (size_t)i * DP + d) = b;
        } else if (c0 + d < p.Vp) {
          *reinterpret_cast<float2*>(wsU + (size_t)i * p.Vp + c0 + d) = make_float2(acc[t][2 * hh], acc[t][2 * hh + 1]);
        }
      }
  }
}

// ----------------------------------------------------------------------------------------------------------------- delta_scan
template <int DP>
struct ScanSmem {
  static constexpr int PD = DP + 8;
  __nv_bfloat16 w[2][C][PD], q[2][C][PD], k[2][C][PD], p[2][C][P64];
  __nv_bfloat16 st[2][DP][PV], nv[2][C][PV];
  float u[C][VT + 4], gc[DP];
};

template <int DP>
__global__ void __launch_bounds__(THREADS) delta_scan_kernel(const DeltaChunkParams p) {
  using SM = ScanSmem<DP>;
  using W_ = Ws<DP>;
  constexpr int PD = SM::PD, MT = DP / 16, NS = MT >= 8 ? 1 : 2, NC = 4 / NS;   // state: MT row tiles x NS column parts of NC n tiles
  extern __shared__ __align__(16) uint8_t raw[];
  SM& s = *reinterpret_cast<SM*>(raw);
  pdl_trigger();
  pdl_wait();
  const int li = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
  const int r = p.long_req[li], c_first = p.long_chunk0[li], nch = p.long_n[li], qs = p.query_start_loc[r], t1 = p.query_start_loc[r + 1];
  const int tbase = p.chunk_t0[c_first], D = p.D, V = p.V;
  float* Sg = p.state + ((size_t)p.state_slots[r] * p.H + h) * D * V;
  const bool owner = warp < MT * NS;
  const int sm_t = warp % MT, sc = (warp / MT) * NC * 8;   // row tile and first column of this warp's part of the state
  const bool init = tbase > qs || p.has_initial_state[r] != 0;   // a later segment of the portion goes on from what the earlier one left
  float S[NC][4];
#pragma unroll
  for (int t = 0; t < NC; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = sm_t * 16 + g8 + 8 * (e >> 1), col = v0 + sc + t * 8 + t4 * 2 + (e & 1);
      S[t][e] = owner && init && row < D && col < V ? Sg[(size_t)row * V + col] : 0.f;
    }
  auto base = [&](int c) { return p.ws + ((size_t)(c_first + c) * p.H + h) * W_::elems(p.Vp); };
  auto tiles = [&](__nv_bfloat16* dst, const __nv_bfloat16* src) {   // two planes [64][DP]
    for (int e = tid; e < 2 * C * (DP / 8); e += THREADS) {
      const int row = e / (DP / 8), c = e % (DP / 8) * 8;
      cp_async16(smem_u32(dst + row * PD + c), src + (size_t)row * DP + c, 16);
    }
  };
  auto fetch_w = [&](int c) {
    tiles(&s.w[0][0][0], base(c) + W_::w);
    const float* u = reinterpret_cast<const float*>(base(c) + W_::u) + v0;
    for (int e = tid; e < C * (VT / 4); e += THREADS) cp_async16(smem_u32(&s.u[e / (VT / 4)][e % (VT / 4) * 4]), u + (size_t)(e / (VT / 4)) * p.Vp + e % (VT / 4) * 4, 16);
    cp_async_commit();
  };
  auto fetch_q = [&](int c) {
    tiles(&s.q[0][0][0], base(c) + W_::q);
    const __nv_bfloat16* pp = base(c) + W_::p;
    for (int e = tid; e < 2 * C * 8; e += THREADS) cp_async16(smem_u32(&s.p[0][0][0] + (e >> 3) * P64 + (e & 7) * 8), pp + (size_t)(e >> 3) * C + (e & 7) * 8, 16);
    cp_async_commit();
  };
  auto fetch_k = [&](int c) {
    tiles(&s.k[0][0][0], base(c) + W_::k);
    const float* gc = reinterpret_cast<const float*>(base(c) + W_::u) + (size_t)C * p.Vp;
    if (tid < DP / 4) cp_async16(smem_u32(&s.gc[tid * 4]), gc + tid * 4, 16);
    cp_async_commit();
  };
  fetch_w(0);
  fetch_q(0);
  fetch_k(0);
  const int mt = warp & 3, nh = (warp >> 2) * 16;   // token-major products: row tile and 16 columns
  const uint32_t wh = smem_u32(&s.w[0][0][0]), wl = smem_u32(&s.w[1][0][0]), qh = smem_u32(&s.q[0][0][0]), ql = smem_u32(&s.q[1][0][0]);
  const uint32_t kh = smem_u32(&s.k[0][0][0]), kl = smem_u32(&s.k[1][0][0]), ph = smem_u32(&s.p[0][0][0]), pl = smem_u32(&s.p[1][0][0]);
  const uint32_t sh = smem_u32(&s.st[0][0][0]), sl = smem_u32(&s.st[1][0][0]), nhh = smem_u32(&s.nv[0][0][0]), nl = smem_u32(&s.nv[1][0][0]);
  auto product = [&](float (&acc)[2][4], uint32_t ah, uint32_t al, int pitch, uint32_t bh, uint32_t bl, int steps) {
    float m1[2][4] = {}, m2[2][4] = {};   // the three products of the planes, apart: a chain of dependent products each
#pragma unroll 4
    for (int ks = 0; ks < steps; ++ks) {
      uint32_t a0[4], a1[4], b0[4], b1[4];
      ldsm_x4(a0, a_addr(ah, pitch, mt * 16, ks * 16, lane));
      ldsm_x4(a1, a_addr(al, pitch, mt * 16, ks * 16, lane));
      ldsm_x4_t(b0, bkn_addr(bh, PV, ks * 16, nh, lane));
      ldsm_x4_t(b1, bkn_addr(bl, PV, ks * 16, nh, lane));
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        mma16816(acc[t], a0, b0[2 * t], b0[2 * t + 1]);
        mma16816(m1[t], a0, b1[2 * t], b1[2 * t + 1]);
        mma16816(m2[t], a1, b0[2 * t], b0[2 * t + 1]);
      }
    }
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[t][e] += m1[t][e] + m2[t][e];
  };
  for (int c = 0; c < nch; ++c) {
    const bool more = c + 1 < nch;
    if (owner) {
#pragma unroll
      for (int t = 0; t < NC; ++t)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int row = sm_t * 16 + g8 + 8 * hh, col = sc + t * 8 + t4 * 2;
          uint32_t a, b;
          split2(S[t][2 * hh], S[t][2 * hh + 1], a, b);
          *reinterpret_cast<uint32_t*>(&s.st[0][row][col]) = a;
          *reinterpret_cast<uint32_t*>(&s.st[1][row][col]) = b;
        }
    }
    cp_async_wait<2>();
    __syncthreads();   // W, U and the state's planes are there
    {
      float acc[2][4] = {};
      product(acc, wh, wl, PD, sh, sl, DP / 16);
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int i = mt * 16 + g8 + 8 * hh, col = nh + t * 8 + t4 * 2;
          uint32_t a, b;
          split2(s.u[i][col] - acc[t][2 * hh], s.u[i][col + 1] - acc[t][2 * hh + 1], a, b);
          *reinterpret_cast<uint32_t*>(&s.nv[0][i][col]) = a;
          *reinterpret_cast<uint32_t*>(&s.nv[1][i][col]) = b;
        }
    }
    cp_async_wait<1>();
    __syncthreads();   // N is complete, Q and P are there, W and U are free
    if (more) fetch_w(c + 1); else cp_async_commit();
    {
      float acc[2][4] = {};
      product(acc, qh, ql, PD, sh, sl, DP / 16);
      product(acc, ph, pl, P64, nhh, nl, mt + 1);   // P is lower triangular
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int tok = tbase + c * C + mt * 16 + g8 + 8 * hh, col = v0 + nh + t * 8 + t4 * 2;
          if (tok < t1) put2(p.out + ((size_t)tok * p.H + h) * V + col, acc[t][2 * hh], acc[t][2 * hh + 1], V - col);
        }
    }
    cp_async_wait<1>();
    __syncthreads();   // K is there, Q and P are free, the state's planes have been read
    if (more) fetch_q(c + 1); else cp_async_commit();
    if (owner) {
      const float ga = s.gc[sm_t * 16 + g8], gb = s.gc[sm_t * 16 + g8 + 8];
#pragma unroll
      for (int t = 0; t < NC; ++t) {
        S[t][0] *= ga; S[t][1] *= ga; S[t][2] *= gb; S[t][3] *= gb;
      }
#pragma unroll
      for (int ks = 0; ks < C / 16; ++ks) {
        uint32_t a0[4], a1[4];
        ldsm_x4_t(a0, at_addr(kh, PD, sm_t * 16, ks * 16, lane));
        ldsm_x4_t(a1, at_addr(kl, PD, sm_t * 16, ks * 16, lane));
#pragma unroll
        for (int np = 0; np < NC / 2; ++np) {
          uint32_t b0[4], b1[4];
          ldsm_x4_t(b0, bkn_addr(nhh, PV, ks * 16, sc + np * 16, lane));
          ldsm_x4_t(b1, bkn_addr(nl, PV, ks * 16, sc + np * 16, lane));
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            mma16816(S[2 * np + t], a0, b0[2 * t], b0[2 * t + 1]);
            mma16816(S[2 * np + t], a0, b1[2 * t], b1[2 * t + 1]);
            mma16816(S[2 * np + t], a1, b0[2 * t], b0[2 * t + 1]);
          }
        }
      }
    }
    __syncthreads();   // K and N have been read
    if (more) fetch_k(c + 1); else cp_async_commit();
  }
  if (!owner) return;
#pragma unroll
  for (int t = 0; t < NC; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = sm_t * 16 + g8 + 8 * (e >> 1), col = v0 + sc + t * 8 + t4 * 2 + (e & 1);
      if (row < D && col < V) Sg[(size_t)row * V + col] = S[t][e];
    }
}

// ------------------------------------------------------------------------------------------------------------------ ssd_chunk
template <int DP>
struct SsdSmem {
  static constexpr int PD = DP + 8;
  __nv_bfloat16 c[2][C][PD], b[2][C][PD], x[2][C][PV];
  __nv_bfloat16 p[2][C][P64], st[2][DP][PV], xs[2][C][PV];
  float G[2][C], dt[2][C];
};

template <int DP>
__global__ void __launch_bounds__(THREADS) ssd_chunk_kernel(const DeltaChunkParams p) {
  using SM = SsdSmem<DP>;
  constexpr int PD = SM::PD, MT = DP / 16, NS = MT >= 8 ? 1 : 2, NC = 4 / NS;
  extern __shared__ __align__(16) uint8_t raw[];
  SM& s = *reinterpret_cast<SM*>(raw);
  pdl_trigger();
  pdl_wait();
  const int li = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3;
  const int r = p.long_req[li], t0 = p.query_start_loc[r], t1 = p.query_start_loc[r + 1], nch = (t1 - t0 + C - 1) / C;
  const int D = p.D, V = p.V, hk = h / (p.H / p.Hk);
  float* Sg = p.state + ((size_t)p.state_slots[r] * p.H + h) * D * V;
  const bool owner = warp < MT * NS, init = p.has_initial_state[r] != 0;
  const int sm_t = warp % MT, sc = (warp / MT) * NC * 8;
  const float nega = -expf(p.A_log[h]) * kLog2e, skip = p.skip[h], dt_bias = p.dt_bias[h];
  float S[NC][4];
#pragma unroll
  for (int t = 0; t < NC; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = sm_t * 16 + g8 + 8 * (e >> 1), col = v0 + sc + t * 8 + t4 * 2 + (e & 1);
      S[t][e] = owner && init && row < D && col < V ? Sg[(size_t)row * V + col] : 0.f;
    }
  float z[2] = {0.f, 0.f};   // warp 0: step logits of the next chunk, loaded a chunk ahead
  auto logits = [&](int c) {
    const int tc = t0 + c * C;
#pragma unroll
    for (int j = 0; j < 2; ++j) z[j] = tc + lane + 32 * j < t1 ? bf(p.b[(size_t)(tc + lane + 32 * j) * p.ld_b + h]) : 0.f;
  };
  if (warp == 0) logits(0);
  auto fetch = [&](int c) {
    const int b = c & 1, tc = t0 + c * C, n = min(C, t1 - tc);
    fetch_rows<THREADS>(&s.c[b][0][0], PD, p.q + (size_t)tc * p.ld + (size_t)hk * D, p.ld, n, D, DP, p.vec);
    fetch_rows<THREADS>(&s.b[b][0][0], PD, p.k + (size_t)tc * p.ld + (size_t)hk * D, p.ld, n, D, DP, p.vec);
    fetch_rows<THREADS>(&s.x[b][0][0], PV, p.v + (size_t)tc * p.ld + (size_t)h * V + v0, p.ld, n, V - v0, VT, p.vec);
    cp_async_commit();
    if (warp == 0) {   // step sizes, and the running sum of the decays' logarithms
      float a[2], g[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int i = lane + 32 * j;
        a[j] = i < n ? fminf(fmaxf(softplus(z[j] + dt_bias), p.dt_min), p.dt_max) : 0.f;
        g[j] = nega * a[j];
      }
      logits(c + 1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, g[0], o), y = __shfl_up_sync(0xffffffffu, g[1], o);
        if (lane >= o) { g[0] += x; g[1] += y; }
      }
      g[1] += __shfl_sync(0xffffffffu, g[0], 31);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        s.dt[b][lane + 32 * j] = a[j];
        s.G[b][lane + 32 * j] = g[j];
      }
    }
  };
  fetch(0);
  const int mt = warp & 3, nh = warp >> 2;
  const uint32_t ph = smem_u32(&s.p[0][0][0]), pl = smem_u32(&s.p[1][0][0]), sh = smem_u32(&s.st[0][0][0]), sl = smem_u32(&s.st[1][0][0]);
  const uint32_t xh = smem_u32(&s.xs[0][0][0]), xl = smem_u32(&s.xs[1][0][0]);
  for (int c = 0; c < nch; ++c) {
    const int b = c & 1;
    const float *G = s.G[b], *dt = s.dt[b];
    const uint32_t sc_ = smem_u32(&s.c[b][0][0]), sb_ = smem_u32(&s.b[b][0][0]), sx_ = smem_u32(&s.x[b][0][0]);
    if (owner) {
#pragma unroll
      for (int t = 0; t < NC; ++t)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int row = sm_t * 16 + g8 + 8 * hh, col = sc + t * 8 + t4 * 2;
          uint32_t u, w;
          split2(S[t][2 * hh], S[t][2 * hh + 1], u, w);
          *reinterpret_cast<uint32_t*>(&s.st[0][row][col]) = u;
          *reinterpret_cast<uint32_t*>(&s.st[1][row][col]) = w;
        }
    }
    cp_async_wait<0>();
    __syncthreads();   // this chunk's rows, steps and the state's planes are there; the other buffers are free
    if (c + 1 < nch) fetch(c + 1);
    if (2 * nh <= mt) {   // P, lower triangular: 16 rows, 32 columns
      float acc[4][4] = {};
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t a[4], x[4], y[4];
        ldsm_x4(a, a_addr(sc_, PD, mt * 16, ks * 16, lane));
        ldsm_x4(x, bnk_addr(sb_, PD, nh * 32, ks * 16, lane));
        ldsm_x4(y, bnk_addr(sb_, PD, nh * 32 + 16, ks * 16, lane));
        mma16816(acc[0], a, x[0], x[1]);
        mma16816(acc[1], a, x[2], x[3]);
        mma16816(acc[2], a, y[0], y[1]);
        mma16816(acc[3], a, y[2], y[3]);
      }
#pragma unroll
      for (int t = 0; t < 4; ++t)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int i = mt * 16 + g8 + 8 * hh, j = nh * 32 + t * 8 + t4 * 2;
          const float v0_ = j <= i ? acc[t][2 * hh] * ex2(G[i] - G[j]) * dt[j] : 0.f;
          const float v1_ = j + 1 <= i ? acc[t][2 * hh + 1] * ex2(G[i] - G[j + 1]) * dt[j + 1] : 0.f;
          uint32_t u, w;
          split2(v0_, v1_, u, w);
          *reinterpret_cast<uint32_t*>(&s.p[0][i][j]) = u;
          *reinterpret_cast<uint32_t*>(&s.p[1][i][j]) = w;
        }
    }
    for (int e = tid; e < C * (VT / 2); e += THREADS) {   // what a token leaves in the state at the chunk's end
      const int i = e / (VT / 2), d = e % (VT / 2) * 2;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&s.x[b][i][d]));
      const float f = ex2(G[C - 1] - G[i]) * dt[i];
      uint32_t u, w;
      split2(x.x * f, x.y * f, u, w);
      *reinterpret_cast<uint32_t*>(&s.xs[0][i][d]) = u;
      *reinterpret_cast<uint32_t*>(&s.xs[1][i][d]) = w;
    }
    __syncthreads();
    {
      float acc[2][4] = {}, low[2][4] = {};
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t a[4], x[4], y[4];
        ldsm_x4(a, a_addr(sc_, PD, mt * 16, ks * 16, lane));
        ldsm_x4_t(x, bkn_addr(sh, PV, ks * 16, nh * 16, lane));
        ldsm_x4_t(y, bkn_addr(sl, PV, ks * 16, nh * 16, lane));
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma16816(acc[t], a, x[2 * t], x[2 * t + 1]);
          mma16816(low[t], a, y[2 * t], y[2 * t + 1]);
        }
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          acc[t][e] += low[t][e];
          low[t][e] = 0.f;
        }
      const float ga = ex2(G[mt * 16 + g8]), gb = ex2(G[mt * 16 + g8 + 8]);
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        acc[t][0] *= ga; acc[t][1] *= ga; acc[t][2] *= gb; acc[t][3] *= gb;
      }
      for (int ks = 0; ks <= mt; ++ks) {
        uint32_t a0[4], a1[4], x[4];
        ldsm_x4(a0, a_addr(ph, P64, mt * 16, ks * 16, lane));
        ldsm_x4(a1, a_addr(pl, P64, mt * 16, ks * 16, lane));
        ldsm_x4_t(x, bkn_addr(sx_, PV, ks * 16, nh * 16, lane));
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma16816(acc[t], a0, x[2 * t], x[2 * t + 1]);
          mma16816(low[t], a1, x[2 * t], x[2 * t + 1]);
        }
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int i = mt * 16 + g8 + 8 * hh, cc = nh * 16 + t * 8 + t4 * 2, tok = t0 + c * C + i;
          if (tok >= t1) continue;
          const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&s.x[b][i][cc]));
          put2(p.out + ((size_t)tok * p.H + h) * V + v0 + cc, fmaf(skip, x.x, acc[t][2 * hh] + low[t][2 * hh]),
               fmaf(skip, x.y, acc[t][2 * hh + 1] + low[t][2 * hh + 1]), V - v0 - cc);
        }
    }
    if (owner) {
      const float gc = ex2(G[C - 1]);
#pragma unroll
      for (int t = 0; t < NC; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[t][e] *= gc;
#pragma unroll
      for (int ks = 0; ks < C / 16; ++ks) {
        uint32_t a[4];
        ldsm_x4_t(a, at_addr(sb_, PD, sm_t * 16, ks * 16, lane));
#pragma unroll
        for (int np = 0; np < NC / 2; ++np) {
          uint32_t x[4], y[4];
          ldsm_x4_t(x, bkn_addr(xh, PV, ks * 16, sc + np * 16, lane));
          ldsm_x4_t(y, bkn_addr(xl, PV, ks * 16, sc + np * 16, lane));
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            mma16816(S[2 * np + t], a, x[2 * t], x[2 * t + 1]);
            mma16816(S[2 * np + t], a, y[2 * t], y[2 * t + 1]);
          }
        }
      }
    }
    __syncthreads();   // P, the planes and this chunk's buffers have been read
  }
  if (!owner) return;
#pragma unroll
  for (int t = 0; t < NC; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = sm_t * 16 + g8 + 8 * (e >> 1), col = v0 + sc + t * 8 + t4 * 2 + (e & 1);
      if (row < D && col < V) Sg[(size_t)row * V + col] = S[t][e];
    }
}

template <typename K>
int prepare(K kernel, size_t smem) {
  return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) == cudaSuccess ? 0 : -4;
}

template <int DP>
int delta_go(const DeltaChunkParams& p, int chunks, int longs, cudaStream_t st) {
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (prepare(delta_prepare_kernel<DP>, sizeof(PrepSmem<DP>)) || prepare(delta_scan_kernel<DP>, sizeof(ScanSmem<DP>))) return -4;
    configured = true;
  }
  launch_k(delta_prepare_kernel<DP>, dim3((unsigned)chunks, (unsigned)p.H), dim3(PREP), sizeof(PrepSmem<DP>), st, true, p);
  launch_k(delta_scan_kernel<DP>, dim3((unsigned)longs, (unsigned)p.H, (unsigned)(p.Vp / VT)), dim3(THREADS), sizeof(ScanSmem<DP>), st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <int DP>
int ssd_go(const DeltaChunkParams& p, int longs, cudaStream_t st) {
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (prepare(ssd_chunk_kernel<DP>, sizeof(SsdSmem<DP>))) return -4;
    configured = true;
  }
  launch_k(ssd_chunk_kernel<DP>, dim3((unsigned)longs, (unsigned)p.H, (unsigned)((p.V + VT - 1) / VT)), dim3(THREADS), sizeof(SsdSmem<DP>), st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

bool recurrence_chunkable(int D, int V) { return D >= 1 && D <= 128 && V >= 1; }
size_t delta_chunk_elems(int D, int Vp) { return D <= 32 ? Ws<32>::elems(Vp) : D <= 64 ? Ws<64>::elems(Vp) : Ws<128>::elems(Vp); }

int delta_chunk_launch(const DeltaChunkParams& p, int chunks, int longs, cudaStream_t st) {
  if (chunks == 0 || longs == 0) return 0;
  if (!recurrence_chunkable(p.D, p.V) || p.H % p.Hk || p.Vp % VT || p.Vp < p.V) return -1;
  return p.D <= 32 ? delta_go<32>(p, chunks, longs, st) : p.D <= 64 ? delta_go<64>(p, chunks, longs, st) : delta_go<128>(p, chunks, longs, st);
}

int ssd_chunk_launch(const DeltaChunkParams& p, int longs, cudaStream_t st) {
  if (longs == 0) return 0;
  if (!recurrence_chunkable(p.D, p.V) || p.H % p.Hk) return -1;
  return p.D <= 32 ? ssd_go<32>(p, longs, st) : p.D <= 64 ? ssd_go<64>(p, longs, st) : ssd_go<128>(p, longs, st);
}

}  // namespace oc
