// Linear recurrences with a matrix state S [D][V] per (sequence, head), fp32, and the gated norm behind them.
//   channel delta:  g = exp(-exp(A) softplus(a + b0)) per key channel, beta = sigmoid(b), q and k unit vectors, q times D^-1/2
//                   S <- g S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q
//   Mamba-2:        dt = softplus(dt + b0) within limits, g = exp(-exp(A) dt);  S <- g S + B (dt x)^T;  o = S^T C + Dskip x
// Recurrent kernel (decoding, short portions, fp32 engines): a CTA owns 32 state columns of one (sequence, head); a column is split over four lanes,
// which keep their rows in registers for the whole portion. Inputs of a few tokens are staged in shared memory together.
#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

template <typename E> __device__ __forceinline__ float to_f(E v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename E> __device__ __forceinline__ E from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

constexpr int VC = 32, NP = 4, THREADS = VC * NP;

// RT: rows of a column per lane (D up to 4 * RT)
template <typename E, bool DELTA, int RT>
__global__ void __launch_bounds__(THREADS, RT == 64 ? 2 : RT == 32 ? 6 : 8) recurrent_kernel(const RecurrenceParams p) {
  constexpr int DP = RT * NP, CH = RT == 64 ? 8 : 16;
  __shared__ __align__(16) float sq[CH][DP], sk[CH][DP];
  __shared__ __align__(16) float sg[DELTA ? CH : 1][DP];
  __shared__ float sv[CH][VC], sdec[CH], sbeta[CH];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * VC;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int lc = warp * 8 + (lane & 7), col = c0 + lc, part = lane >> 3;
  const int t0 = p.query_start_loc[r], t1 = p.query_start_loc[r + 1];
  if (t1 <= t0 || (p.skip_min_len > 0 && t1 - t0 >= p.skip_min_len)) return;
  const int hk = h / (p.H / p.Hk), D = p.D, V = p.V;
  float* Sg = p.state + ((size_t)p.state_slots[r] * p.H + h) * D * V;
  const bool init = p.has_initial_state[r] != 0, mine = col < V;
  float S[RT];
  const bool whole = D == DP && c0 + VC <= V;   // no padding in this CTA's rows and columns
  float* mineg = Sg + (size_t)part * RT * V + col;
  if (whole && init) {
#pragma unroll
    for (int k = 0; k < RT; ++k) S[k] = mineg[(size_t)k * V];
  } else {
#pragma unroll
    for (int k = 0; k < RT; ++k) S[k] = init && mine && part * RT + k < D ? mineg[(size_t)k * V] : 0.f;
  }
  const float nega = -expf(p.A_log[h]);
  const float skip = DELTA ? 0.f : p.skip[h], dt_bias = DELTA ? 0.f : p.dt_bias[h];
  for (int tc = t0; tc < t1; tc += CH) {
    const int n = min(CH, t1 - tc);
    __syncthreads();   // the previous tokens' rows have been read
    if (tid < n) {
      const float z = to_f<E>(reinterpret_cast<const E*>(p.b)[(size_t)(tc + tid) * p.ld_b + h]);
      if (DELTA) sbeta[tid] = 1.f / (1.f + expf(-z));
      else {
        const float dt = fminf(fmaxf(softplus(z + dt_bias), p.dt_min), p.dt_max);
        sbeta[tid] = dt;
        sdec[tid] = expf(nega * dt);
      }
    }
    for (int i = warp; i < n; i += THREADS / 32) {
      const size_t t = tc + i;
      const E* q = reinterpret_cast<const E*>(p.q) + t * p.ld + (size_t)hk * D;
      const E* k = reinterpret_cast<const E*>(p.k) + t * p.ld + (size_t)hk * D;
      float qv[DP / 32], kv[DP / 32], q2 = 0.f, k2 = 0.f;
#pragma unroll
      for (int e = 0; e < DP / 32; ++e) {
        const int d = lane + 32 * e;
        qv[e] = d < D ? to_f<E>(q[d]) : 0.f;
        kv[e] = d < D ? to_f<E>(k[d]) : 0.f;
        q2 = fmaf(qv[e], qv[e], q2);
        k2 = fmaf(kv[e], kv[e], k2);
        if (DELTA) {
          const size_t ch = (size_t)h * D + d;
          sg[i][d] = d < D ? expf(nega * softplus(p.a[t * p.ld_a + ch] + p.dt_bias[ch])) : 0.f;
        }
      }
      float fq = 1.f, fk = 1.f;
      if (DELTA) {
        fq = 1.f / sqrtf(warp_sum(q2) + 1e-6f) * p.scale;
        fk = 1.f / sqrtf(warp_sum(k2) + 1e-6f);
      }
#pragma unroll
      for (int e = 0; e < DP / 32; ++e) {
        sq[i][lane + 32 * e] = qv[e] * fq;
        sk[i][lane + 32 * e] = kv[e] * fk;
      }
      sv[i][lane] = c0 + lane < V ? to_f<E>(reinterpret_cast<const E*>(p.v)[t * p.ld + (size_t)h * V + c0 + lane]) : 0.f;
    }
    __syncthreads();
#pragma unroll 1
    for (int i = 0; i < n; ++i) {
      const float beta = sbeta[i], v = sv[i][lc];
      const float4* k4 = reinterpret_cast<const float4*>(&sk[i][part * RT]);
      const float4* q4 = reinterpret_cast<const float4*>(&sq[i][part * RT]);
      float u, o[4] = {0.f, 0.f, 0.f, 0.f};
      if (DELTA) {
        const float4* g4 = reinterpret_cast<const float4*>(&sg[i][part * RT]);
        float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int k = 0; k < RT; k += 4) {
          const float4 kk = k4[k >> 2], gg = g4[k >> 2];
          S[k] *= gg.x; S[k + 1] *= gg.y; S[k + 2] *= gg.z; S[k + 3] *= gg.w;
          a[0] = fmaf(kk.x, S[k], a[0]); a[1] = fmaf(kk.y, S[k + 1], a[1]); a[2] = fmaf(kk.z, S[k + 2], a[2]); a[3] = fmaf(kk.w, S[k + 3], a[3]);
        }
        float s = (a[0] + a[1]) + (a[2] + a[3]);
        s += __shfl_xor_sync(0xffffffffu, s, 8);
        s += __shfl_xor_sync(0xffffffffu, s, 16);
        u = beta * (v - s);
      } else {
        const float dec = sdec[i];
        u = beta * v;
#pragma unroll
        for (int k = 0; k < RT; ++k) S[k] *= dec;
      }
#pragma unroll
      for (int k = 0; k < RT; k += 4) {
        const float4 kk = k4[k >> 2], qq = q4[k >> 2];
        S[k] = fmaf(kk.x, u, S[k]); S[k + 1] = fmaf(kk.y, u, S[k + 1]); S[k + 2] = fmaf(kk.z, u, S[k + 2]); S[k + 3] = fmaf(kk.w, u, S[k + 3]);
        o[0] = fmaf(qq.x, S[k], o[0]); o[1] = fmaf(qq.y, S[k + 1], o[1]); o[2] = fmaf(qq.z, S[k + 2], o[2]); o[3] = fmaf(qq.w, S[k + 3], o[3]);
      }
      float y = (o[0] + o[1]) + (o[2] + o[3]);
      y += __shfl_xor_sync(0xffffffffu, y, 8);
      y += __shfl_xor_sync(0xffffffffu, y, 16);
      if (!DELTA) y = fmaf(skip, v, y);
      if (part == 0 && mine) reinterpret_cast<E*>(p.out)[((size_t)(tc + i) * p.H + h) * V + col] = from_f<E>(y);
    }
  }
  int W = V;   // opaque: the rows' addresses are computed again rather than kept in registers since the loads
  asm volatile("" : "+r"(W));
  if (whole) {
#pragma unroll
    for (int k = 0; k < RT; ++k) mineg[(size_t)k * W] = S[k];
  } else {
#pragma unroll
    for (int k = 0; k < RT; ++k)
      if (mine && part * RT + k < D) mineg[(size_t)k * W] = S[k];
  }
}

template <typename E, bool DELTA>
int recurrent_go(const RecurrenceParams& p, cudaStream_t st) {
  const dim3 grid((unsigned)p.R, (unsigned)p.H, (unsigned)((p.V + VC - 1) / VC));
  auto run = [&](auto kernel) { launch_k(kernel, grid, dim3(THREADS), 0, st, true, p); };
  if (p.D <= 32) run(recurrent_kernel<E, DELTA, 8>);
  else if (p.D <= 64) run(recurrent_kernel<E, DELTA, 16>);
  else if (p.D <= 128) run(recurrent_kernel<E, DELTA, 32>);
  else if (p.D <= 256) run(recurrent_kernel<E, DELTA, 64>);
  else return -1;
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// LANES lanes own a part of a row and keep it in registers: IT vectors of N elements each. Parts of at least LANES == 32 vectors take a warp, wide
// ones (LANES == 256) a CTA; parts that are wider still are read twice.
template <typename E> __device__ __forceinline__ float sigmoid(float x);
template <> __device__ __forceinline__ float sigmoid<float>(float x) { return 1.f / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float sigmoid<__nv_bfloat16>(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

template <typename E, int N, int LANES, int IT>
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedNormParams p) {
  struct alignas(sizeof(E) * N) Vec { E e[N]; };
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x % LANES, n = p.n / p.groups;
  const long long item = (long long)blockIdx.x * (256 / LANES) + threadIdx.x / LANES;
  const bool live = item < (long long)p.T * p.groups;
  const size_t t = live ? item / p.groups : 0;
  const int g = live ? (int)(item % p.groups) : 0;
  const E* x = reinterpret_cast<const E*>(p.x) + t * p.ld_x + (size_t)g * n;
  const E* z = reinterpret_cast<const E*>(p.gate) + t * p.ld_g + (size_t)g * n;
  const E* w = reinterpret_cast<const E*>(p.w) + (p.w_shared ? 0 : (size_t)g * n);
  E* y = reinterpret_cast<E*>(p.y) + t * p.n + (size_t)g * n;
  float v[IT][N], s[IT][N], ss = 0.f;
  auto value = [&](int c, float (&a)[N], float (&b)[N]) {   // what is normalised, and the factor behind the norm
    const Vec vx = *reinterpret_cast<const Vec*>(x + c), vz = *reinterpret_cast<const Vec*>(z + c);
#pragma unroll
    for (int j = 0; j < N; ++j) {
      const float q = to_f<E>(vz.e[j]), sg = sigmoid<E>(q);
      a[j] = to_f<E>(vx.e[j]) * (p.gate_first ? q * sg : 1.f);
      b[j] = p.gate_first ? 1.f : sg;
    }
  };
  auto total = [&](float a) {
#pragma unroll
    for (int o = (LANES < 32 ? LANES : 32) / 2; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
    if (LANES > 32) {
      if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = a;
      __syncthreads();
      a = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) a += red[i];
    }
    return a;
  };
  auto write = [&](int c, const float (&a)[N], const float (&b)[N], float inv) {
    const Vec vw = *reinterpret_cast<const Vec*>(w + c);
    Vec o;
#pragma unroll
    for (int j = 0; j < N; ++j) o.e[j] = from_f<E>(a[j] * inv * to_f<E>(vw.e[j]) * b[j]);
    *reinterpret_cast<Vec*>(y + c) = o;
  };
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int c = (i * LANES + lane) * N;
    if (live && c < n) {
      value(c, v[i], s[i]);
#pragma unroll
      for (int j = 0; j < N; ++j) ss = fmaf(v[i][j], v[i][j], ss);
    }
  }
  float a[N], b[N];
  for (int c = (IT * LANES + lane) * N; live && c < n; c += LANES * N) {
    value(c, a, b);
#pragma unroll
    for (int j = 0; j < N; ++j) ss = fmaf(a[j], a[j], ss);
  }
  const float inv = 1.f / sqrtf(total(ss) / (float)n + p.eps);
  if (!live) return;
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int c = (i * LANES + lane) * N;
    if (c < n) write(c, v[i], s[i], inv);
  }
  for (int c = (IT * LANES + lane) * N; c < n; c += LANES * N) {
    value(c, a, b);
    write(c, a, b, inv);
  }
}

template <typename E, int N>
int gated_norm_go(const GatedNormParams& p, cudaStream_t st) {
  const long long items = (long long)p.T * p.groups;
  const int vecs = (p.n / p.groups + N - 1) / N;
  auto run = [&](auto kernel, int lanes) { launch_k(kernel, dim3((unsigned)((items * lanes + 255) / 256)), dim3(256), 0, st, true, p); };
  if (vecs <= 8) run(gated_norm_kernel<E, N, 8, 1>, 8);
  else if (vecs <= 16) run(gated_norm_kernel<E, N, 16, 1>, 16);
  else if (vecs <= 32) run(gated_norm_kernel<E, N, 32, 1>, 32);
  else if (vecs <= 64) run(gated_norm_kernel<E, N, 32, 2>, 32);
  else if (vecs <= 128) run(gated_norm_kernel<E, N, 32, 4>, 32);
  else run(gated_norm_kernel<E, N, 256, 2>, 256);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

int recurrence_launch(const RecurrenceParams& p, cudaStream_t st) {
  if (p.T == 0 || p.R == 0) return 0;
  if (p.H % p.Hk || p.D < 1 || p.V < 1) return -1;
  if (p.delta) return p.f32 ? recurrent_go<float, true>(p, st) : recurrent_go<__nv_bfloat16, true>(p, st);
  return p.f32 ? recurrent_go<float, false>(p, st) : recurrent_go<__nv_bfloat16, false>(p, st);
}

int gated_norm_launch(const GatedNormParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  if (p.groups < 1 || p.n % p.groups) return -1;
  const int n = p.n / p.groups;
  const int v = p.f32 ? 4 : 8;   // elements of a 16-byte vector
  auto ok = [&](const void* q) { return ((uintptr_t)q & 15) == 0; };
  const bool vec = n % v == 0 && p.n % v == 0 && p.ld_x % v == 0 && p.ld_g % v == 0 && ok(p.x) && ok(p.gate) && ok(p.w) && ok(p.y);
  if (p.f32) return vec ? gated_norm_go<float, 4>(p, st) : gated_norm_go<float, 1>(p, st);
  return vec ? gated_norm_go<__nv_bfloat16, 8>(p, st) : gated_norm_go<__nv_bfloat16, 1>(p, st);
}

}  // namespace oc
