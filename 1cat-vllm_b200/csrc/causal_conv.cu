// Causal convolution per channel over variable-length batches with a rolling per-sequence state, optional bias, SiLU and residual add.
//   y[t, c] = act(b[c] + sum_j w[c, j] x[t - (taps - 1) + j, c]) (+ x[t, c]); inputs ahead of a portion come from state[slot][j][c] (j = 0 oldest).
// A thread owns a few channels and walks a tile of consecutive tokens with the last taps - 1 inputs in registers, so an input is read once per
// tile. The thread that processes a portion's first token has read the old state, and it writes the new one; the taps - 1 tokens that still
// look into the old state belong to the same thread, whatever tile they fall into, so nobody reads what it overwrites.
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

template <typename E, int N> struct alignas(sizeof(E) * N) Vec { E e[N]; };
template <typename E, int N>
__device__ __forceinline__ void load_vec(const E* p, float (&v)[N]) {
  const Vec<E, N> t = *reinterpret_cast<const Vec<E, N>*>(p);
#pragma unroll
  for (int j = 0; j < N; ++j) v[j] = to_f<E>(t.e[j]);
}
template <typename E, int N>
__device__ __forceinline__ void store_vec(E* p, const float (&v)[N]) {
  Vec<E, N> t;
#pragma unroll
  for (int j = 0; j < N; ++j) t.e[j] = from_f<E>(v[j]);
  *reinterpret_cast<Vec<E, N>*>(p) = t;
}

constexpr int kMaxTaps = 16, kTile = 8;   // most taps; tokens per tile of a long step

// TAPS 0: any number of taps up to kMaxTaps
template <typename E, int N, int TAPS>
__global__ void __launch_bounds__(128) causal_conv_kernel(const CausalConvParams p, int tile) {
  constexpr int KT = TAPS ? TAPS : kMaxTaps;
  pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * N;
  if (c >= p.C) return;
  const int taps = TAPS ? TAPS : p.taps, m = taps - 1;
  const int start = blockIdx.y * tile, stop = min(start + tile, p.T);
  const int* qsl = p.query_start_loc;
  int lo = 0, hi = p.R;   // qsl[lo] <= start < qsl[hi]
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (qsl[mid] <= start) lo = mid; else hi = mid;
  }
  int r = lo, t0 = qsl[r], t1 = qsl[r + 1];
  const E* x = reinterpret_cast<const E*>(p.x) + c;
  E* state = reinterpret_cast<E*>(p.state) + c;
  float w[KT][N], b[N], h[KT][N];   // h[j]: the input j + 1 tokens back
  E wt[N * KT];   // [channel][tap]: a few vector loads where the taps are whole vectors
  if constexpr (TAPS == 4 && N > 1) {
#pragma unroll
    for (int i = 0; i < TAPS; ++i) *reinterpret_cast<Vec<E, N>*>(wt + i * N) = *reinterpret_cast<const Vec<E, N>*>(reinterpret_cast<const E*>(p.w) + (size_t)c * 4 + i * N);
  } else {
#pragma unroll
    for (int e = 0; e < N * KT; ++e)
      if (e < N * taps) wt[e] = reinterpret_cast<const E*>(p.w)[(size_t)c * taps + e];
  }
#pragma unroll
  for (int j = 0; j < KT; ++j)
    if (j < taps) {
#pragma unroll
      for (int e = 0; e < N; ++e) w[j][e] = to_f<E>(wt[e * taps + j]);
    }
#pragma unroll
  for (int e = 0; e < N; ++e) b[e] = 0.f;
  if (p.bias != nullptr) load_vec<E, N>(reinterpret_cast<const E*>(p.bias) + c, b);

  const int rows = m > 0 ? m : 1;
  auto history = [&](int t) {   // the m inputs ahead of token t of request r
    const E* st = state + (size_t)p.state_slots[r] * rows * p.C;
    const bool init = p.has_initial_state[r] != 0;
#pragma unroll
    for (int j = 0; j < KT - 1; ++j)
      if (j < m) {
        const int tt = t - 1 - j;
        if (tt >= t0) load_vec<E, N>(x + (size_t)tt * p.ldx, h[j]);
        else if (init) load_vec<E, N>(st + (size_t)(m + tt - t0) * p.C, h[j]);
        else {
#pragma unroll
          for (int e = 0; e < N; ++e) h[j][e] = 0.f;
        }
      }
  };
  // A whole tile inside a portion, away from its first tokens: all rows are loaded before the first one is used.
  if constexpr (TAPS > 0 && N > 1) {
    if (start - t0 >= m && stop <= t1 && stop - start == kTile) {
      Vec<E, N> raw[kTile + TAPS - 1];
#pragma unroll
      for (int i = 0; i < kTile + TAPS - 1; ++i) raw[i] = *reinterpret_cast<const Vec<E, N>*>(x + (size_t)(start - (TAPS - 1) + i) * p.ldx);
#pragma unroll
      for (int i = 0; i < kTile; ++i) {
        float y[N];
#pragma unroll
        for (int e = 0; e < N; ++e) {
          y[e] = b[e];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) y[e] = fmaf(w[j][e], to_f<E>(raw[i + j].e[e]), y[e]);
          if (p.silu) y[e] = y[e] * (p.f32 ? 1.f / (1.f + expf(-y[e])) : __fdividef(1.f, 1.f + __expf(-y[e])));
          if (p.residual) y[e] += to_f<E>(raw[i + TAPS - 1].e[e]);
        }
        store_vec<E, N>(reinterpret_cast<E*>(p.y) + (size_t)(start + i) * p.C + c, y);
      }
      return;
    }
  }
  int t = start;
  if (t > t0 && t - t0 < m) t = min(t1, t0 + m);   // these belong to the thread of the portion's first token
  bool fresh = true;
  while (true) {
    while (r < p.R && t >= t1) {
      ++r;
      if (r < p.R) { t0 = t1; t1 = qsl[r + 1]; }
      fresh = true;
    }
    if (r >= p.R || t >= p.T) break;
    if (t >= stop && !(t0 >= start && t0 < stop && t - t0 < m)) break;
    if (fresh) {
      history(t);
      fresh = false;
      if (t == t0 && m > 0) {
        E* st = state + (size_t)p.state_slots[r] * rows * p.C;
        const int n = t1 - t0;
        float v[KT][N];
#pragma unroll
        for (int j = 0; j < KT - 1; ++j)
          if (j < m) {
            const int idx = n - m + j;
            if (idx >= 0) load_vec<E, N>(x + (size_t)(t0 + idx) * p.ldx, v[j]);
            else {
#pragma unroll
              for (int i = 0; i < KT - 1; ++i)   // the input -idx tokens ahead of the portion
                if (i == -idx - 1) {
#pragma unroll
                  for (int e = 0; e < N; ++e) v[j][e] = h[i][e];
                }
            }
          }
#pragma unroll
        for (int j = 0; j < KT - 1; ++j)
          if (j < m) store_vec<E, N>(st + (size_t)j * p.C, v[j]);
      }
    }
    float cur[N], y[N];
    load_vec<E, N>(x + (size_t)t * p.ldx, cur);
#pragma unroll
    for (int e = 0; e < N; ++e) y[e] = b[e];
#pragma unroll
    for (int j = KT - 2; j >= 0; --j)
      if (j < m) {
#pragma unroll
        for (int i = 0; i < KT; ++i)
          if (i == m - 1 - j) {
#pragma unroll
            for (int e = 0; e < N; ++e) y[e] = fmaf(w[i][e], h[j][e], y[e]);
          }
      }
#pragma unroll
    for (int i = 0; i < KT; ++i)
      if (i == m) {
#pragma unroll
        for (int e = 0; e < N; ++e) y[e] = fmaf(w[i][e], cur[e], y[e]);
      }
    if (p.silu) {
#pragma unroll
      for (int e = 0; e < N; ++e) y[e] = y[e] / (1.f + (p.f32 ? expf(-y[e]) : __expf(-y[e])));
    }
    if (p.residual) {
#pragma unroll
      for (int e = 0; e < N; ++e) y[e] += cur[e];
    }
    store_vec<E, N>(reinterpret_cast<E*>(p.y) + (size_t)t * p.C + c, y);
#pragma unroll
    for (int j = KT - 2; j > 0; --j) {
#pragma unroll
      for (int e = 0; e < N; ++e) h[j][e] = h[j - 1][e];
    }
#pragma unroll
    for (int e = 0; e < N; ++e) h[0][e] = cur[e];
    ++t;
  }
}

template <typename E, int N>
int go(const CausalConvParams& p, cudaStream_t st) {
  const int threads = 128, tile = p.T <= 2048 ? 1 : kTile;
  const dim3 grid((unsigned)((p.C / N + threads - 1) / threads), (unsigned)((p.T + tile - 1) / tile));
  auto run = [&](auto kernel) { launch_k(kernel, grid, dim3(threads), 0, st, true, p, tile); };
  if (p.taps == 4) run(causal_conv_kernel<E, N, 4>);
  else if (p.taps == 3) run(causal_conv_kernel<E, N, 3>);
  else if (p.taps == 2) run(causal_conv_kernel<E, N, 2>);
  else run(causal_conv_kernel<E, 1, 0>);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

int causal_conv_launch(const CausalConvParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  if (p.taps < 1 || p.taps > kMaxTaps || p.C < 1 || p.R < 1) return -1;
  const int n = p.f32 ? 4 : 8;
  auto ok = [&](const void* q) { return ((uintptr_t)q & 15) == 0; };
  const bool vec = p.taps >= 2 && p.taps <= 4 && p.C % n == 0 && p.ldx % n == 0 && ok(p.x) && ok(p.y) && ok(p.state) && ok(p.bias) && ok(p.w);
  if (p.f32) return vec ? go<float, 4>(p, st) : go<float, 1>(p, st);
  return vec ? go<__nv_bfloat16, 8>(p, st) : go<__nv_bfloat16, 1>(p, st);
}

}  // namespace oc
