// Talking-heads attention over a paged cache whose rows are keys and values at once.
//   s_h(i, j) = (q_h(i) . k(j)) f(j) - r1_h ln(1 + r2_h (i - j)),  a_h = softmax_j s_h,  o_h = sum_j (sum_g T[h, g] a_g(i, j)) k(j)
// q carries the norms' weights, the score's scale and the temperature; f(j) is the row's RMS factor, cached beside the pages.
//
//   talk_prepare: query norm, gain and temperature, key rows and their factors into the cache, one CTA per token.
//   talk_plain:   any head sizes, fp32 or bf16 in and out, fp32 arithmetic; one CTA per token, two walks over the keys (the mix needs the weights
//                 normalised, so the first walk finds every head's maximum and sum).
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

__device__ __forceinline__ float block_total(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += red[i];
  return t;
}

template <typename E, int N>
__global__ void __launch_bounds__(256) talk_prepare_kernel(const TalkPrepareParams p) {
  struct alignas(sizeof(E) * N) Vec { E e[N]; };
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int nq = p.H * p.dim, nk = p.G * p.dim;
  const E* q = reinterpret_cast<const E*>(p.qk) + t * p.ld;
  const E* k = q + nq;
  float qq = 0.f, kk = 0.f;
  auto square = [&](const E* row, int n) {
    float s = 0.f;
    for (int c = threadIdx.x * N; c < n; c += blockDim.x * N) {
      const Vec v = *reinterpret_cast<const Vec*>(row + c);
#pragma unroll
      for (int j = 0; j < N; ++j) s = fmaf(to_f<E>(v.e[j]), to_f<E>(v.e[j]), s);
    }
    return s;
  };
  qq = block_total(square(q, nq), red);
  kk = block_total(square(k, nk), red);
  float f = 1.f / sqrtf(qq / (float)nq + p.eps);
  if (p.every > 0) f *= 1.f + p.coef * logf((float)((p.positions[t] + 1) / p.every) + 1.f);
  E* qo = reinterpret_cast<E*>(p.q_out) + t * p.H * p.row;
  const int per = p.row / N;
  for (int i = threadIdx.x; i < p.H * per; i += blockDim.x) {
    const int d = i % per * N, head = i / per;
    Vec o;
    if (d < p.dim) {
      const Vec v = *reinterpret_cast<const Vec*>(q + head * p.dim + d);
#pragma unroll
      for (int j = 0; j < N; ++j) o.e[j] = from_f<E>(to_f<E>(v.e[j]) * f * p.gain[head * p.dim + d + j]);
    } else {
#pragma unroll
      for (int j = 0; j < N; ++j) o.e[j] = from_f<E>(0.f);
    }
    *reinterpret_cast<Vec*>(qo + (size_t)head * p.row + d) = o;
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  const int blk = slot / p.bs, at = slot % p.bs;
  for (int i = threadIdx.x; i < p.G * per; i += blockDim.x) {
    const int d = i % per * N, g = i / per;
    Vec v;
    if (d < p.dim) v = *reinterpret_cast<const Vec*>(k + g * p.dim + d);
    else {
#pragma unroll
      for (int j = 0; j < N; ++j) v.e[j] = from_f<E>(0.f);
    }
    *reinterpret_cast<Vec*>(reinterpret_cast<E*>(p.pages) + (((size_t)blk * p.G + g) * p.bs + at) * p.row + d) = v;
  }
  if (threadIdx.x == 0) p.k_scale[(size_t)blk * p.bs + at] = 1.f / sqrtf(kk / (float)nk + p.eps);
}

constexpr int kPlainThreads = 256;

__host__ __device__ inline size_t plain_smem_floats(int H, int G, int D, int kt) {
  return (size_t)kt * (G * (D + 1)) + 2 * (size_t)H * D + 2 * (size_t)H * kt + 2 * H + kt;
}

template <typename E>
__global__ void __launch_bounds__(kPlainThreads) talk_plain_kernel(const TalkParams p, int kt) {
  extern __shared__ float sm[];
  const int H = p.H, G = p.G, D = p.dim, share = H / G, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pitch = D + 1;
  float* sk = sm;                              // [kt][G][D + 1]
  float* sq = sk + (size_t)kt * G * pitch;     // [H][D]
  float* so = sq + H * D;                      // [H][D]
  float* sp = so + H * D;                      // [H][kt] weights
  float* sx = sp + H * kt;                     // [H][kt] mixed weights
  float* smx = sx + H * kt;                    // [H] maximum, then [H] sum
  float* ssum = smx + H;
  float* sf = ssum + H;                        // [kt]
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  int r = 0;
  {
    int lo = 0, hi = p.R;
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.query_start_loc[mid] <= t) lo = mid; else hi = mid;
    }
    r = lo;
  }
  if (t >= p.query_start_loc[p.R]) return;
  const int qs = p.query_start_loc[r], qlen = p.query_start_loc[r + 1] - qs, pos = p.seq_lens[r] - qlen + (t - qs);
  const int* bt = p.block_table + (size_t)r * p.bt_stride;
  for (int i = threadIdx.x; i < H * D; i += kPlainThreads) {
    sq[i] = to_f<E>(reinterpret_cast<const E*>(p.q)[(size_t)t * H * D + i]);
    so[i] = 0.f;
  }
  for (int i = threadIdx.x; i < H; i += kPlainThreads) {
    smx[i] = -INFINITY;
    ssum[i] = 0.f;
  }
  const int keys = pos + 1;
  for (int pass = 0; pass < 2; ++pass) {
    for (int k0 = 0; k0 < keys; k0 += kt) {
      __syncthreads();
      for (int i = threadIdx.x; i < kt * G * D; i += kPlainThreads) {
        const int d = i % D, g = i / D % G, kr = i / (D * G), key = k0 + kr;
        float v = 0.f;
        if (key < keys)
          v = to_f<E>(reinterpret_cast<const E*>(p.pages)[(((size_t)bt[key / p.bs] * G + g) * p.bs + key % p.bs) * D + d]);
        sk[(kr * G + g) * pitch + d] = v;
      }
      if ((int)threadIdx.x < kt) {
        const int key = k0 + threadIdx.x;
        sf[threadIdx.x] = key < keys ? p.k_scale[(size_t)bt[key / p.bs] * p.bs + key % p.bs] : 0.f;
      }
      __syncthreads();
      for (int h = warp; h < H; h += kPlainThreads / 32) {
        const int key = k0 + lane;
        const bool live = lane < kt && key < keys;
        float s = -INFINITY;
        if (live) {
          const float* kp = sk + (lane * G + h / share) * pitch;
          const float* qp = sq + h * D;
          float a = 0.f;
          for (int d = 0; d < D; ++d) a = fmaf(qp[d], kp[d], a);
          s = a * sf[lane] - p.bias[h] * logf(fmaf(p.bias[H + h], (float)(pos - key), 1.f));
        }
        if (pass == 0) {
          const float m = smx[h], nm = fmaxf(m, warp_max(s));
          const float sum = warp_sum(live ? expf(s - nm) : 0.f);
          __syncwarp();
          if (lane == 0) {
            smx[h] = nm;
            ssum[h] = ssum[h] * expf(m - nm) + sum;
          }
          __syncwarp();
        } else if (lane < kt) {
          sp[h * kt + lane] = live ? expf(s - smx[h]) / ssum[h] : 0.f;
        }
      }
      if (pass == 0) continue;
      __syncthreads();
      for (int i = threadIdx.x; i < H * kt; i += kPlainThreads) {
        const int h = i / kt, kr = i % kt;
        float a = 0.f;
        for (int g = 0; g < H; ++g) a = fmaf(to_f<E>(reinterpret_cast<const E*>(p.mix)[h * H + g]), sp[g * kt + kr], a);
        sx[i] = a;
      }
      __syncthreads();
      for (int i = threadIdx.x; i < H * D; i += kPlainThreads) {
        const int h = i / D, d = i % D;
        float a = so[i];
        for (int kr = 0; kr < kt; ++kr) a = fmaf(sx[h * kt + kr], sk[(kr * G + h / share) * pitch + d], a);
        so[i] = a;
      }
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < H * D; i += kPlainThreads) reinterpret_cast<E*>(p.out)[(size_t)t * H * D + i] = from_f<E>(so[i]);
}

template <typename E>
int plain_go(const TalkParams& p, cudaStream_t st) {
  const size_t most = 227 * 1024;
  int kt = 32;
  while (kt > 4 && plain_smem_floats(p.H, p.G, p.dim, kt) * 4 > most) kt /= 2;
  const size_t smem = plain_smem_floats(p.H, p.G, p.dim, kt) * 4;
  if (smem > most) return -3;
  static int configured_dev[kMaxDevices] = {};
  int& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (cudaFuncSetAttribute(talk_plain_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)most) != cudaSuccess) return -4;
    configured = 1;
  }
  launch_k(talk_plain_kernel<E>, dim3((unsigned)p.T), dim3(kPlainThreads), smem, st, true, p, kt);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace

int talk_prepare_launch(const TalkPrepareParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  if (p.H < 1 || p.G < 1 || p.H % p.G || p.row < p.dim || p.bs < 1) return -1;
  const int n = p.f32 ? 4 : 8;
  auto ok = [&](const void* q) { return ((uintptr_t)q & 15) == 0; };
  const bool vec = p.dim % n == 0 && p.row % n == 0 && p.ld % n == 0 && ok(p.qk) && ok(p.q_out) && ok(p.pages);
  auto go = [&](auto kernel) { launch_k(kernel, dim3((unsigned)p.T), dim3(256), 0, st, true, p); };
  if (p.f32) vec ? go(talk_prepare_kernel<float, 4>) : go(talk_prepare_kernel<float, 1>);
  else vec ? go(talk_prepare_kernel<__nv_bfloat16, 8>) : go(talk_prepare_kernel<__nv_bfloat16, 1>);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

int talk_plain_launch(const TalkParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  if (p.H < 1 || p.G < 1 || p.H % p.G || p.dim < 1 || p.bs < 1 || p.R < 1) return -1;
  return p.f32 ? plain_go<float>(p, st) : plain_go<__nv_bfloat16>(p, st);
}

}  // namespace oc
