// Mixture-of-experts plumbing around the grouped tcgen05 GEMM: count tokens per local expert, lay the (token, expert) pairs out
// expert-major ("slots"), build the GEMM work lists on the device, gather activations into slot order, and combine the expert
// outputs back per token with the routing weights. Nothing here needs the host to know how tokens were routed, so a whole MoE
// layer is a fixed sequence of launches (CUDA-graph friendly).
//   count -> plan (1 CTA: prefix sum + work lists for both GEMMs) -> scatter (slot assignment + gather of X rows)
//   -> grouped GEMM w13 with SiLU*mul epilogue -> grouped GEMM w2 -> combine (weighted sum over each token's experts)
// With expert parallelism a rank owns experts [e_off, e_off + E_local); pairs routed elsewhere get slot -1 and contribute nothing,
// so the layer output is a partial sum that the tensor-parallel reduction completes.
// (reference: csrc/moe/moe_align_sum_kernels.cu:22-456, moe_permute_unpermute_op.cu:240; layers/fused_moe/modular_kernel.py:1236-1461)
#include <type_traits>

#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

__global__ void moe_count_kernel(const int* __restrict__ ids, int n_pairs, int e_off, int E, int* __restrict__ counts) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n_pairs) return;
  const int e = ids[i] - e_off;
  if (e >= 0 && e < E) atomicAdd(&counts[e], 1);
}

// One CTA. offsets[e] = first slot of expert e; work lists for GEMM 1 (n1 row tiles per expert) and GEMM 2 (n2 row tiles).
__global__ void __launch_bounds__(1024) moe_plan_kernel(MoePlanParams p) {
  __shared__ int s_off[1025];
  const int E = p.E;
  if (threadIdx.x == 0) {
    int acc = 0;
    for (int e = 0; e < E; ++e) { s_off[e] = acc; acc += p.counts[e]; }
    s_off[E] = acc;
    p.total_slots[0] = acc;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) p.offsets[e] = s_off[e];
  for (int e = threadIdx.x; e < E; e += blockDim.x) p.cursor[e] = 0;
  // item base per expert for both lists (sequential scan by thread 0; E <= 1024)
  __shared__ int s_tiles[1025];
  if (threadIdx.x == 0) {
    int acc = 0;
    for (int e = 0; e < E; ++e) { s_tiles[e] = acc; acc += (p.counts[e] + p.tn - 1) / p.tn; }
    s_tiles[E] = acc;
    p.work_count[0] = acc * p.n1;
    p.work_count[1] = acc * p.n2;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int cnt = p.counts[e], tt0 = s_tiles[e], ntt = s_tiles[e + 1] - tt0;
    for (int tt = 0; tt < ntt; ++tt) {
      const int t0 = s_off[e] + tt * p.tn, rows = min(p.tn, cnt - tt * p.tn);
      for (int n = 0; n < p.n1; ++n) p.work1[(size_t)(tt0 + tt) * p.n1 + n] = make_int4(e * p.n1 + n, t0, rows, n * 128);
      for (int n = 0; n < p.n2; ++n) p.work2[(size_t)(tt0 + tt) * p.n2 + n] = make_int4(e * p.n2 + n, t0, rows, n * 128);
    }
  }
}

template <typename E> __device__ __forceinline__ float ldf(const E* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename E> __device__ __forceinline__ E from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// One warp per (token, j) pair: claim a slot in the pair's expert, remember it, copy the token's activation row there (rows of Hp >= H
// elements, zeros past H). W: the unit of the copy, 16 bytes or one element.
template <typename W>
__global__ void moe_scatter_kernel(const int* __restrict__ ids, int n_pairs, int k, int e_off, int E, const int* __restrict__ offsets,
                                   int* __restrict__ cursor, int* __restrict__ slot_of, const W* __restrict__ x, long long ldx,
                                   W* __restrict__ xs, int H, int Hp) {
  const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (pair >= n_pairs) return;
  const int lane = threadIdx.x & 31;
  const int e = ids[pair] - e_off;
  int slot = -1;
  if (e >= 0 && e < E) {
    if (lane == 0) slot = offsets[e] + atomicAdd(&cursor[e], 1);
    slot = __shfl_sync(0xffffffffu, slot, 0);
  }
  if (lane == 0) slot_of[pair] = slot;
  if (slot < 0) return;
  const W* src = x + (size_t)(pair / k) * ldx;
  W* dst = xs + (size_t)slot * Hp;
  for (int i = lane; i < H; i += 32) dst[i] = src[i];
  for (int i = H + lane; i < Hp; i += 32) dst[i] = W{};
}

// y[t] = sum_j w[t, j] * a2[slot_of[t, j]]   (fixed j order: bit-stable), N columns per thread
template <typename E, int N>
__global__ void moe_combine_kernel(const E* __restrict__ a2, int lda, const int* __restrict__ slot_of, const float* __restrict__ w,
                                   E* __restrict__ y, int T, int k, int H) {
  struct alignas(sizeof(E) * N) Vec { E e[N]; };
  const int t = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * N;
  if (c >= H) return;
  float acc[N];
#pragma unroll
  for (int i = 0; i < N; ++i) acc[i] = 0.f;
  for (int j = 0; j < k; ++j) {
    const int slot = slot_of[t * k + j];
    if (slot < 0) continue;
    const float wj = w[t * k + j];
    const Vec v = *reinterpret_cast<const Vec*>(a2 + (size_t)slot * lda + c);
#pragma unroll
    for (int i = 0; i < N; ++i) acc[i] += wj * ldf<E>(&v.e[i]);
  }
  Vec o;
#pragma unroll
  for (int i = 0; i < N; ++i) o.e[i] = from_f<E>(acc[i]);
  *reinterpret_cast<Vec*>(y + (size_t)t * H + c) = o;
}

// fp32 grouped product for engines that run in 32 bits: 64 x 64 output tiles, 16 input columns at a time through shared memory, a 4 x 4
// block per thread. Work items are those of the tensor-core kernel (128 weight rows of an expert x a run of slots).
template <bool SILU>
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ w, float* __restrict__ out, int N,
                                                           int K, const int4* __restrict__ work, const int* __restrict__ work_count, int n_tiles) {
  __shared__ float sx[16][65], sw[16][65];
  const int tid = threadIdx.x, ti = tid >> 4, tj = tid & 15, items = work_count[0];
  for (int item = blockIdx.x; item < items; item += gridDim.x) {
    const int4 it = work[item];   // {row tile over all experts, first slot, slots, first row inside the expert}
    const float* we = w + (size_t)(it.x / n_tiles) * N * K;
    for (int s0 = 0; s0 < it.z; s0 += 64)
      for (int n0 = it.w; n0 < min(it.w + 128, N); n0 += 64) {
        float acc[4][4] = {};
        for (int k0 = 0; k0 < K; k0 += 16) {
          __syncthreads();
          for (int e = tid; e < 64 * 16; e += 256) {
            const int i = e >> 4, kk = e & 15, k = k0 + kk;
            float a = 0.f, b = 0.f;
            if (k < K && s0 + i < it.z) {
              const float* src = x + (size_t)(it.y + s0 + i) * ldx + k;
              a = SILU ? src[0] / (1.f + expf(-src[0])) * src[K] : src[0];
            }
            if (k < K && n0 + i < N) b = we[(size_t)(n0 + i) * K + k];
            sx[kk][i] = a;
            sw[kk][i] = b;
          }
          __syncthreads();
#pragma unroll
          for (int kk = 0; kk < 16; ++kk)
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
              for (int b = 0; b < 4; ++b) acc[a][b] = fmaf(sx[kk][ti + 16 * a], sw[kk][tj + 16 * b], acc[a][b]);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
          for (int b = 0; b < 4; ++b)
            if (s0 + ti + 16 * a < it.z && n0 + tj + 16 * b < N) out[(size_t)(it.y + s0 + ti + 16 * a) * N + n0 + tj + 16 * b] = acc[a][b];
      }
  }
}

}  // namespace

int moe_prepare_launch(const MoePlanParams& p, const int* ids, int n_pairs, int k, int e_off, int* slot_of, const void* x, long long ldx,
                       void* xs, int H, int Hp, int f32, cudaStream_t st) {
  if (p.E > 1024 || Hp < H) return -1;
  if (cudaMemsetAsync(p.counts, 0, sizeof(int) * p.E, st) != cudaSuccess) return -2;
  if (n_pairs > 0) moe_count_kernel<<<(n_pairs + 255) / 256, 256, 0, st>>>(ids, n_pairs, e_off, p.E, p.counts);
  moe_plan_kernel<<<1, 1024, 0, st>>>(p);
  if (n_pairs > 0) {
    const int per = f32 ? 4 : 8;   // elements of a 16-byte unit
    const dim3 grid((n_pairs + 7) / 8);
    if (H % per == 0 && Hp % per == 0 && ldx % per == 0 && (((uintptr_t)x | (uintptr_t)xs) & 15) == 0)
      moe_scatter_kernel<uint4><<<grid, 256, 0, st>>>(ids, n_pairs, k, e_off, p.E, p.offsets, p.cursor, slot_of, (const uint4*)x, ldx / per, (uint4*)xs, H / per, Hp / per);
    else if (f32)
      moe_scatter_kernel<uint32_t><<<grid, 256, 0, st>>>(ids, n_pairs, k, e_off, p.E, p.offsets, p.cursor, slot_of, (const uint32_t*)x, ldx, (uint32_t*)xs, H, Hp);
    else
      moe_scatter_kernel<unsigned short><<<grid, 256, 0, st>>>(ids, n_pairs, k, e_off, p.E, p.offsets, p.cursor, slot_of, (const unsigned short*)x, ldx,
                                                               (unsigned short*)xs, H, Hp);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

int moe_gemm_f32_launch(const float* x, int ldx, const float* w, float* out, int N, int K, int silu, const int4* work, const int* work_count, int n_tiles,
                        int num_sms, cudaStream_t st) {
  if (silu) moe_gemm_f32_kernel<true><<<4 * num_sms, 256, 0, st>>>(x, ldx, w, out, N, K, work, work_count, n_tiles);
  else moe_gemm_f32_kernel<false><<<4 * num_sms, 256, 0, st>>>(x, ldx, w, out, N, K, work, work_count, n_tiles);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

// Work lists only, from counts that are already on the device (expert-parallel exchange: the rows arrive in slot order).
int moe_plan_launch(const MoePlanParams& p, cudaStream_t st) {
  if (p.E > 1024) return -1;
  moe_plan_kernel<<<1, 1024, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

int moe_combine_launch(const void* a2, int lda, const int* slot_of, const float* w, void* y, int T, int k, int H, int f32, cudaStream_t st) {
  if (T == 0) return 0;
  auto go = [&](auto kernel, auto* typed, int n) {
    using E = std::remove_pointer_t<decltype(typed)>;
    kernel<<<dim3(((H + n - 1) / n + 127) / 128, T), 128, 0, st>>>((const E*)a2, lda, slot_of, w, (E*)y, T, k, H);
  };
  const int per = f32 ? 4 : 8;
  const bool vec = H % per == 0 && lda % per == 0 && (((uintptr_t)a2 | (uintptr_t)y) & 15) == 0;
  if (f32) {
    if (vec) go(moe_combine_kernel<float, 4>, (float*)nullptr, 4);
    else go(moe_combine_kernel<float, 1>, (float*)nullptr, 1);
  } else {
    if (vec) go(moe_combine_kernel<__nv_bfloat16, 8>, (__nv_bfloat16*)nullptr, 8);
    else go(moe_combine_kernel<__nv_bfloat16, 1>, (__nv_bfloat16*)nullptr, 1);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

unsigned int moe_read_status(bool clear) { return read_status_tu(clear); }
void moe_read_status_async(unsigned int* dst, cudaStream_t st) { read_status_tu_async(dst, st); }

}  // namespace oc
