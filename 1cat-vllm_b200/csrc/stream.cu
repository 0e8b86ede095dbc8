// Kernels around the fp32 residual stream and the un-rotated paged cache.
//   stream_join: x' = x + mul * scale * post(part) (+ add), y = next(x'): a sub-block's output is normalised, scaled, added to the stream and the
//                sum normalised for the next sub-block in one pass; optionally x' also leaves in the model's element type.
//   embed_stream: the stream's start from scaled token embeddings and hashed-bigram rows or learned position rows.
//   kv_insert:   key (and value) rows into their pages.
#include <type_traits>

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

__device__ __forceinline__ float block_total(float v, float* red) {
  v = warp_sum(v);
  const int nw = blockDim.x >> 5;
  if (nw == 1) return v;
  __syncthreads();                       // the previous total has been read
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += red[i];   // same order in every thread
  return t;
}

// One CTA per token. A thread holds elements (it * blockDim + tid) * N .. + N - 1 in registers; the variance is taken over the deviations
// from the mean (two passes over registers).
template <typename E, typename PE, int N, int IT>
__global__ void __launch_bounds__(256) stream_join_kernel(const StreamJoinParams p) {
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int H = p.H;
  const PE* part = reinterpret_cast<const PE*>(p.part) + t * p.ld_part;
  float v[IT][N];
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * N;
    if (c < H) load_vec<PE, N>(part + c, v[i]);
  }
  auto normalise = [&](const StreamNorm& n) {
    if (n.kind == 3) {   // dynamic tanh: no statistics
      const float al = to_f<E>(*reinterpret_cast<const E*>(n.alpha));
#pragma unroll
      for (int i = 0; i < IT; ++i) {
        const int c = (i * blockDim.x + threadIdx.x) * N;
        if (c < H) {
          float w[N], b[N];
          load_vec<E, N>(reinterpret_cast<const E*>(n.w) + c, w);
          load_vec<E, N>(reinterpret_cast<const E*>(n.b) + c, b);
#pragma unroll
          for (int j = 0; j < N; ++j) v[i][j] = fmaf(tanhf(al * v[i][j]), w[j], b[j]);
        }
      }
      return;
    }
    float mean = 0.f;
    if (n.kind == 2) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < IT; ++i)
        if ((i * blockDim.x + threadIdx.x) * N < H) {
#pragma unroll
          for (int j = 0; j < N; ++j) s += v[i][j];
        }
      mean = block_total(s, red) / (float)H;
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < IT; ++i)
      if ((i * blockDim.x + threadIdx.x) * N < H) {
#pragma unroll
        for (int j = 0; j < N; ++j) {
          v[i][j] -= mean;
          ss = fmaf(v[i][j], v[i][j], ss);
        }
      }
    const float inv = 1.f / sqrtf(block_total(ss, red) / (float)H + n.eps);
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * N;
      if (c < H) {
        float w[N], b[N];
        if (n.w != nullptr) load_vec<E, N>(reinterpret_cast<const E*>(n.w) + c, w);
        if (n.b != nullptr) load_vec<E, N>(reinterpret_cast<const E*>(n.b) + c, b);
#pragma unroll
        for (int j = 0; j < N; ++j) {
          float y = v[i][j] * inv;
          if (n.w != nullptr) y *= n.plus_one ? 1.f + w[j] : w[j];
          v[i][j] = n.b != nullptr ? y + b[j] : y;
        }
      }
    }
  };
  if (p.post.kind != 0) normalise(p.post);
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * N;
    if (c < H) {
      float a[N];
      if (p.scale != nullptr) {
        load_vec<E, N>(reinterpret_cast<const E*>(p.scale) + c, a);
#pragma unroll
        for (int j = 0; j < N; ++j) v[i][j] *= a[j];
      }
      if (p.mul != 1.f) {
#pragma unroll
        for (int j = 0; j < N; ++j) v[i][j] *= p.mul;
      }
      if (p.add != nullptr) {
        load_vec<E, N>(reinterpret_cast<const E*>(p.add) + c, a);
#pragma unroll
        for (int j = 0; j < N; ++j) v[i][j] += a[j];
      }
      if (p.x_in != nullptr) {
        load_vec<float, N>(p.x_in + t * H + c, a);
#pragma unroll
        for (int j = 0; j < N; ++j) v[i][j] += a[j];
      }
      store_vec<float, N>(p.x_out + t * H + c, v[i]);
      if (p.copy_out != nullptr) store_vec<E, N>(reinterpret_cast<E*>(p.copy_out) + t * p.ld_copy + c, v[i]);
    }
  }
  if (p.next.kind == 0) return;
  normalise(p.next);
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * N;
    if (c < H) store_vec<E, N>(reinterpret_cast<E*>(p.y) + t * H + c, v[i]);
  }
}

template <typename E, typename PE, int N>
int stream_join_n(const StreamJoinParams& p, cudaStream_t st) {
  const int vecs = (p.H + N - 1) / N;
  int threads = ((vecs + 31) / 32) * 32;
  if (threads > 256) threads = 256;
  const int it = (vecs + threads - 1) / threads;
  auto go = [&](auto kernel) { launch_k(kernel, dim3((unsigned)p.T), dim3((unsigned)threads), 0, st, true, p); };
  if (it <= 1) go(stream_join_kernel<E, PE, N, 1>);
  else if (it <= 2) go(stream_join_kernel<E, PE, N, 2>);
  else if (it <= 4) go(stream_join_kernel<E, PE, N, 4>);
  else if (it <= 8) go(stream_join_kernel<E, PE, N, 8>);
  else if (it <= 32 && N == 1) go(stream_join_kernel<E, PE, N, N == 1 ? 32 : 8>);
  else return -1;
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename E, int N>
__global__ void __launch_bounds__(256) embed_stream_kernel(const EmbedParams p) {
  pdl_trigger();
  pdl_wait();
  const size_t t = blockIdx.x;
  const int id = p.ids[t];
  const E* row = reinterpret_cast<const E*>(p.table) + (p.gathered ? t : (size_t)min(max(id, 0), p.vocab - 1)) * p.H;
  const E* big = nullptr;
  if (p.bigram != nullptr) {
    const int prev = p.prev[t];
    const long long h = prev < 0 ? p.buckets : ((long long)prev * p.mul_prev + (long long)id * p.mul_cur) % p.buckets;
    big = reinterpret_cast<const E*>(p.bigram) + (h < 0 ? h + p.buckets : h) * p.H;
  }
  for (int c = threadIdx.x * N; c < p.H; c += blockDim.x * N) {
    float v[N], b[N];
    load_vec<E, N>(row + c, v);
    if (big != nullptr) load_vec<E, N>(big + c, b);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = big != nullptr ? fmaf(v[j], p.scale, b[j]) : v[j] * p.scale;
    if (p.rows != nullptr) {
      load_vec<E, N>(reinterpret_cast<const E*>(p.rows) + (size_t)min(max(p.positions[t], 0), p.num_rows - 1) * p.H + c, b);
#pragma unroll
      for (int j = 0; j < N; ++j) v[j] += b[j];
    }
    store_vec<float, N>(p.x + t * p.H + c, v);
    if (p.y != nullptr) store_vec<E, N>(reinterpret_cast<E*>(p.y) + t * p.H + c, v);
  }
}

template <typename W>
__global__ void __launch_bounds__(256) kv_insert_kernel(const KvInsertParams p) {
  pdl_trigger();
  pdl_wait();
  const int per = p.row_bytes / (int)sizeof(W), tensors = p.v != nullptr ? 2 : 1;
  const long long total = (long long)p.T * tensors * p.H * per;
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const int w = (int)(i % per);
  const long long hh = i / per;
  const int h = (int)(hh % p.H), kv = (int)((hh / p.H) % tensors), t = (int)(hh / p.H / tensors);
  const int slot = p.slot_mapping[t];
  if (slot < 0) return;
  const char* src = (kv == 0 ? p.k + (size_t)t * p.k_st : p.v + (size_t)t * p.v_st) + (size_t)h * p.row_bytes;
  const size_t row = (((size_t)(slot / p.bs) * tensors + kv) * p.H + h) * p.bs + slot % p.bs;
  reinterpret_cast<W*>(p.cache + row * p.row_bytes)[w] = reinterpret_cast<const W*>(src)[w];
}

}  // namespace

int stream_join_launch(const StreamJoinParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  auto incomplete = [](const StreamNorm& n) { return n.kind == 3 && (n.w == nullptr || n.b == nullptr || n.alpha == nullptr); };
  if (incomplete(p.post) || incomplete(p.next)) return -1;
  if (p.H < 1 || p.x_out == nullptr || (p.next.kind != 0 && p.y == nullptr) || (p.f32 && !p.part_f32)) return -1;
  // vectors of four elements when every row starts on a vector boundary
  const uintptr_t esz = p.f32 ? 4 : 2, psz = p.part_f32 ? 4 : 2;
  auto ok = [](const void* q, uintptr_t a) { return ((uintptr_t)q & (a - 1)) == 0; };
  const bool vec = p.H % 4 == 0 && p.ld_part % 4 == 0 && (p.copy_out == nullptr || p.ld_copy % 4 == 0) && ok(p.part, 4 * psz) && ok(p.x_in, 16) &&
                   ok(p.x_out, 16) && ok(p.y, 4 * esz) && ok(p.copy_out, 4 * esz) && ok(p.scale, 4 * esz) && ok(p.add, 4 * esz) &&
                   ok(p.post.w, 4 * esz) && ok(p.post.b, 4 * esz) && ok(p.next.w, 4 * esz) && ok(p.next.b, 4 * esz);
  if (p.f32) return vec ? stream_join_n<float, float, 4>(p, st) : stream_join_n<float, float, 1>(p, st);
  if (p.part_f32) return vec ? stream_join_n<__nv_bfloat16, float, 4>(p, st) : stream_join_n<__nv_bfloat16, float, 1>(p, st);
  return vec ? stream_join_n<__nv_bfloat16, __nv_bfloat16, 4>(p, st) : stream_join_n<__nv_bfloat16, __nv_bfloat16, 1>(p, st);
}

int embed_stream_launch(const EmbedParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  if (p.H < 1 || p.vocab < 1 || (p.bigram != nullptr && (p.prev == nullptr || p.buckets < 1)) ||
      (p.rows != nullptr && (p.positions == nullptr || p.num_rows < 1))) return -1;
  const uintptr_t a = p.f32 ? 16 : 8;
  auto ok = [](const void* q, uintptr_t n) { return ((uintptr_t)q & (n - 1)) == 0; };
  const bool vec = p.H % 4 == 0 && ok(p.table, a) && ok(p.bigram, a) && ok(p.rows, a) && ok(p.x, 16) && ok(p.y, a);
  int threads = ((vec ? (p.H + 3) / 4 : p.H) + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  auto go = [&](auto kernel) { launch_k(kernel, dim3((unsigned)p.T), dim3((unsigned)threads), 0, st, true, p); };
  if (p.f32) vec ? go(embed_stream_kernel<float, 4>) : go(embed_stream_kernel<float, 1>);
  else vec ? go(embed_stream_kernel<__nv_bfloat16, 4>) : go(embed_stream_kernel<__nv_bfloat16, 1>);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

int kv_insert_launch(const KvInsertParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  auto fits = [&](long long n) {
    return p.row_bytes % n == 0 && p.k_st % n == 0 && p.v_st % n == 0 && ((uintptr_t)p.k % n) == 0 && ((uintptr_t)p.v % n) == 0 &&
           ((uintptr_t)p.cache % n) == 0;
  };
  auto go = [&](auto kernel, int n) {
    const long long total = (long long)p.T * (p.v != nullptr ? 2 : 1) * p.H * (p.row_bytes / n);
    launch_k(kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st, true, p);
  };
  if (fits(16)) go(kv_insert_kernel<uint4>, 16);
  else if (fits(4)) go(kv_insert_kernel<uint32_t>, 4);
  else if (fits(2)) go(kv_insert_kernel<unsigned short>, 2);
  else return -1;
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace oc
