// Differential attention, between the QKV projection and the attention kernel: every map of every query and key head is RMS-normalised
// and rotated in fp32, queries leave padded for the kernel, keys (both maps of a head side by side) and values go into their pages.
// A lane holds the pairs lane, lane + 32, ... of a row, so both elements of a rotated pair are in one thread.
#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

template <typename E> __device__ __forceinline__ float ld1(const E* p);
template <> __device__ __forceinline__ float ld1<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld1<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename E> __device__ __forceinline__ void st1(E* p, float v);
template <> __device__ __forceinline__ void st1<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void st1<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
// neighbours (2i, 2i + 1) as one access
__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ld2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void st2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }

// A warp takes kRows neighbouring (head, map) rows of one token - all their loads are in flight before the first reduction - or one value row.
// NP: pairs per lane and row. VEC: rows have an even number of elements and start on pairs.
constexpr int kRows = 4;
template <typename E, int NP, bool VEC>
__global__ void __launch_bounds__(256) diff_prepare_kernel(const DiffPrepareParams p) {
  pdl_trigger();
  pdl_wait();
  const int maps = 2 * (p.H + p.G), groups = (maps + kRows - 1) / kRows, units = groups + p.G, lane = threadIdx.x & 31;
  const unsigned wid = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int t = (int)(wid / (unsigned)units), unit = (int)(wid - (unsigned)t * units);
  if (t >= p.T) return;
  const E* x = reinterpret_cast<const E*>(p.x) + (size_t)t * p.ld;
  const int hd = p.D / 2, slot = p.slots[t];
  auto cache_row = [&](int which, int g) {
    return reinterpret_cast<E*>(p.cache) + ((((size_t)(slot / p.bs) * 2 + which) * p.G + g) * p.bs + slot % p.bs) * p.D;
  };
  if (unit >= groups) {
    if (slot < 0) return;
    const int g = unit - groups;
    const E* v = x + (size_t)maps * p.dim + (size_t)g * p.vdim;
    E* dst = cache_row(1, g);
    if (VEC) {
      for (int c = lane * 2; c < p.D; c += 64) st2(dst + c, c < p.vdim ? ld2(v + c) : make_float2(0.f, 0.f));
    } else {
      for (int c = lane; c < p.D; c += 32) st1<E>(dst + c, c < p.vdim ? ld1<E>(v + c) : 0.f);
    }
    return;
  }
  const int u0 = unit * kRows, half = p.rot / 2, pairs = (p.dim + 1) / 2;
  // elements of pair i: neighbours, or (i, i + rot / 2) inside the rotated part of the half-split layout
  const bool split = !VEC || !p.interleaved;
  auto first = [&](int i) { return p.interleaved || i >= half ? 2 * i : i; };
  auto second = [&](int i) { return p.interleaved || i >= half ? 2 * i + 1 : i + half; };
  float2 v[kRows][NP], cs[NP];
#pragma unroll
  for (int r = 0; r < kRows; ++r)   // queries and keys follow one another
#pragma unroll
    for (int k = 0; k < NP; ++k) {
      const int i = lane + 32 * k;
      const E* row = x + (size_t)(u0 + r) * p.dim;
      v[r][k] = make_float2(0.f, 0.f);
      if (i < pairs && u0 + r < maps) {
        if (split) {
          v[r][k].x = ld1<E>(row + first(i));
          if (second(i) < p.dim) v[r][k].y = ld1<E>(row + second(i));
        } else {
          v[r][k] = ld2(row + 2 * i);
        }
      }
    }
  const float* angles = p.cos_sin + (size_t)p.positions[t] * p.rot;
#pragma unroll
  for (int k = 0; k < NP; ++k) {
    const int i = lane + 32 * k;
    cs[k] = i < half ? make_float2(angles[i], angles[half + i]) : make_float2(1.f, 0.f);
  }
  float ss[kRows];
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    ss[r] = 0.f;
#pragma unroll
    for (int k = 0; k < NP; ++k) ss[r] = fmaf(v[r][k].x, v[r][k].x, fmaf(v[r][k].y, v[r][k].y, ss[r]));
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int r = 0; r < kRows; ++r) ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], o);
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const int u = u0 + r, kv = u - 2 * p.H;
    if (u >= maps || (kv >= 0 && slot < 0)) continue;
    const E* w = reinterpret_cast<const E*>(kv < 0 ? p.q_w : p.k_w);
    E* dst = kv < 0 ? reinterpret_cast<E*>(p.q_out) + ((size_t)t * 2 * p.H + u) * hd : cache_row(0, kv >> 1) + (kv & 1) * hd;
    const float inv = 1.f / sqrtf(ss[r] / (float)p.dim + p.eps);
#pragma unroll
    for (int k = 0; k < NP; ++k) {
      const int i = lane + 32 * k;
      if (i >= pairs) continue;
      const int e0 = first(i), e1 = second(i);
      float2 wv;
      if (split) wv = make_float2(ld1<E>(w + e0), e1 < p.dim ? ld1<E>(w + e1) : 0.f);
      else wv = make_float2(ld1<E>(w + 2 * i), ld1<E>(w + 2 * i + 1));
      const float a0 = v[r][k].x * inv * wv.x, b0 = v[r][k].y * inv * wv.y;
      const float a = i < half ? a0 * cs[k].x - b0 * cs[k].y : a0, b = i < half ? b0 * cs[k].x + a0 * cs[k].y : b0;
      if (split) {
        st1<E>(dst + e0, a);
        if (e1 < p.dim) st1<E>(dst + e1, b);
      } else {
        st2(dst + 2 * i, make_float2(a, b));
      }
    }
    for (int c = p.dim + lane; c < hd; c += 32) st1<E>(dst + c, 0.f);
  }
}

template <typename E>
int prepare_e(const DiffPrepareParams& p, cudaStream_t st) {
  const long long warps = (long long)p.T * ((2 * (p.H + p.G) + kRows - 1) / kRows + p.G);
  if (warps >= (1ll << 31)) return -1;
  const uintptr_t pair = 2 * sizeof(E);
  auto ok = [&](const void* q) { return ((uintptr_t)q & (pair - 1)) == 0; };
  const bool vec = p.dim % 2 == 0 && p.vdim % 2 == 0 && p.D % 4 == 0 && p.ld % 2 == 0 && ok(p.x) && ok(p.q_out) && ok(p.cache);
  auto go = [&](auto kernel) { launch_k(kernel, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0, st, true, p); };
  if (p.dim <= 64) vec ? go(diff_prepare_kernel<E, 1, true>) : go(diff_prepare_kernel<E, 1, false>);
  else if (p.dim <= 128) vec ? go(diff_prepare_kernel<E, 2, true>) : go(diff_prepare_kernel<E, 2, false>);
  else if (p.dim <= 512) vec ? go(diff_prepare_kernel<E, 8, true>) : go(diff_prepare_kernel<E, 8, false>);
  else return -1;
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

int diff_prepare_launch(const DiffPrepareParams& p, cudaStream_t st) {
  if (p.T == 0) return 0;
  if (p.dim < 1 || p.D < 2 * p.dim || p.D < p.vdim || p.D % 2 || p.rot % 2 || p.rot > p.dim || p.bs < 1) return -1;
  return p.f32 ? prepare_e<float>(p, st) : prepare_e<__nv_bfloat16>(p, st);
}

}  // namespace oc
