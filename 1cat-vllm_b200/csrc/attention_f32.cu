// Paged attention with fp32 queries, cache and arithmetic: causal, GQA, variable-length batches, sliding window with kept first tokens,
// soft cap, sinks, distance bias, output gate per head, separate or shared keys and values (see AttnParams). It is the full-precision
// form of the kernels in attention.cu for engines that run in 32 bits, written for exactness rather than speed. Differential attention
// (DIFF): rows (head, map) lie next to one another, so both maps of a head belong to one warp, which takes the difference and normalises it.
// Its bf16 form (bf16 in and out, fp32 arithmetic) serves rows that are wider than the tensor-core kernels' 256 columns.
//
// A CTA owns 16 (token, query head of the group) rows of one request and KV head; each of its four warps owns four of them. Tiles of 32
// keys stream through shared memory: a lane scores one key of the tile for each of the warp's rows, the online softmax is reduced over
// the lanes, and for the value product a lane owns the output columns lane, lane + 32, ...
#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

constexpr int kTile = 32, kRows = 16, kRowsPerWarp = 4;

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// NC: 32-column blocks of a value row that a lane owns one column of (row widths up to 32 * NC)
template <typename E, int NC, bool DIFF>
__global__ void __launch_bounds__(128) attn_f32_kernel(const AttnParams p) {
  extern __shared__ float sm[];
  __shared__ int s_req, s_row0;
  pdl_trigger();
  pdl_wait();
  const int D = p.D, G = p.Hq / p.Hkv, hkv = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pitch = D + 1;                       // odd: lanes of a warp read different keys of a column without bank conflicts when D is even
  const int QD = DIFF ? D / 2 : D;               // a map's queries see its half of the key columns
  float* sq = sm;                                // [kRows][QD]
  float* sk = sq + kRows * QD;                   // [kTile][pitch]
  float* sv = p.kv_shared ? sk : sk + kTile * pitch;
  if (threadIdx.x == 0) {
    int b = blockIdx.x, found = -1, r0 = 0;
    for (int i = 0; i < p.R; ++i) {
      const int nt = ((p.query_start_loc[i + 1] - p.query_start_loc[i]) * G + kRows - 1) / kRows;
      if (b < nt) { found = i; r0 = b * kRows; break; }
      b -= nt;
    }
    s_req = found;
    s_row0 = r0;
  }
  __syncthreads();
  const int r = s_req, row0 = s_row0;
  if (r < 0) return;
  const int qs = p.query_start_loc[r], qlen = p.query_start_loc[r + 1] - qs, S = p.seq_lens[r], ctx0 = S - qlen;
  const int nrows = min(kRows, qlen * G - row0);
  const int q_first = ctx0 + row0 / G, kv_end = min(S, ctx0 + (row0 + nrows - 1) / G + 1);
  const int* bt = p.block_table + (size_t)r * p.bt_stride;
  const E* cache = reinterpret_cast<const E*>(p.kv_cache);
  const size_t page = (size_t)p.bs * D, blk_stride = (size_t)(p.kv_shared ? 1 : 2) * p.Hkv * page;
  const E* q = reinterpret_cast<const E*>(p.q);

  for (int idx = threadIdx.x; idx < kRows * QD; idx += 128) {
    const int row = idx / QD, d = idx - row * QD, fr = row0 + row;
    sq[idx] = row < nrows ? ld(q + (size_t)(qs + fr / G) * p.q_st + (size_t)(hkv * G + fr % G) * p.q_sh + d) : 0.f;
  }
  float m[kRowsPerWarp], l[kRowsPerWarp], o[kRowsPerWarp][NC];
#pragma unroll
  for (int i = 0; i < kRowsPerWarp; ++i) {
    m[i] = -INFINITY;
    l[i] = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c) o[i][c] = 0.f;
  }
  // earliest key that a position sees (kept tokens aside)
  auto first_key = [&](int pos) {
    int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    return p.chunk > 0 ? max(lo, pos - pos % p.chunk) : lo;
  };
  const int ntiles = (kv_end + kTile - 1) / kTile;
  const int first = first_key(q_first) / kTile;
  const int keep_tiles = min((p.keep + kTile - 1) / kTile, first);
  for (int v = first - keep_tiles; v < ntiles; ++v) {
    const int k0 = (v < first ? v - (first - keep_tiles) : v) * kTile;
    __syncthreads();
    for (int idx = threadIdx.x; idx < kTile * D; idx += 128) {
      const int kr = idx / D, d = idx - kr * D, key = k0 + kr;
      float kx = 0.f, vx = 0.f;
      if (key < kv_end) {
        const E* src = cache + (size_t)bt[key >> p.bs_shift] * blk_stride + (size_t)hkv * page + (size_t)(key & (p.bs - 1)) * D + d;
        kx = ld(src);
        if (!p.kv_shared) vx = ld(src + (size_t)p.Hkv * page);
      }
      sk[kr * pitch + d] = kx;
      if (!p.kv_shared) sv[kr * pitch + d] = vx;
    }
    __syncthreads();
    float s[kRowsPerWarp] = {0.f, 0.f, 0.f, 0.f};
    const float* kp = sk + lane * pitch;
    const float* qp = sq + warp * kRowsPerWarp * QD;
    for (int d = 0; d < QD; ++d) {
      const float kx = kp[d], ky = DIFF ? kp[QD + d] : kx;   // odd rows are second maps
#pragma unroll
      for (int i = 0; i < kRowsPerWarp; ++i) s[i] = fmaf(qp[i * QD + d], (i & 1) ? ky : kx, s[i]);
    }
    const int key = k0 + lane;
#pragma unroll
    for (int i = 0; i < kRowsPerWarp; ++i) {
      const int fr = row0 + warp * kRowsPerWarp + i, qpos = ctx0 + fr / G;
      float x = s[i] * p.scale;
      if (p.softcap > 0.f) x = tanhf(x / p.softcap) * p.softcap;
      if (p.bias != nullptr) x += __ldg(p.bias + (size_t)(hkv * G + fr % G) * p.bias_len + min(max(qpos - key, 0), p.bias_len - 1));
      if (!(key <= qpos && key < kv_end && (key >= first_key(qpos) || key < p.keep))) x = -INFINITY;
      const float m_new = fmaxf(m[i], warp_max(x)), m_use = m_new == -INFINITY ? 0.f : m_new;
      const float alpha = expf(m[i] - m_use);
      s[i] = expf(x - m_use);
      l[i] = l[i] * alpha + warp_sum(s[i]);
      m[i] = m_new;
#pragma unroll
      for (int c = 0; c < NC; ++c) o[i][c] *= alpha;
    }
    for (int kr = 0; kr < kTile; ++kr) {
      float w[kRowsPerWarp];
#pragma unroll
      for (int i = 0; i < kRowsPerWarp; ++i) w[i] = __shfl_sync(0xffffffffu, s[i], kr);
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const int d = lane + 32 * c;
        if (d < D) {
          const float vx = sv[kr * pitch + d];
#pragma unroll
          for (int i = 0; i < kRowsPerWarp; ++i) o[i][c] = fmaf(w[i], vx, o[i][c]);
        }
      }
    }
  }
  if constexpr (DIFF) {
    const float lam = *p.lam;
#pragma unroll
    for (int i = 0; i < kRowsPerWarp; i += 2) {
      const int row = warp * kRowsPerWarp + i;
      if (row >= nrows) continue;
      const float ia = l[i] > 0.f ? 1.f / l[i] : 0.f, ib = l[i + 1] > 0.f ? lam / l[i + 1] : 0.f;
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        o[i][c] = lane + 32 * c < p.vdim ? o[i][c] * ia - o[i + 1][c] * ib : 0.f;
        ss = fmaf(o[i][c], o[i][c], ss);
      }
      const float f = p.out_scale / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
      const int fr = row0 + row;
      E* dst = reinterpret_cast<E*>(p.out) + ((size_t)(qs + fr / G) * (p.Hq / 2) + (hkv * G + fr % G) / 2) * p.vdim;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (lane + 32 * c < p.vdim) put(dst + lane + 32 * c, o[i][c] * f);
    }
  } else {
#pragma unroll
    for (int i = 0; i < kRowsPerWarp; ++i) {
      const int row = warp * kRowsPerWarp + i;
      if (row >= nrows) continue;
      const int fr = row0 + row, head = hkv * G + fr % G;
      const size_t tok = (size_t)(qs + fr / G);
      const float den = l[i] + (p.sinks != nullptr ? expf(p.sinks[head] - m[i]) : 0.f);
      float inv = den > 0.f ? 1.f / den : 0.f;
      if (p.gate != nullptr) inv *= 1.f / (1.f + expf(-ld(reinterpret_cast<const E*>(p.gate) + tok * p.gate_st + head)));
      E* dst = reinterpret_cast<E*>(p.out) + (tok * p.Hq + head) * D;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (lane + 32 * c < D) put(dst + lane + 32 * c, o[i][c] * inv);
      if (p.lse != nullptr && lane == 0) p.lse[tok * p.Hq + head] = m[i] + logf(l[i]);
    }
  }
}

// 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))), in place
__global__ void gelu_tanh_f32_kernel(float* x, long long n) {
  pdl_trigger();
  pdl_wait();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float z = x[i];
  x[i] = 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename E, int NC, bool DIFF>
int plain_go(const AttnParams& p, cudaStream_t st) {
  const int smem_max = (kRows * 32 * NC + 2 * kTile * (32 * NC + 1)) * 4;
  const int smem = (kRows * p.D + (p.kv_shared ? 1 : 2) * kTile * (p.D + 1)) * 4;
  static int configured_dev[kMaxDevices] = {};
  int& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (cudaFuncSetAttribute(attn_f32_kernel<E, NC, DIFF>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_max) != cudaSuccess) return -4;
    configured = 1;
  }
  if (p.num_q_tiles == 0) return 0;
  launch_k(attn_f32_kernel<E, NC, DIFF>, dim3((unsigned)p.num_q_tiles, (unsigned)p.Hkv), dim3(128), (size_t)smem, st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace

int attention_f32_launch(const AttnParams& p, bool bf16, cudaStream_t st) {
  if (p.Hq % p.Hkv || p.bs < 1 || (p.bs & (p.bs - 1)) || p.D < 1 || p.D > 512 || p.kv_fp8) return -1;
  if (p.bias != nullptr && p.bias_len < 1) return -1;
  if (p.maps == 2) {
    if (p.D % 2 || (p.Hq / p.Hkv) % 2 || p.vdim < 1 || p.vdim > p.D || p.lam == nullptr || p.kv_shared || p.bias != nullptr || p.gate != nullptr ||
        p.sinks != nullptr || p.lse != nullptr) return -1;
    if (bf16) return plain_go<__nv_bfloat16, 16, true>(p, st);
    return p.D <= 256 ? plain_go<float, 8, true>(p, st) : plain_go<float, 16, true>(p, st);
  }
  return bf16 || p.D > 256 ? -1 : plain_go<float, 8, false>(p, st);
}

int gelu_tanh_f32_launch(float* x, long long n, cudaStream_t st) {
  if (n == 0) return 0;
  launch_k(gelu_tanh_f32_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, true, x, n);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace oc
