// Talking-heads attention of single tokens (bf16 queries and cache, fp32 scores and weights), and the mix over heads for both tensor-core kernels.
// Definitions in talk_attention.cu.
//
// The mix is linear, so it may follow the value products: with O_g the product of head g's weights with the rows of ALL key heads,
// o_h = sum_g T[h, g] O_g[columns of h's own key head] / sum_g. The keys are read once, the heads' softmax stays independent (running maximum, partial
// results of key splits merge as usual), and what is mixed is one row per head instead of one weight per key.
//   talk_decode: one CTA per (request, split of the keys). A tile of keys, all key heads, serves both products:
//     scores S^T [keys][heads of the key head] = K Q^T;   weights per head, lanes over keys;   O [heads][all columns] += P K, accumulators in registers.
//   talk_join:   merges the splits, divides by the sums and mixes; one CTA per token.
// Weights enter the value product as two bf16 terms.
#include "kernels.h"
#include "mma_sync.cuh"

namespace oc {
namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr int MT = 512, WARPS = MT / 32;

__device__ __forceinline__ void ldsm_x2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
}
__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct Geom {   // sizes of the shared-memory areas, in elements
  int tg, nt, rows, ps, pp;   // tiles of eight heads per key head and in all; rows of the value product; pitches of the scores and weights
  size_t k, q, s, p;
};
__host__ __device__ inline Geom geom(int H, int G, int dp, int kt) {
  Geom m;
  m.tg = (H / G + 7) / 8;
  m.nt = G * m.tg;
  m.rows = (H + 15) / 16 * 16;
  m.ps = kt + 4;
  m.pp = kt + 8;
  m.k = (size_t)G * kt * (dp + 8);
  m.q = (size_t)m.nt * 8 * (dp + 8);
  m.s = (size_t)m.nt * 8 * m.ps;
  m.p = (size_t)m.rows * m.pp;
  return m;
}
inline size_t smem_bytes(const Geom& m, int H, int kt) { return (2 * m.k + m.q + 2 * m.p) * 2 + (m.s + 2 * kt + m.rows + 2 * H) * 4 + 64; }

// KT keys a tile; MH tiles of 16 heads; NTC pairs of eight-column tiles per warp
template <int DP, int KT, int MH, int NTC>
__global__ void __launch_bounds__(MT) talk_decode_kernel(const TalkTcParams p) {
  constexpr int PD = DP + 8, KL = (KT + 31) / 32, MTS = KT / 16;
  extern __shared__ __align__(16) uint8_t raw[];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, r = blockIdx.x, split = blockIdx.y;
  const int H = p.t.H, G = p.t.G, share = H / G, bs = p.bs_shift, bsm = p.t.bs - 1, GD = G * DP;
  const int qs = p.t.query_start_loc[r], n = p.t.query_start_loc[r + 1] - qs;
  if (n != 1) return;
  const Geom m = geom(H, G, DP, KT);
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(raw);   // [2][G][KT][PD]
  __nv_bfloat16* sq = sk + 2 * m.k;                            // [nt * 8][PD]
  __nv_bfloat16* sp = sq + m.q;                                // [2][rows][pp]
  float* ss = reinterpret_cast<float*>(sp + 2 * m.p);          // [nt * 8][ps] scores
  float* sf = ss + m.s;                                        // [2][KT]
  float* sal = sf + 2 * KT;                                    // [rows] what the tile scales earlier results by
  int* moved = reinterpret_cast<int*>(sal + m.rows);           // last tile that scales anything
  const int keys = p.t.seq_lens[r], tiles = (keys + KT - 1) / KT;
  const int each = (tiles + p.splits - 1) / p.splits, first = split * each, last = min(tiles, first + each);
  const int* bt = p.t.block_table + (size_t)r * p.t.bt_stride;
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.t.q) + (size_t)qs * H * DP;
  const __nv_bfloat16* pages = reinterpret_cast<const __nv_bfloat16*>(p.t.pages);
  for (int e = tid; e < m.nt * 8 * (DP / 8); e += MT) {
    const int c = e % (DP / 8) * 8, row = e / (DP / 8), g = row / (8 * m.tg), h = row % (8 * m.tg);
    const bool live = h < share;
    cp_async16(smem_u32(sq + row * PD + c), q + (size_t)(live ? g * share + h : 0) * DP + c, live ? 16 : 0);
  }
  for (int i = tid; i < (int)(2 * m.p); i += MT) sp[i] = __float2bfloat16(0.f);
  for (int i = tid; i < m.rows; i += MT) sal[i] = 1.f;
  if (tid == 0) *moved = -1;
  auto fetch = [&](int tile) {
    if (tile < last) {
      constexpr int RPI = MT / (DP / 8);   // rows of the tile that the threads copy at a time
      const int st = tile & 1, c = tid % (DP / 8) * 8;
#pragma unroll
      for (int k0 = 0; k0 < KT; k0 += RPI) {
        const int row = k0 + tid / (DP / 8);
        if (row >= KT) break;
        const int key = tile * KT + row, at = key < keys ? key : 0, bytes = key < keys ? 16 : 0;
        const __nv_bfloat16* src = pages + ((((size_t)bt[at >> bs] * G) << bs) + (at & bsm)) * DP + c;
        uint32_t dst = smem_u32(sk + st * m.k) + (uint32_t)((row * PD + c) * 2);
        for (int g = 0; g < G; ++g) {
          cp_async16(dst, src, bytes);
          dst += KT * PD * 2;
          src += (size_t)DP << bs;
        }
      }
      if (tid < KT) {
        const int key = tile * KT + tid, at = key < keys ? key : 0;
        cp_async4(smem_u32(sf + st * KT + tid), p.t.k_scale + ((size_t)bt[at >> bs] << bs) + (at & bsm), key < keys ? 4 : 0);
      }
    }
    cp_async_commit();
  };
  fetch(first);

  float acc[MH][NTC][2][4];
#pragma unroll
  for (int a = 0; a < MH; ++a)
#pragma unroll
    for (int b = 0; b < NTC; ++b)
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[a][b][t][e] = 0.f;
  const int col0 = warp * NTC * 16;   // this warp's columns of all key heads' rows
  // heads warp, warp + 16, ...: reference of the exponents (it moves when a score exceeds it by 2^8), this lane's part of the sum
  constexpr int HW = MH;
  float mx[HW], l[HW], r1[HW], r2[HW];
  int srow[HW];
#pragma unroll
  for (int i = 0; i < HW; ++i) {
    const int h = warp + i * WARPS;
    mx[i] = -INFINITY;
    l[i] = 0.f;
    r1[i] = h < H ? p.t.bias[h] : 0.f;
    r2[i] = h < H ? p.t.bias[H + h] : 0.f;
    srow[i] = h < H ? (h / share) * m.tg * 8 + h % share : 0;
  }
  const uint32_t aq = smem_u32(sq), ap = smem_u32(sp), plane = (uint32_t)(m.p * 2);
  const uint32_t lane_q = (uint32_t)(((lane & 7) * PD + ((lane >> 3) & 1) * 8) * 2), lane_k = a_addr(0, PD, 0, 0, lane);

  for (int tile = first; tile < last; ++tile) {
    const int st = tile & 1;
    cp_async_wait<0>();
    __syncthreads();   // the tile is there, and every warp is done with the previous one
    fetch(tile + 1);
    const uint32_t ak = smem_u32(sk + st * m.k);
    for (int u = warp; u < m.nt * MTS; u += WARPS) {
      const int t = u / MTS, mt = u % MTS, g = t / m.tg;
      const uint32_t ka = ak + (uint32_t)((g * KT + mt * 16) * PD * 2) + lane_k, qa = aq + (uint32_t)(t * 8 * PD * 2) + lane_q;
      float sa[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) sa[i][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t a[4], b0, b1;
        ldsm_x4(a, ka + ks * 32);
        ldsm_x2(b0, b1, qa + ks * 32);
        mma16816(sa[ks & 3], a, b0, b1);
      }
      float s[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] = (sa[0][e] + sa[1][e]) + (sa[2][e] + sa[3][e]);
      float* d = ss + (size_t)(t * 8 + 2 * t4) * m.ps + mt * 16 + g8;
      d[0] = s[0];
      d[m.ps] = s[1];
      d[8] = s[2];
      d[m.ps + 8] = s[3];
    }
    __syncthreads();   // the scores are there
#pragma unroll
    for (int i = 0; i < HW; ++i) {
      const int h = warp + i * WARPS;
      if (h >= H) break;
      float x[KL], top = -INFINITY;
#pragma unroll
      for (int k = 0; k < KL; ++k) {
        const int kr = lane + 32 * k;
        const float d = (float)(keys - 1 - tile * KT - kr);
        x[k] = -INFINITY;
        if (kr < KT && d >= 0.f) x[k] = fmaf(ss[(size_t)srow[i] * m.ps + kr], sf[st * KT + kr] * kLog2e, -r1[i] * lg2(fmaf(r2[i], d, 1.f)));
        top = fmaxf(top, x[k]);
      }
      float sum = l[i];
      if (__any_sync(0xffffffffu, top > mx[i] + 8.f)) {
        top = fmaxf(warp_max(top), mx[i]);
        const float al = ex2(mx[i] - top);
        sum *= al;
        mx[i] = top;
        if (lane == 0) {
          sal[h] = al;
          *moved = tile;
        }
      } else if (lane == 0) sal[h] = 1.f;
#pragma unroll
      for (int k = 0; k < KL; ++k) {
        const int kr = lane + 32 * k;
        if (kr < KT) {
          const float w = ex2(x[k] - mx[i]);   // a tile of a split holds at least one key, so the reference is a number
          const __nv_bfloat16 hi = __float2bfloat16(w);
          sum += w;
          sp[h * m.pp + kr] = hi;
          sp[m.p + h * m.pp + kr] = __float2bfloat16(w - __bfloat162float(hi));
        }
      }
      l[i] = sum;
    }
    __syncthreads();   // weights and factors are there
    if (col0 < GD) {
if (*moved == tile) {
#pragma unroll
        for (int a = 0; a < MH; ++a) {
          const float f0 = sal[a * 16 + g8], f1 = sal[a * 16 + g8 + 8];
#pragma unroll
          for (int b = 0; b < NTC; ++b)
#pragma unroll
            for (int t = 0; t < 2; ++t) {
              acc[a][b][t][0] *= f0; acc[a][b][t][1] *= f0;
              acc[a][b][t][2] *= f1; acc[a][b][t][3] *= f1;
            }
        }
      }
#pragma unroll
      for (int ks = 0; ks < MTS; ++ks) {
        uint32_t hi[MH][4], lo[MH][4];
#pragma unroll
        for (int a = 0; a < MH; ++a) {
          ldsm_x4(hi[a], a_addr(ap, m.pp, a * 16, ks * 16, lane));
          ldsm_x4(lo[a], a_addr(ap + plane, m.pp, a * 16, ks * 16, lane));
        }
#pragma unroll
        for (int b = 0; b < NTC; ++b) {
          const int col = col0 + b * 16;
          if (col >= GD) break;
          uint32_t v[4];
          ldsm_x4_t(v, bkn_addr(ak + (uint32_t)((col / DP) * KT * PD * 2), PD, ks * 16, col % DP, lane));
#pragma unroll
          for (int a = 0; a < MH; ++a) {
            mma16816(acc[a][b][0], hi[a], v[0], v[1]);
            mma16816(acc[a][b][1], hi[a], v[2], v[3]);
          }
#pragma unroll
          for (int a = 0; a < MH; ++a) {
            mma16816(acc[a][b][0], lo[a], v[0], v[1]);
            mma16816(acc[a][b][1], lo[a], v[2], v[3]);
          }
        }
      }
    }
  }
  cp_async_wait<0>();
  const size_t out = (size_t)split * p.t.R + r;
#pragma unroll
  for (int i = 0; i < HW; ++i) {
    const int h = warp + i * WARPS;
    if (h >= H) break;
    const float sum = warp_sum(l[i]);
    if (lane == 0) reinterpret_cast<float2*>(p.ws_ml)[out * H + h] = make_float2(mx[i], sum);
  }
  float* o = p.ws_o + out * H * GD;
#pragma unroll
  for (int a = 0; a < MH; ++a)
#pragma unroll
    for (int b = 0; b < NTC; ++b)
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int h = a * 16 + g8 + 8 * hh, col = col0 + b * 16 + t * 8 + 2 * t4;
          if (h < H && col < GD) *reinterpret_cast<float2*>(o + (size_t)h * GD + col) = make_float2(acc[a][b][t][2 * hh], acc[a][b][t][2 * hh + 1]);
        }
}

// One CTA per row of the partial results and block of columns; rows are requests (dec), or the tokens of the tiles tile0, tile0 + 1, ... of 128 over
// the longer portions. A thread owns a column of one key head's rows and up to eight of the heads that read it.
constexpr int kJoinHeads = 8, kJoinThreads = 128;

template <bool DEC>
__global__ void __launch_bounds__(kJoinThreads) talk_join_kernel(const TalkTcParams p) {
  extern __shared__ __align__(16) float jm[];
  const int H = p.t.H, G = p.t.G, share = H / G, dim = p.t.dim, DP = p.t.row, GD = G * DP, splits = DEC ? p.splits : 1;
  const int blocks = (share + kJoinHeads - 1) / kJoinHeads, wide = G * blocks * kJoinHeads;
  float* st = jm;             // [from][key head, block, eight heads] mix
  float* sc = jm + H * wide;  // [splits][H] factors
  __shared__ int s_tok;
  pdl_trigger();
  pdl_wait();
  const size_t row = blockIdx.x;
  if (threadIdx.x == 0) {
    int tok = -1;
    if (DEC) {
      const int qs = p.t.query_start_loc[row];
      if (p.t.query_start_loc[row + 1] - qs == 1) tok = qs;
    } else {
      int b = p.tile0 + (int)(row / 128);
      for (int i = 0; i < p.t.R; ++i) {
        const int qs = p.t.query_start_loc[i], n = p.t.query_start_loc[i + 1] - qs;
        if (n < p.min_len) continue;
        const int nt = (n + 127) / 128;
        if (b < nt) {
          const int at = b * 128 + (int)(row % 128);
          if (at < n) tok = qs + at;
          break;
        }
        b -= nt;
      }
    }
    s_tok = tok;
  }
  __syncthreads();
  const int tok = s_tok;
  if (tok < 0) return;
  const size_t plane = DEC ? (size_t)p.t.R : 0;   // rows of a split
  for (int g = threadIdx.x; g < H; g += kJoinThreads) {
    const float2* ml = reinterpret_cast<const float2*>(p.ws_ml) + row * H + g;
    float m = -INFINITY, sum = 0.f;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, ml[s * plane * H].x);
    for (int s = 0; s < splits; ++s) {
      const float2 v = ml[s * plane * H];
      sum += v.x == -INFINITY ? 0.f : v.y * ex2(v.x - m);
    }
    for (int s = 0; s < splits; ++s) {
      const float x = ml[s * plane * H].x;
      sc[s * H + g] = x == -INFINITY ? 0.f : ex2(x - m) / sum;
    }
  }
  for (int i = threadIdx.x; i < H * wide; i += kJoinThreads) {
    const int from = i / wide, a = i % wide / (blocks * kJoinHeads), k = i % (blocks * kJoinHeads);
    st[i] = k < share ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.t.mix)[(a * share + k) * H + from]) : 0.f;
  }
  __syncthreads();
  const float* o = p.ws_o + row * H * GD;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.t.out) + (size_t)tok * H * dim;
  const int step = gridDim.y * kJoinThreads;
  for (int i = blockIdx.y * kJoinThreads + threadIdx.x; i < G * dim; i += step) {
    const int a = i / dim, d = i % dim;
    const float* src = o + a * DP + d;
    for (int blk = 0; blk < blocks; ++blk) {
      const float* w = st + (a * blocks + blk) * kJoinHeads;
      float acc[kJoinHeads];
#pragma unroll
      for (int k = 0; k < kJoinHeads; ++k) acc[k] = 0.f;
      auto add = [&](int g, float x) {
        const float4 t0 = *reinterpret_cast<const float4*>(w + g * wide), t1 = *reinterpret_cast<const float4*>(w + g * wide + 4);
        acc[0] = fmaf(t0.x, x, acc[0]); acc[1] = fmaf(t0.y, x, acc[1]); acc[2] = fmaf(t0.z, x, acc[2]); acc[3] = fmaf(t0.w, x, acc[3]);
        acc[4] = fmaf(t1.x, x, acc[4]); acc[5] = fmaf(t1.y, x, acc[5]); acc[6] = fmaf(t1.z, x, acc[6]); acc[7] = fmaf(t1.w, x, acc[7]);
      };
      int g = 0;
      for (; g + 8 <= H; g += 8) {   // eight loads in flight
        float x[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) x[k] = sc[g + k] * src[(size_t)(g + k) * GD];
        for (int s = 1; s < splits; ++s) {
#pragma unroll
          for (int k = 0; k < 8; ++k) x[k] = fmaf(sc[s * H + g + k], src[(s * plane * H + g + k) * GD], x[k]);
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) add(g + k, x[k]);
      }
      for (; g < H; ++g) {
        float x = 0.f;
        for (int s = 0; s < splits; ++s) x = fmaf(sc[s * H + g], src[(s * plane * H + g) * GD], x);
        add(g, x);
      }
#pragma unroll
      for (int k = 0; k < kJoinHeads; ++k)
        if (blk * kJoinHeads + k < share) out[(a * share + blk * kJoinHeads + k) * dim + d] = __float2bfloat16(acc[k]);
    }
  }
}

constexpr size_t kMaxSmem = 227 * 1024 - 64;

int key_tile(int H, int G, int dp) {
  for (int kt : {64, 32, 16})
    if (G * kt <= 256 && smem_bytes(geom(H, G, dp, kt), H, kt) <= kMaxSmem) return kt;
  return 0;
}

template <int DP, int KT, int MH, int NTC>
int decode_go(const TalkTcParams& p, cudaStream_t st) {
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (cudaFuncSetAttribute(talk_decode_kernel<DP, KT, MH, NTC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMaxSmem) != cudaSuccess) return -4;
    configured = true;
  }
  launch_k(talk_decode_kernel<DP, KT, MH, NTC>, dim3((unsigned)p.t.R, (unsigned)p.splits), dim3(MT), smem_bytes(geom(p.t.H, p.t.G, DP, KT), p.t.H, KT), st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}
template <int DP, int KT, int MH>
int decode_cols(const TalkTcParams& p, cudaStream_t st) {
  const int n = (p.t.G * DP + WARPS * 16 - 1) / (WARPS * 16);   // pieces of 16 columns per warp
  if (n <= 1) return decode_go<DP, KT, MH, 1>(p, st);
  if (n <= 2) return decode_go<DP, KT, MH, 2>(p, st);
  if constexpr (MH <= 2)
    if (n <= 4) return decode_go<DP, KT, MH, 4>(p, st);
  if constexpr (MH == 1)
    if (n <= 8) return decode_go<DP, KT, MH, 8>(p, st);
  return -3;
}
template <int DP, int KT>
int decode_heads(const TalkTcParams& p, cudaStream_t st) {
  const int n = (p.t.H + 15) / 16;
  return n <= 1 ? decode_cols<DP, KT, 1>(p, st) : n <= 2 ? decode_cols<DP, KT, 2>(p, st) : decode_cols<DP, KT, 4>(p, st);
}
template <int DP>
int decode_tile(const TalkTcParams& p, cudaStream_t st) {
  switch (key_tile(p.t.H, p.t.G, DP)) {
    case 64: return decode_heads<DP, 64>(p, st);
    case 32: return decode_heads<DP, 32>(p, st);
    case 16: return decode_heads<DP, 16>(p, st);
  }
  return -3;
}

}  // namespace

int talk_tc_row(int H, int G, int dim) {
  if (H < 1 || H > 64 || G < 1 || H % G || dim < 1 || dim > 128) return 0;
  const int dp = dim <= 64 ? 64 : 128, pieces = (G * dp + WARPS * 16 - 1) / (WARPS * 16), mh = (H + 15) / 16;
  return key_tile(H, G, dp) && pieces * (mh > 2 ? 4 : mh) <= 8 ? dp : 0;
}

int talk_decode_launch(const TalkTcParams& p_, cudaStream_t st) {
  TalkTcParams p = p_;
  if (p.t.R == 0 || p.t.T == 0) return 0;
  if (p.t.f32 || talk_tc_row(p.t.H, p.t.G, p.t.dim) != p.t.row || (p.t.bs & (p.t.bs - 1)) || p.splits < 1 || p.ws_ml == nullptr || p.ws_o == nullptr) return -1;
  p.bs_shift = __builtin_ctz((unsigned)p.t.bs);
  const int rc = p.t.row == 64 ? decode_tile<64>(p, st) : decode_tile<128>(p, st);
  return rc ? rc : talk_join_launch(p, true, p.t.R, st);
}

int talk_join_launch(const TalkTcParams& p, bool dec, int rows, cudaStream_t st) {
  const int share = p.t.H / p.t.G, wide = p.t.G * ((share + kJoinHeads - 1) / kJoinHeads) * kJoinHeads;
  const size_t smem = ((size_t)p.t.H * wide + (size_t)(dec ? p.splits : 1) * p.t.H) * 4;
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {   // up to 64 key heads of one head each: 64 x 512 numbers
    if (cudaFuncSetAttribute(talk_join_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(talk_join_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess) return -4;
    configured = true;
  }
  if (smem > 160 * 1024) return -6;
  const int cols = (p.t.G * p.t.dim + kJoinThreads - 1) / kJoinThreads;
  const dim3 grid((unsigned)rows, (unsigned)(dec ? cols : (cols + 3) / 4));   // few rows: more blocks of columns
  if (dec) launch_k(talk_join_kernel<true>, grid, dim3(kJoinThreads), smem, st, true, p);
  else launch_k(talk_join_kernel<false>, grid, dim3(kJoinThreads), smem, st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace oc
