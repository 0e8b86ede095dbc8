// Talking-heads attention on tensor cores (bf16 queries and cache, fp32 scores and weights); definitions in talk_attention.cu.
//
// The mix over heads needs normalised weights, so the keys are walked twice:
//   talk_stats: every head's maximum and sum, per (queries, key head, split of the keys); scores only.
//   talk_mix:   scores again, exact weights, mix, value product. A CTA holds all heads of a few tokens: tiles of keys (all key heads) stream through
//               shared memory and serve both products. Splits of the keys add up, since the weights are already normalised.
//
// Query rows are laid out per key head as (token, head), heads padded to hp = 1, 2, 4, 8, 16 or 32: eight columns of a product are one "tile" of a
// query block of QB = max(1, 8 / hp) tokens, and the tiles of all key heads together are the columns of the block. talk_mix, per tile of KT keys:
//   scores   S^T [keys][columns] = K Q^T per key head, weights as two bf16 planes into shared memory
//   mix      [keys][columns] = weights x T', T' the mix matrix with zeros between different tokens; transposed stores
//   values   O [rows][dim] += mixed [rows][keys] x K per key head, accumulators in registers for the whole walk
// 32-bit weights enter the products as two bf16 terms; a block of eight rows (decoding) carries the second terms in its unused rows.
#include "kernels.h"
#include "mma_sync.cuh"

namespace oc {
namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ void ldsm_x2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr) : "memory");
}
__device__ __forceinline__ void stsm_x4_t(uint32_t addr, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};" ::"r"(addr), "r"(r0), "r"(r1), "r"(r2), "r"(r3) : "memory");
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

struct Where { int req, tok0, ntok, qs, ctx0; };   // request, first token of the tile in its portion, tokens, row of the portion, context ahead of it

// dec: block x is a request, single tokens only; otherwise block x counts tiles of `per` tokens over the longer portions, last tiles first
__device__ __forceinline__ Where locate(const TalkTcParams& p, int x, int per, bool dec) {
  Where w{-1, 0, 0, 0, 0};
  if (dec) {
    const int qs = p.t.query_start_loc[x], n = p.t.query_start_loc[x + 1] - qs;
    if (n >= 1 && n <= p.short_len) w = Where{x, 0, n, qs, p.t.seq_lens[x] - n};
    return w;
  }
  int b = x;
  for (int i = 0; i < p.t.R; ++i) {
    const int qs = p.t.query_start_loc[i], n = p.t.query_start_loc[i + 1] - qs;
    if (n <= p.short_len) continue;
    const int nt = (n + per - 1) / per;
    if (b < nt) {
      const int k = nt - 1 - b;
      return Where{i, k * per, min(per, n - k * per), qs, p.t.seq_lens[i] - n};
    }
    b -= nt;
  }
  return w;
}

// ----------------------------------------------------------------------------------------------------------------- talk_stats
constexpr int SK = 64, SST = 3;   // keys per tile, stages

// !DEC: 64 rows (token, head) over four warps. DEC: up to 16 rows, the warps take 16 keys of a tile each.
template <int DP, bool DEC>
__global__ void __launch_bounds__(128) talk_stats_kernel(const TalkTcParams p) {
  constexpr int PD = DP + 8, ROWS = DEC ? 16 : 64, NB = DEC ? 2 : 8;
  extern __shared__ __align__(16) uint8_t raw[];
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(raw);          // [SST][SK][PD]
  __nv_bfloat16* sq = sk + SST * SK * PD;                             // [ROWS][PD]
  float* sf = reinterpret_cast<float*>(sq + ROWS * PD);               // [SST][SK]
  float* sm = sf + SST * SK;                                          // [4][16][2] (DEC)
  __shared__ Where s_w;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, g = blockIdx.y, split = blockIdx.z;
  const int hp = p.t.group_rows, share = p.t.H / p.t.G, per = DEC ? 1 : ROWS / hp, bs = p.bs_shift, bsm = p.t.bs - 1;
  if (tid == 0) s_w = locate(p, blockIdx.x, per, DEC);
  __syncthreads();
  const Where w = s_w;
  if (w.req < 0) return;
  const int* bt = p.t.block_table + (size_t)w.req * p.t.bt_stride;
  const int keys = w.ctx0 + w.tok0 + w.ntok, tiles = (keys + SK - 1) / SK;
  const int each = (tiles + p.splits - 1) / p.splits, first = split * each, last = min(tiles, first + each);
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.t.q);
  const __nv_bfloat16* pages = reinterpret_cast<const __nv_bfloat16*>(p.t.pages);
  for (int e = tid; e < ROWS * (DP / 8); e += 128) {
    const int row = e / (DP / 8), c = e % (DP / 8) * 8, tok = row / hp;
    const bool live = tok < w.ntok;
    cp_async16(smem_u32(sq + row * PD + c), q + (((size_t)(w.qs + w.tok0 + (live ? tok : 0)) * p.t.G + g) * hp + row % hp) * DP + c, live ? 16 : 0);
  }
  auto fetch = [&](int tile) {
    if (tile < last) {
      const int st = tile % SST;
      for (int e = tid; e < SK * (DP / 8); e += 128) {
        const int kr = e / (DP / 8), c = e % (DP / 8) * 8, key = tile * SK + kr;
        const bool live = key < keys;
        const int at = live ? key : 0;
        cp_async16(smem_u32(sk + (st * SK + kr) * PD + c), pages + ((((size_t)bt[at >> bs] * p.t.G + g) << bs) + (at & bsm)) * DP + c, live ? 16 : 0);
      }
      if (tid < SK) {
        const int key = tile * SK + tid, at = key < keys ? key : 0;
        cp_async4(smem_u32(sf + st * SK + tid), p.t.k_scale + ((size_t)bt[at >> bs] << bs) + (at & bsm), key < keys ? 4 : 0);
      }
    }
    cp_async_commit();
  };
  fetch(first);
  fetch(first + 1);
  const int row0 = DEC ? 0 : warp * 16;
  float r1[2], r2[2], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float pos[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int row = row0 + g8 + 8 * i, h = row % hp, tok = row / hp;
    const bool live = h < share && tok < w.ntok;
    r1[i] = live ? p.t.bias[g * share + h] : 0.f;
    r2[i] = live ? p.t.bias[p.t.H + g * share + h] : 0.f;
    pos[i] = live ? (float)(w.ctx0 + w.tok0 + tok) : -1.f;
  }
  const uint32_t aq = smem_u32(sq);
  for (int tile = first; tile < last; ++tile) {
    cp_async_wait<1>();
    __syncthreads();
    fetch(tile + 2);   // into the stage that every warp has left
    const int st = tile % SST;
    const uint32_t ak = smem_u32(sk + st * SK * PD);
    float acc[NB][4];
#pragma unroll
    for (int t = 0; t < NB; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[t][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks) {
      uint32_t a[4];
      ldsm_x4(a, a_addr(aq, PD, row0, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < NB / 2; ++np) {
        uint32_t b[4];
        ldsm_x4(b, bnk_addr(ak, PD, (DEC ? warp * 16 : np * 16), ks * 16, lane));
        mma16816(acc[2 * np], a, b[0], b[1]);
        mma16816(acc[2 * np + 1], a, b[2], b[3]);
      }
    }
    float nm[2] = {m[0], m[1]};
    const int kr0 = (DEC ? warp * 16 : 0) + 2 * t4;
    const float k0 = (float)(tile * SK + kr0);
    const float d0[2] = {pos[0] - k0, pos[1] - k0};   // distance to this lane's first key
#pragma unroll
    for (int t = 0; t < NB; ++t) {
      const float2 f = *reinterpret_cast<const float2*>(sf + st * SK + kr0 + t * 8);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = e >> 1;
        const float d = d0[i] - (float)(t * 8 + (e & 1));
        const float s = fmaf(acc[t][e], ((e & 1) ? f.y : f.x) * kLog2e, -r1[i] * lg2(fmaf(r2[i], d, 1.f)));
        acc[t][e] = d >= 0.f ? s : -INFINITY;
        nm[i] = fmaxf(nm[i], acc[t][e]);
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float base = nm[i] == -INFINITY ? 0.f : nm[i];
      float sum = l[i] * ex2(m[i] - base);
#pragma unroll
      for (int t = 0; t < NB; ++t) sum += ex2(acc[t][2 * i] - base) + ex2(acc[t][2 * i + 1] - base);
      l[i] = sum;
      m[i] = nm[i];
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {   // the four lanes of a row
      const float om = __shfl_xor_sync(0xffffffffu, m[i], o), ol = __shfl_xor_sync(0xffffffffu, l[i], o);
      const float x = fmaxf(m[i], om), base = x == -INFINITY ? 0.f : x;
      l[i] = l[i] * ex2(m[i] - base) + ol * ex2(om - base);
      m[i] = x;
    }
  }
  auto put = [&](int row, float mm, float ll) {
    const int h = row % hp, tok = row / hp;
    if (h < share && tok < w.ntok)
      reinterpret_cast<float2*>(p.ws_ml)[((size_t)split * p.t.T + w.qs + w.tok0 + tok) * p.t.H + g * share + h] = make_float2(mm, ll);
  };
  if (!DEC) {
    if (t4 == 0) {
      put(row0 + g8, m[0], l[0]);
      put(row0 + g8 + 8, m[1], l[1]);
    }
  } else {
    if (t4 == 0) {
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        sm[(warp * 16 + g8 + 8 * i) * 2] = m[i];
        sm[(warp * 16 + g8 + 8 * i) * 2 + 1] = l[i];
      }
    }
    __syncthreads();
    if (tid < 16) {
      float x = -INFINITY, sum = 0.f;
#pragma unroll
      for (int k = 0; k < 4; ++k) x = fmaxf(x, sm[(k * 16 + tid) * 2]);
      const float base = x == -INFINITY ? 0.f : x;
#pragma unroll
      for (int k = 0; k < 4; ++k) sum += sm[(k * 16 + tid) * 2 + 1] * ex2(sm[(k * 16 + tid) * 2] - base);
      put(tid, x, sum);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------- talk_mix
constexpr int MT = 512;   // threads

struct MixGeom {   // sizes of the shared-memory areas, in elements
  int tg, nt, nte, qb, rg, rgp, pp, pw;   // tiles per key head, per block; rounded up to even; tokens per block; rows per key head (and padded); pitches
  size_t k, q, p, w, t, f;
};
__host__ __device__ inline MixGeom mix_geom(int G, int hp, int pd, int nqb, int kt) {
  MixGeom m;
  m.tg = hp <= 8 ? 1 : hp / 8;
  m.nt = G * m.tg;
  m.nte = (m.nt + 1) / 2 * 2;
  m.qb = hp <= 8 ? 8 / hp : 1;
  m.rg = nqb * 8 * m.tg;
  m.rgp = m.rg < 16 ? 16 : m.rg;
  m.pp = 8 * m.nte + 8;
  m.pw = kt + 8;
  m.k = (size_t)G * kt * pd;
  m.q = (size_t)G * m.rg * pd;
  m.p = (size_t)nqb * kt * m.pp;
  m.w = (size_t)G * m.rgp * m.pw;
  m.t = (size_t)8 * m.nt * m.pp;
  m.f = (size_t)2 * kt + nqb * 8 * m.nt + 16 * m.nt + 32 + 4 * ((size_t)m.nt * (kt / 16) * nqb + (size_t)m.nte * (kt / 16) * nqb);
  return m;
}
inline size_t mix_smem(const MixGeom& m, bool pack) { return (2 * m.k + m.q + 2 * m.p + (pack ? 1 : 2) * m.w + m.t) * 2 + m.f * 4; }

// NQB: query blocks of a tile; ACC: pieces of 16 output columns per warp
template <int DP, int NQB, int ACC>
__global__ void __launch_bounds__(MT) talk_mix_kernel(const TalkTcParams p) {
  constexpr int PD = DP + 8, QPU = NQB >= 2 ? 2 : 1, NPU = NQB >= 2 ? 2 : 1, DC = DP / 16;
  constexpr bool DEC = NQB == 1;
  extern __shared__ __align__(16) uint8_t raw[];
  __shared__ Where s_w;
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g8 = lane >> 2, t4 = lane & 3, split = blockIdx.y;
  const int H = p.t.H, G = p.t.G, hp = p.t.group_rows, share = H / G, kts = p.kt_shift, KT = 1 << kts, bs = p.bs_shift, bsm = p.t.bs - 1;
  const MixGeom m = mix_geom(G, hp, PD, NQB, KT);
  const bool pack = m.rg < 16;
  const int cols = 8 * m.nt, per = DEC ? 1 : NQB * m.qb;
  if (tid == 0) s_w = locate(p, blockIdx.x, per, DEC);
  __syncthreads();
  const Where w = s_w;
  if (w.req < 0) return;
  __nv_bfloat16* sk = reinterpret_cast<__nv_bfloat16*>(raw);   // [2][G][KT][PD]
  __nv_bfloat16* sq = sk + 2 * m.k;                            // [G][rg][PD]
  __nv_bfloat16* sp = sq + m.q;                                // [2][NQB][KT][pp]
  __nv_bfloat16* sw = sp + 2 * m.p;                            // [2 or 1][G][rgp][pw]
  __nv_bfloat16* stt = sw + (pack ? 1 : 2) * m.w;              // [cols][pp]
  float* sf = reinterpret_cast<float*>(stt + m.t);             // [2][KT]
  float* slse = sf + 2 * KT;                                   // [NQB][cols]
  float* sr1 = slse + NQB * cols;                              // [cols]
  float* sr2 = sr1 + cols;
  float* spos = sr2 + cols;                                    // [NQB * qb]
  int4* units = reinterpret_cast<int4*>(spos + 32);            // what the warps do, for the scores and then for the mix

  const int* bt = p.t.block_table + (size_t)w.req * p.t.bt_stride;
  const int keys = w.ctx0 + w.tok0 + w.ntok, tiles = (keys + KT - 1) / KT;
  const int each = (tiles + p.mix_splits - 1) / p.mix_splits, first = split * each, last = min(tiles, first + each);
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.t.q);
  const __nv_bfloat16* pages = reinterpret_cast<const __nv_bfloat16*>(p.t.pages);
  const __nv_bfloat16* mix = reinterpret_cast<const __nv_bfloat16*>(p.t.mix);
  for (int e = tid; e < G * m.rg * (DP / 8); e += MT) {
    const int c = e % (DP / 8) * 8, row = e / (DP / 8) % m.rg, g = e / (DP / 8 * m.rg), tok = row / hp;
    const bool live = tok < w.ntok;
    cp_async16(smem_u32(sq + (size_t)(g * m.rg + row) * PD + c), q + (((size_t)(w.qs + w.tok0 + (live ? tok : 0)) * G + g) * hp + row % hp) * DP + c, live ? 16 : 0);
  }
  auto fetch = [&](int tile) {
    if (tile < last) {
      const int st = tile & 1;
      const uint32_t dst = smem_u32(sk + st * m.k);
      for (int e = tid; e < G * KT * (DP / 8); e += MT) {
        const int c = e % (DP / 8) * 8, row = e / (DP / 8), kr = row & (KT - 1), g = row >> kts, key = tile * KT + kr;
        const bool live = key < keys;
        const int at = live ? key : 0;
        cp_async16(dst + (uint32_t)((row * PD + c) * 2), pages + ((((size_t)bt[at >> bs] * G + g) << bs) + (at & bsm)) * DP + c, live ? 16 : 0);
      }
      if (tid < KT) {
        const int key = tile * KT + tid, at = key < keys ? key : 0;
        cp_async4(smem_u32(sf + st * KT + tid), p.t.k_scale + ((size_t)bt[at >> bs] << bs) + (at & bsm), key < keys ? 4 : 0);
      }
    }
    cp_async_commit();
  };
  fetch(first);
  // column -> (token of its block, head); columns that are none have a logarithm of the sum of +inf, so their weights are zero
  auto head_of = [&](int col) {
    const int t = col >> 3, c = col & 7, g = t / m.tg, h = hp <= 8 ? c % hp : (t % m.tg) * 8 + c;
    return h < share ? g * share + h : -1;
  };
  auto token_of = [&](int c) { return hp <= 8 ? c / hp : 0; };
  for (int i = tid; i < NQB * m.qb; i += MT) spos[i] = i < w.ntok ? (float)(w.ctx0 + w.tok0 + i) : -1.f;
  for (int i = tid; i < cols; i += MT) {
    const int h = head_of(i);
    sr1[i] = h >= 0 ? p.t.bias[h] : 0.f;
    sr2[i] = h >= 0 ? p.t.bias[H + h] : 0.f;
  }
  for (int i = tid; i < NQB * cols; i += MT) {
    const int h = head_of(i % cols), tok = i / cols * m.qb + token_of(i & 7);
    float lse = INFINITY;
    if (h >= 0 && tok < w.ntok) {
      const float2* ml = reinterpret_cast<const float2*>(p.ws_ml) + (size_t)(w.qs + w.tok0 + tok) * H + h;
      float x = -INFINITY, sum = 0.f;
      for (int s = 0; s < p.splits; ++s) x = fmaxf(x, ml[(size_t)s * p.t.T * H].x);
      for (int s = 0; s < p.splits; ++s) {
        const float2 v = ml[(size_t)s * p.t.T * H];
        sum += v.x == -INFINITY ? 0.f : v.y * ex2(v.x - x);
      }
      lse = x + log2f(sum);
    }
    slse[i] = lse;
  }
  for (int i = tid; i < cols * m.pp; i += MT) {
    const int to = i / m.pp, from = i % m.pp;
    float v = 0.f;
    if (from < cols && token_of(to & 7) == token_of(from & 7)) {
      const int a = head_of(to), b = head_of(from);
      if (a >= 0 && b >= 0) v = __bfloat162float(mix[a * H + b]);
    }
    stt[i] = __float2bfloat16(v);
  }
  const int mts = KT / 16, nu1 = m.nt * mts * (NQB / QPU), nu2 = mts * NQB * (m.nte / NPU);
  for (int u = tid; u < nu1; u += MT) {   // byte offsets of the key rows and query rows, row in the tile, column, query block
    const int t = u % m.nt, mt = u / m.nt % mts, qb = u / (m.nt * mts) * QPU, g = t / m.tg, part = t % m.tg;
    units[u] = make_int4((g * KT + mt * 16) * PD * 2, (g * m.rg + (qb * m.tg + part) * 8) * PD * 2, mt * 16 | t << 16, qb);
  }
  for (int u = tid; u < nu2; u += MT) {   // offset of the weights, first column tile, offsets of the stores of its tiles (-1: none)
    const int mt = u % mts, qb = u / mts % NQB, n0 = u / (mts * NQB) * NPU;
    auto out = [&](int t) { return t < m.nt ? (((t / m.tg) * m.rgp + (qb * m.tg + t % m.tg) * 8) * m.pw + mt * 16) * 2 : -1; };
    units[nu1 + u] = make_int4((qb * KT + mt * 16) * m.pp * 2, min(n0, m.nt - 1), out(n0), NPU == 2 ? out(n0 + 1) : -1);
  }
  if (m.nte != m.nt)   // the columns that round the mix's inner dimension up
    for (int i = tid; i < 2 * NQB * KT * 8; i += MT) sp[(size_t)(i >> 3) * m.pp + cols + (i & 7)] = __float2bfloat16(0.f);

  float acc[ACC][2][4];
#pragma unroll
  for (int a = 0; a < ACC; ++a)
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[a][t][e] = 0.f;
  const int mtiles = m.rgp / 16, pieces = G * mtiles * DC, piece0 = warp * ACC;
  uint32_t woff[ACC], koff[ACC];   // byte offsets of a piece's rows of the mixed weights and of its key columns, this lane's address included
#pragma unroll
  for (int a = 0; a < ACC; ++a) {
    const int gm = min(piece0 + a, pieces - 1) / DC, c = min(piece0 + a, pieces - 1) % DC, g = gm / mtiles;
    woff[a] = a_addr((uint32_t)(g * m.rgp * m.pw * 2), m.pw, gm % mtiles * 16, 0, lane);
    koff[a] = bkn_addr((uint32_t)(g * KT * PD * 2), PD, 0, c * 16, lane);
  }
  const uint32_t aw = smem_u32(sw), aq = smem_u32(sq), ap = smem_u32(sp), plane_p = (uint32_t)(m.p * 2), plane_w = (uint32_t)(m.w * 2);
  const uint32_t lane_a = a_addr(0, PD, 0, 0, lane), lane_p = a_addr(0, m.pp, 0, 0, lane);
  // columns of a pair of query blocks, one block above the other
  const uint32_t lane_q = (uint32_t)((((QPU == 2 ? (lane >> 4) * m.tg * 8 : 0) + (lane & 7)) * PD + ((lane >> 3) & 1) * 8) * 2);
  const uint32_t lane_t = (uint32_t)(((lane & 7) * m.pp + ((lane >> 3) & 1) * 8) * 2), next_t = NPU == 2 && lane >= 16 ? (uint32_t)(8 * m.pp * 2) : 0;
  const uint32_t lane_w = (uint32_t)(((lane & 7) * m.pw + ((lane >> 3) & 1) * 8) * 2) + (lane >= 16 ? (pack ? (uint32_t)(8 * m.pw * 2) : plane_w) : 0);
  const int tk0 = token_of(2 * t4), tk1 = token_of(2 * t4 + 1);

  for (int tile = first; tile < last; ++tile) {
    const int st = tile & 1;
    cp_async_wait<0>();
    __syncthreads();   // the tile is there, and every warp is done with the previous one
    fetch(tile + 1);
    const uint32_t ak = smem_u32(sk + st * m.k);
    const float key0 = (float)(tile * KT);
    // ---- scores and weights
    for (int u = warp; u < nu1; u += MT / 32) {
      const int4 un = units[u];
      const int mt16 = un.z & 0xffff, col = (un.z >> 16) * 8 + 2 * t4;
      const uint32_t ka = ak + un.x + lane_a, qa = aq + un.y + lane_q;
      float s[QPU][4];
#pragma unroll
      for (int i = 0; i < QPU; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t a[4], b[4];
        ldsm_x4(a, ka + ks * 32);
        if (QPU == 2) ldsm_x4(b, qa + ks * 32);
        else ldsm_x2(b[0], b[1], qa + ks * 32);
#pragma unroll
        for (int i = 0; i < QPU; ++i) mma16816(s[i], a, b[2 * i], b[2 * i + 1]);
      }
      const int kr = mt16 + g8;
      const float f[2] = {sf[st * KT + kr] * kLog2e, sf[st * KT + kr + 8] * kLog2e};
      const float2 ra = *reinterpret_cast<const float2*>(sr1 + col), rb = *reinterpret_cast<const float2*>(sr2 + col);
      const float key = key0 + (float)kr;
#pragma unroll
      for (int i = 0; i < QPU; ++i) {
        const int qb = un.w + i;
        const float d0 = spos[qb * m.qb + tk0] - key, d1 = spos[qb * m.qb + tk1] - key;
        const float2 lse = *reinterpret_cast<const float2*>(slse + qb * cols + col);
        const uint32_t dst = ap + (uint32_t)(((qb * KT + kr) * m.pp + col) * 2);
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const float e0 = d0 - 8.f * hh, e1 = d1 - 8.f * hh;
          const float x0 = fmaf(s[i][2 * hh], f[hh], -fmaf(ra.x, lg2(fmaf(rb.x, e0, 1.f)), lse.x));
          const float x1 = fmaf(s[i][2 * hh + 1], f[hh], -fmaf(ra.y, lg2(fmaf(rb.y, e1, 1.f)), lse.y));
          uint32_t hi, lo;
          split2(e0 >= 0.f ? ex2(x0) : 0.f, e1 >= 0.f ? ex2(x1) : 0.f, hi, lo);
          const uint32_t at = dst + (uint32_t)(hh * 8 * m.pp * 2);
          asm volatile("st.shared.b32 [%0], %1;" ::"r"(at), "r"(hi) : "memory");
          asm volatile("st.shared.b32 [%0], %1;" ::"r"(at + plane_p), "r"(lo) : "memory");
        }
      }
    }
    __syncthreads();   // the weights are there
    // ---- mix over the heads, transposed into rows of the value product
    for (int u = warp; u < nu2; u += MT / 32) {
      const int4 un = units[nu1 + u];
      if (un.z < 0) continue;
      const uint32_t pa = ap + un.x + lane_p, ta = smem_u32(stt) + (uint32_t)(un.y * 8 * m.pp * 2) + lane_t + (un.w >= 0 ? next_t : 0);
      float x[NPU][4];
#pragma unroll
      for (int i = 0; i < NPU; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) x[i][e] = 0.f;
#pragma unroll 4
      for (int ks = 0; ks < m.nte / 2; ++ks) {
        uint32_t a0[4], a1[4], b[4];
        ldsm_x4(a0, pa + ks * 32);
        ldsm_x4(a1, pa + plane_p + ks * 32);
        if (NPU == 2) ldsm_x4(b, ta + ks * 32);
        else ldsm_x2(b[0], b[1], ta + ks * 32);
#pragma unroll
        for (int i = 0; i < NPU; ++i) mma16816(x[i], a0, b[2 * i], b[2 * i + 1]);
#pragma unroll
        for (int i = 0; i < NPU; ++i) mma16816(x[i], a1, b[2 * i], b[2 * i + 1]);
      }
#pragma unroll
      for (int i = 0; i < NPU; ++i) {
        const int off = i ? un.w : un.z;
        if (off < 0) break;
        uint32_t h0, l0, h1, l1;
        split2(x[i][0], x[i][1], h0, l0);
        split2(x[i][2], x[i][3], h1, l1);
        stsm_x4_t(aw + off + lane_w, h0, h1, l0, l1);
      }
    }
    __syncthreads();
    // ---- values
#pragma unroll 2
    for (int ks = 0; ks < mts; ++ks) {
      uint32_t a0[4], a1[4];
#pragma unroll
      for (int a = 0; a < ACC; ++a) {
        if (piece0 + a >= pieces) break;
        if (a == 0 || woff[a] != woff[a - 1]) {
          ldsm_x4(a0, aw + woff[a] + ks * 32);
          if (!pack) ldsm_x4(a1, aw + plane_w + woff[a] + ks * 32);
        }
        uint32_t b[4];
        ldsm_x4_t(b, ak + koff[a] + (uint32_t)(ks * 16 * PD * 2));
        mma16816(acc[a][0], a0, b[0], b[1]);
        mma16816(acc[a][1], a0, b[2], b[3]);
        if (!pack) {
          mma16816(acc[a][0], a1, b[0], b[1]);
          mma16816(acc[a][1], a1, b[2], b[3]);
        }
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int a = 0; a < ACC; ++a) {
    const int piece = piece0 + a;
    if (piece >= pieces) break;
    const int gm = piece / DC, c = piece % DC, g = gm / mtiles, r0 = gm % mtiles * 16;
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        float v0 = acc[a][t][2 * hh], v1 = acc[a][t][2 * hh + 1];
        if (pack) {   // rows 8 .. 15 hold the second terms of rows 0 .. 7
          if (hh) continue;
          v0 += acc[a][t][2];
          v1 += acc[a][t][3];
        }
        const int row = r0 + g8 + 8 * hh, tok = row / hp, h = row % hp, d = c * 16 + t * 8 + 2 * t4;
        if (h >= share || tok >= w.ntok) continue;
        const size_t at = ((size_t)(w.qs + w.tok0 + tok) * H + g * share + h) * p.t.dim + d;
        if (p.mix_splits > 1) {
          float* o = p.ws_o + (size_t)split * p.t.T * H * p.t.dim + at;
          if (d < p.t.dim) o[0] = v0;
          if (d + 1 < p.t.dim) o[1] = v1;
        } else {
          __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(p.t.out) + at;
          if (d < p.t.dim) o[0] = __float2bfloat16(v0);
          if (d + 1 < p.t.dim) o[1] = __float2bfloat16(v1);
        }
      }
  }
}

// sum over the splits, for the tokens of this launch's requests
template <bool DEC>
__global__ void __launch_bounds__(256) talk_sum_kernel(const TalkTcParams p) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  int lo = 0, hi = p.t.R;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (p.t.query_start_loc[mid] <= t) lo = mid; else hi = mid;
  }
  const int n = p.t.query_start_loc[lo + 1] - p.t.query_start_loc[lo];
  if (t >= p.t.query_start_loc[lo + 1] || (n <= p.short_len) != DEC) return;
  const int row = p.t.H * p.t.dim;
  const size_t plane = (size_t)p.t.T * row;
  for (int i = threadIdx.x; i < row; i += 256) {
    const float* x = p.ws_o + (size_t)t * row + i;
    float s = 0.f;
    for (int k = 0; k < p.mix_splits; ++k) s += x[k * plane];
    reinterpret_cast<__nv_bfloat16*>(p.t.out)[(size_t)t * row + i] = __float2bfloat16(s);
  }
}

constexpr size_t kMaxSmem = 227 * 1024 - 256;

// the largest key tile that fits (0: none), and how many pieces a warp holds
int mix_tile(int G, int hp, int dp, int nqb, int& acc) {
  const MixGeom probe = mix_geom(G, hp, dp + 8, nqb, 16);
  const int pieces = G * probe.rgp / 16 * (dp / 16), warps = MT / 32;
  acc = pieces <= 4 * warps ? 4 : 8;
  if (pieces > 8 * warps) return 0;
  for (int kt = 128; kt >= 16; kt /= 2)
    if (G * kt <= 256 && mix_smem(mix_geom(G, hp, dp + 8, nqb, kt), probe.rg < 16) <= kMaxSmem) return kt;
  return 0;
}
int group_rows(int share) {
  for (int r = 1; r <= 32; r *= 2)
    if (r >= share) return r;
  return 0;
}
int prefill_blocks(int G, int hp, int dp) {
  int acc;
  for (int nqb : {4, 2})
    if (mix_tile(G, hp, dp, nqb, acc) >= 32) return nqb;
  return mix_tile(G, hp, dp, 2, acc) ? 2 : 0;
}

template <typename K> int allow(K kernel) { return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMaxSmem) == cudaSuccess ? 0 : -4; }

template <int DP, bool DEC>
int stats_go(const TalkTcParams& p, int blocks, cudaStream_t st) {
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (allow(talk_stats_kernel<DP, DEC>)) return -4;
    configured = true;
  }
  const size_t smem = (size_t)(SST * SK + (DEC ? 16 : 64)) * (DP + 8) * 2 + (SST * SK + 128) * 4;
  launch_k(talk_stats_kernel<DP, DEC>, dim3((unsigned)blocks, (unsigned)p.t.G, (unsigned)p.splits), dim3(128), smem, st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

template <int DP, int NQB, int ACC>
int mix_go(const TalkTcParams& p, int blocks, cudaStream_t st) {
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (allow(talk_mix_kernel<DP, NQB, ACC>)) return -4;
    configured = true;
  }
  const MixGeom m = mix_geom(p.t.G, p.t.group_rows, DP + 8, NQB, 1 << p.kt_shift);
  launch_k(talk_mix_kernel<DP, NQB, ACC>, dim3((unsigned)blocks, (unsigned)p.mix_splits), dim3(MT), mix_smem(m, m.rg < 16), st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

template <int DP>
int run(TalkTcParams p, bool dec, cudaStream_t st) {
  const int hp = p.t.group_rows, nqb = dec ? 1 : prefill_blocks(p.t.G, hp, DP);
  int acc;
  const int kt = mix_tile(p.t.G, hp, DP, nqb, acc);
  if (kt == 0) return -3;
  p.kt_shift = __builtin_ctz((unsigned)kt);
  p.bs_shift = __builtin_ctz((unsigned)p.t.bs);
  int rc = dec ? stats_go<DP, true>(p, p.t.R, st) : stats_go<DP, false>(p, p.stats_tiles, st);
  if (rc) return rc;
  const int blocks = dec ? p.t.R : p.mix_tiles;
  if (dec) rc = acc == 4 ? mix_go<DP, 1, 4>(p, blocks, st) : mix_go<DP, 1, 8>(p, blocks, st);
  else if (nqb == 4) rc = acc == 4 ? mix_go<DP, 4, 4>(p, blocks, st) : mix_go<DP, 4, 8>(p, blocks, st);
  else rc = acc == 4 ? mix_go<DP, 2, 4>(p, blocks, st) : mix_go<DP, 2, 8>(p, blocks, st);
  if (rc || p.mix_splits == 1) return rc;
  if (dec) launch_k(talk_sum_kernel<true>, dim3((unsigned)p.t.T), dim3(256), 0, st, true, p);
  else launch_k(talk_sum_kernel<false>, dim3((unsigned)p.t.T), dim3(256), 0, st, true, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace

bool talk_tc_sizes(int H, int G, int dim, TalkSizes* s) {
  if (H < 1 || G < 1 || H % G || dim < 1 || dim > 128) return false;
  const int hp = group_rows(H / G), dp = dim <= 64 ? 64 : 128;
  int acc;
  if (hp == 0) return false;
  const int nqb = prefill_blocks(G, hp, dp);
  // single tokens have a variant of their own where their rows fit one operand tile
  const bool dec = hp <= 16 && mix_tile(G, hp, dp, 1, acc) > 0;
  if (nqb == 0) return false;
  s->row = dp;
  s->group_rows = hp;
  s->stats_tokens = 64 / hp;
  s->mix_tokens = nqb * (hp <= 8 ? 8 / hp : 1);
  s->short_len = dec ? 1 : 0;
  return true;
}

int talk_tc_launch(const TalkTcParams& p, bool dec, cudaStream_t st) {
  TalkSizes s;
  if (p.t.T == 0) return 0;
  if (!talk_tc_sizes(p.t.H, p.t.G, p.t.dim, &s) || s.row != p.t.row || s.group_rows != p.t.group_rows || p.t.f32 || (p.t.bs & (p.t.bs - 1)) || p.splits < 1 || p.mix_splits < 1 ||
      p.short_len != s.short_len || (dec && s.short_len == 0) || p.ws_ml == nullptr || (p.mix_splits > 1 && p.ws_o == nullptr)) return -1;
  return p.t.row == 64 ? run<64>(p, dec, st) : run<128>(p, dec, st);
}

}  // namespace oc
