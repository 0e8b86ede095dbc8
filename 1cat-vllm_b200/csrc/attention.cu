// Paged-KV flash attention for head sizes 64, 128 and 256: causal, GQA-packed, variable-length batches where each
// request's queries are the last rows of its context (so decode, multi-token verify and chunked prefill over a cached
// prefix are one kernel family).
//   mode 0 (prefill): a CTA owns a tile of 64 (token, q-head-in-group) rows of one KV head; its 4 warps own 16 rows each
//                     and stream 64-key tiles of K and V through double-buffered shared memory.
//   mode 1 (decode / verify): rows fit in 16 or 32; the 4 warps split each 64-key tile by keys, grid.z splits the context
//                     (split-KV), partial (max, sum, O) are merged across warps in shared memory and across splits by a
//                     second small kernel.
// K/V pages are [block][2][Hkv][block_size][D] so one (page, head) is contiguous. Tensor-core math is bf16
// mma.sync.m16n8k16 with fp32 accumulation (softmax in the exp2 domain).
// Options for the Gemma / GPT-OSS / Mistral families: a sliding window (a query at position i sees keys i-window+1 .. i; key tiles
// wholly before the window are skipped), tanh soft-capping of the scaled scores, and per-head attention sinks (a learned logit that
// joins the softmax denominator only).
// FP8 KV cache (KV8): pages hold e4m3 bytes in the same layout; tiles stream through a byte-wide cp.async ring and are widened to
// bf16 into one working tile per operand before the MMAs; the per-tensor scales fold into the softmax scale (K) and the output (V).
// Extended variants (EXT, bf16 cache): first tokens that stay visible outside the window (their tiles are walked ahead of the window's),
// a bias by distance added to the scores in fp32, values that are the keys (one tensor per page: the ring holds one tile per stage and
// both products read it), one output gate per head. The softmax weights enter the value product as two bf16 terms (p and the rest of
// p after rounding), so that they keep about 16 bits of mantissa. In a decode tile of at most eight rows the second terms ride in the
// unused rows 8..15 of the same operand and cost no extra product.
// Chunks (EXT): a query sees the keys of its own chunk of the sequence; tiles before the chunk of a CTA's first row are skipped.
// Differential attention (DIFF, an extended variant): a head has two maps over the same values. A cached key row holds both maps' keys side
// by side and a query row belongs to one map. (Prompts with soft-capped scores run diff_prefill_tc.cu instead.) Prefill: warps 0 and 1 own the first map's rows, warps 2 and 3 the same rows of the
// second map, each multiplying its half of the key columns; the second map's output crosses over in shared memory. Decode: rows (head, map)
// lie next to one another with zeros in the other map's half (the tile has rows to spare), and the merge of the warps or splits takes
// the difference. Either way the difference, the head norm and the scale are part of the epilogue.
// (reference: flash-attention-v100/kernel/fused_mha_forward_paged.cu:364, flash_decode_paged.cu:667,831,1301;
//  v1/attention/backends/flash_attn_v100.py:2216 for the math)
#include <cuda_fp8.h>
#include <stdlib.h>

#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

constexpr int kKeysPerTile = 64;

__device__ __forceinline__ void cp_async16(void* smem, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
// byte offset of the 16-byte chunk `chunk` of row `row` in a [rows][D] bf16 tile with XOR swizzle
template <int D>
__device__ __forceinline__ uint32_t sw_off(int row, int chunk) {
  return (uint32_t)(row * D * 2 + ((chunk ^ (row & 7)) << 4));
}

// 16 e4m3 bytes -> 16 bf16, exactly (every e4m3 value is a bf16 value). A byte's sign goes to bit 15 and its exponent and mantissa
// four places below the top of the bf16 exponent field, which reads as value * 2^-120 (e4m3 subnormals become bf16 subnormals);
// one bf16x2 multiply by 2^120 restores the value.
__device__ __forceinline__ uint32_t widen_fp8_pair(uint32_t w, uint32_t sel) {
  uint32_t t;
  asm("prmt.b32 %0, %1, %2, %3;" : "=r"(t) : "r"(w), "r"(0u), "r"(sel));
  uint32_t v = (t & 0x80008000u) | ((t >> 4) & 0x07f007f0u);
  const uint32_t two120 = 0x7b807b80u;
  __nv_bfloat162 r = __hmul2(*reinterpret_cast<__nv_bfloat162*>(&v), *reinterpret_cast<const __nv_bfloat162*>(&two120));
  return *reinterpret_cast<uint32_t*>(&r);
}
__device__ __forceinline__ void widen_fp8x16(const uint4& in, uint4& lo, uint4& hi) {
  lo = make_uint4(widen_fp8_pair(in.x, 0x1404u), widen_fp8_pair(in.x, 0x3424u), widen_fp8_pair(in.y, 0x1404u), widen_fp8_pair(in.y, 0x3424u));
  hi = make_uint4(widen_fp8_pair(in.z, 0x1404u), widen_fp8_pair(in.z, 0x3424u), widen_fp8_pair(in.w, 0x1404u), widen_fp8_pair(in.w, 0x3424u));
}

constexpr float kLog2e = 1.4426950408889634f;

// sigmoid of the output gate of (token, head); 1 without a gate
__device__ __forceinline__ float head_gate(const AttnParams& p, size_t tok, int head) {
  if (p.gate == nullptr) return 1.f;
  return 1.f / (1.f + __expf(-__bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.gate)[tok * p.gate_st + head])));
}

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// tanh for soft caps in fp32: an odd polynomial (the series up to x^11, 3e-8 off at 0.4) near zero, (1 - e^-2x) / (1 + e^-2x) elsewhere
constexpr float kTanhSmall = 0.4f;
__device__ __forceinline__ float tanh_small(float x) {
  const float y = x * x;
  return x * fmaf(y, fmaf(y, fmaf(y, fmaf(y, fmaf(y, -1382.f / 155925.f, 62.f / 2835.f), -17.f / 315.f), 2.f / 15.f), -1.f / 3.f), 1.f);
}
__device__ __forceinline__ float tanh_any(float x) {
  const float e = ex2(-2.f * kLog2e * fabsf(x));
  return fabsf(x) < kTanhSmall ? tanh_small(x) : copysignf(__fdividef(1.f - e, 1.f + e), x);
}

// columns c and c + 1 (c even) of an output row of n elements
__device__ __forceinline__ void store_pair(__nv_bfloat16* dst, int c, int n, float x, float y) {
  if ((n & 1) == 0) {
    if (c < n) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(x, y);
  } else {
    if (c < n) dst[c] = __float2bfloat16(x);
    if (c + 1 < n) dst[c + 1] = __float2bfloat16(y);
  }
}

// CTAs per SM that the extended variants are compiled for (0: the compiler's choice)
template <int D, int MODE, int MB, bool EXT, bool DIFF>
constexpr int ext_min_ctas() {
  if (!EXT) return 0;
  if (DIFF) return D == 64 ? 3 : D == 128 ? 2 : 0;
  if (D == 64) return MODE == 0 ? 4 : (MB == 1 ? 5 : 3);
  if (D == 128) return MODE == 0 ? 3 : (MB == 1 ? 4 : 2);
  return 0;
}

template <int D, int MODE, int MB, bool KV8, int ST = 3, bool EXT = false, bool DIFF = false>
__global__ void __launch_bounds__(128, ext_min_ctas<D, MODE, MB, EXT, DIFF>()) attn_kernel(const AttnParams p) {
  static_assert(!DIFF || EXT, "differential attention is an extended variant");
  constexpr bool BY_MAP = DIFF && MODE == 0;    // rows 0..31 are the first map's, 32..63 the same rows of the second map
  pdl_trigger();
  pdl_wait();
  constexpr int STAGES = ST;                    // K/V tiles in the cp.async ring (a fourth stage of byte tiles measured no faster)
  constexpr int MBW = (MODE == 0) ? 1 : MB;     // 16-row blocks per warp
  constexpr int NB2 = (MODE == 0) ? 4 : 1;      // 16-key groups per warp per tile
  constexpr int ROWS = (MODE == 0) ? 64 : 16 * MB;
  constexpr int CH = D / 8;                     // 16-byte chunks per row
  extern __shared__ __align__(128) uint8_t smem[];
  // bf16 cache: sK / sV are the cp.async rings of bf16 tiles. fp8 cache: they are rings of byte tiles, followed by one bf16
  // working tile per operand (sKb / sVb)
  constexpr int ESZ = KV8 ? 1 : 2;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + ROWS * D * 2;
  const bool shared_kv = EXT && p.kv_shared;    // one tile per stage serves both products
  uint8_t* sV = shared_kv ? sK : sK + STAGES * kKeysPerTile * D * ESZ;
  uint8_t* sKb = sV + STAGES * kKeysPerTile * D * ESZ;
  uint8_t* sVb = sKb + kKeysPerTile * D * 2;
  __shared__ int s_req, s_tile0;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = p.Hq / p.Hkv;
  const int hkv = blockIdx.y;
  int r, tq0, tq1;
  if (MODE == 0) {
    const int TQ = 64 / G;
    if (threadIdx.x == 0) {
      int b = blockIdx.x, found = -1, t0 = 0;
      for (int i = 0; i < p.R; ++i) {
        int ql = p.query_start_loc[i + 1] - p.query_start_loc[i];
        int nt = (ql > p.short_q_len) ? (ql + TQ - 1) / TQ : 0;  // short queries belong to the decode kernel
        if (b < nt) { found = i; t0 = b * TQ; break; }
        b -= nt;
      }
      s_req = found;
      s_tile0 = t0;
    }
    __syncthreads();
    r = s_req;
    if (r < 0) return;
    tq0 = s_tile0;
    int ql = p.query_start_loc[r + 1] - p.query_start_loc[r];
    tq1 = min(tq0 + TQ, ql);
  } else {
    r = blockIdx.x;
    tq0 = 0;
    tq1 = p.query_start_loc[r + 1] - p.query_start_loc[r];
    if (tq1 > p.short_q_len) return;  // long queries belong to the prefill kernel (uniform exit: before any barrier)
  }
  const int qs = p.query_start_loc[r];
  const int qlen = p.query_start_loc[r + 1] - qs;
  const int S = p.seq_lens[r];
  if (qlen <= 0 || S <= 0) return;
  const int ctx0 = S - qlen;
  const int Gr = BY_MAP ? G / 2 : G;            // rows per token of a block of rows
  const int nrows = (tq1 - tq0) * Gr;
  auto row_tok = [&](int row) { return (BY_MAP ? row & 31 : row) / Gr; };
  const int kv_end = min(S, ctx0 + tq1);
  const int ntiles = (kv_end + kKeysPerTile - 1) / kKeysPerTile;
  // sliding window: the first row of the tile sees the earliest key, ctx0 + tq0 - window + 1
  const int wlo = p.window > 0 ? p.window : 0x3fffffff;
  // earliest key that a position sees (kept tokens aside)
  auto first_key = [&](int pos) {
    int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    if (EXT && p.chunk > 0) lo = max(lo, pos - pos % p.chunk);
    return lo;
  };
  const int tile_first = first_key(ctx0 + tq0) / kKeysPerTile;
  int tile_lo = tile_first, tile_hi = ntiles;
  // kept first tokens: their tiles that lie wholly before the window are walked first (tile index - tile_shift for those)
  int keep_tiles = 0;
  if (EXT) {
    keep_tiles = min((p.keep + kKeysPerTile - 1) / kKeysPerTile, tile_first);
    tile_lo -= keep_tiles;
  }
  const int tile_shift = tile_first - keep_tiles, tile_first_v = tile_lo;
  auto tile_of = [&](int v) { return (EXT && v < tile_first) ? v - tile_shift : v; };
  if (MODE == 1 && p.splits > 1) {
    int per = (ntiles - tile_first_v + p.splits - 1) / p.splits;
    tile_lo = tile_first_v + blockIdx.z * per;
    tile_hi = min(ntiles, tile_lo + per);
  }
  const int* bt = p.block_table + (size_t)r * p.bt_stride;
  const size_t page_elems = (size_t)p.bs * D;

  // each thread always copies the same 16-byte column chunk of rows (tid / CH) + i * (128 / CH); pages are a power of
  // two tokens long, so the block-table lookup is a shift and a mask
  constexpr int LCH = KV8 ? D / 16 : CH;        // 16-byte chunks per cache row
  const int ld_ch = threadIdx.x % LCH, ld_row0 = threadIdx.x / LCH;
  constexpr int kRowStep = 128 / LCH;
  const int bs_shift = p.bs_shift, bs_mask = p.bs - 1;
  // byte addressing covers both element sizes
  const uint8_t* kv_head = reinterpret_cast<const uint8_t*>(p.kv_cache) + ((size_t)hkv * page_elems) * ESZ + ld_ch * 16;
  const size_t blk_stride = (size_t)(shared_kv ? 1 : 2) * p.Hkv * page_elems * ESZ, v_off = (size_t)p.Hkv * page_elems * ESZ;
  // One block-table lookup per 16-key chunk of the tile: pages are at least 16 keys long and tiles start at multiples of 64, so
  // the 16 / kRowStep rows that a thread copies inside a chunk share a page.
  auto load_tile = [&](int tile, int buf) {
    const int k0 = tile * kKeysPerTile;
    uint8_t* dk = sK + (size_t)buf * kKeysPerTile * D * ESZ;
    uint8_t* dv = sV + (size_t)buf * kKeysPerTile * D * ESZ;
    if constexpr (kRowStep <= 16) {
      constexpr int RPC = 16 / kRowStep;
#pragma unroll
      for (int c = 0; c < kKeysPerTile / 16; ++c) {
        const int key_c = k0 + c * 16;
        const uint8_t* src = kv_head;
        if (key_c < kv_end) src += (size_t)bt[key_c >> bs_shift] * blk_stride + (size_t)((key_c & bs_mask) + ld_row0) * (D * ESZ);
#pragma unroll
        for (int j = 0; j < RPC; ++j) {
          const int row = c * 16 + ld_row0 + j * kRowStep;
          const uint32_t off = KV8 ? (uint32_t)(row * D + ld_ch * 16) : sw_off<D>(row, ld_ch);
          if (k0 + row < kv_end) {
            cp_async16(dk + off, src + (size_t)j * (kRowStep * D * ESZ));
            if (!shared_kv) cp_async16(dv + off, src + (size_t)j * (kRowStep * D * ESZ) + v_off);
          } else {
            *reinterpret_cast<uint4*>(dk + off) = make_uint4(0, 0, 0, 0);
            *reinterpret_cast<uint4*>(dv + off) = make_uint4(0, 0, 0, 0);
          }
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < kKeysPerTile / kRowStep; ++i) {
        const int row = ld_row0 + i * kRowStep;
        const int key = k0 + row;
        const uint32_t off = KV8 ? (uint32_t)(row * D + ld_ch * 16) : sw_off<D>(row, ld_ch);
        if (key < kv_end) {
          const int blk = bt[key >> bs_shift];
          const uint8_t* src = kv_head + (size_t)blk * blk_stride + (size_t)(key & bs_mask) * D * ESZ;
          cp_async16(dk + off, src);
          if (!shared_kv) cp_async16(dv + off, src + v_off);
        } else {
          *reinterpret_cast<uint4*>(dk + off) = make_uint4(0, 0, 0, 0);
          *reinterpret_cast<uint4*>(dv + off) = make_uint4(0, 0, 0, 0);
        }
      }
    }
  };

  // Decode: the four warps see disjoint keys, so each warp streams its own 16 keys of every tile through its own cp.async groups
  // (and widens its own e4m3 bytes) and the main loop needs no CTA-wide barrier: the warps drift apart and hide one another's
  // latencies (measured in lock step, a CTA took 1.9 us per tile, a dependent chain of copy wait, barrier, QK, softmax, PV).
  constexpr bool WARP_PIPE = (MODE == 1);
  constexpr int WCH = KV8 ? D / 16 : CH;        // 16-byte chunks per cache row
  const uint8_t* kv_warp = reinterpret_cast<const uint8_t*>(p.kv_cache) + ((size_t)hkv * page_elems) * ESZ;
  // Extended variants read a tile's block-table entry one iteration before its copies are issued, so that its latency is not in the way
  // of this iteration's products.
  int next_blk = 0;
  auto peek_blk = [&](int v) {
    const int key0 = tile_of(v) * kKeysPerTile + warp * 16;
    next_blk = (v < tile_hi && key0 < kv_end) ? __ldg(bt + (key0 >> bs_shift)) : 0;
  };
  auto load_tile_w = [&](int tile, int buf, int blk) {
    const int key0 = tile * kKeysPerTile + warp * 16;
    uint8_t* dk = sK + (size_t)buf * kKeysPerTile * D * ESZ;
    uint8_t* dv = sV + (size_t)buf * kKeysPerTile * D * ESZ;
    const uint8_t* src = kv_warp;
    if (key0 < kv_end) src += (size_t)(EXT ? blk : bt[key0 >> bs_shift]) * blk_stride + (size_t)(key0 & bs_mask) * (D * ESZ);
#pragma unroll
    for (int i = 0; i < 16 * WCH / 32; ++i) {
      const int idx = lane + 32 * i, rl = idx / WCH, ch = idx % WCH;
      const uint32_t off = KV8 ? (uint32_t)((warp * 16 + rl) * D + ch * 16) : sw_off<D>(warp * 16 + rl, ch);
      if (key0 + rl < kv_end) {
        cp_async16(dk + off, src + (size_t)rl * (D * ESZ) + ch * 16);
        if (!shared_kv) cp_async16(dv + off, src + (size_t)rl * (D * ESZ) + ch * 16 + v_off);
      } else {
        *reinterpret_cast<uint4*>(dk + off) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(dv + off) = make_uint4(0, 0, 0, 0);
      }
    }
  };

  float o[MBW][D / 8][4];
  float mrow[MBW][2], lrow[MBW][2];
#pragma unroll
  for (int b = 0; b < MBW; ++b) {
    mrow[b][0] = mrow[b][1] = -INFINITY;
    lrow[b][0] = lrow[b][1] = 0.f;
#pragma unroll
    for (int i = 0; i < D / 8; ++i) o[b][i][0] = o[b][i][1] = o[b][i][2] = o[b][i][3] = 0.f;
  }
  // plain: s * scale * log2(e); soft-capped: cap * tanh(s * scale / cap) * log2(e)
  const bool capped = p.softcap > 0.f;
  const float qk_scale = KV8 ? p.scale * p.k_scale : p.scale;   // K was stored as k / k_scale
  const float sc = capped ? qk_scale / p.softcap : qk_scale * 1.4426950408889634f;
  const float sc_post = p.softcap * 1.4426950408889634f;
  const int row_base = (MODE == 0) ? warp * 16 : 0;
  const int key_base = (MODE == 0) ? 0 : warp * 16;
  const int g_ = lane >> 2, tg = lane & 3;

  // extended variants: what the rows of this thread need in every tile
  int row_pos[MBW][2], row_lo[MBW][2];
  const float* row_bias[MBW][2];
  float row_far[MBW][2];
  int pos_lo = 0, pos_hi = 0, lo_hi = 0;
  const bool paired = EXT && MODE == 1 && MB == 1 && nrows <= 8;   // rows 8..15 carry the second terms of rows 0..7
  if constexpr (EXT) {
    pos_lo = ctx0 + tq0 + row_tok(row_base);
    pos_hi = ctx0 + tq0 + row_tok(row_base + 16 * MBW - 1);
    lo_hi = first_key(pos_hi);
#pragma unroll
    for (int b = 0; b < MBW; ++b)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int row = row_base + b * 16 + g_ + h * 8, tok = row_tok(row);
        row_pos[b][h] = ctx0 + tq0 + tok;
        row_lo[b][h] = first_key(row_pos[b][h]);
        row_bias[b][h] = p.bias != nullptr ? p.bias + (size_t)(hkv * G + row - tok * G) * p.bias_len : nullptr;
        row_far[b][h] = p.bias != nullptr ? __ldg(row_bias[b][h] + p.bias_len - 1) * kLog2e : 0.f;
      }
  }
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) {
    if (tile_lo + i < tile_hi) {
      if constexpr (WARP_PIPE) {
        if constexpr (EXT) peek_blk(tile_lo + i);
        load_tile_w(tile_of(tile_lo + i), i, next_blk);
      }
      else load_tile(tile_of(tile_lo + i), i);
    }
    cp_async_commit();
  }
  // ---- Q tile -> shared memory (zero rows past the end), behind the first K/V copies so that its latency overlaps theirs; the
  // first barrier of the loop publishes it
  for (int idx = threadIdx.x; idx < ROWS * CH; idx += 128) {
    int row = idx / CH, ch = idx % CH;
    uint4 v = make_uint4(0, 0, 0, 0);
    if constexpr (DIFF) {
      const int rr = BY_MAP ? row & 31 : row, tok = tq0 + rr / Gr, gh = BY_MAP ? (rr % Gr) * 2 + (row >> 5) : rr % Gr;
      if (rr < nrows && ch / (CH / 2) == (gh & 1))
        v = *reinterpret_cast<const uint4*>(p.q + (size_t)(qs + tok) * p.q_st + (size_t)(hkv * G + gh) * p.q_sh + (ch % (CH / 2)) * 8);
    } else if (row < nrows) {
      int tok = tq0 + row / G, gh = row % G;
      v = *reinterpret_cast<const uint4*>(p.q + (size_t)(qs + tok) * p.q_st + (size_t)(hkv * G + gh) * p.q_sh + ch * 8);
    }
    *reinterpret_cast<uint4*>(sQ + sw_off<D>(row, ch)) = v;
  }
  if constexpr (WARP_PIPE && EXT) peek_blk(tile_lo + STAGES - 1);
  if constexpr (WARP_PIPE) __syncthreads();  // publishes the Q tile; the loop below has no CTA-wide barrier

  for (int tile = tile_lo; tile < tile_hi; ++tile) {
    const int buf = (tile - tile_lo) % STAGES;
    cp_async_wait<STAGES - 2>();  // the group of this tile has landed (one group is committed per iteration)
    if constexpr (WARP_PIPE) {
      __syncwarp();                // ...for every lane of this warp, whose ldmatrix reads of the buffer refilled below are done
      if (tile + STAGES - 1 < tile_hi) load_tile_w(tile_of(tile + STAGES - 1), (tile - tile_lo + STAGES - 1) % STAGES, next_blk);
      if constexpr (EXT) peek_blk(tile + STAGES);
    } else {
      __syncthreads();             // ...for every thread, and everybody has finished the buffer refilled below
      if (tile + STAGES - 1 < tile_hi) load_tile(tile_of(tile + STAGES - 1), (tile - tile_lo + STAGES - 1) % STAGES);
    }
    cp_async_commit();
    if (KV8) {
      const uint8_t* k8 = sK + (size_t)buf * kKeysPerTile * D;
      const uint8_t* v8 = sV + (size_t)buf * kKeysPerTile * D;
      if constexpr (WARP_PIPE) {
        // this warp's 16 keys -> its rows of the bf16 working tiles (its own MMAs of the previous tile are done: program order)
#pragma unroll
        for (int i = 0; i < 16 * WCH / 32; ++i) {
          const int idx = lane + 32 * i, row = warp * 16 + idx / WCH, ch = idx % WCH;
          uint4 lo, hi;
          widen_fp8x16(*reinterpret_cast<const uint4*>(k8 + row * D + ch * 16), lo, hi);
          *reinterpret_cast<uint4*>(sKb + sw_off<D>(row, ch * 2)) = lo;
          *reinterpret_cast<uint4*>(sKb + sw_off<D>(row, ch * 2 + 1)) = hi;
          widen_fp8x16(*reinterpret_cast<const uint4*>(v8 + row * D + ch * 16), lo, hi);
          *reinterpret_cast<uint4*>(sVb + sw_off<D>(row, ch * 2)) = lo;
          *reinterpret_cast<uint4*>(sVb + sw_off<D>(row, ch * 2 + 1)) = hi;
        }
        __syncwarp();
      } else {
        // widen this tile's bytes into the bf16 working tiles (everyone is past the previous tile's MMAs: barrier above)
#pragma unroll
        for (int i = 0; i < kKeysPerTile / kRowStep; ++i) {
          const int row = ld_row0 + i * kRowStep;
          uint4 lo, hi;
          widen_fp8x16(*reinterpret_cast<const uint4*>(k8 + row * D + ld_ch * 16), lo, hi);
          *reinterpret_cast<uint4*>(sKb + sw_off<D>(row, ld_ch * 2)) = lo;
          *reinterpret_cast<uint4*>(sKb + sw_off<D>(row, ld_ch * 2 + 1)) = hi;
          widen_fp8x16(*reinterpret_cast<const uint4*>(v8 + row * D + ld_ch * 16), lo, hi);
          *reinterpret_cast<uint4*>(sVb + sw_off<D>(row, ld_ch * 2)) = lo;
          *reinterpret_cast<uint4*>(sVb + sw_off<D>(row, ld_ch * 2 + 1)) = hi;
        }
        __syncthreads();
      }
    }
    const uint32_t kb = smem_u32(KV8 ? sKb : sK + (size_t)buf * kKeysPerTile * D * 2);
    const uint32_t vb = smem_u32(KV8 ? sVb : sV + (size_t)buf * kKeysPerTile * D * 2);
    const uint32_t qb = smem_u32(sQ);
    const int k0 = tile_of(tile) * kKeysPerTile + key_base;

    // ---- S = Q K^T
    float s[MBW][NB2 * 2][4];
#pragma unroll
    for (int b = 0; b < MBW; ++b)
#pragma unroll
      for (int n = 0; n < NB2 * 2; ++n) s[b][n][0] = s[b][n][1] = s[b][n][2] = s[b][n][3] = 0.f;
    const int ch0 = BY_MAP ? (warp >> 1) * (CH / 2) : 0;   // this warp's half of the key columns
#pragma unroll
    for (int kk = 0; kk < (BY_MAP ? D / 32 : D / 16); ++kk) {
      uint32_t a[MBW][4];
#pragma unroll
      for (int b = 0; b < MBW; ++b) {
        int row = row_base + b * 16 + (lane & 15);
        ldsm_x4(a[b], qb + sw_off<D>(row, ch0 + kk * 2 + (lane >> 4)));
      }
#pragma unroll
      for (int n2 = 0; n2 < NB2; ++n2) {
        uint32_t bfr[4];
        int krow = key_base + n2 * 16 + (lane & 7) + ((lane >> 4) << 3);
        ldsm_x4(bfr, kb + sw_off<D>(krow, ch0 + kk * 2 + ((lane >> 3) & 1)));
#pragma unroll
        for (int b = 0; b < MBW; ++b) {
          mma_bf16(s[b][n2 * 2], a[b], bfr[0], bfr[1]);
          mma_bf16(s[b][n2 * 2 + 1], a[b], bfr[2], bfr[3]);
        }
      }
    }
    // ---- mask, online softmax
    float alpha_r[MBW][2];
    // whole tiles of this warp that need neither masking nor a per-key bias
    bool no_mask = false, far_bias = false;
    if constexpr (EXT) {
      const int k_hi = k0 + NB2 * 16 - 1;
      no_mask = k_hi <= pos_lo && k_hi < kv_end && (k0 >= lo_hi || k_hi < p.keep);
      far_bias = p.bias == nullptr || pos_lo - k_hi >= p.bias_len - 1;   // one value per row (0 without a bias)
    }
#pragma unroll
    for (int b = 0; b < MBW; ++b) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        if (paired && h == 1) {
          alpha_r[b][1] = alpha_r[b][0];
          continue;
        }
        const int row = row_base + b * 16 + g_ + h * 8;
        const int qpos = EXT ? row_pos[b][h] : ctx0 + tq0 + row / G;  // rows past nrows are never stored
        if constexpr (EXT) {
          // one decision per tile and row instead of one per score
          auto each = [&](auto f) {
#pragma unroll
            for (int n = 0; n < NB2 * 2; ++n)
#pragma unroll
              for (int e = 0; e < 2; ++e) s[b][n][h * 2 + e] = f(s[b][n][h * 2 + e], k0 + n * 8 + tg * 2 + e);
          };
          const float far = row_far[b][h];
          if (far_bias && !capped) {
            each([&](float v, int) { return fmaf(v, sc, far); });
          } else {
            if (capped) {
              float top = 0.f;
              each([&](float v, int) { top = fmaxf(top, fabsf(v)); return v; });
              if (__any_sync(0xffffffffu, top * fabsf(sc) >= kTanhSmall)) each([&](float v, int) { return tanh_any(v * sc) * sc_post; });
              else each([&](float v, int) { return tanh_small(v * sc) * sc_post; });
            } else {
              each([&](float v, int) { return v * sc; });
            }
            if (far_bias) each([&](float v, int) { return v + far; });
            else each([&](float v, int key) { return fmaf(__ldg(row_bias[b][h] + min(max(qpos - key, 0), p.bias_len - 1)), kLog2e, v); });
          }
          if (!no_mask)
            each([&](float v, int key) { return (key <= qpos && key < kv_end && (key >= row_lo[b][h] || key < p.keep)) ? v : -INFINITY; });
        }
        float mx = -INFINITY;
#pragma unroll
        for (int n = 0; n < NB2 * 2; ++n) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            int key = k0 + n * 8 + tg * 2 + e;
            float v = s[b][n][h * 2 + e];
            if constexpr (!EXT) {
              v *= sc;
              if (capped) v = tanhf(v) * sc_post;
              v = (key <= qpos && key < kv_end && key + wlo > qpos) ? v : -INFINITY;
            }
            s[b][n][h * 2 + e] = v;
            mx = fmaxf(mx, v);
          }
        }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(mrow[b][h], mx);
        const float m_use = (m_new == -INFINITY) ? 0.f : m_new;
        const float alpha = exp2f(mrow[b][h] - m_use);
        float sum = 0.f;
#pragma unroll
        for (int n = 0; n < NB2 * 2; ++n) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float pv = exp2f(s[b][n][h * 2 + e] - m_use);
            s[b][n][h * 2 + e] = pv;
            sum += pv;
          }
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        lrow[b][h] = lrow[b][h] * alpha + sum;
        mrow[b][h] = m_new;
        alpha_r[b][h] = alpha;
      }
    }
    // the running maxima settle after a few tiles: rescale the accumulator only when some row of the warp moved
#pragma unroll
    for (int b = 0; b < MBW; ++b) {
      if (__any_sync(0xffffffffu, alpha_r[b][0] != 1.f || alpha_r[b][1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < D / 8; ++i) {
          o[b][i][0] *= alpha_r[b][0];
          o[b][i][1] *= alpha_r[b][0];
          o[b][i][2] *= alpha_r[b][1];
          o[b][i][3] *= alpha_r[b][1];
        }
      }
    }
    // ---- O += P V
#pragma unroll
    for (int n2 = 0; n2 < NB2; ++n2) {
      uint32_t a[MBW][4];
#pragma unroll
      for (int b = 0; b < MBW; ++b) {
        a[b][0] = pack_bf16(s[b][n2 * 2][0], s[b][n2 * 2][1]);
        a[b][1] = pack_bf16(s[b][n2 * 2][2], s[b][n2 * 2][3]);
        a[b][2] = pack_bf16(s[b][n2 * 2 + 1][0], s[b][n2 * 2 + 1][1]);
        a[b][3] = pack_bf16(s[b][n2 * 2 + 1][2], s[b][n2 * 2 + 1][3]);
      }
      uint32_t lo[MBW][4];   // what rounding took from the weights, as a second bf16 term
      if constexpr (EXT) {
        auto rest = [](uint32_t hi, float x, float y) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(&hi));
          return pack_bf16(x - f.x, y - f.y);
        };
        if (paired) {
          a[0][1] = rest(a[0][0], s[0][n2 * 2][0], s[0][n2 * 2][1]);
          a[0][3] = rest(a[0][2], s[0][n2 * 2 + 1][0], s[0][n2 * 2 + 1][1]);
        } else {
#pragma unroll
          for (int b = 0; b < MBW; ++b) {
            lo[b][0] = rest(a[b][0], s[b][n2 * 2][0], s[b][n2 * 2][1]);
            lo[b][1] = rest(a[b][1], s[b][n2 * 2][2], s[b][n2 * 2][3]);
            lo[b][2] = rest(a[b][2], s[b][n2 * 2 + 1][0], s[b][n2 * 2 + 1][1]);
            lo[b][3] = rest(a[b][3], s[b][n2 * 2 + 1][2], s[b][n2 * 2 + 1][3]);
          }
        }
      }
#pragma unroll
      for (int d2 = 0; d2 < D / 16; ++d2) {
        uint32_t bfr[4];
        int krow = key_base + n2 * 16 + (lane & 15);
        ldsm_x4_t(bfr, vb + sw_off<D>(krow, d2 * 2 + (lane >> 4)));
#pragma unroll
        for (int b = 0; b < MBW; ++b) {
          mma_bf16(o[b][d2 * 2], a[b], bfr[0], bfr[1]);
          mma_bf16(o[b][d2 * 2 + 1], a[b], bfr[2], bfr[3]);
          if (EXT && !paired) {
            mma_bf16(o[b][d2 * 2], lo[b], bfr[0], bfr[1]);
            mma_bf16(o[b][d2 * 2 + 1], lo[b], bfr[2], bfr[3]);
          }
        }
      }
    }
  }
  cp_async_wait<0>();

  if constexpr (BY_MAP) {
    // the second map's output crosses over to the warps of the first one: same rows, same registers
    float inv[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) inv[h] = lrow[0][h] > 0.f ? 1.f / lrow[0][h] : 0.f;
    __syncthreads();   // everyone is done reading K/V tiles
    float2* xch = reinterpret_cast<float2*>(sK) + (warp & 1) * (D / 8) * 2 * 32 + lane;
    if (warp >= 2) {
#pragma unroll
      for (int i = 0; i < D / 8; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) xch[(i * 2 + h) * 32] = make_float2(o[0][i][h * 2] * inv[h], o[0][i][h * 2 + 1] * inv[h]);
    }
    __syncthreads();
    if (warp >= 2) return;
    const float lam = *p.lam;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < D / 8; ++i) {
        const float2 b = xch[(i * 2 + h) * 32];
        const float x = o[0][i][h * 2] * inv[h] - lam * b.x, y = o[0][i][h * 2 + 1] * inv[h] - lam * b.y;
        o[0][i][h * 2] = x;
        o[0][i][h * 2 + 1] = y;
        ss = fmaf(x, x, fmaf(y, y, ss));
      }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      const int row = row_base + g_ + h * 8;
      if (row >= nrows) continue;
      const float f = p.out_scale / sqrtf(ss / (float)p.vdim + p.eps);
      __nv_bfloat16* dst = p.out + ((size_t)(qs + tq0 + row / Gr) * (p.Hq / 2) + hkv * Gr + row % Gr) * p.vdim;
#pragma unroll
      for (int i = 0; i < D / 8; ++i) store_pair(dst, i * 8 + tg * 2, p.vdim, o[0][i][h * 2] * f, o[0][i][h * 2 + 1] * f);
    }
    return;
  }
  if (MODE == 0) {
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int row = row_base + g_ + h * 8;
      if (row >= nrows) continue;
      const int tok = tq0 + row / G, gh = row % G;
      const float den = lrow[0][h] + (p.sinks != nullptr ? exp2f(p.sinks[hkv * G + gh] * 1.4426950408889634f - mrow[0][h]) : 0.f);
      float inv = den > 0.f ? (KV8 ? p.v_scale : 1.f) / den : 0.f;
      if constexpr (EXT) inv *= head_gate(p, (size_t)(qs + tok), hkv * G + gh);
      __nv_bfloat16* dst = p.out + ((size_t)(qs + tok) * p.Hq + hkv * G + gh) * D;
#pragma unroll
      for (int i = 0; i < D / 8; ++i)
        *reinterpret_cast<uint32_t*>(dst + i * 8 + tg * 2) = pack_bf16(o[0][i][h * 2] * inv, o[0][i][h * 2 + 1] * inv);
      if (p.lse != nullptr && tg == 0)
        p.lse[(size_t)(qs + tok) * p.Hq + hkv * G + gh] = (mrow[0][h] + log2f(lrow[0][h])) * 0.6931471805599453f;
    }
    return;
  }

  // ---- mode 1: merge the four warps' partial results (they saw disjoint keys), then store or hand to the split combine
  __syncthreads();  // everyone is done reading K/V tiles; reuse that memory
  if (paired) {
#pragma unroll
    for (int i = 0; i < D / 8; ++i) {
      o[0][i][0] += o[0][i][2];
      o[0][i][1] += o[0][i][3];
    }
  }
  float* mo = reinterpret_cast<float*>(sK);             // [4][ROWS][D]
  float* mm = reinterpret_cast<float*>(sQ);             // [4][ROWS][2] (the Q tile is no longer needed)
#pragma unroll
  for (int b = 0; b < MBW; ++b)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int row = b * 16 + g_ + h * 8;
      float* dst = mo + ((size_t)warp * ROWS + row) * D;
#pragma unroll
      for (int i = 0; i < D / 8; ++i) {
        dst[i * 8 + tg * 2] = o[b][i][h * 2];
        dst[i * 8 + tg * 2 + 1] = o[b][i][h * 2 + 1];
      }
      if (tg == 0) {
        mm[((size_t)warp * ROWS + row) * 2] = mrow[b][h];
        mm[((size_t)warp * ROWS + row) * 2 + 1] = lrow[b][h];
      }
    }
  __syncthreads();
  if constexpr (DIFF) {
    if (p.splits == 1) {   // one warp per (token, head): rows 2 * pair and 2 * pair + 1 are its maps
      const float lam = *p.lam;
      for (int pair = warp; pair * 2 < nrows; pair += 4) {
        float f[2][4];
#pragma unroll
        for (int m = 0; m < 2; ++m) {
          float M = -INFINITY, L = 0.f;
#pragma unroll
          for (int w = 0; w < 4; ++w) M = fmaxf(M, mm[((size_t)w * ROWS + pair * 2 + m) * 2]);
#pragma unroll
          for (int w = 0; w < 4; ++w) {
            const float* ml = mm + ((size_t)w * ROWS + pair * 2 + m) * 2;
            f[m][w] = ml[0] == -INFINITY ? 0.f : exp2f(ml[0] - M);
            L += ml[1] * f[m][w];
          }
          const float inv = L > 0.f ? (m == 0 ? 1.f : -lam) / L : 0.f;
#pragma unroll
          for (int w = 0; w < 4; ++w) f[m][w] *= inv;
        }
        float x[D / 32], ss = 0.f;
#pragma unroll
        for (int i = 0; i < D / 32; ++i) {
          x[i] = 0.f;
#pragma unroll
          for (int w = 0; w < 4; ++w) {
            const float* src = mo + ((size_t)w * ROWS + pair * 2) * D + lane + 32 * i;
            x[i] = fmaf(src[0], f[0][w], fmaf(src[D], f[1][w], x[i]));
          }
          ss = fmaf(x[i], x[i], ss);
        }
        const float g = p.out_scale / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
        const int tok = pair / (G / 2), gh = pair % (G / 2);
        __nv_bfloat16* dst = p.out + ((size_t)(qs + tok) * (p.Hq / 2) + hkv * (G / 2) + gh) * p.vdim;
#pragma unroll
        for (int i = 0; i < D / 32; ++i)
          if (lane + 32 * i < p.vdim) dst[lane + 32 * i] = __float2bfloat16(x[i] * g);
      }
      return;
    }
  }
  for (int idx = threadIdx.x; idx < nrows * (D / 4); idx += 128) {
    const int row = idx / (D / 4), c4 = (idx % (D / 4)) * 4;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) M = fmaxf(M, mm[((size_t)w * ROWS + row) * 2]);
    float L = 0.f, acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      float mw = mm[((size_t)w * ROWS + row) * 2];
      float f = (mw == -INFINITY) ? 0.f : exp2f(mw - M);
      L += mm[((size_t)w * ROWS + row) * 2 + 1] * f;
      const float4 v = *reinterpret_cast<const float4*>(mo + ((size_t)w * ROWS + row) * D + c4);
      acc[0] += v.x * f; acc[1] += v.y * f; acc[2] += v.z * f; acc[3] += v.w * f;
    }
    const int tok = row / G, gh = row % G;
    const size_t orow = (size_t)(qs + tok) * p.Hq + hkv * G + gh;
    if (p.splits > 1) {
      float* wo = p.ws_o + ((size_t)blockIdx.z * p.T * p.Hq + orow) * D + c4;
      *reinterpret_cast<float4*>(wo) = make_float4(acc[0], acc[1], acc[2], acc[3]);
      if (c4 == 0) {
        float* wm = p.ws_ml + ((size_t)blockIdx.z * p.T * p.Hq + orow) * 2;
        wm[0] = M;
        wm[1] = L;
      }
    } else {
      const float den = L + (p.sinks != nullptr ? exp2f(p.sinks[hkv * G + gh] * 1.4426950408889634f - M) : 0.f);
      float inv = den > 0.f ? (KV8 ? p.v_scale : 1.f) / den : 0.f;
      if constexpr (EXT) inv *= head_gate(p, (size_t)(qs + tok), hkv * G + gh);
      __nv_bfloat16* dst = p.out + orow * D + c4;
      *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16(acc[0] * inv, acc[1] * inv), pack_bf16(acc[2] * inv, acc[3] * inv));
      if (p.lse != nullptr && c4 == 0) p.lse[orow] = (M + log2f(L)) * 0.6931471805599453f;
    }
  }
}

// merges split-KV partials: one warp per (token, head)
template <int D>
__global__ void attn_combine_kernel(const AttnParams p) {
  pdl_trigger();
  pdl_wait();
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  const int rows = p.T * p.Hq;
  if (warp >= rows) return;
  float M = -INFINITY;
  for (int s = 0; s < p.splits; ++s) M = fmaxf(M, p.ws_ml[((size_t)s * rows + warp) * 2]);
  float L = 0.f;
  float acc[D / 32];
#pragma unroll
  for (int i = 0; i < D / 32; ++i) acc[i] = 0.f;
  for (int s = 0; s < p.splits; ++s) {
    const float ms = p.ws_ml[((size_t)s * rows + warp) * 2];
    const float f = (ms == -INFINITY) ? 0.f : exp2f(ms - M);
    L += p.ws_ml[((size_t)s * rows + warp) * 2 + 1] * f;
    const float* src = p.ws_o + ((size_t)s * rows + warp) * D;
#pragma unroll
    for (int i = 0; i < D / 32; ++i) acc[i] += src[lane + 32 * i] * f;
  }
  const float den = L + (p.sinks != nullptr ? exp2f(p.sinks[warp % p.Hq] * 1.4426950408889634f - M) : 0.f);
  const float inv = (den > 0.f ? (p.kv_fp8 ? p.v_scale : 1.f) / den : 0.f) * head_gate(p, (size_t)(warp / p.Hq), warp % p.Hq);
#pragma unroll
  for (int i = 0; i < D / 32; ++i) p.out[(size_t)warp * D + lane + 32 * i] = __float2bfloat16(acc[i] * inv);
  if (p.lse != nullptr && lane == 0) p.lse[warp] = (M + log2f(L)) * 0.6931471805599453f;
}

// the same for the two maps of a head: one warp per (token, head)
template <int D>
__global__ void diff_combine_kernel(const AttnParams p) {
  pdl_trigger();
  pdl_wait();
  const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  const size_t rows = (size_t)p.T * p.Hq;
  if ((size_t)warp * 2 >= rows) return;
  const float lam = *p.lam;
  float x[D / 32];
#pragma unroll
  for (int i = 0; i < D / 32; ++i) x[i] = 0.f;
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const size_t row = (size_t)warp * 2 + m;
    const float mine = lane < p.splits ? p.ws_ml[((size_t)lane * rows + row) * 2] : -INFINITY;   // at most 32 splits
    const float M = warp_max(mine), f_mine = mine == -INFINITY ? 0.f : exp2f(mine - M);
    const float L = warp_sum(lane < p.splits ? p.ws_ml[((size_t)lane * rows + row) * 2 + 1] * f_mine : 0.f);
    const float inv = L > 0.f ? (m == 0 ? 1.f : -lam) / L : 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float f = __shfl_sync(0xffffffffu, f_mine, s) * inv;
      if (f == 0.f) continue;
      const float* src = p.ws_o + (s * rows + row) * D;
#pragma unroll
      for (int i = 0; i < D / 32; ++i) x[i] = fmaf(src[lane + 32 * i], f, x[i]);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < D / 32; ++i) ss = fmaf(x[i], x[i], ss);
  const float g = p.out_scale / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
#pragma unroll
  for (int i = 0; i < D / 32; ++i)
    if (lane + 32 * i < p.vdim) p.out[(size_t)warp * p.vdim + lane + 32 * i] = __float2bfloat16(x[i] * g);
}

template <int D, int MODE, int MB, bool KV8, int ST = 3, bool EXT = false, bool DIFF = false>
int launch_one(const AttnParams& p, cudaStream_t st) {
  constexpr int ROWS = (MODE == 0) ? 64 : 16 * MB;
  const int smem_max = ROWS * D * 2 + (KV8 ? 2 * ST * kKeysPerTile * D + 2 * kKeysPerTile * D * 2 : 2 * ST * kKeysPerTile * D * 2);
  int smem = smem_max;
  if (EXT && p.kv_shared) {  // one ring; the decode kernel's merge of its warps' fp32 partials lies over it
    const int ring = ST * kKeysPerTile * D * 2, merge = (MODE == 1) ? 4 * ROWS * D * 4 : 0;
    smem = ROWS * D * 2 + (ring > merge ? ring : merge);
  }
  static int configured_dev[kMaxDevices] = {};
  int& configured = configured_dev[current_device_slot()];  // the limit is an attribute of (kernel, device)
  if (!configured) {
    if (cudaFuncSetAttribute(attn_kernel<D, MODE, MB, KV8, ST, EXT, DIFF>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_max) != cudaSuccess) return -4;
    configured = 1;
  }
  dim3 grid(MODE == 0 ? p.num_q_tiles : p.R, p.Hkv, MODE == 0 ? 1 : p.splits);
  if (grid.x == 0) return 0;
  launch_k(attn_kernel<D, MODE, MB, KV8, ST, EXT, DIFF>, grid, dim3(128), (size_t)smem, st, true, p);
  if (MODE == 1 && p.splits > 1) {
    int rows = p.T * p.Hq;
    if constexpr (DIFF) launch_k(diff_combine_kernel<D>, dim3((rows / 2 * 32 + 255) / 256), dim3(256), 0, st, true, p);
    else launch_k(attn_combine_kernel<D>, dim3((rows * 32 + 255) / 256), dim3(256), 0, st, true, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -5;
}

}  // namespace

int attention_launch(const AttnParams& p, int mode, cudaStream_t st) {
  if (p.Hq % p.Hkv || p.bs < 16 || (p.bs & (p.bs - 1)) || (p.D != 64 && p.D != 128 && p.D != 256)) return -1;
  const int G = p.Hq / p.Hkv;
  if (G > 64) return -1;
  const bool f8 = p.kv_fp8 != 0;
  if (p.maps == 2) {
    if (f8 || p.keep > 0 || p.kv_shared || p.bias != nullptr || p.gate != nullptr || p.sinks != nullptr || p.lse != nullptr || p.lam == nullptr || G % 2 ||
        p.vdim < 1 || p.vdim > p.D || p.splits > 32) return -8;
    if (mode == 1) {
      const int rows = p.short_q_len * G;
      if (p.D == 64) {
        if (rows <= 16) return launch_one<64, 1, 1, false, 3, true, true>(p, st);
        if (rows <= 32) return launch_one<64, 1, 2, false, 3, true, true>(p, st);
      } else if (p.D == 128) {
        if (rows <= 16) return launch_one<128, 1, 1, false, 3, true, true>(p, st);
        if (rows <= 32) return launch_one<128, 1, 2, false, 3, true, true>(p, st);
      } else if (rows <= 16) {
        return launch_one<256, 1, 1, false, 3, true, true>(p, st);
      }
      return -6;
    }
    return p.D == 64 ? launch_one<64, 0, 1, false, 3, true, true>(p, st) : p.D == 128 ? launch_one<128, 0, 1, false, 3, true, true>(p, st)
                                                                                      : launch_one<256, 0, 1, false, 3, true, true>(p, st);
  }
  if (p.chunk > 0 || p.keep > 0 || p.kv_shared || p.bias != nullptr || p.gate != nullptr) {
    if (f8 || (p.bias != nullptr && p.bias_len < 1)) return -7;
    const int rows = p.short_q_len * G;
    if (mode == 1) {
      if (p.D == 64) {
        if (rows <= 16) return launch_one<64, 1, 1, false, 3, true>(p, st);
        if (rows <= 32) return launch_one<64, 1, 2, false, 3, true>(p, st);
      } else if (p.D == 128) {
        if (rows <= 16) return launch_one<128, 1, 1, false, 3, true>(p, st);
        if (rows <= 32) return launch_one<128, 1, 2, false, 3, true>(p, st);
      } else if (rows <= 16) {
        return launch_one<256, 1, 1, false, 3, true>(p, st);
      }
      return -6;
    }
    return p.D == 64 ? launch_one<64, 0, 1, false, 3, true>(p, st) : p.D == 128 ? launch_one<128, 0, 1, false, 3, true>(p, st)
                                                                               : launch_one<256, 0, 1, false, 3, true>(p, st);
  }
  if (mode == 1) {
    const int rows = p.short_q_len * G;
    if (p.D == 64) {
      if (rows <= 16) return f8 ? launch_one<64, 1, 1, true>(p, st) : launch_one<64, 1, 1, false>(p, st);
      if (rows <= 32) return f8 ? launch_one<64, 1, 2, true>(p, st) : launch_one<64, 1, 2, false>(p, st);
    } else if (p.D == 128) {
      if (rows <= 16) {
        if (f8) return launch_one<128, 1, 1, true>(p, st);
        // two ring stages leave room for a third CTA per SM (experiment switch; three stages and two CTAs are the default)
        static const int two_stage = getenv("ONECAT_ATTN_STAGES") && atoi(getenv("ONECAT_ATTN_STAGES")) == 2;
        return two_stage ? launch_one<128, 1, 1, false, 2>(p, st) : launch_one<128, 1, 1, false>(p, st);
      }
      if (rows <= 32) return f8 ? launch_one<128, 1, 2, true>(p, st) : launch_one<128, 1, 2, false>(p, st);
    } else {
      if (rows <= 16) return f8 ? launch_one<256, 1, 1, true>(p, st) : launch_one<256, 1, 1, false>(p, st);
    }
    return -6;  // caller must use mode 0 for longer queries
  }
  if (p.D == 64) return f8 ? launch_one<64, 0, 1, true>(p, st) : launch_one<64, 0, 1, false>(p, st);
  if (p.D == 128) return f8 ? launch_one<128, 0, 1, true>(p, st) : launch_one<128, 0, 1, false>(p, st);
  return f8 ? launch_one<256, 0, 1, true>(p, st) : launch_one<256, 0, 1, false>(p, st);
}

unsigned int attention_read_status(bool clear) { return read_status_tu(clear); }
void attention_read_status_async(unsigned int* dst, cudaStream_t st) { read_status_tu_async(dst, st); }

}  // namespace oc
