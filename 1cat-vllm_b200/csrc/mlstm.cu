// mLSTM (matrix memory with exponential gates): recurrence, per-head RMS norm and sigmoid output gate.
//   i = cap tanh((gi + bi) / cap)      f = logsigmoid(cap tanh((gf + bf) / cap))
//   m' = max(f + m, i)      S' = e^(f + m - m') S + e^(i - m') k v^T      n' = e^(f + m - m') n + e^(i - m') k
//   o = S'^T q / (max(|n' . q|, e^-m') + 1e-6)      y = o / rms(o) * w * sigmoid(gate)
// State per (slot, head), all fp32: S [D][V], n [D], m.
//
// Recurrent kernel (decoding, short portions, fp32 engines): a CTA owns 64 state columns of one (sequence, head); a head with more columns
// is a thread-block cluster, whose CTAs exchange the sums of squares for the head norm through distributed shared memory and share n and m
// (the cluster barrier orders everybody's reads of the old values before the one write of the new ones).
//
// Chunked kernels (bf16, portions of at least 64 tokens): unlike the delta rule, a chunk's contribution to the state does not depend on the
// state before it, so nothing but an elementwise scan is sequential. With F the running sum of the log forget gates inside a chunk of 64
// tokens, b_s = i_s - F_s, M_t = max(m0, max_{s<=t} b_s) (so that m_t = F_t + M_t):
//   chunk kernel:  dS = sum_s e^(F_C + b_s - mloc) k_s v_s^T, dn likewise, mloc = F_C + max_s b_s           (per chunk and head)
//   scan kernel:   m' = max(F_C + m, mloc), S' = e^(F_C + m - m') S + e^(mloc - m') dS                        (elements in parallel)
//   output kernel: num_t = e^(m0 - M_t) S0^T q_t + sum_{s<=t} e^(b_s - M_t) (q_t . k_s) v_s, den likewise, norm, gate
// Products run on bf16 mma.sync; whatever is 32-bit by definition (S0, the weights) enters them as two bf16 terms (the rounded value and
// what rounding took from it). The host cuts the chunk list into segments, which bounds the memory of the chunk states.
#include <type_traits>

#include "common.cuh"
#include "kernels.h"

namespace oc {
namespace {

template <typename E> __device__ __forceinline__ float ldf(const E* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename E> __device__ __forceinline__ void stf(E* p, float v);
template <> __device__ __forceinline__ void stf<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stf<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float gate_in(float g, float b, float cap) { return cap * tanhf((g + b) / cap); }
__device__ __forceinline__ float gate_forget(float g, float b, float cap) {
  const float z = cap * tanhf((g + b) / cap);
  return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));   // log of the sigmoid
}
__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
}

constexpr int RCH = 8;    // tokens staged together by the recurrent kernel, one per warp in its last step
constexpr int RV = 64;    // state columns per CTA

// HK: state rows per thread; a column is split over four lanes (lane = column + 8 * part, part p holds rows p * HK ..).
template <typename E, int HK>
__global__ void __launch_bounds__(256, HK <= 32 ? 3 : HK <= 64 ? 2 : 1) mlstm_recurrent_kernel(const MlstmParams p) {
  constexpr int KP = 4 * HK, NH = HK / 8;
  __shared__ __align__(16) float sq[RCH][KP], sk[RCH][KP];
  __shared__ float sv[RCH][RV], so[RCH][RV], si[RCH], sf[RCH], part_ss[2][RCH];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * RV, nz = gridDim.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, part = lane >> 3, lc = warp * 8 + (lane & 7), col = c0 + lc;
  const int t0 = p.query_start_loc[r], t1 = p.query_start_loc[r + 1];
  if (t1 <= t0 || (p.skip_min_len > 0 && t1 - t0 >= p.skip_min_len)) return;   // the same decision in every CTA of a cluster
  const int D = p.D, V = p.V, H = p.H, slot = p.state_slots[r];
  const bool init = p.has_initial_state[r] != 0, own = col < V;
  float* Sg = p.S + ((size_t)slot * H + h) * D * V;
  float* ng = p.n + ((size_t)slot * H + h) * D;
  float* mg = p.m + (size_t)slot * H + h;
  float S[HK], nn[NH];
#pragma unroll
  for (int j = 0; j < HK; ++j) {
    const int row = part * HK + j;
    S[j] = init && own && row < D ? Sg[(size_t)row * V + col] : 0.f;
  }
  const int nrow = part * HK + (lane & 7) * NH;   // every warp carries n, spread over its lanes
#pragma unroll
  for (int j = 0; j < NH; ++j) nn[j] = init && nrow + j < D ? ng[nrow + j] : 0.f;
  float m = init ? *mg : 0.f;
  const E* x = reinterpret_cast<const E*>(p.x);
  const E* w = reinterpret_cast<const E*>(p.norm_w) + (size_t)h * V;
  E* out = reinterpret_cast<E*>(p.out);
  int buf = 0;
  for (int tc = t0; tc < t1; tc += RCH, buf ^= 1) {
    const int cnt = min(RCH, t1 - tc);
    __syncthreads();   // the previous tokens' outputs have left
    for (int e = tid; e < cnt * KP; e += 256) {
      const int i = e / KP, d = e - i * KP;
      const E* row = x + (size_t)(tc + i) * p.ld + h * D + d;
      sq[i][d] = d < D ? ldf<E>(row) * p.scale : 0.f;
      sk[i][d] = d < D ? ldf<E>(row + (size_t)H * D) : 0.f;
    }
    for (int e = tid; e < cnt * RV; e += 256) {
      const int i = e / RV, c = e - i * RV;
      sv[i][c] = c0 + c < V ? ldf<E>(x + (size_t)(tc + i) * p.ld + 2 * (size_t)H * D + (size_t)h * V + c0 + c) : 0.f;
    }
    if (tid < cnt) {
      const float* g = p.gates + (size_t)(tc + tid) * p.ld_g;
      si[tid] = gate_in(g[h], p.i_bias[h], p.cap);
      sf[tid] = gate_forget(g[H + h], p.f_bias[h], p.cap);
    }
    __syncthreads();
#pragma unroll 1
    for (int i = 0; i < cnt; ++i) {
      const float f = sf[i] + m, li = si[i], mn = fmaxf(f, li), keep = expf(f - mn), put = expf(li - mn), v = sv[i][lc] * put;
      m = mn;
      const float4* k4 = reinterpret_cast<const float4*>(&sk[i][part * HK]);
      const float4* q4 = reinterpret_cast<const float4*>(&sq[i][part * HK]);
      float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < HK; j += 4) {
        const float4 kk = k4[j >> 2], qq = q4[j >> 2];
        S[j] = fmaf(kk.x, v, S[j] * keep); S[j + 1] = fmaf(kk.y, v, S[j + 1] * keep);
        S[j + 2] = fmaf(kk.z, v, S[j + 2] * keep); S[j + 3] = fmaf(kk.w, v, S[j + 3] * keep);
        a[0] = fmaf(qq.x, S[j], a[0]); a[1] = fmaf(qq.y, S[j + 1], a[1]); a[2] = fmaf(qq.z, S[j + 2], a[2]); a[3] = fmaf(qq.w, S[j + 3], a[3]);
      }
      float o = (a[0] + a[1]) + (a[2] + a[3]), dot = 0.f;
#pragma unroll
      for (int j = 0; j < NH; ++j) {
        nn[j] = fmaf(sk[i][nrow + j], put, nn[j] * keep);
        dot = fmaf(sq[i][nrow + j], nn[j], dot);
      }
      o += __shfl_xor_sync(0xffffffffu, o, 8);
      o += __shfl_xor_sync(0xffffffffu, o, 16);
      dot = warp_sum(dot);
      if (part == 0) so[i][lc] = o / (fmaxf(fabsf(dot), expf(-m)) + 1e-6f);
    }
    __syncthreads();
    // head norm and gate: warp i finishes token i (columns beyond V hold zeros)
    const float o0 = warp < cnt ? so[warp][lane] : 0.f, o1 = warp < cnt ? so[warp][lane + 32] : 0.f;
    float ss = warp_sum(o0 * o0 + o1 * o1);
    if (nz > 1) {
      if (lane == 0) part_ss[buf][warp] = ss;
      cluster_sync_all();
      float v = 0.f;
      if (lane < nz) asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(mapa_shared(smem_u32(&part_ss[buf][warp]), lane)) : "memory");
      ss = warp_sum(v);
    }
    if (warp < cnt) {
      const float inv = 1.f / sqrtf(ss / (float)V + p.eps);
      const size_t t = tc + warp;
      const E* g = x + t * p.ld + 2 * (size_t)H * D + (size_t)H * V + (size_t)h * V;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = c0 + lane + 32 * e;
        if (c < V) stf<E>(out + t * H * V + (size_t)h * V + c, (e ? o1 : o0) * inv * ldf<E>(w + c) * sigmoid(ldf<E>(g + c)));
      }
    }
  }
  int pitch = V;
  asm volatile("" : "+r"(pitch));   // the addresses are formed anew: keeping those of the loads would take two registers a row
  float* Sw = Sg + (size_t)part * HK * pitch + col;
#pragma unroll
  for (int j = 0; j < HK; ++j)
    if (own && part * HK + j < D) Sw[(size_t)j * pitch] = S[j];
  if (nz > 1) cluster_sync_all();   // the old n and m have been read, and nobody still reads this CTA's shared memory
  if (blockIdx.z == 0 && warp == 0) {
#pragma unroll
    for (int j = 0; j < NH; ++j)
      if (nrow + j < D) ng[nrow + j] = nn[j];
    if (lane == 0) *mg = m;
  }
}

// ---------------------------------------------------------------------------------------------------------------- chunked form
constexpr int C = 64;     // tokens per chunk
constexpr int KV = 64;    // value columns per CTA of the chunk kernel
constexpr int PV = 72;    // shared-memory pitch of a [*][64] bf16 tile
constexpr int NS = 32;    // value columns per pass of the output kernel
constexpr int PS = 40;    // and the pitch of a [*][32] tile

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float rounded(float v) { return __bfloat162float(__float2bfloat16(v)); }
// fragment addresses: A from a row-major [m][k] tile; A^T from a [k][m] tile (loaded transposed); B pairs from [n][k]; B pairs from [k][n]
__device__ __forceinline__ uint32_t a_addr(uint32_t base, int pitch, int m0, int k0, int lane) {
  return base + (uint32_t)(((m0 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + k0 + (lane >> 4) * 8) * 2);
}
__device__ __forceinline__ uint32_t at_addr(uint32_t base, int pitch, int m0, int k0, int lane) {
  return base + (uint32_t)(((k0 + (lane & 7) + (lane >> 4) * 8) * pitch + m0 + ((lane >> 3) & 1) * 8) * 2);
}
__device__ __forceinline__ uint32_t bnk_addr(uint32_t base, int pitch, int n0, int k0, int lane) {
  return base + (uint32_t)(((n0 + (lane & 7) + (lane >> 4) * 8) * pitch + k0 + ((lane >> 3) & 1) * 8) * 2);
}
__device__ __forceinline__ uint32_t bkn_addr(uint32_t base, int pitch, int k0, int n0, int lane) {
  return base + (uint32_t)(((k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + n0 + (lane >> 4) * 8) * 2);
}

__device__ __forceinline__ void cp16(void* smem, const void* g) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(g) : "memory");
}
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// rows x cols bf16 tile from global (row pitch ld) into shared memory (pitch `pitch`), zeros outside [vr) x [vc); pc: columns to fill
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, int pitch, const __nv_bfloat16* src, long long ld, int rows, int pc, int vr, int vc, bool vec,
                                          int tid, int nt) {
  if (vec) {   // whole 16-byte segments: vc % 8 == 0, aligned rows
    const int per = pc / 8;
    for (int e = tid; e < rows * per; e += nt) {
      const int i = e / per, s = (e - i * per) * 8;
      if (i < vr && s < vc) cp16(dst + i * pitch + s, src + (size_t)i * ld + s);   // the caller waits for the copies
      else *reinterpret_cast<uint4*>(dst + i * pitch + s) = make_uint4(0, 0, 0, 0);
    }
  } else {
    for (int e = tid; e < rows * pc; e += nt) {
      const int i = e / pc, s = e - i * pc;
      dst[i * pitch + s] = i < vr && s < vc ? src[(size_t)i * ld + s] : __float2bfloat16(0.f);
    }
  }
}

// Gates of a chunk, by warp 0: sF[t] = running sum of f, sb[t] = i_t - F_t (-inf past the end of the sequence).
__device__ __forceinline__ void chunk_gates(const MlstmParams& p, int tc, int n, int h, float* sF, float* sb, int lane) {
  float f[2], li[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int t = lane + 32 * e;
    f[e] = 0.f;
    li[e] = -INFINITY;
    if (t < n) {
      const float* g = p.gates + (size_t)(tc + t) * p.ld_g;
      li[e] = gate_in(g[h], p.i_bias[h], p.cap);
      f[e] = gate_forget(g[p.H + h], p.f_bias[h], p.cap);
    }
  }
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float y0 = __shfl_up_sync(0xffffffffu, f[0], o), y1 = __shfl_up_sync(0xffffffffu, f[1], o);
    if (lane >= o) { f[0] += y0; f[1] += y1; }
  }
  f[1] += __shfl_sync(0xffffffffu, f[0], 31);
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    sF[lane + 32 * e] = f[e];
    sb[lane + 32 * e] = li[e] - f[e];
  }
}

// grid (chunks of the segment, H, column groups), 128 threads.
__global__ void __launch_bounds__(128) mlstm_chunk_kernel(const MlstmParams p) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float sF[C], sb[C], sw[C];
  const int ci = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * KV, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = p.D, V = p.V, H = p.H, Dp = (D + 15) & ~15, PD = Dp + 8;
  __nv_bfloat16* kt = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* vh = kt + C * PD;
  __nv_bfloat16* vl = vh + C * PV;
  const int r = p.chunk_req[ci], tc = p.chunk_t0[ci], n = min(C, p.query_start_loc[r + 1] - tc);
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)tc * p.ld;
  if (warp == 0) {
    chunk_gates(p, tc, n, h, sF, sb, lane);
    __syncwarp();
    const float FC = sF[C - 1];
    float mx = fmaxf(sb[lane], sb[lane + 32]);
    mx = warp_max(mx);
    sw[lane] = expf(sb[lane] - mx);
    sw[lane + 32] = expf(sb[lane + 32] - mx);
    if (blockIdx.z == 0 && lane == 0) {
      float* g = p.ws_g + ((size_t)ci * H + h) * 2;
      g[0] = FC;
      g[1] = FC + mx;
      const int li = p.chunk_long[ci];
      if (p.long_chunk0[li] == ci) {   // the maximum that this segment starts from
        const bool init = p.has_initial_state[r] != 0 || tc > p.query_start_loc[r];
        p.ws_m[(size_t)ci * H + h] = init ? p.m[(size_t)p.state_slots[r] * H + h] : 0.f;
      }
    }
  }
  load_tile(kt, PD, x + (size_t)H * D + (size_t)h * D, p.ld, C, Dp, n, D, p.vec_qk, tid, 128);
  load_tile(vl, PV, x + 2 * (size_t)H * D + (size_t)h * V + c0, p.ld, C, KV, n, min(KV, V - c0), p.vec_v, tid, 128);
  cp_wait();
  __syncthreads();
  for (int e = tid; e < C * KV / 2; e += 128) {   // weighted value rows as two terms, pairs of columns
    const int i = e / (KV / 2), c = (e - i * (KV / 2)) * 2;
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vl + i * PV + c));
    const float a = sw[i] * v.x, b = sw[i] * v.y;
    *reinterpret_cast<uint32_t*>(vh + i * PV + c) = pack2(a, b);
    *reinterpret_cast<uint32_t*>(vl + i * PV + c) = pack2(a - rounded(a), b - rounded(b));
  }
  if (blockIdx.z == 0)
    for (int d = tid; d < D; d += 128) {
      float a = 0.f;
      for (int i = 0; i < n; ++i) a = fmaf(sw[i], __bfloat162float(kt[i * PD + d]), a);
      p.ws_n[((size_t)ci * H + h) * D + d] = a;
    }
  __syncthreads();
  const uint32_t sk = smem_u32(kt), svh = smem_u32(vh), svl = smem_u32(vl);
  float* dS = p.ws_s + ((size_t)ci * H + h) * D * V;
  const int g = lane >> 2, t4 = lane & 3;
  for (int m0 = warp * 16; m0 < Dp; m0 += 64) {
    float acc[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[nt][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < C / 16; ++ks) {
      uint32_t a[4];
      ldsm_x4_t(a, at_addr(sk, PD, m0, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4];
        ldsm_x4_t(b, bkn_addr(svh, PV, ks * 16, np * 16, lane));
        mma16816(acc[2 * np], a, b[0], b[1]);
        mma16816(acc[2 * np + 1], a, b[2], b[3]);
        ldsm_x4_t(b, bkn_addr(svl, PV, ks * 16, np * 16, lane));
        mma16816(acc[2 * np], a, b[0], b[1]);
        mma16816(acc[2 * np + 1], a, b[2], b[3]);
      }
    }
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int row = m0 + g + 8 * hh, c = c0 + nt * 8 + t4 * 2;
        if (row >= D) continue;
        float* dst = dS + (size_t)row * V + c;
        if (c + 1 < V && (V & 1) == 0) *reinterpret_cast<float2*>(dst) = make_float2(acc[nt][2 * hh], acc[nt][2 * hh + 1]);
        else {
          if (c < V) dst[0] = acc[nt][2 * hh];
          if (c + 1 < V) dst[1] = acc[nt][2 * hh + 1];
        }
      }
  }
}

// grid (sequences of the segment, H, element groups + 1): every thread scans VEC elements of S over the segment's chunks and leaves the
// state ahead of each chunk as two bf16 terms; the last group scans n and the maxima.
template <int VEC>
__global__ void __launch_bounds__(256) mlstm_scan_kernel(const MlstmParams p) {
  const int li = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, H = p.H, D = p.D;
  const int r = p.long_req[li], cb = p.long_chunk0[li], nc = p.long_n[li], slot = p.state_slots[r];
  const bool init = p.has_initial_state[r] != 0 || p.chunk_t0[cb] > p.query_start_loc[r];
  const size_t DV = (size_t)D * p.V;
  float m = p.ws_m[(size_t)cb * H + h];
  if (blockIdx.z + 1 < gridDim.z) {
    const size_t e = ((size_t)blockIdx.z * 256 + tid) * VEC;
    if (e >= DV) return;
    float* Sg = p.S + ((size_t)slot * H + h) * DV + e;
    float s[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) s[j] = init ? Sg[j] : 0.f;
    float d[VEC], dn[VEC];
    auto fetch = [&](int c, float (&v)[VEC]) {
      const float* src = p.ws_s + ((size_t)c * H + h) * DV + e;
      if (VEC == 4) {
        const float4 q = *reinterpret_cast<const float4*>(src);
        v[0] = q.x; v[1 % VEC] = q.y; v[2 % VEC] = q.z; v[3 % VEC] = q.w;
      } else {
        v[0] = src[0];
      }
    };
    fetch(cb, d);
    for (int c = cb; c < cb + nc; ++c) {
      if (c + 1 < cb + nc) fetch(c + 1, dn);
      const float* g = p.ws_g + ((size_t)c * H + h) * 2;
      const float F = g[0] + m, ml = g[1], mn = fmaxf(F, ml), ka = expf(F - mn), kb = expf(ml - mn);
      m = mn;
      __nv_bfloat16* ph = p.ws_h + ((size_t)c * H + h) * 2 * DV + e;
      if (VEC == 4) {
        *reinterpret_cast<uint2*>(ph) = make_uint2(pack2(s[0], s[1 % VEC]), pack2(s[2 % VEC], s[3 % VEC]));
        *reinterpret_cast<uint2*>(ph + DV) = make_uint2(pack2(s[0] - rounded(s[0]), s[1 % VEC] - rounded(s[1 % VEC])),
                                                        pack2(s[2 % VEC] - rounded(s[2 % VEC]), s[3 % VEC] - rounded(s[3 % VEC])));
      } else {
        ph[0] = __float2bfloat16(s[0]);
        ph[DV] = __float2bfloat16(s[0] - rounded(s[0]));
      }
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        s[j] = fmaf(ka, s[j], kb * d[j]);
        d[j] = dn[j];
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) Sg[j] = s[j];
    return;
  }
  float* ng = p.n + ((size_t)slot * H + h) * D;
  for (int d = tid; d < D; d += 256) {
    float s = init ? ng[d] : 0.f, mm = m;
    for (int c = cb; c < cb + nc; ++c) {
      const float* g = p.ws_g + ((size_t)c * H + h) * 2;
      const float F = g[0] + mm, ml = g[1], mn = fmaxf(F, ml);
      float* q = p.ws_n + ((size_t)c * H + h) * D + d;
      const float add = *q;
      *q = s;   // n ahead of the chunk
      s = fmaf(expf(F - mn), s, expf(ml - mn) * add);
      mm = mn;
    }
    ng[d] = s;
  }
  if (tid == 0) {
    for (int c = cb; c < cb + nc; ++c) {
      const float* g = p.ws_g + ((size_t)c * H + h) * 2;
      if (c > cb) p.ws_m[(size_t)c * H + h] = m;
      m = fmaxf(g[0] + m, g[1]);
    }
    p.m[(size_t)slot * H + h] = m;
  }
}

__host__ __device__ __forceinline__ size_t out_smem(int D, int V) {
  const int Dp = (D + 15) & ~15, PD = Dp + 8;
  size_t kb = (size_t)C * PD * 2, pb = (size_t)2 * Dp * PS * 2;
  return (size_t)C * PD * 2 + (kb > pb ? kb : pb) + (size_t)C * PS * 2 + (size_t)C * (((V + NS - 1) / NS) * NS + 4) * 4;   // the last part holds n first
}

// grid (chunks of the segment, H), 128 threads; warp w owns tokens 16 w .. 16 w + 15.
__global__ void __launch_bounds__(128) mlstm_output_kernel(const MlstmParams p) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float sF[C], sb[C], sM[C], snq[C], sinv[C];
  const int ci = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int D = p.D, V = p.V, H = p.H, Dp = (D + 15) & ~15, PD = Dp + 8, PO = ((V + NS - 1) / NS) * NS + 4;
  __nv_bfloat16* qt = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* kt = qt + C * PD;        // keys, later the state's two planes [Dp][PS]
  const size_t kb = (size_t)C * PD, pb = (size_t)2 * Dp * PS;
  __nv_bfloat16* vt = kt + (kb > pb ? kb : pb);
  float* so = reinterpret_cast<float*>(vt + C * PS);
  const int r = p.chunk_req[ci], tc = p.chunk_t0[ci], n = min(C, p.query_start_loc[r + 1] - tc);
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.x) + (size_t)tc * p.ld;
  const float m0 = p.ws_m[(size_t)ci * H + h];
  if (warp == 0) {
    chunk_gates(p, tc, n, h, sF, sb, lane);
    __syncwarp();
    float a = sb[lane], b = sb[lane + 32];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float ya = __shfl_up_sync(0xffffffffu, a, o), yb = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) { a = fmaxf(a, ya); b = fmaxf(b, yb); }
    }
    b = fmaxf(b, __shfl_sync(0xffffffffu, a, 31));
    sM[lane] = fmaxf(a, m0);
    sM[lane + 32] = fmaxf(b, m0);
  }
  load_tile(qt, PD, x + (size_t)h * D, p.ld, C, Dp, n, D, p.vec_qk, tid, 128);
  load_tile(kt, PD, x + (size_t)H * D + (size_t)h * D, p.ld, C, Dp, n, D, p.vec_qk, tid, 128);
  for (int d = tid; d < Dp; d += 128) so[d] = d < D ? p.ws_n[((size_t)ci * H + h) * D + d] : 0.f;   // n ahead of the chunk
  cp_wait();
  __syncthreads();
  {
    const int row = tid >> 1, half = tid & 1;
    float a[2] = {0.f, 0.f};
    for (int d = half * 8; d < Dp; d += 16) {
      const uint4 raw = *reinterpret_cast<const uint4*>(qt + row * PD + d);
      const __nv_bfloat162* q2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 q = __bfloat1622float2(q2[e]);
        a[0] = fmaf(q.x, so[d + 2 * e], a[0]);
        a[1] = fmaf(q.y, so[d + 2 * e + 1], a[1]);
      }
    }
    a[0] += a[1];
    a[0] += __shfl_xor_sync(0xffffffffu, a[0], 1);
    if (half == 0) snq[row] = a[0];
  }
  __syncthreads();
  const uint32_t sq = smem_u32(qt), sk = smem_u32(kt), sv = smem_u32(vt);
  const int r0 = warp * 16;
  uint32_t ph[4][4], pl[4][4];   // weights of this warp's 16 tokens over the chunk's 64, as A operands in two terms
  float carry[2], inv[2];
  {
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = 0.f;
    for (int ks = 0; ks < Dp / 16; ++ks) {
      uint32_t a[4];
      ldsm_x4(a, a_addr(sq, PD, r0, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        uint32_t b[4];
        ldsm_x4(b, bnk_addr(sk, PD, np * 16, ks * 16, lane));
        mma16816(s[2 * np], a, b[0], b[1]);
        mma16816(s[2 * np + 1], a, b[2], b[3]);
      }
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int i = r0 + g + 8 * hh;
      const float M = sM[i];
      float dot = 0.f;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = nt * 8 + t4 * 2 + e;
          const float v = j <= i ? s[nt][2 * hh + e] * p.scale * expf(sb[j] - M) : 0.f;   // b_j = -inf past the end: weight 0
          s[nt][2 * hh + e] = v;
          dot += v;
        }
      dot += __shfl_xor_sync(0xffffffffu, dot, 1);
      dot += __shfl_xor_sync(0xffffffffu, dot, 2);
      carry[hh] = expf(m0 - M) * p.scale;
      inv[hh] = 1.f / (fmaxf(fabsf(fmaf(carry[hh], snq[i], dot)), expf(-(sF[i] + M))) + 1e-6f);
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)
#pragma unroll
      for (int e = 0; e < 4; ++e) {   // a0: row g, a1: row g + 8, a2 / a3: the same rows, next 8 columns
        const float* q = s[2 * ks + (e >> 1)];
        const float u = q[2 * (e & 1)], v = q[2 * (e & 1) + 1];
        ph[ks][e] = pack2(u, v);
        pl[ks][e] = pack2(u - rounded(u), v - rounded(v));
      }
  }
  float ss[2] = {0.f, 0.f};
  const size_t DV = (size_t)D * V;
  const __nv_bfloat16* plane = p.ws_h + ((size_t)ci * H + h) * 2 * DV;
  const uint32_t sh = sk, sl = sk + (uint32_t)(Dp * PS * 2);
  for (int c0 = 0; c0 < V; c0 += NS) {
    const int vc = min(NS, V - c0);
    __syncthreads();   // the keys, or the previous pass's tiles, have been read
    load_tile(kt, PS, plane + c0, V, Dp, NS, D, vc, p.vec_v, tid, 128);
    load_tile(kt + Dp * PS, PS, plane + DV + c0, V, Dp, NS, D, vc, p.vec_v, tid, 128);
    load_tile(vt, PS, x + 2 * (size_t)H * D + (size_t)h * V + c0, p.ld, C, NS, n, vc, p.vec_v, tid, 128);
    cp_wait();
    __syncthreads();
    float in[4][4], out[4][4];
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) in[nt][e] = out[nt][e] = 0.f;
    for (int ks = 0; ks < Dp / 16; ++ks) {
      uint32_t a[4];
      ldsm_x4(a, a_addr(sq, PD, r0, ks * 16, lane));
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t b[4];
        ldsm_x4_t(b, bkn_addr(sh, PS, ks * 16, np * 16, lane));
        mma16816(in[2 * np], a, b[0], b[1]);
        mma16816(in[2 * np + 1], a, b[2], b[3]);
        ldsm_x4_t(b, bkn_addr(sl, PS, ks * 16, np * 16, lane));
        mma16816(in[2 * np], a, b[0], b[1]);
        mma16816(in[2 * np + 1], a, b[2], b[3]);
      }
    }
#pragma unroll
    for (int ks = 0; ks < 4; ++ks)
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        if (ks > warp) continue;   // keys past this warp's last token weigh nothing
        uint32_t b[4];
        ldsm_x4_t(b, bkn_addr(sv, PS, ks * 16, np * 16, lane));
        mma16816(out[2 * np], ph[ks], b[0], b[1]);
        mma16816(out[2 * np + 1], ph[ks], b[2], b[3]);
        mma16816(out[2 * np], pl[ks], b[0], b[1]);
        mma16816(out[2 * np + 1], pl[ks], b[2], b[3]);
      }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const float u = fmaf(in[nt][2 * hh], carry[hh], out[nt][2 * hh]) * inv[hh], v = fmaf(in[nt][2 * hh + 1], carry[hh], out[nt][2 * hh + 1]) * inv[hh];
        *reinterpret_cast<float2*>(so + (r0 + g + 8 * hh) * PO + c0 + nt * 8 + t4 * 2) = make_float2(u, v);
        ss[hh] = fmaf(u, u, fmaf(v, v, ss[hh]));
      }
  }
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    ss[hh] += __shfl_xor_sync(0xffffffffu, ss[hh], 1);
    ss[hh] += __shfl_xor_sync(0xffffffffu, ss[hh], 2);
    if (t4 == 0) sinv[r0 + g + 8 * hh] = 1.f / sqrtf(ss[hh] / (float)V + p.eps);
  }
  __syncwarp();
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.norm_w) + (size_t)h * V;
  __nv_bfloat16* y = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)tc * H * V + (size_t)h * V;
  const __nv_bfloat16* gate = x + 2 * (size_t)H * D + (size_t)H * V + (size_t)h * V;
  const int rows = min(16, n - r0);
  if (p.vec_v && (V & 1) == 0) {
    for (int c = lane * 2; c < V; c += 64) {
      const float2 wg = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(w + c));
      for (int i0 = 0; i0 < rows; i0 += 8) {   // the gates of eight rows are in flight together
        uint32_t gr[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) gr[e] = i0 + e < rows ? *reinterpret_cast<const uint32_t*>(gate + (size_t)(r0 + i0 + e) * p.ld + c) : 0u;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const int i = r0 + i0 + e;
          if (i0 + e >= rows) continue;
          const float2 o = *reinterpret_cast<const float2*>(so + i * PO + c), gg = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gr[e]));
          *reinterpret_cast<uint32_t*>(y + (size_t)i * H * V + c) = pack2(o.x * sinv[i] * wg.x * sigmoid(gg.x), o.y * sinv[i] * wg.y * sigmoid(gg.y));
        }
      }
    }
  } else {
    for (int i = r0; i < r0 + rows; ++i)
      for (int c = lane; c < V; c += 32)
        y[(size_t)i * H * V + c] = __float2bfloat16(so[i * PO + c] * sinv[i] * __bfloat162float(w[c]) * sigmoid(__bfloat162float(gate[(size_t)i * p.ld + c])));
  }
}

// x * sigmoid(gate), one thread per VEC elements
template <typename E, int VEC>
__global__ void __launch_bounds__(256) sigmoid_mul_kernel(const E* __restrict__ x, long long ldx, const E* __restrict__ gate, long long ldg, E* __restrict__ y,
                                                          int T, int N) {
  pdl_trigger();
  pdl_wait();
  const int per = N / VEC;
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= (long long)T * per) return;
  const long long t = i / per;
  const int c = (int)(i - t * per) * VEC;
  struct alignas(sizeof(E) * VEC) Vc { E e[VEC]; };
  const Vc a = *reinterpret_cast<const Vc*>(x + t * ldx + c), b = *reinterpret_cast<const Vc*>(gate + t * ldg + c);
  Vc o;
#pragma unroll
  for (int j = 0; j < VEC; ++j) stf<E>(&o.e[j], ldf<E>(&a.e[j]) * sigmoid(ldf<E>(&b.e[j])));
  *reinterpret_cast<Vc*>(y + t * N + c) = o;
}

template <typename E, int HK>
int recurrent_go(const MlstmParams& p, cudaStream_t st) {
  const int nz = (p.V + RV - 1) / RV;
  if (nz > 8) return -1;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.R, p.H, nz);
  cfg.blockDim = dim3(256);
  cfg.stream = st;
  cudaLaunchAttribute at[2];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim = {1, 1, (unsigned)nz};
  at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  at[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = at;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, mlstm_recurrent_kernel<E, HK>, p) == cudaSuccess ? 0 : -2;
}
template <typename E>
int recurrent_e(const MlstmParams& p, cudaStream_t st) {
  if (p.D <= 32) return recurrent_go<E, 8>(p, st);
  if (p.D <= 64) return recurrent_go<E, 16>(p, st);
  if (p.D <= 128) return recurrent_go<E, 32>(p, st);
  if (p.D <= 256) return recurrent_go<E, 64>(p, st);
  if (p.D <= 512) return recurrent_go<E, 128>(p, st);
  return -1;
}

}  // namespace

int mlstm_recurrent_launch(const MlstmParams& p, cudaStream_t st) {
  if (p.R == 0 || p.T == 0) return 0;
  return p.f32 ? recurrent_e<float>(p, st) : recurrent_e<__nv_bfloat16>(p, st);
}

bool mlstm_chunkable(int D, int V) { return D >= 1 && D <= 512 && V >= 1 && V <= 512 && out_smem(D, V) <= 220 * 1024; }

int mlstm_chunk_launch(const MlstmParams& p, int num_chunks, int num_long, cudaStream_t st) {
  if (num_chunks == 0 || num_long == 0) return 0;
  if (p.f32 || !mlstm_chunkable(p.D, p.V)) return -1;
  static bool configured_dev[kMaxDevices] = {};
  bool& configured = configured_dev[current_device_slot()];
  if (!configured) {
    if (cudaFuncSetAttribute(mlstm_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return -4;
    if (cudaFuncSetAttribute(mlstm_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return -4;
    configured = true;
  }
  const int Dp = (p.D + 15) & ~15;
  const size_t smem = ((size_t)C * (Dp + 8) + 2 * (size_t)C * PV) * 2;
  mlstm_chunk_kernel<<<dim3(num_chunks, p.H, (p.V + KV - 1) / KV), 128, smem, st>>>(p);
  const size_t DV = (size_t)p.D * p.V;
  if (DV % 4 == 0) mlstm_scan_kernel<4><<<dim3(num_long, p.H, (unsigned)((DV / 4 + 255) / 256 + 1)), 256, 0, st>>>(p);
  else mlstm_scan_kernel<1><<<dim3(num_long, p.H, (unsigned)((DV + 255) / 256 + 1)), 256, 0, st>>>(p);
  mlstm_output_kernel<<<dim3(num_chunks, p.H), 128, out_smem(p.D, p.V), st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

int sigmoid_mul_launch(const void* x, long long ldx, const void* gate, long long ldg, void* y, int T, int N, int f32, cudaStream_t st) {
  if (T == 0 || N == 0) return 0;
  const int esz = f32 ? 4 : 2;
  auto fits = [&](int v) {
    const uintptr_t a = (uintptr_t)v * esz;
    return N % v == 0 && ldx % v == 0 && ldg % v == 0 && ((uintptr_t)x % a) == 0 && ((uintptr_t)gate % a) == 0 && ((uintptr_t)y % a) == 0;
  };
  auto go = [&](auto kernel, auto* typed, int v) {
    using E = std::remove_pointer_t<decltype(typed)>;
    const long long total = (long long)T * (N / v);
    launch_k(kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st, true, (const E*)x, ldx, (const E*)gate, ldg, (E*)y, T, N);
  };
  if (f32) {
    if (fits(4)) go(sigmoid_mul_kernel<float, 4>, (float*)nullptr, 4);
    else go(sigmoid_mul_kernel<float, 1>, (float*)nullptr, 1);
  } else {
    if (fits(8)) go(sigmoid_mul_kernel<__nv_bfloat16, 8>, (__nv_bfloat16*)nullptr, 8);
    else go(sigmoid_mul_kernel<__nv_bfloat16, 1>, (__nv_bfloat16*)nullptr, 1);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace oc
