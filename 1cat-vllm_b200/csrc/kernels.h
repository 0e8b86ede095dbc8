// Host launchers of the non-GEMM kernels. All take raw device pointers and a stream; return 0 on success.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace oc {

struct RopeCacheParams {
  __nv_bfloat16 *q, *k, *v;
  long long q_st, q_sh, k_st, v_st;  // element strides: token / head (k and v heads are D apart)
  const int* positions;
  const float* cos_sin;  // [max_pos][rot]: cos | sin
  __nv_bfloat16* kv_cache;  // [blocks][2][Hkv][bs][D] or null
  const int* slot_mapping;
  const __nv_bfloat16 *q_norm, *k_norm;  // per-head RMSNorm weights or null
  int T, Hq, Hkv, D, rot, bs, gemma;
  float eps;
  int kv_fp8;                    // kv_cache holds e4m3 bytes: k / k_scale and v / v_scale, saturated
  float k_scale_inv, v_scale_inv;
  // rotary sections (0 = off): frequencies below mrope_s0 rotate by positions[t], below mrope_s1 by positions[pos_stride + t], the
  // rest by positions[2 * pos_stride + t]
  int mrope_s0, mrope_s1;
  long long pos_stride;
};

int rms_norm_launch(const void* x, const void* res_in, const void* w, void* y, void* res_out, int T, int H, int ldx, float eps,
                    int gemma, cudaStream_t st);
int rms_norm_gated_launch(const void* x, const void* z, const void* w, void* y, int rows, int D, int ldx, int ldz, int heads,
                          float eps, cudaStream_t st);
int silu_and_mul_launch(const void* x, void* y, int T, int I, cudaStream_t st);
int rope_cache_launch(const RopeCacheParams& p, cudaStream_t st);
// k (and v) rows [T][H][D] into pages [blocks][tensors][H][bs][D]; strides and widths in bytes
struct KvInsertParams {
  const char *k, *v;            // v null: one cached tensor per page
  char* cache;
  const int* slot_mapping;      // negative: skip
  long long k_st, v_st;         // bytes between tokens (heads are row_bytes apart)
  int T, H, row_bytes, bs;
};
int kv_insert_launch(const KvInsertParams& p, cudaStream_t st);

// fp32 residual stream: x' = x + scale * post(part) (+ add); y = next(x'). Norm kinds: 0 none, 1 RMS, 2 mean-and-variance.
struct StreamNorm {
  int kind, plus_one;
  const void *w, *b;            // null: ones / zeros
  float eps;
  const void* alpha;            // dynamic tanh: the scalar inside
};
struct StreamJoinParams {
  const void* part;             // [T][H], pitch ld_part
  long long ld_part;
  int part_f32;                 // part is fp32 (else the model's element type)
  const float* x_in;            // [T][H] or null: the stream starts from part
  float* x_out;                 // [T][H], may be x_in
  StreamNorm post, next;
  const void *scale, *add;      // [H] or null
  float mul;                    // number on the normalised, scaled part
  void* y;                      // [T][H] in the model's element type, or null (next.kind 0)
  void* copy_out;               // x' in the model's element type, pitch ld_copy, or null
  long long ld_copy;
  int T, H;
  int f32;                      // the model's element type (part, weights, y, copy_out): 1 fp32, 0 bf16
};
int stream_join_launch(const StreamJoinParams& p, cudaStream_t st);
// Start of the stream: x = table[id] * scale (+ bigram[hash of (previous token, token)]), y = x in the model's element type.
struct EmbedParams {
  const void *table, *bigram;   // [vocab][H], [buckets + 1][H] or null
  const int *ids, *prev;        // [T]; prev < 0: no previous token (the last row)
  float* x;                     // [T][H]
  void* y;                      // [T][H] or null
  float scale;
  int T, H, vocab, buckets, mul_prev, mul_cur, gathered, f32;   // gathered: the table's rows are the tokens' own
  const void* rows;             // [num_rows][H] learned position rows or null
  const int* positions;         // [T]
  int num_rows;
};
int embed_stream_launch(const EmbedParams& p, cudaStream_t st);
int gelu_tanh_f32_launch(float* x, long long n, cudaStream_t st);  // in place

int argmax_launch(const void* x, int is_fp32, long long* out, unsigned long long* packed, int B, int V, long long ld, cudaStream_t st);
int merge_attn_states_launch(const void* o1, const float* lse1, const void* o2, const float* lse2, void* out, float* lse_out, int rows, int D,
                             cudaStream_t st);
unsigned int elementwise_read_status(bool clear);
void elementwise_read_status_async(unsigned int* dst, cudaStream_t st);

struct AttnParams {
  const __nv_bfloat16* q;     // [T][Hq][D] with strides
  long long q_st, q_sh;
  const __nv_bfloat16* kv_cache;  // [blocks][2][Hkv][bs][D]
  __nv_bfloat16* out;         // [T][Hq][D] contiguous
  float* lse;                 // [T][Hq] or null
  const int* query_start_loc; // [R+1]
  const int* seq_lens;        // [R]
  const int* block_table;     // [R][bt_stride]
  int bt_stride;
  int R, T, Hq, Hkv, D, bs, bs_shift;  // bs: tokens per page (power of two, >= 16)
  float scale;
  int num_q_tiles;            // grid.x for prefill mode (host: sum over requests of ceil(q_len / tokens per tile))
  int splits;                 // decode mode: KV splits per (request, kv head)
  float* ws_o;                // [splits][T][Hq][D] fp32 partial outputs
  float* ws_ml;               // [splits][T][Hq][2]  running max (log2 domain) and sum
  int max_q_len;
  int short_q_len;            // requests with at most this many query tokens run in mode 1, the others in mode 0
  int window;                 // sliding window in tokens (0 = full causal attention); mma.sync kernels only
  float softcap;              // tanh soft-capping of the scaled scores (0 = off); mma.sync kernels only
  const float* sinks;         // [Hq] attention-sink logits or null; mma.sync kernels only
  int kv_fp8;                 // the cache holds e4m3 bytes (value / scale) instead of bf16; mma.sync kernels only
  float k_scale, v_scale;     // per-tensor scales of an fp8 cache
  // Extended variants of the mma.sync kernels (and the fp32 kernel), taken when any of these is set; not with an fp8 cache:
  int keep;                   // keys at positions below it stay visible outside the window
  int kv_shared;              // the cache is [blocks][1][Hkv][bs][D]: the values are the keys
  const float* bias;          // [Hq][bias_len] added to the scaled score by distance (the last entry for all distances past it), or null
  int bias_len;
  const void* gate;           // [T][Hq] (row pitch gate_st, element type of q): outputs are multiplied by its sigmoid, or null
  long long gate_st;
  int chunk;                  // > 0: only keys of the query's own chunk of that many positions are visible
  // Differential attention (maps == 2): Hq counts (head, map) rows, q is [T][Hq][D / 2], a key row holds both maps side by side, out is
  // [T][Hq / 2][vdim]: the first map's output minus *lam times the second's, divided by its root mean square over vdim, times out_scale.
  int maps;
  const float* lam;
  float out_scale, eps;
  int vdim;
};
// fp32 queries, cache and outputs (attention_f32.cu; bf16: differential attention only, with fp32 arithmetic): q / kv_cache / out / gate
// point at floats, num_q_tiles counts tiles of 16
// (token, query head of the group) rows over all requests; splits, short_q_len and the workspaces are not used.
int attention_f32_launch(const AttnParams& p, bool bf16, cudaStream_t st);
// mode 0: rows of a query tile are spread over warps (prefill / long queries); mode 1: keys are spread over warps
// (decode and short verify queries, with split-KV + combine).
int attention_launch(const AttnParams& p, int mode, cudaStream_t st);
unsigned int attention_read_status(bool clear);
void attention_read_status_async(unsigned int* dst, cudaStream_t st);
// Differential attention ahead of its kernels: per (token, head, map) RMS norm and rotation of queries and keys, cache insert.
struct DiffPrepareParams {
  const void* x;              // [T][ld]: q [2 H dim] | k [2 G dim] | v [G vdim]
  long long ld;
  const void *q_w, *k_w;      // norm weights [dim]
  float eps;
  const int *positions, *slots;   // slots negative: nothing is inserted
  const float* cos_sin;       // [positions][rot]
  void* q_out;                // [T][2 H][D / 2], zeros past dim
  void* cache;                // [blocks][2][G][bs][D]: key rows (map 1 | map 2), value rows, zeros in the padding
  int T, H, G, dim, vdim, D, rot, bs, interleaved, f32;
};
int diff_prepare_launch(const DiffPrepareParams& p, cudaStream_t st);
// tcgen05 prefill of differential attention (diff_prefill_tc.cu): requests with more than short_q_len new tokens, num_q_tiles counts their
// 128-token tiles; q contiguous.
bool diff_prefill_tc_sizes(int D, float softcap);
int diff_prefill_tc_launch(const AttnParams& p, long long num_blocks, cudaStream_t st);
unsigned int diff_prefill_read_status(bool clear);
void diff_prefill_read_status_async(unsigned int* dst, cudaStream_t st);

// tcgen05 prefill (attention_tc.cu): D == 128, 128-token query tiles; num_q_tiles counts those tiles.
int attention_prefill_tc_launch(const AttnParams& p, long long num_blocks, cudaStream_t st);
unsigned int attention_tc_read_status(bool clear);
void attention_tc_read_status_async(unsigned int* dst, cudaStream_t st);


struct RowStats {
  float p_draft;  // target probability of the draft token at the row's temperature
  int arg_all;    // arg-max of the row
  int arg_ex;     // recovered token: arg-max over v != draft of logit/T (+ Gumbel noise for random rows)
};
int rejection_launch(const void* logits, int is_fp32, const long long* draft_ids, const long long* num_draft, const long long* bonus,
                     const double* uniforms, const float* temperature, const float* synth_rates, RowStats* stats, long long* out, int B, int k, int V,
                     long long ld_b, long long ld_pos, unsigned long long seed, int use_noise, cudaStream_t st);

struct SampleParams {
  const void* logits;        // [B][ld] fp32 or bf16
  int is_fp32;
  long long ld;
  int B, V;
  const float* temperature;  // [B]; below 1e-5 the row takes its arg-max
  const int* top_k;          // [B] or null; <= 0 or >= V: off
  const float* top_p;        // [B] or null; >= 1: off
  const float* min_p;        // [B] or null; <= 0: off
  const unsigned long long* seeds;  // [B] one random 64-bit word per row and step
  long long* out;            // [B] sampled token ids
  unsigned char* kept;       // [B][V] or null: 1 where the token survived the filters
};
int sample_launch(const SampleParams& p, cudaStream_t st);

struct RouteParams {
  const void* logits;           // [T][ld] bf16 or fp32
  int is_fp32;
  long long ld;
  const float* bias;            // e_score_correction_bias [E] or null
  float* topk_w;                // [T][k]
  int* topk_ids;                // [T][k]
  int T, E, k, n_group, topk_group, sigmoid, renormalize;
  int whole_lanes;              // filled by the launcher: a group's scores lie in whole lanes of the warp
  float scaling;
};
int route_launch(const RouteParams& p, cudaStream_t st);
unsigned int sampling_read_status(bool clear);
void sampling_read_status_async(unsigned int* dst, cudaStream_t st);

struct MoePlanParams {
  int* counts;        // [E] scratch
  int* offsets;       // [E+1] first slot of each local expert
  int* cursor;        // [E] scratch
  int* total_slots;   // [1]
  int* work_count;    // [2] number of work items of the two grouped GEMMs
  int4* work1;        // GEMM 1 items {row tile in stacked w13, first slot, valid rows, output column base}
  int4* work2;        // GEMM 2 items (stacked w2)
  int E, tn, n1, n2;  // local experts, token tile, 128-row tiles per expert in w13 / w2
};
// xs: rows of Hp >= H elements, zeros past H
int moe_prepare_launch(const MoePlanParams& p, const int* ids, int n_pairs, int k, int e_off, int* slot_of, const void* x, long long ldx,
                       void* xs, int H, int Hp, int f32, cudaStream_t st);
// fp32 grouped product over the work list: out[slot][n] = sum_k a[slot][k] w[expert][n][k]; silu: a = silu(x[k]) * x[K + k]
int moe_gemm_f32_launch(const float* x, int ldx, const float* w, float* out, int N, int K, int silu, const int4* work, const int* work_count, int n_tiles,
                        int num_sms, cudaStream_t st);
int moe_plan_launch(const MoePlanParams& p, cudaStream_t st);
int moe_combine_launch(const void* a2, int lda, const int* slot_of, const float* w, void* y, int T, int k, int H, int f32, cudaStream_t st);
unsigned int moe_read_status(bool clear);
void moe_read_status_async(unsigned int* dst, cudaStream_t st);

struct MlaParams {
  const void* q_abs;            // [T][H][kv_lora] query with W_UK absorbed, contiguous
  const void* q_rope;           // [T][H][rope] with strides (elements)
  long long qr_st, qr_sh;
  const float* cos_sin;         // [positions][rope] (cos | sin): the kernel rotates q_rope; null: it is rotated already
  int interleaved;              // rotary pairs (2i, 2i + 1) instead of (i, i + rope / 2)
  const void* cache;            // [blocks][bs][kv_lora + rope_pad] latent | shared key part, zeros in the padding
  void* out;                    // [T][H][kv_lora]
  const int* query_start_loc;
  const int* seq_lens;
  const int* block_table;
  int bt_stride, R, T, H, kv_lora, rope, rope_pad, bs, bs_shift, max_q_len, splits;
  int skip_min_len;             // > 0: requests with at least this many new tokens are left to the prefill kernel
  int fine;                     // softmax weights enter the value product as two bf16 terms
  int f32;                      // element type of everything: fp32 instead of bf16
  float scale;
  float* ws_o;                  // [splits][T][H][kv_lora]
  float* ws_ml;                 // [splits][T][H][2]
  const float* sinks;           // [H] logits that join the softmax denominator only, or null
  const void* gate;             // [T][H] (row pitch gate_st): outputs are multiplied by its sigmoid, or null
  long long gate_st;
};
int mla_decode_launch(const MlaParams& p, cudaStream_t st);
bool mla_tensor_core_sizes(int kv_lora, int rope_pad);
// Prefill in the expanded form: gathered latents -> per-head keys and values (a GEMM in between) -> causal attention.
struct MlaPrefillParams {
  const __nv_bfloat16* cache;   // [blocks][bs][lora_pad + rope_pad]
  __nv_bfloat16 *lat, *rot;     // [rows][lora_pad], [rows][RC * 64]: the contexts of the listed requests, one after another
  const __nv_bfloat16* q;       // [T][q_st] rows of H x (nope + rope)
  long long q_st;
  __nv_bfloat16* q_out;         // [T][H][(NC + RC) * 64]
  const __nv_bfloat16* kv;      // [rows][H][(NC + VC) * 64] keys | values
  __nv_bfloat16* out;           // [T][H][vd]
  const int *query_start_loc, *seq_lens, *block_table, *positions;
  const int *long_req, *long_ctx;   // per listed request: its index, its first row in the gathered buffers
  const float* cos_sin;
  int bt_stride, bs, T, H, rows, num_long, num_q_tiles, lora_pad, rope_pad, nope, rope, vd, NC, RC, interleaved, fine;
  float scale;
  const float* sinks;           // as in MlaParams
  const __nv_bfloat16* gate;
  long long gate_st;
};
bool mla_prefill_sizes(int nope, int rope, int vd);
int mla_prefill_inputs_launch(const MlaPrefillParams& p, cudaStream_t st);   // gather + query rows
int mla_prefill_launch(const MlaPrefillParams& p, cudaStream_t st);
unsigned int mla_prefill_read_status(bool clear);
void mla_prefill_read_status_async(unsigned int* dst, cudaStream_t st);
struct MlaPrepareParams {
  const void *q, *kv;           // query latent [T][nq] or null; [T][lora + rope], pitches ld_q / ld_kv
  long long ld_q, ld_kv;
  const void *q_w, *kv_w;       // norm weights
  float eps;
  const int* positions;
  const float* cos_sin;         // [positions][rope]
  const int* slots;             // cache row per token, negative: none
  void* q_out;                  // [T][nq]
  void* cache;                  // rows of `width` elements: latent at 0, key part at lora_pad
  int T, nq, lora, lora_pad, rope, width, interleaved, f32;
};
int mla_prepare_launch(const MlaPrepareParams& p, cudaStream_t st);
struct MlstmParams {
  const void* x;                // [T][ld] q [H D] | k [H D] | v [H V] | output gate [H V]
  long long ld;
  const float* gates;           // [T][ld_g] input | forget gate logits
  long long ld_g;
  const float *i_bias, *f_bias; // [H]
  const void* norm_w;           // [H V]
  float eps, cap, scale;        // scale: of the queries
  float *S, *n, *m;             // [slots][H][D][V], [slots][H][D], [slots][H]
  void* out;                    // [T][H V]
  const int *query_start_loc, *state_slots, *has_initial_state;
  int T, R, H, D, V, f32, skip_min_len;
  // chunked form: one segment of the step's chunk list
  const int *chunk_req, *chunk_t0, *chunk_long;      // per chunk: request, first token, entry of the sequence list
  const int *long_req, *long_chunk0, *long_n;        // per sequence of the segment: request, first chunk, chunks
  float *ws_s, *ws_n, *ws_g, *ws_m;                  // [chunks][H][D V], [chunks][H][D], [chunks][H][2], [chunks][H]
  __nv_bfloat16* ws_h;                               // [chunks][H][2][D V] state ahead of the chunk in two terms
  int vec_qk, vec_v;                                 // rows of q / k, and of v / the state planes, start on 16-byte boundaries
};
int mlstm_recurrent_launch(const MlstmParams& p, cudaStream_t st);
bool mlstm_chunkable(int D, int V);
int mlstm_chunk_launch(const MlstmParams& p, int num_chunks, int num_long, cudaStream_t st);
int sigmoid_mul_launch(const void* x, long long ldx, const void* gate, long long ldg, void* y, int T, int N, int f32, cudaStream_t st);
unsigned int mla_read_status(bool clear);
void mla_read_status_async(unsigned int* dst, cudaStream_t st);

struct GdnConvParams {
  const __nv_bfloat16* x;   // [T][ldx] pre-conv mixed q|k|v (column slice allowed)
  long long ldx;
  const __nv_bfloat16* w;   // [C][kw]
  __nv_bfloat16* y;         // [T][C] contiguous
  __nv_bfloat16* conv_state;  // [slots][C][kw-1], updated in place
  const int* query_start_loc;
  const int* state_slots;
  const int* has_initial_state;
  int T, R, C, kw;
  const int* n_valid;              // optional [R]: count only this many tokens of each chunk (speculative commit)
  const __nv_bfloat16* prev_state; // optional [R][C][kw-1]: snapshot of the state before the chunk (speculative commit)
};

struct GdnParams {
  const __nv_bfloat16 *q, *k, *v;  // post-conv tensors: q,k [T][Hk*K], v [T][Hv*V] with a common row pitch ld_qkv
  long long ld_qkv;
  const __nv_bfloat16 *a, *b;      // [T][Hv] gate inputs with row pitch ld_ba
  long long ld_ba;
  const float *A_log, *dt_bias;    // [Hv]
  float* state;                    // [slots][Hv][K][V] fp32
  __nv_bfloat16* out;              // [T][Hv*V]
  const int* query_start_loc;
  const int* state_slots;
  const int* has_initial_state;
  int R, Hk, Hv, K, V;
  int write_state;                 // 0: leave the slot untouched (speculative verification commits later)
  float* spec_state;               // optional [R][spec_q][Hv][K][V]: state after each token
  int spec_q;
  int skip_min_len;                // > 0: sequences with at least this many tokens are left to the chunked kernels
};

// Chunked prefill (gdn_chunk.cu): sequences of at least `GdnParams::skip_min_len` tokens are split into 64-token chunks listed by
// the host; the recurrent kernel skips them.
struct GdnChunkParams {
  const __nv_bfloat16 *q, *k, *v;
  long long ld_qkv;
  const __nv_bfloat16 *a, *b;
  long long ld_ba;
  const float *A_log, *dt_bias;
  float* state;
  __nv_bfloat16* out;
  const int* query_start_loc;
  const int* state_slots;
  const int* has_initial_state;
  int Hk, Hv, K, V, write_state;
  __nv_bfloat16* ws;          // gdn_chunk_workspace_elems(num_chunks, Hv) elements
  const int* chunk_req;       // [num_chunks] request of each chunk
  const int* chunk_t0;        // [num_chunks] first token of each chunk
  int num_chunks;
  const int* long_req;        // [num_long] requests on the chunked path
  const int* long_chunk0;     // [num_long] index of the request's first chunk
  int num_long;
};
size_t gdn_chunk_workspace_elems(int num_chunks, int Hv);
int gdn_chunk_launch(const GdnChunkParams& p, cudaStream_t st);

int gdn_conv_launch(const GdnConvParams& p, cudaStream_t st);
int gdn_conv_commit_launch(const GdnConvParams& p, cudaStream_t st);
int gdn_recurrent_launch(const GdnParams& p, cudaStream_t st);
unsigned int gdn_read_status(bool clear);
void gdn_read_status_async(unsigned int* dst, cudaStream_t st);

struct CausalConvParams {
  const void* x;                // [T][C], row pitch ldx
  long long ldx;
  const void *w, *bias;         // [C][taps], [C] or null
  void* y;                      // [T][C]
  void* state;                  // [slots][max(taps - 1, 1)][C], updated in place
  const int *query_start_loc, *state_slots, *has_initial_state;
  int T, R, C, taps, silu, residual, f32;
};
int causal_conv_launch(const CausalConvParams& p, cudaStream_t st);

// Recurrences with a matrix state (recurrence.cu). channel delta: q, k [Hk D], v [H V], a decay logits, b step logits; Mamba-2 (delta = 0): q = C and
// k = B [Hk D] (Hk groups, D the state size), v = x [H V], b the dt logits.
struct RecurrenceParams {
  const void *q, *k, *v;        // rows of a common pitch ld
  long long ld;
  const float* a;               // [T][H D], pitch ld_a
  long long ld_a;
  const void* b;                // [T][H], pitch ld_b
  long long ld_b;
  const float *A_log, *dt_bias, *skip;   // [H]; [H D] (delta) or [H]; [H]
  float dt_min, dt_max, scale;
  float* state;                 // [slots][H][D][V]
  void* out;                    // [T][H V]
  const int *query_start_loc, *state_slots, *has_initial_state;
  int T, R, Hk, H, D, V, delta, f32, skip_min_len;
};
int recurrence_launch(const RecurrenceParams& p, cudaStream_t st);
// Chunked forms for bf16 portions of at least 64 tokens (recurrence_chunk.cu); the recurrent kernel skips those (skip_min_len).
struct DeltaChunkParams {
  const __nv_bfloat16 *q, *k, *v;
  long long ld;
  const float* a;
  long long ld_a;
  const __nv_bfloat16* b;
  long long ld_b;
  const float *A_log, *dt_bias, *skip;
  float dt_min, dt_max, scale;
  float* state;
  __nv_bfloat16* out;
  const int *query_start_loc, *state_slots, *has_initial_state;
  const int *chunk_req, *chunk_t0, *long_req, *long_chunk0, *long_n;   // one segment of the step's chunk list, see MlstmParams
  __nv_bfloat16* ws;            // delta: [chunks][H] x delta_chunk_elems
  int Hk, H, D, V, Vp, vec;     // Vp: V rounded up to 32; vec: every row of q, k, v starts on a 16-byte boundary
};
bool recurrence_chunkable(int D, int V);
size_t delta_chunk_elems(int D, int Vp);
int delta_chunk_launch(const DeltaChunkParams& p, int chunks, int longs, cudaStream_t st);
int ssd_chunk_launch(const DeltaChunkParams& p, int longs, cudaStream_t st);
struct GatedNormParams {
  const void *x, *gate, *w;     // [T][n], [T][n], [n] or one part's
  long long ld_x, ld_g;
  void* y;                      // [T][n]
  float eps;
  int T, n, groups, w_shared, gate_first, f32;
};
int gated_norm_launch(const GatedNormParams& p, cudaStream_t st);

struct TalkPrepareParams {
  const void* qk;               // [T][H dim | G dim], pitch ld
  long long ld;
  const float* gain;            // [H dim]
  float eps, coef;
  int every;                    // 0: no temperature
  const int *positions, *slots;
  void *q_out, *pages;          // [T][H][row]; [blocks][G][bs][row]
  float* k_scale;               // [blocks][bs]
  int T, H, G, dim, row, bs, f32;
};
int talk_prepare_launch(const TalkPrepareParams& p, cudaStream_t st);
struct TalkParams {
  const void *q, *pages, *mix;  // as talk_prepare leaves them; [H][H] (to, from)
  const float *k_scale, *bias;  // [blocks][bs]; [2][H]: r1, r2
  void* out;                    // [T][H][dim]
  const int *query_start_loc, *seq_lens, *block_table;
  int bt_stride, T, R, H, G, dim, row, bs, f32;
};
int talk_plain_launch(const TalkParams& p, cudaStream_t st);
// Tensor-core forms: single tokens (talk_decode.cu) and portions of at least min_len tokens (talk_prefill_tc.cu), launched apart.
int talk_tc_row(int H, int G, int dim);   // width of a query row and of a cached row, zeros behind dim; 0: only the plain kernel takes the sizes
struct TalkTcParams {
  TalkParams t;
  float* ws_ml;                 // [rows][H][2] reference (log2 domain) and sum; rows: [splits][R] (single tokens), or tokens of a segment's tiles
  float* ws_o;                  // [rows][H][G row] unnormalised results over the rows of all key heads
  int splits, min_len;
  int tile0, bs_shift;          // set by the launchers
};
int talk_decode_launch(const TalkTcParams& p, cudaStream_t st);
int talk_join_launch(const TalkTcParams& p, bool dec, int rows, cudaStream_t st);
// tiles: 128-token tiles over the portions; `segment` of them at a time go through the workspace
int talk_prefill_launch(const TalkTcParams& p, int tiles, int segment, long long num_blocks, cudaStream_t st);
unsigned int talk_prefill_read_status(bool clear);
void talk_prefill_read_status_async(unsigned int* dst, cudaStream_t st);

}  // namespace oc
