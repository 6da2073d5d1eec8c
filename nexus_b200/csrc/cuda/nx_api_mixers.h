// C ABI of the building blocks of decoders with heterogeneous layers: pre / post norms around a sublayer, residuals of several
// streams, norms of queries and keys, heads that mix, rotary
// embedding fused with the cache append, windowed and soft-capped paged attention for any head sizes, the short causal
// convolution with its carried tail, the Mamba-2 (SSD), gated-delta-rule and gated-linear-attention recurrences with their
// carried FP32 state, gated norms, gated activations, the per-layer token input and soft-capping of logits.
//
// Activations are BF16 or FP32 (`dtype`: NX_BF16 / NX_F32); weights of norms, decays and convolutions are FP32.
//
// A batch is a packed list of rows (tokens); a segment is the run of consecutive rows that one sequence contributes to
// the step: seg_row0 (first row), seg_len (rows; 0 marks a padding entry of a captured batch), seg_pos (position of
// the first row in its sequence) and seg_seq (sequence slot: the row of the block table and of every state tensor).
// A segment that starts at position 0 starts from a zero state, whatever the slot held before.
#pragma once
#include "nx_api.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef struct NxSegments {
  const int32_t* row0;
  const int32_t* len;
  const int32_t* pos;
  const int32_t* seq;
  int32_t count;
  int32_t max_len;    // largest len of the list (host copy)
  int32_t total_len;  // sum of len (host copy)
} NxSegments;

typedef struct NxResidualNormArgs {
  float* x;                // [rows, cols] residual stream, updated in place (written when `table`, `y` or `experts` is given)
  const int32_t* tokens;   // with `table`: x = embed_scale * table[tokens[row]]
  const void* table;       // [vocab, cols] dtype, may be null
  const void* y;           // [rows, ldy] sublayer output, may be null: x += res_mult * rms(y) * w_post
  const float* w_post;     // may be null: x += res_mult * y
  const float* w_next;     // may be null; else h = rms(x) * w_next
  void* h;                 // [rows, ldh]; columns cols..ldh are zeroed
  void* x_cast;            // [rows, ldh], may be null: x in the activation dtype
  int64_t ldy, ldh;
  int32_t rows, cols, dtype;
  float eps, embed_scale, res_mult;
  // Sublayer output of a layer of experts, may be null: expert_scale * sum_j w_j experts[expert_slots[row * top + j]] with w_j =
  // expert_weights[row * top + j] (null: 1), plus y_gate[row] * y[row] when `y` is given too (y_gate null: plain y).
  const void* experts;     // [slots, ld_experts]
  const int32_t* expert_slots;
  const float* y_gate;
  int64_t ld_experts;
  int32_t top;
  float expert_scale;
  // dot_out[row] = sigmoid(x . w_dot), may be null
  const float* w_dot;
  float* dot_out;
  // copies of the x_cast row at scatter[scatter_slots[row * top + j]], may be null (pitch ldh)
  void* scatter;
  const int32_t* scatter_slots;
  const float* expert_weights;
  // with `table`: x += pos_table[positions[row]], may be null
  const int32_t* positions;
  const void* pos_table;   // [positions, cols] dtype
} NxResidualNormArgs;
int nx_residual_norm(const NxResidualNormArgs* args, nx_stream_t stream);

// Residual of several streams x_s.  table: every stream becomes embed_scale * table[token] + pos_table[position]; else with y the
// streams become x_t <- sum_s mix[s][t] x_s + out[t] y.  Then h = rms(sum_s in[s] x_s) * w_next of the new streams.
typedef struct NxStreamResidualArgs {
  float* x;                // [rows, streams, cols], updated in place
  const int32_t* tokens;
  const void* table;       // [vocab, cols] dtype, may be null
  const int32_t* positions;
  const void* pos_table;   // [positions, cols] dtype, may be null
  const void* y;           // [rows, ldy], may be null
  const float* mix;        // [streams, streams]: from, to
  const float* out;        // [streams]
  const float* in;         // [streams]; null: ones
  const float* w_next;     // [cols]
  void* h;                 // [rows, ldh], may be null; columns cols..ldh are zeroed
  int64_t ldy, ldh;
  int32_t rows, cols, streams, dtype;   // up to 8 streams of up to 49152 columns
  float eps, embed_scale;
} NxStreamResidualArgs;
int nx_stream_residual(const NxStreamResidualArgs* args, nx_stream_t stream);

// What lies between the projections and the scores of attention on normed queries and keys, in place in `proj`: RMS norms of q and
// k (over each head with one shared weight, or norm_all: over all heads at once), q also times q_scale * head_scale[head] * (1 + coef
// ln(floor((p + 1) / every) + 1)), unit_values: v divided by its root mean square per head; k and v go to the cache (with store_kv
// back to proj too), gate = sigmoid.  Heads are dim / vdim columns wide, of which the leading norm_dim / norm_vdim count (the rest
// are zeros).
typedef struct NxHeadPrepArgs {
  void* proj;              // [rows, ld]; the parts of a row start at q_off, k_off, v_off, g_off
  int64_t ld;
  int32_t q_off, k_off, v_off, g_off;
  int32_t rows, heads, kv_heads, dim, vdim, norm_dim, norm_vdim, norm_all, unit_values, store_kv, every, dtype;   // every 0: none
  float eps, q_scale, coef;
  const float* w_q;        // [dim], or [heads * dim] with norm_all
  const float* w_k;        // [dim], or [kv_heads * dim]
  const float* head_scale; // [heads], may be null
  const int32_t* positions;
  const int32_t* slots;    // cache slot per row, negative: nothing is appended
  void* k_cache;           // [slots, kv_heads, dim]
  void* v_cache;           // [slots, kv_heads, vdim]
  float* gate;             // [rows, heads], may be null
} NxHeadPrepArgs;
int nx_head_prep(const NxHeadPrepArgs* args, nx_stream_t stream);

// Heads that mix their weights after the softmax, on the outputs: wide [rows, heads, kv_heads, vdim] holds what every head's weights
// give with the values of every KV head; out [rows, heads, vdim]: out_h = gate_h sum_g talk[h][g] wide[g][KV head of h].
int nx_head_mix(const void* wide, int64_t ldw, const float* talk, const float* gate, void* out, int64_t ldo, int rows, int heads,
                int kv_heads, int vdim, int dtype, nx_stream_t stream);

typedef struct NxRopeAppendArgs {
  void* proj;              // [rows, ld]; q, k, v of a row start at q_off, k_off, v_off; q and k are rotated in place
  int64_t ld;
  int32_t q_off, k_off, v_off;
  int32_t rows, heads, kv_heads, dim, vdim, rot_dims, dtype;
  const int32_t* positions;
  const int32_t* slots;    // cache slot per row, negative: nothing is appended
  const float* cos_t;      // [max_pos, rot_dims / 2]
  const float* sin_t;
  void* k_cache;           // [slots, kv_heads, dim]
  void* v_cache;           // [slots, kv_heads, vdim]
} NxRopeAppendArgs;
int nx_rope_append(const NxRopeAppendArgs* args, nx_stream_t stream);

// What lies between the down projections of latent attention and its cache: the query latent and the key / value latent
// are normed, the shared key part is rotated, latent and key part go to the cache (and to `lat`), the output gate's
// sigmoid is taken.  q_rank 0: queries have no latent; gate null: no output gate.
typedef struct NxLatentPrepArgs {
  const void* proj;        // [rows, ld]; the parts of a row start at q_off, c_off, r_off, g_off
  int64_t ld;
  int32_t q_off, c_off, r_off, g_off;
  int32_t rows, q_rank, kv_rank, rot_dims, heads, dtype;
  float eps;
  const float* w_q;        // [q_rank]
  const float* w_kv;       // [kv_rank]
  const int32_t* positions;
  const int32_t* slots;    // cache slot per row, negative: nothing is appended
  const float* cos_t;      // [max_pos, rot_dims / 2]
  const float* sin_t;
  void* cq;                // [rows, ldq]: normed query latent, columns q_rank..ldq are zeroed
  int64_t ldq;
  void* cache;             // [slots, ld_cache]: latent, at column rot_col the rotated key part; other columns stay as they are
  int64_t ld_cache;
  int32_t rot_col;
  void* lat;               // [rows, ld_cache], may be null: the cache row, its other columns zero
  float* gate;             // [rows, heads]: sigmoid
} NxLatentPrepArgs;
int nx_latent_prep(const NxLatentPrepArgs* args, nx_stream_t stream);
// Rotates `rot_dims` columns of every head: src [rows, ld_src], head h at h * src_head + src_off; dst likewise (the same
// place is allowed).  Columns rot_dims..width of dst become zeros.
int nx_rope_heads(const void* src, int64_t ld_src, int src_head, int src_off, void* dst, int64_t ld_dst, int dst_head,
                  int dst_off, int rows, int heads, int rot_dims, int width, const int32_t* positions, const float* cos_t,
                  const float* sin_t, int dtype, nx_stream_t stream);

// y = silu(causal_conv(x) + bias) per channel; state [slots, taps - 1, channels] holds the last taps - 1 inputs.
typedef struct NxConvArgs {
  const void* x;           // [rows, ldx]
  void* y;                 // [rows, ldy]
  const float* w;          // [taps, channels], last row: the current token
  const float* bias;       // [channels] or null
  void* state;             // dtype
  int64_t ldx, ldy;
  int32_t channels, taps, dtype;
  NxSegments seg;
} NxConvArgs;
int nx_conv_silu(const NxConvArgs* args, nx_stream_t stream);

// The convolution without an activation over the packed projections q (heads * dim) | k (kv_heads * dim) | v (kv_heads *
// vdim), then what attention needs of them: pairs of neighbouring columns (2 i, 2 i + 1) of q and k rotate for i < rot_dims / 2,
// v becomes (1 - mix) v + mix first, k and v go to the cache and q (with store_kv also k and v) to y.  dim and vdim are
// multiples of 4.
typedef struct NxConvRopeArgs {
  NxConvArgs conv;         // channels = heads * dim + kv_heads * (dim + vdim)
  int32_t heads, kv_heads, dim, vdim, rot_dims, store_kv;
  const int32_t* slots;    // cache slot per row, negative: nothing is appended
  const float* cos_t;      // [max_pos, rot_dims / 2]
  const float* sin_t;
  void* k_cache;           // [slots, kv_heads, dim]
  void* v_cache;           // [slots, kv_heads, vdim]
  const float* mix;        // one value, may be null
  void* first;             // [rows, kv_heads * vdim]: read with `mix`, otherwise written; may be null without `mix`
} NxConvRopeArgs;
int nx_conv_rope_append(const NxConvRopeArgs* args, nx_stream_t stream);

// Mamba-2: S = exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x,  dt = softplus(dt_raw + dt_bias).
typedef struct NxSsdArgs {
  const void* xbc;         // [rows, ld_xbc]: x (heads * vdim) | B (groups * state) | C (groups * state)
  const void* dt;          // [rows, ld_dt]: heads raw step sizes
  void* y;                 // [rows, ldy]: heads * vdim
  const float* dt_bias;
  const float* a_log;
  const float* d_skip;
  float* state;            // [slots, heads, state, vdim]
  int64_t ld_xbc, ld_dt, ldy;
  int32_t heads, groups, n_state, vdim, dtype;
  NxSegments seg;
  // Long segments on the tensor cores only: the segment list is cut into `parts` spans of `span` tokens per segment
  // (span a multiple of 64); part_state [seg.count, parts, heads, state, vdim] and part_decay [seg.count, parts, heads]
  // are scratch.  parts == 1: no scratch.
  float* part_state;
  float* part_decay;
  int32_t parts, span;
} NxSsdArgs;
// token by token, any sizes and both dtypes
int nx_ssd_step(const NxSsdArgs* args, nx_stream_t stream);
// chunks of 64 tokens on the tensor cores, BF16 activations, state <= 256, vdim <= 256
int nx_ssd_chunk(const NxSsdArgs* args, nx_stream_t stream);

// Gated delta rule: S = g S;  u = beta (v - S^T k);  S += k u^T;  o = S^T q, with unit q / k (q also times dim^-1/2),
// beta = sigmoid(b), g = exp(-exp(A_log) softplus(a + dt_bias)).
typedef struct NxDeltaArgs {
  const void* qkv;         // [rows, ld_qkv]: q (kv_heads * dim) | k (kv_heads * dim) | v (heads * vdim)
  const void* b;           // [rows, ld_ba]: heads
  const void* a;           // [rows, ld_ba]: heads
  void* o;                 // [rows, ldo]: heads * vdim
  const float* dt_bias;
  const float* a_log;
  float* state;            // [slots, heads, dim, vdim]
  int64_t ld_qkv, ld_ba, ldo;
  int32_t heads, kv_heads, dim, vdim, dtype;
  float unit_eps, q_scale;
  NxSegments seg;
  void* scratch;           // chunked form: nx_delta_scratch_bytes
} NxDeltaArgs;
// token by token, any sizes and both dtypes
int nx_delta_step(const NxDeltaArgs* args, nx_stream_t stream);
// chunks of 64 tokens on the tensor cores, BF16 activations, dim <= 256
int64_t nx_delta_scratch_bytes(int heads, int segments, int max_len);
int nx_delta_chunk(const NxDeltaArgs* args, nx_stream_t stream);

// Gated linear attention: S = diag(2^a) S + k v^T,  o = S^T (q_scale q), a decay per key channel.
typedef struct NxGlaArgs {
  const void* q;           // [rows, ld]: heads * dim
  const void* k;           // [rows, ld]: heads * dim
  const void* v;           // [rows, ld]: heads * vdim
  const float* decay;      // [rows, ld_decay]: log2 of the decays (<= 0), heads * dim
  void* o;                 // [rows, ldo]: heads * vdim
  float* state;            // [slots, heads, dim, vdim]
  int64_t ld, ld_decay, ldo;
  int32_t heads, dim, vdim, dtype;
  float q_scale;
  NxSegments seg;
  // Chunked form only: spans of a segment that run at the same time (as in NxSsdArgs); part_state [seg.count, parts, heads, dim,
  // vdim], part_decay [seg.count, parts, heads, dim].
  float* part_state;
  float* part_decay;
  int32_t parts, span;
} NxGlaArgs;
// token by token, any sizes and both dtypes
int nx_gla_step(const NxGlaArgs* args, nx_stream_t stream);
// chunks of 64 tokens on the tensor cores, BF16 activations, dim <= 256
int nx_gla_chunk(const NxGlaArgs* args, nx_stream_t stream);
// out[r][c] = log2(sigmoid(z)) / tau (FP32, [rows, ldo]), z = sum_j a[r][j] w[c][j] + bias[c]: a [rows, lda] activations, w FP32
// [cols, rank]
int nx_decay_gate(const void* a, int64_t lda, const float* w, const float* bias, float* out, int64_t ldo, int rows, int cols,
                  int rank, float tau, int dtype, nx_stream_t stream);

// gate_first: out = rms(y * silu(z)) * w * out_scale, else out = rms(y) * w * silu(z) * out_scale; statistics over each
// of `groups` equal parts of a row.  w has groups * group_size entries, or group_size shared by every part (w_shared).
typedef struct NxGatedNormArgs {
  const void* y;
  const void* z;
  const float* w;
  void* out;
  int64_t ldy, ldz, ldo;
  int32_t rows, groups, group_size, gate_first, w_shared, dtype;
  float eps, out_scale;
} NxGatedNormArgs;
int nx_gated_norm(const NxGatedNormArgs* args, nx_stream_t stream);

// out[r][j] = gelu_tanh(a[r][j]) * table[tokens[r]][offset + j], j < dim; columns dim..ldo are zeroed.  `a` is FP32: far
// out on the negative side the relative slope of GELU is its argument, so a rounded argument would show in the product.
int nx_token_side_gate(const float* a, int64_t lda, const int32_t* tokens, const void* table, int64_t ld_table, int offset,
                       void* out, int64_t ldo, int rows, int dim, int dtype, nx_stream_t stream);
// out[r][j] = silu(h[r][j]) * h[r][half + j], j < half
int nx_silu_mul(const void* h, int64_t ldh, void* out, int64_t ldo, int rows, int half, int dtype, nx_stream_t stream);
// Gated activation; half: columns of the output; gates and values lie in two halves of h, or (interleaved) in turns of eight
// columns, gates first.
int nx_glu(const void* h, int64_t ldh, void* out, int64_t ldo, int rows, int half, int interleaved, NxGlu glu, int dtype,
           nx_stream_t stream);
// x = cap * tanh(scale * x / cap) in place on FP32 [rows, ld]; cap 0: x = scale * x
int nx_softcap(float* x, int64_t ld, int rows, int cols, float cap, float scale, nx_stream_t stream);

// Causal attention of packed query rows over a paged cache.  Row at position p sees keys p - window + 1 .. p (window <= 0:
// 0 .. p), with chunk > 0 only those of its own chunk (p / chunk), and the first keep_first keys; score = scale * q.k, soft-capped
// when softcap > 0, plus bias[head][min(distance, bias_len - 1)].  sink: a score per head (not scaled) that counts in the denominator
// only.  The rows' own keys are in the cache already.  all_values: every query head meets the values of every KV head, out is
// [rows, heads, kv_heads, vdim] (prompt and FP32 kernels).
typedef struct NxPagedWindowArgs {
  const void* q;           // [rows, ldq]: heads * dim
  const void* k_cache;     // [blocks * block_size, kv_heads, dim]
  const void* v_cache;     // [blocks * block_size, kv_heads, vdim]
  const int32_t* block_table;  // [slots, max_blocks]
  void* out;               // [rows, ldo]: heads * vdim, times out_scale
  int64_t ldq, ldo;
  float* part_o;           // decode with splits > 1: [count, heads, splits, vdim]
  float* part_ml;          // decode with splits > 1: [count, heads, splits, 2]
  int32_t heads, kv_heads, dim, vdim, block_size, max_blocks, window, splits, dtype;
  float scale, softcap, out_scale;
  NxSegments seg;
  int64_t k_pitch, v_pitch;  // elements between cache slots: kv_heads * dim and kv_heads * vdim, or the row of a latent cache,
                             // whose values are the leading columns of its keys
  const float* gate;         // [rows, heads] factor of the output, may be null
  const float* sink;         // [heads], may be null
  int32_t keep_first;
  int32_t chunk, bias_len, all_values;
  const float* bias;         // [heads, bias_len], may be null
} NxPagedWindowArgs;
// one-row segments, BF16: tensor-core tiles of up to 16 query heads of a KV head against 64 keys, split over the keys
int nx_paged_window_decode(const NxPagedWindowArgs* args, nx_stream_t stream);
// longer segments, BF16: 128 (row, head) pairs of one KV head against tiles of 64 keys
int nx_paged_window_prefill(const NxPagedWindowArgs* args, nx_stream_t stream);
// any segments, FP32
int nx_paged_window_f32(const NxPagedWindowArgs* args, nx_stream_t stream);
// One-row and short segments, BF16, of heads that mix their weights: weight_h <- sum_g talk[h][g] weight_g, FP32, before the values of
// the KV head of h.  Scratch has `rows` = nx_talk_rows(..) rows: scores [rows, heads, pitch] and weights of the same shape, part_ml
// [rows, heads, splits, 2], with splits > 1 part_o [rows, heads, splits, vdim].  No sink, no all_values; up to 96 heads of up to 256
// columns.
typedef struct NxTalkPagedArgs {
  NxPagedWindowArgs base;
  const float* talk;         // [heads, heads]
  float* scores;
  void* weights;             // BF16
  int64_t pitch;             // a multiple of 64, at least the keys that rows of one tile (64 / query heads per KV head) can see
  int32_t rows;
} NxTalkPagedArgs;
int nx_talk_rows(int heads, int kv_heads, int count, int max_len, int total_len);
int nx_talk_paged(const NxTalkPagedArgs* args, nx_stream_t stream);


// Attention of packed query rows over a latent cache, BF16: every head meets the same cache row [latent (rank) | rotated key
// part], whose leading `rank` columns are the values.  score = scale * q . row; out = gate * softmax-weighted sum of the
// latents.  Windows as above.
typedef struct NxLatentAttnArgs {
  const void* q;           // [rows, ldq]: heads * row
  const void* cache;       // [blocks * block_size, row]
  const int32_t* block_table;  // [slots, max_blocks]
  void* out;               // [rows, ldo]: heads * rank
  const float* gate;       // [rows, heads], may be null
  float* part_o;           // splits > 1: [rows, heads, splits, rank]
  float* part_ml;          // splits > 1: [rows, heads, splits, 2]
  int* status;
  int64_t ldq, ldo;
  int32_t heads, row, rank, block_size, max_blocks, window, splits;   // row a multiple of 64 up to 768, rank of 16 up to 512,
  int32_t n_slots;                                                    // block_size of 8; n_slots = blocks * block_size
  float scale;
  NxSegments seg;
} NxLatentAttnArgs;
int nx_latent_attention(const NxLatentAttnArgs* args, nx_stream_t stream);

// The same attention for prompts, BF16, on keys and values formed from the latents: a head's key is its own part (dim) beside
// the shared rotated part (rot).  q [q_rows, ldq]: head h at h * q_head, own part then rotated part; kv [kv_rows, ldkv]:
// heads * dim keys, heads * vdim values; lat [kv_rows, ld_lat]: latent rows, the shared key part at column `rank`.
// blocks [n_blocks, 4]: first row of q, rows (1..256), position of the first row, row of kv / lat that position 0 would have
// (rows of positions no row can see need not exist); most expensive blocks first.  out [., ldo]: heads * vdim, times the gate.
typedef struct NxLatentPromptArgs {
  const void* q;
  const void* kv;
  const void* lat;
  void* out;
  const float* gate;       // [rows, heads], may be null
  const int32_t* blocks;   // 16-byte aligned
  int* status;
  int64_t ldq, ldkv, ld_lat, ldo;
  int32_t n_blocks, q_rows, kv_rows, q_head, rank, heads, dim, rot, vdim, window;  // dim <= 128, rot <= 64: multiples of 16;
  float scale;                                                                     // vdim <= 128: multiple of 8; scale > 0
} NxLatentPromptArgs;
int nx_latent_prompt(const NxLatentPromptArgs* args, nx_stream_t stream);

// The same kernel on plain grouped keys and values: q [q_rows, ldq]: heads * dim; k [kv_rows, ldk]: kv_heads * dim; v [kv_rows,
// ldv]: kv_heads * vdim; query head h reads KV head h / (heads / kv_heads).  Windows, kept first keys and sinks as in
// NxPagedWindowArgs, chunks and biases (up to 3072 distances) too.  blocks as above; kept [n_blocks]: row that position 0
// has among the kept keys (null: the fourth entry of the block).  dim <= 128: multiple of 16; vdim <= 128: multiple of 8; scale > 0.
typedef struct NxWindowPromptArgs {
  const void* q;
  const void* k;
  const void* v;
  void* out;               // [., ldo]: heads * vdim
  const float* sink;       // [heads], may be null
  const int32_t* blocks;
  const int32_t* kept;
  int* status;
  int64_t ldq, ldk, ldv, ldo;
  int32_t n_blocks, q_rows, kv_rows, heads, kv_heads, dim, vdim, window, keep_first;
  float scale;
  const float* gate;       // [rows, heads], may be null
  const float* bias;       // [heads, bias_len], may be null
  int32_t bias_len, chunk;
} NxWindowPromptArgs;
int nx_window_prompt(const NxWindowPromptArgs* args, nx_stream_t stream);

// The same for heads that mix: every query head with the values of every KV head, out [., ldo]: heads * kv_heads * vdim.  Layouts,
// sizes and blocks as above, without kept keys and sinks.  bias [heads, bias_pitch], may be null: entry NX_TALK_BIAS_NEAR + distance in
// units of log2, for the distances -NX_TALK_BIAS_NEAR .. bias_len + NX_TALK_BIAS_FAR - 1 (any finite value below 0, the last one from
// bias_len on); bias_pitch a multiple of 4.
enum { NX_TALK_BIAS_NEAR = 256, NX_TALK_BIAS_FAR = 256, NX_TALK_BIAS_MAX = 3072 };
typedef struct NxTalkPromptArgs {
  const void* q;
  const void* k;
  const void* v;
  void* out;
  const float* bias;
  const int32_t* blocks;
  int* status;
  int64_t ldq, ldk, ldv, ldo;
  int32_t n_blocks, q_rows, kv_rows, heads, kv_heads, dim, vdim, window, chunk, bias_len, bias_pitch;
  float scale;
} NxTalkPromptArgs;
int nx_talk_prompt(const NxTalkPromptArgs* args, nx_stream_t stream);
// Cache rows of `segments` runs of positions into one packed buffer.  list [segments, 4]: first destination row, rows, first
// position, sequence; `longest`: most rows of a run.
int nx_latent_gather(const void* cache, void* dst, const int32_t* block_table, const int32_t* list, int segments, int longest,
                     int max_blocks, int block_size, int row, nx_stream_t stream);

#ifdef __cplusplus
}
#endif
