/* quickdraw_b200 — C ABI of the kernels for models with bf16 weights and an fp32 residual stream
 * (libquickdraw_b200_hybrid.so): dense products, the residual stream, grouped-query attention over bounded spans.  Mechanisms
 * that only some of these models have are libraries of their own: gated linear recurrences
 * (libquickdraw_b200_recurrent.so), latent attention (libquickdraw_b200_latent.so).
 *
 * The conventions of quickdraw_b200.h hold: device pointers, sizes and a stream (as void*), asynchronous, nothing
 * allocated, a QD_* code returned.  Weights, norm weights, biases, taps and sinks are bf16.  dtype selects the
 * activation type: QD_BF16 or QD_F32 (everything in true fp32).
 */
#ifndef QUICKDRAW_B200_HYBRID_H
#define QUICKDRAW_B200_HYBRID_H

#include "quickdraw_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

enum { QD_BF16 = 0, QD_F32 = 1 };
enum { QD_GREEDY_BLOCKS = 128 };

/* y[t, n] = sum_k x[t, k] w[n, k] (+ bias[n], fp32, where given) with bf16 weights [rows, width] (contiguous) and fp32
 * accumulation.  The first gelu_cols outputs pass through the exact GELU.  glu: weight rows 2i and 2i + 1 are a gate and
 * its linear partner, y[t, i] = relu(gate) * partner, rows / 2 outputs.  add: the result is added to y.  x: [tokens,
 * width], rows ldx elements apart; y: [tokens, outputs], ldy apart; each bf16 or fp32.  Many bf16 token rows run on
 * tcgen05 (TMA needs width, ldx, ldy and rows to be multiples of eight), up to eight token rows stream the weights,
 * anything else takes FMA tiles.  norm (bf16 [width], or NULL): x enters as x / rms(x) * (norm_offset + norm); up to
 * eight token rows with width and ldx multiples of eight only.
 * status: device word, bit 0 is set if a bounded wait ran out. */
int qd_linear(const void* x, long long ldx, int x_dtype, const void* w, void* y, long long ldy, int y_dtype, int
    tokens, int rows, int width, int gelu_cols, int glu, const float* bias, int add, const void* norm, float norm_offset,
    float eps, unsigned int* status, void* stream);

/* token (int64) = index of the largest of `count` fp32 logits, the lowest among equals.  keys: QD_GREEDY_BLOCKS
 * 64-bit words, counter: one word, zero before the first call. */
int qd_greedy(const float* logits, int count, void* keys, unsigned int* counter, void* token, void* stream);

/* x[t] = table[tokens[t]] as fp32 (tokens int64, clamped to the vocabulary) and normed[t] = layer_norm(x[t]) * w + b. */
int qd_embed_norm(const void* tokens, const void* table, int vocab, float* x, const void* norm_w, const void* norm_b,
    void* normed, int count, int width, float eps, int dtype, void* stream);

/* out[r] = layer_norm(x[index[r]]) * w + b; index == NULL: row r. */
int qd_layer_norm_rows(const float* x, const int* index, const void* w, const void* b, void* out, int rows, int
    width, float eps, int dtype, void* stream);

/* The end of a sublayer: v = x_in + layer_norm(y * sigmoid(gate + gate_bias)) * post_w + post_b.  With older >= 0 the
 * result is stored as results[older] (results: layers of [tokens, width], result_stride elements apart) and
 * x_out = sum over j = 0 .. older of depth[j] * results[j]; otherwise x_out = v.  With next_w the norm in front of the
 * next sublayer, layer_norm(x_out) * next_w + next_b, goes to normed.  x_out may be x_in. */
int qd_sublayer_close(const void* y, const void* gate, long long ld_gate, const void* gate_bias, const void* post_w,
    const void* post_b, const float* x_in, float* x_out, float* results, long long result_stride, const void* depth,
    int older, const void* next_w, const void* next_b, void* normed, int tokens, int width, float eps, int dtype,
    void* stream);

/* v = table[tokens[r]] (tokens int64, clamped to the vocabulary) or, without table, x_in[index[r]] (index == NULL: row
 * r); + y[r] and + step (bf16 [width]) where given.  x_out[r] = v and normed[r] = v / rms(v) * (norm_offset + norm),
 * each where given.  x_out may be x_in without index. */
int qd_stream_norm(const void* tokens, const void* table, int vocab, const float* x_in, const int* index, const void* y,
    const void* step, float* x_out, const void* norm, float norm_offset, void* normed, int rows, int width, float eps, int
    dtype, void* stream);

/* fp32 operands of gated linear attention from a chunk's projections (rows ld apart): oq = q / sqrt(dim), ok = k,
 * ov = v, og = sigmoid(z + z_bias)^(1 / tau) - 1.  og may be z. */
int qd_gla_prepare(const void* q, const void* k, const void* v, long long ld, const float* z, const void* z_bias,
    float tau, float* oq, float* ok, float* og, float* ov, int tokens, int heads, int dim, int vdim, int dtype, void*
    stream);

/* fp32 operands of the channel-decay delta rule: q, k, v through a causal convolution of `taps` taps (history ring
 * [taps, channels q | k | v], position p in row p mod taps; updated with the chunk's last inputs) and SiLU, q and k as
 * not yet unit vectors: oscales [tokens, kv_heads, 3] = the factors that make k and
 * q unit vectors (q's also / sqrt(dim)) and k . q of the results, og = exp(-exp(a_log) softplus(z + z_bias)) - 1 (og may be z), obeta = sigmoid(beta).
 * The position of the chunk's first token is *position_ptr, or `position` if that is NULL. */
int qd_channel_delta_prepare(const void* q, const void* k, const void* v, const void* beta, long long ld, const
    float* z, const void* z_bias, const void* a_log, const void* q_taps, const void* k_taps, const void* v_taps,
    void* history, int taps, const int* position_ptr, int position, float* oq, float* ok, float* og, float* ov,
    float* obeta, float* oscales, int tokens, int heads, int kv_heads, int dim, int vdim, int dtype, void* stream);

/* The recurrence over a chunk; q, k [tokens, kv_heads, dim], g [tokens, heads, dim], v, out [tokens, heads, vdim], state
 * [heads, dim, vdim] fp32, updated in place.  delta = 0: S = diag(1 + g) S + k v^T; 1: S = diag(1 + g) S,
 * u = beta (v - S^T k), S += k u^T, with k and q times their scales; out = S^T q.  dim <= 256. */
int qd_linear_recurrence(const float* q, const float* k, const float* g, const float* v, const float* beta, const
    float* kq, float* state, float* out, int tokens, int heads, int kv_heads, int dim, int vdim, int delta, void*
    stream);

/* out[t, h] = x[t, h] / rms(x[t, h]) * w * act(gate[t, h]), act 0 = SiLU, 1 = sigmoid; w [vdim] shared by the heads. */
int qd_head_norm_gate(const float* x, const void* w, const void* gate, long long ld_gate, void* out, int tokens, int
    heads, int vdim, float eps, int act, int dtype, void* stream);

/* Everything between the projections and the output projection of one token (gated linear attention); low = the
 * rank-sized inner product of the decay, up [heads * dim, rank].  dim, vdim <= 256. */
int qd_gla_step(const void* q, const void* k, const void* v, const void* low, const void* up, const void* up_bias,
    int rank, float tau, const void* gate, const void* norm, float eps, float* state, void* out, int heads, int dim,
    int vdim, int dtype, void* stream);

/* The same for the channel-decay delta rule; the output gate is sigmoid(gate_up gate_low). */
int qd_channel_delta_step(const void* q, const void* k, const void* v, const void* beta, const void* low, const void*
    up, const void* up_bias, int rank, const void* a_log, const void* q_taps, const void* k_taps, const void* v_taps,
    void* history, int taps, const int* position_ptr, int position, const void* gate_low, const void* gate_up, int
    gate_rank, const void* norm, float eps, float* state, void* out, int heads, int kv_heads, int dim, int vdim, int
    dtype, void* stream);

/* Grouped-query attention over a bounded span of positions.  Query head h uses key/value head h / (heads / kv_heads); the
 * position of the first token is *position_ptr, or `position` if that is NULL; position p's rows are k_cache[p mod
 * capacity] and v_cache[p mod capacity], ld_k and ld_v elements apart, heads next to one another.
 * A field that a kind of norm, sink or gate does not use may be NULL. */
enum { QD_MASK_WINDOW = 0, QD_MASK_CHUNK = 1 };      /* sees the last `span` positions / those of its chunk of `span` positions */
enum { QD_NORM_NONE = 0, QD_NORM_ROW = 1, QD_NORM_HEAD = 2 };        /* RMS over the projection (weight per element) / per head */
enum { QD_SINK_NONE = 0, QD_SINK_LEARNED = 1, QD_SINK_ZERO = 2 };    /* exp(sink) / one in the softmax's denominator */
enum { QD_GATE_NONE = 0, QD_GATE_HEAD = 1, QD_GATE_VALUE = 2 };      /* sigmoid(gate) per head / per value column */

typedef struct qd_attention_args {
    const void* q; const void* k; const void* v; const void* gate;   /* projection rows, ld (gate: ld_gate) elements apart */
    const void* q_norm; const void* k_norm;
    const float* freq;                  /* [2][rot / 2]: high and low parts of the rotation's frequencies (interleaved pairs) */
    const void* sink;                   /* [heads] */
    const float* slopes;                /* [heads]: slope * distance is taken off the scaled scores; NULL: not */
    void* k_cache; void* v_cache;
    const void* k_shared;               /* key columns that all heads share, behind the head's own `dim`: rows as of the cache */
    const int* position_ptr;
    void* q_rows;                       /* [tokens, heads, dim + shared_dim]: normed, rotated queries; scratch if q is given */
    void* out;                          /* [tokens, heads, vdim] */
    float* partial; unsigned int* counters;      /* one token: qd_attention_step_floats, kv_heads words (zero before the first call) */
    long long ld, ld_gate, ld_k, ld_v, ld_shared;
    float scale, eps;
    int norm, rot, sink_kind, gate_kind, mask, span, capacity, position, tokens, heads, kv_heads, dim, vdim, shared_dim;
    int splits;                         /* one token: blocks per key/value head, at most 64 */
    int dtype;
} qd_attention_args;

/* A chunk.  With q: norm and rotation, rows into the ring, attention (shared_dim 0).  Without: q_rows holds the queries
 * and the ring the keys.  tokens + span - 1 <= capacity, unless the sequence has not filled the ring. */
int qd_attention(const qd_attention_args* args, void* stream);

/* Floats of `partial` (16-byte aligned). */
long long qd_attention_step_floats(int heads, int vdim, int splits);

/* One token in one launch (q given, shared_dim 0, capacity >= span); with q_rows in two where a group of heads exceeds
 * what one launch holds. */
int qd_attention_step(const qd_attention_args* args, void* stream);

/* Latent attention over the last `span` positions (libquickdraw_b200_latent.so).  The cache row of position p is
 * cache[p mod capacity], ld_cache elements: the normed latent (kv_rank), zeros up to rot_column, the rotated key columns
 * that all heads share (rot, pairs i, i + rot / 2), zeros. */
typedef struct qd_latent_args {
    const void* q;                      /* one token: [heads, dim + rot], not rotated */
    const void* dq; const void* dkv;    /* projection rows, ld elements apart: query latent (q_rank); latent and rotated columns (kv_rank + rot) */
    const void* gate;                   /* one token: [heads * vdim], sigmoid(gate) on the result; NULL: none */
    const void* dq_norm; const void* dkv_norm;
    const float* freq;                  /* [2][rot / 2] as for qd_attention */
    const void* uk; const void* uv;     /* [heads * dim, kv_rank], [heads * vdim, kv_rank] */
    void* cache;
    const int* position_ptr;
    void* q_latent;                     /* chunk: [tokens, q_rank], normed */
    float* absorbed; float* partial;    /* one token: scratch [heads, ld_cache] (8-byte aligned), qd_latent_step_floats (16-byte aligned) */
    void* out;                          /* one token: [heads, vdim] */
    long long ld, ld_cache;
    float scale, eps;
    int span, capacity, position, tokens, heads, dim, rot, vdim, q_rank, kv_rank, rot_column;
    int splits;                         /* one token: blocks per 16 heads, at most 64 */
    int dtype;
} qd_latent_args;

/* A chunk: q_latent and the cache rows.  The heads' keys and values are then products of the cached latents. */
int qd_latent_prepare(const qd_latent_args* args, void* stream);

/* The last `rot` of the `dim` columns of every head rotated in place, x [tokens, heads, dim]. */
int qd_rotate_half(void* x, const float* freq, const int* position_ptr, int position, int tokens, int heads, int dim, int
    rot, int dtype, void* stream);

/* Floats of `partial`. */
long long qd_latent_step_floats(int heads, int kv_rank, int splits);

/* One token from its query to the gated heads, on the latents themselves (span <= capacity); writes its cache row. */
int qd_latent_step(const qd_latent_args* args, void* stream);

#ifdef __cplusplus
}
#endif
#endif
