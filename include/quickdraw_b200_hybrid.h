/* quickdraw_b200 — C ABI of the kernels for models with bf16 weights and an fp32 residual stream
 * (libquickdraw_b200_hybrid.so): dense products, windowed attention with sinks, gated linear recurrences.
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

/* y[t, n] = sum_k x[t, k] w[n, k] with bf16 weights [rows, width] (contiguous) and fp32 accumulation; the first
 * gelu_cols outputs pass through the exact GELU.  x: [tokens, width], rows ldx elements apart; y: [tokens, rows], ldy
 * apart; dtypes bf16 -> bf16, bf16 -> fp32 or fp32 -> fp32.  Many bf16 token rows run on tcgen05 (TMA needs width, ldx,
 * ldy and rows to be multiples of eight), up to eight token rows stream the weights, anything else takes FMA tiles.
 * status: device word, bit 0 is set if a bounded wait ran out. */
int qd_linear(const void* x, long long ldx, int x_dtype, const void* w, void* y, long long ldy, int y_dtype, int
    tokens, int rows, int width, int gelu_cols, unsigned int* status, void* stream);

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

/* Sliding-window attention of a chunk: RMS norm over the whole query and key projections, interleaved rotation of the
 * first `rot` dimensions (freq: [2][rot / 2] fp32, high and low parts of the frequencies), rows into the ring
 * (k_cache [capacity, kv_heads, dim], v_cache [capacity, kv_heads, vdim], position p in row p mod capacity), softmax of
 * score * scale over the last `window` positions with exp(sink) added to the denominator, heads multiplied by
 * sigmoid(gate).  q, k, v, gate: projection rows ld elements apart.  tokens + window - 1 <= capacity, unless the
 * sequence has not filled the ring. */
int qd_window_attention(const void* q, const void* k, const void* v, const void* gate, long long ld, const void*
    q_norm, const void* k_norm, const float* freq, int rot, const void* sink, float scale, float eps, void* k_cache,
    void* v_cache, int capacity, int window, const int* position_ptr, int position, void* q_scratch, void* out, int
    tokens, int heads, int kv_heads, int dim, int vdim, int dtype, void* stream);

/* Floats of `partial` below (16-byte aligned). */
long long qd_window_attention_step_floats(int heads, int vdim, int splits);

/* The same for one token in one launch; counters: kv_heads words, zero before the first call.
 * splits (of the window, at most 64): blocks per key/value head. */
int qd_window_attention_step(const void* q, const void* k, const void* v, const void* gate, const void* q_norm, const
    void* k_norm, const float* freq, int rot, const void* sink, float scale, float eps, void* k_cache, void* v_cache,
    int capacity, int window, const int* position_ptr, int position, float* partial, unsigned int* counters, int
    splits, void* out, int heads, int kv_heads, int dim, int vdim, int dtype, void* stream);

#ifdef __cplusplus
}
#endif
#endif
