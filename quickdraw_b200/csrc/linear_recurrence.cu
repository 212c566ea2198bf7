// Gated linear recurrences with one decay per head and key channel, state S [dim, vdim] per head in fp32:
//   gated linear attention   S = diag(a) S + k v^T,                               o = S^T q
//   channel-decay delta rule S = diag(g) S, u = beta (v - S^T k), S = S + k u^T,  o = S^T q
// (gdn.cu has the delta rule with one decay per head.)  Everything that enters the recurrence is fp32.
//
// Prompt chunks: a prepare kernel (all tokens in parallel: short convolution, SiLU, decays) writes q, k,
// decay, v, beta as fp32 rows, unit_scales_kernel the factors that make q and k unit vectors; linear_recurrence_kernel walks the tokens with the state in
// registers.  A warp owns eight value columns; a lane a group of key rows and a few columns, held as row
// pairs for the packed fp32 FMA.  Both read-outs of the delta rule use the decayed state before the
// write, o = (gS)^T q + (k . q) u, so that the second one hides in the first one's shuffles.
// Latency-bound: one warp per scheduler, a dependent chain per token.
// Decode: recurrence_step_kernel does everything between the projections and the output projection in
// one launch: low-rank decay (and output gate), convolution, unit norms, recurrence, per-head RMS norm,
// gate.  A cluster of blocks shares a head (32 value columns each) and adds its sums of squares over
// distributed shared memory.  HBM-bound by the state.
#include <cooperative_groups.h>

#include "typed.cuh"

namespace cg = cooperative_groups;

namespace qd {
namespace {

constexpr float kUnitEps = 1e-6f;

QD_DEVINL float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// Decays are carried as decay - 1, S + S (decay - 1) in one FMA: a slow channel's decay is so close to one
// that its own rounding, the same at every token, would add up over a long sequence.
QD_DEVINL float gla_decay_less_one(float z, float inv_tau) { return expm1f(log_sigmoid(z) * inv_tau); }
QD_DEVINL float delta_decay_less_one(float z, float rate) { return expm1f(-rate * softplus_precise(z)); }      // rate = exp(A_log)

// Convolution input history: ring of `taps` rows, position p in row p mod taps.  A step reads the rows of
// the taps - 1 positions before it and writes its own, which is none of those.
struct ConvSource {
    const void* history;      // [taps, channels]
    int taps, channels;
};
// sum over taps of w[j] * input(position - (taps - 1 - j)) of one channel at chunk token t; x: the channel's
// input at the chunk's first token (row stride ld), older inputs from the history, zeros before position 0.
template <typename T>
QD_DEVINL float conv_at(const T* x, long long ld, int t, int position, const bf16* w, const ConvSource& src, int channel) {
    float acc = 0.f;
    for (int back = src.taps - 1; back >= 0; --back) {
        const int p = position - back;
        float v = 0.f;
        if (back <= t) v = load_f(x + (long long)(t - back) * ld);
        else if (p >= 0) v = load_f(reinterpret_cast<const T*>(src.history) + (size_t)(p % src.taps) * src.channels + channel);
        acc = fmaf(v, ld_bf16(w + src.taps - 1 - back), acc);
    }
    return acc;
}

// ----------------------------------------------------------------------------------- prepare
struct PrepareParams {
    const void* q; const void* k; const void* v; long long ld;      // this chunk's projections, rows ld apart
    const float* z; const bf16* z_bias;                             // decay logits [tokens, heads * dim], bias [heads * dim]
    const void* beta; const bf16* a_log;                            // delta rule: [tokens] rows ld apart; [heads]
    const bf16* q_taps; const bf16* k_taps; const bf16* v_taps; ConvSource conv;
    float tau;
    const int* position_ptr; int position;
    float* oq; float* ok; float* og; float* ov; float* obeta; float* oscales;
    int tokens, heads, kv_heads, dim, vdim;
};

template <typename T>
__global__ void __launch_bounds__(256) gla_prepare_kernel(const __grid_constant__ PrepareParams p) {
    chain_enter();
    const size_t t = blockIdx.x;
    const int keys = p.heads * p.dim, values = p.heads * p.vdim;
    const T* q = reinterpret_cast<const T*>(p.q) + t * p.ld;
    const T* k = reinterpret_cast<const T*>(p.k) + t * p.ld;
    const T* v = reinterpret_cast<const T*>(p.v) + t * p.ld;
    const float scale = 1.0f / sqrtf((float)p.dim), inv_tau = 1.0f / p.tau;
    for (int i = threadIdx.x; i < keys; i += blockDim.x) {
        p.oq[t * keys + i] = load_f(q + i) * scale;
        p.ok[t * keys + i] = load_f(k + i);
        p.og[t * keys + i] = gla_decay_less_one(p.z[t * keys + i] + ld_bf16(p.z_bias + i), inv_tau);
    }
    for (int i = threadIdx.x; i < values; i += blockDim.x) p.ov[t * values + i] = load_f(v + i);
}

constexpr int kPrepareTokens = 8;    // tokens of one channel per thread, all their inputs requested at once

// blockIdx.y: groups of 256 convolution channels (q | k | v), then groups of 256 decay channels (the
// first of these also the step sizes).  TAPS == 0: any number of taps.
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) delta_prepare_kernel(const __grid_constant__ PrepareParams p) {
    chain_enter();
    const int t0 = blockIdx.x * kPrepareTokens, count = min(kPrepareTokens, p.tokens - t0);
    const int base = p.position_ptr ? *p.position_ptr : p.position;
    const int keys = p.heads * p.dim, values = p.heads * p.vdim, kv_keys = p.kv_heads * p.dim, channels = 2 * kv_keys + values;
    const int conv_groups = (channels + 255) / 256;
    int group = blockIdx.y;
    if (group < conv_groups) {
        const int channel = group * 256 + threadIdx.x;
        if (channel >= channels) return;
        const int which = channel < kv_keys ? 0 : (channel < 2 * kv_keys ? 1 : 2), c = channel - which * kv_keys;
        const T* x = reinterpret_cast<const T*>(which == 0 ? p.q : (which == 1 ? p.k : p.v)) + c;
        const bf16* taps = (which == 0 ? p.q_taps : (which == 1 ? p.k_taps : p.v_taps)) + (size_t)c * p.conv.taps;
        float* out = which == 0 ? p.oq : (which == 1 ? p.ok : p.ov);
        const int width = which == 2 ? values : kv_keys;
        out += (size_t)t0 * width + c;
        if (TAPS == 0) {
            for (int i = 0; i < count; ++i)
                out[(size_t)i * width] = silu_precise(conv_at(x, p.ld, t0 + i, base + t0 + i, taps, p.conv, channel));
            return;
        }
        constexpr int kBack = TAPS ? TAPS - 1 : 0;
        float w[kBack + 1], in[kBack + kPrepareTokens];
#pragma unroll
        for (int j = 0; j <= kBack; ++j) w[j] = ld_bf16(taps + j);
#pragma unroll
        for (int j = 0; j < kBack + kPrepareTokens; ++j) {
            const int t = t0 + j - kBack, at = base + t;
            in[j] = 0.f;
            if (t >= 0) { if (t < p.tokens) in[j] = load_f(x + (long long)t * p.ld); }
            else if (at >= 0) in[j] = load_f(reinterpret_cast<const T*>(p.conv.history) + (size_t)(at % p.conv.taps) * channels + channel);
        }
#pragma unroll
        for (int i = 0; i < kPrepareTokens; ++i) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j <= kBack; ++j) acc = fmaf(in[i + j], w[j], acc);
            if (i < count) out[(size_t)i * width] = silu_precise(acc);
        }
        return;
    }
    group -= conv_groups;
    const int c = group * 256 + threadIdx.x;
    if (c < keys) {
        const float bias = ld_bf16(p.z_bias + c), rate = expf(ld_bf16(p.a_log + c / p.dim));
        float z[kPrepareTokens];
#pragma unroll
        for (int i = 0; i < kPrepareTokens; ++i) z[i] = i < count ? p.z[(size_t)(t0 + i) * keys + c] : 0.f;
#pragma unroll
        for (int i = 0; i < kPrepareTokens; ++i)
            if (i < count) p.og[(size_t)(t0 + i) * keys + c] = delta_decay_less_one(z[i] + bias, rate);
    }
    if (group == 0)
        for (int i = threadIdx.x; i < count * p.heads; i += 256) {
            const int t = t0 + i / p.heads, h = i % p.heads;
            p.obeta[(size_t)t * p.heads + h] = sigmoid_precise(load_f(reinterpret_cast<const T*>(p.beta) + (long long)t * p.ld + h));
        }
}

// Per token and key/value head: the factors that make k and q unit vectors (q's with 1 / sqrt(dim)) and
// k . q of the results.  A warp each.
__global__ void __launch_bounds__(256)
unit_scales_kernel(const float* __restrict__ q, const float* __restrict__ k, float* __restrict__ scales, long long rows, int dim) {
    chain_enter();
    const long long row = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (row >= rows) return;
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int d = lane; d < dim; d += 32) {
        const float a = q[row * dim + d], b = k[row * dim + d];
        qq = fmaf(a, a, qq); kk = fmaf(b, b, kk); kq = fmaf(a, b, kq);
    }
    qq = warp_sum(qq); kk = warp_sum(kk); kq = warp_sum(kq);
    if (lane == 0) {
        const float ks = 1.0f / sqrtf(kk + kUnitEps), qs = 1.0f / (sqrtf(qq + kUnitEps) * sqrtf((float)dim));
        scales[row * 3] = ks;
        scales[row * 3 + 1] = qs;
        scales[row * 3 + 2] = kq * ks * qs;
    }
}

template <typename T>
int launch_delta_prepare(const PrepareParams& p, cudaStream_t s) {
    const int groups = (2 * p.kv_heads * p.dim + p.heads * p.vdim + 255) / 256 + (p.heads * p.dim + 255) / 256;
    const dim3 grid((p.tokens + kPrepareTokens - 1) / kPrepareTokens, groups);
    int rc;
    switch (p.conv.taps) {
        case 2: rc = qd_launch(delta_prepare_kernel<T, 2>, grid, dim3(256), 0, s, 1, p); break;
        case 3: rc = qd_launch(delta_prepare_kernel<T, 3>, grid, dim3(256), 0, s, 1, p); break;
        case 4: rc = qd_launch(delta_prepare_kernel<T, 4>, grid, dim3(256), 0, s, 1, p); break;
        default: rc = qd_launch(delta_prepare_kernel<T, 0>, grid, dim3(256), 0, s, 1, p); break;
    }
    if (rc != QD_OK) return rc;
    const long long rows = (long long)p.tokens * p.kv_heads;
    return qd_launch(unit_scales_kernel, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, s, 1, p.oq, p.ok, p.oscales, rows, p.dim);
}

// The chunk's last `taps` inputs into the history ring.
template <typename T>
__global__ void __launch_bounds__(256)
conv_history_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, long long ld, T* __restrict__ history,
                    int taps, int kv_keys, int values, int tokens, const int* position_ptr, int position) {
    chain_enter();
    const int channels = 2 * kv_keys + values, back = blockIdx.y, t = tokens - 1 - back;
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (t < 0 || c >= channels) return;
    const int at = (position_ptr ? *position_ptr : position) + t;
    const T* src = c < kv_keys ? q + c : (c < 2 * kv_keys ? k + (c - kv_keys) : v + (c - 2 * kv_keys));
    history[(size_t)(at % taps) * channels + c] = src[(long long)t * ld];
}

// -------------------------------------------------------------------------------- recurrence
typedef unsigned long long u64;
QD_DEVINL u64 fma2(u64 a, u64 b, u64 c) { u64 d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
QD_DEVINL u64 pack2(float lo, float hi) { return (u64)__float_as_uint(lo) | ((u64)__float_as_uint(hi) << 32); }
QD_DEVINL float lo2(u64 v) { return __uint_as_float((uint32_t)v); }
QD_DEVINL float hi2(u64 v) { return __uint_as_float((uint32_t)(v >> 32)); }

QD_DEVINL void copy16(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
QD_DEVINL void copy4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
QD_DEVINL void copies_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> QD_DEVINL void copies_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

constexpr int kRecCols = 32, kRecTile = 16;      // value columns of a block; tokens per staged tile

struct RecurrenceParams {
    const float* q; const float* k; const float* g; const float* v; const float* beta;
    const float* scales;          // delta rule: per token and key/value head the factors that make k and q unit vectors (q's / sqrt(dim)), k . q of the unit vectors
    float* state; float* out;
    int tokens, heads, kv_heads, dim, vdim, vectors;
};

// floats of one staged token: q, k, decay - 1 (padded to `row`), v columns, step size and the three scales
constexpr int rec_token_floats(int row) { return 3 * row + kRecCols + 4; }

// A token's vectors, this lane's rows, and values, this lane's columns.
template <int J, int CC> struct RecVectors { ulonglong2 q[J], k[J], g[J]; float v[CC]; };

// Sums of NV values over the KL lanes of a key group, NV <= KL: a round exchanges half of what is left, lane
// kl ends up with the sum of value kl / (KL / NV).
template <int KL, int NV>
QD_DEVINL float scatter_sum(float (&v)[NV], int kl) {
    int lanes = KL / 2;
#pragma unroll
    for (int n = NV / 2; n >= 1; n >>= 1, lanes >>= 1) {
        const bool upper = kl & lanes;
#pragma unroll
        for (int i = 0; i < n; ++i)
            v[i] = (upper ? v[i + n] : v[i]) + __shfl_xor_sync(0xffffffffu, upper ? v[i] : v[i + n], lanes);
    }
#pragma unroll
    for (; lanes >= 1; lanes >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], lanes);
    return v[0];
}
// The inverse: v[0] of lane kl is value kl / (KL / NV); every lane gets all values.
template <int KL, int NV>
QD_DEVINL void gather_values(float (&v)[NV], int kl) {
#pragma unroll
    for (int n = 1; n < NV; n <<= 1) {
        const int lanes = KL / NV * n;
        const bool upper = kl & lanes;
#pragma unroll
        for (int i = 0; i < n; ++i) {
            const float other = __shfl_xor_sync(0xffffffffu, v[i], lanes), own = v[i];
            v[i] = upper ? other : own;
            v[i + n] = upper ? own : other;
        }
    }
}
template <int N> QD_DEVINL void load_columns(const float* p, float (&v)[N]) {
    if (N % 4 == 0) {
#pragma unroll
        for (int i = 0; i < N / 4; ++i) {
            const float4 x = *reinterpret_cast<const float4*>(p + 4 * i);
            v[4 * i] = x.x; v[(4 * i + 1) % N] = x.y; v[(4 * i + 2) % N] = x.z; v[(4 * i + 3) % N] = x.w;
        }
    } else if (N == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        v[0] = x.x; v[1 % N] = x.y;
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = p[i];
    }
}

// KL lanes share a column's keys (rows 4 KL j + 4 kl + {0..3}), a lane holds CC columns; a warp (32 / KL) CC,
// a block kRecCols.  GATHER: the delta rule's predictions are summed by scatter and gather (fewer shuffles,
// more rounds) instead of a butterfly per column.
template <int KL, int CC> constexpr int rec_threads() { return kRecCols / (32 / KL * CC) * 32; }

template <int KL, int CC, int J, bool DELTA, bool GATHER>
__global__ void __launch_bounds__(rec_threads<KL, CC>()) linear_recurrence_kernel(const __grid_constant__ RecurrenceParams p) {
    chain_enter();
    extern __shared__ __align__(16) float tiles[];
    constexpr int kRow = 4 * KL * J, kToken = rec_token_floats(kRow), kThreads = rec_threads<KL, CC>();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, kl = lane % KL, cl = lane / KL;
    const int head = blockIdx.x, kv = head / (p.heads / p.kv_heads), c0 = blockIdx.y * kRecCols;
    const int local = (warp * (32 / KL) + cl) * CC, col = c0 + local;
    const int dim = p.dim, vdim = p.vdim;
    float* state = p.state + (size_t)head * dim * vdim;

    for (int i = tid; i < 2 * kRecTile * kToken; i += kThreads) tiles[i] = 0.f;      // padding rows stay zero
    u64 s[J][2][CC];
#pragma unroll
    for (int j = 0; j < J; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int c = 0; c < CC; ++c) {
                const int r = j * 4 * KL + kl * 4 + h * 2;
                const bool ok = col + c < vdim;
                s[j][h][c] = pack2(ok && r < dim ? state[(size_t)r * vdim + col + c] : 0.f,
                                   ok && r + 1 < dim ? state[(size_t)(r + 1) * vdim + col + c] : 0.f);
            }
    __syncthreads();

    // a thread copies the same piece of every token of a tile
    const int cols = min(kRecCols, vdim - c0), unit = p.vectors ? 4 : 1;
    const int kp = dim / unit, per = 3 * kp + cols / unit;
    auto stage = [&](int tile) {
        const int t0 = tile * kRecTile, count = min(kRecTile, p.tokens - t0);
        float* base = tiles + (tile & 1) * kRecTile * kToken;
        for (int piece = tid; piece < per; piece += kThreads) {
            const int which = piece / kp, e = (which < 3 ? piece - which * kp : piece - 3 * kp) * unit;
            const float* src;
            float* dst = base + (which < 3 ? which : 3) * kRow + e;
            size_t stride;
            if (which < 2) { stride = (size_t)p.kv_heads * dim; src = (which ? p.k : p.q) + t0 * stride + (size_t)kv * dim + e; }
            else if (which == 2) { stride = (size_t)p.heads * dim; src = p.g + t0 * stride + (size_t)head * dim + e; }
            else { stride = (size_t)p.heads * vdim; src = p.v + t0 * stride + (size_t)head * vdim + c0 + e; }
            if (p.vectors) {
#pragma unroll 4
                for (int tt = 0; tt < count; ++tt, src += stride, dst += kToken) copy16(dst, src);
            } else {
                for (int tt = 0; tt < count; ++tt, src += stride, dst += kToken) copy4(dst, src);
            }
        }
        if (DELTA && tid < count) {
            float* dst = base + tid * kToken + 3 * kRow + kRecCols;
            copy4(dst, p.beta + (size_t)(t0 + tid) * p.heads + head);
            for (int i = 0; i < 3; ++i) copy4(dst + 1 + i, p.scales + ((size_t)(t0 + tid) * p.kv_heads + kv) * 3 + i);
        }
        copies_commit();
    };
    auto fetch = [&](const float* token, RecVectors<J, CC>& f) {
#pragma unroll
        for (int j = 0; j < J; ++j) {
            f.g[j] = *reinterpret_cast<const ulonglong2*>(token + 2 * kRow + j * 4 * KL + kl * 4);
            f.k[j] = *reinterpret_cast<const ulonglong2*>(token + kRow + j * 4 * KL + kl * 4);
            f.q[j] = *reinterpret_cast<const ulonglong2*>(token + j * 4 * KL + kl * 4);
        }
        load_columns<CC>(token + 3 * kRow + local, f.v);
    };
    float* out = p.out + (size_t)head * vdim;
    const size_t out_stride = (size_t)p.heads * vdim;
    // one token; o: the read-outs of this lane's rows
    auto advance = [&](const RecVectors<J, CC>& f, const float* token, float* o) {
        u64 oa[CC], ob[CC];
#pragma unroll
        for (int c = 0; c < CC; ++c) oa[c] = ob[c] = 0ull;
        if (DELTA) {
            const float4 w = *reinterpret_cast<const float4*>(token + 3 * kRow + kRecCols);      // step size, scale of k, of q, k . q
            u64 pa[CC], pb[CC];
            float pred[CC];
#pragma unroll
            for (int c = 0; c < CC; ++c) pa[c] = pb[c] = 0ull;
#pragma unroll
            for (int j = 0; j < J; ++j)
#pragma unroll
                for (int c = 0; c < CC; ++c) {
                    s[j][0][c] = fma2(s[j][0][c], f.g[j].x, s[j][0][c]);
                    s[j][1][c] = fma2(s[j][1][c], f.g[j].y, s[j][1][c]);
                    pa[c] = fma2(s[j][0][c], f.k[j].x, pa[c]);
                    pb[c] = fma2(s[j][1][c], f.k[j].y, pb[c]);
                }
#pragma unroll
            for (int c = 0; c < CC; ++c) pred[c] = (lo2(pa[c]) + hi2(pa[c])) + (lo2(pb[c]) + hi2(pb[c]));
            if (GATHER) {
                scatter_sum<KL, CC>(pred, kl);
                gather_values<KL, CC>(pred, kl);
            } else {
#pragma unroll
                for (int x = 1; x < KL; x <<= 1)
#pragma unroll
                    for (int c = 0; c < CC; ++c) pred[c] += __shfl_xor_sync(0xffffffffu, pred[c], x);
            }
#pragma unroll
            for (int j = 0; j < J; ++j)               // fills the shuffles' latency
#pragma unroll
                for (int c = 0; c < CC; ++c) {
                    oa[c] = fma2(s[j][0][c], f.q[j].x, oa[c]);
                    ob[c] = fma2(s[j][1][c], f.q[j].y, ob[c]);
                }
#pragma unroll
            for (int c = 0; c < CC; ++c) {
                const float u = w.x * fmaf(-w.y, pred[c], f.v[c]), ku = w.y * u;
                const u64 uu = pack2(ku, ku);
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    s[j][0][c] = fma2(f.k[j].x, uu, s[j][0][c]);
                    s[j][1][c] = fma2(f.k[j].y, uu, s[j][1][c]);
                }
                o[c] = fmaf(w.z, (lo2(oa[c]) + hi2(oa[c])) + (lo2(ob[c]) + hi2(ob[c])), kl == 0 ? u * w.w : 0.f);
            }
        } else {
#pragma unroll
            for (int c = 0; c < CC; ++c) {
                const u64 vv = pack2(f.v[c], f.v[c]);
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    s[j][0][c] = fma2(f.k[j].x, vv, fma2(s[j][0][c], f.g[j].x, s[j][0][c]));
                    s[j][1][c] = fma2(f.k[j].y, vv, fma2(s[j][1][c], f.g[j].y, s[j][1][c]));
                    oa[c] = fma2(s[j][0][c], f.q[j].x, oa[c]);
                    ob[c] = fma2(s[j][1][c], f.q[j].y, ob[c]);
                }
                o[c] = (lo2(oa[c]) + hi2(oa[c])) + (lo2(ob[c]) + hi2(ob[c]));
            }
        }
    };

    const int ntiles = (p.tokens + kRecTile - 1) / kRecTile;
    stage(0);
    for (int tile = 0; tile < ntiles; ++tile) {
        if (tile + 1 < ntiles) { stage(tile + 1); copies_wait<1>(); } else { copies_wait<0>(); }
        __syncthreads();
        const float* token = tiles + (tile & 1) * kRecTile * kToken;
        const int count = min(kRecTile, p.tokens - tile * kRecTile);
        RecVectors<J, CC> even, odd;                     // the next token's vectors are read while this one is reduced
        fetch(token, even);
        for (int tt = 0; tt < count; tt += 4, token += 4 * kToken) {
            float o[4 * CC];
#pragma unroll
            for (int i = 0; i < 4 * CC; ++i) o[i] = 0.f;
            if (tt + 1 < count) fetch(token + kToken, odd);
            advance(even, token, o);
            if (tt + 2 < count) fetch(token + 2 * kToken, even);
            if (tt + 1 < count) advance(odd, token + kToken, o + CC);
            if (tt + 3 < count) fetch(token + 3 * kToken, odd);
            if (tt + 2 < count) advance(even, token + 2 * kToken, o + 2 * CC);
            if (tt + 4 < count) fetch(token + 4 * kToken, even);
            if (tt + 3 < count) advance(odd, token + 3 * kToken, o + 3 * CC);
            const float mine = scatter_sum<KL, 4 * CC>(o, kl);
            const int value = kl / (KL / (4 * CC)), t = value / CC, c = value % CC;
            if (kl % (KL / (4 * CC)) == 0 && tt + t < count && col + c < vdim) out[t * out_stride + col + c] = mine;
            out += 4 * out_stride;
        }
        __syncthreads();                 // the buffer may be refilled
    }
#pragma unroll
    for (int j = 0; j < J; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int c = 0; c < CC; ++c) {
                const int r = j * 4 * KL + kl * 4 + h * 2;
                if (col + c < vdim) {
                    if (r < dim) state[(size_t)r * vdim + col + c] = lo2(s[j][h][c]);
                    if (r + 1 < dim) state[(size_t)(r + 1) * vdim + col + c] = hi2(s[j][h][c]);
                }
            }
}

// Launched ordinarily: started as a dependent while the kernel before it still fills the SMs, the blocks
// gather on the few SMs that free up first (1.1 ms instead of 0.58 and 0.45 ms at 2048 tokens).
template <int KL, int CC, int J, bool DELTA, bool GATHER>
int launch_recurrence(const RecurrenceParams& p, cudaStream_t stream) {
    const size_t smem = 2ull * kRecTile * rec_token_floats(4 * KL * J) * 4;
    if (!allow_smem(linear_recurrence_kernel<KL, CC, J, DELTA, GATHER>, smem)) return QD_ERR_LAUNCH;
    return qd_launch(linear_recurrence_kernel<KL, CC, J, DELTA, GATHER>, dim3(p.heads, (p.vdim + kRecCols - 1) / kRecCols),
                     dim3(rec_threads<KL, CC>()), smem, stream, 0, p);
}
// Layouts by measurement (2048 tokens, 32 heads of 128): the delta rule 584 us with sixteen lanes and four
// columns (630 with 8 x 2, 642 with 16 x 2, 679 with 32 x 4), gated linear attention 393 us with 32 x 8.
int delta_recurrence(const RecurrenceParams& p, cudaStream_t stream) {
    if (p.dim <= 64) return launch_recurrence<16, 4, 1, true, false>(p, stream);
    if (p.dim <= 128) return launch_recurrence<16, 4, 2, true, false>(p, stream);
    if (p.dim <= 192) return launch_recurrence<16, 4, 3, true, false>(p, stream);
    if (p.dim <= 256) return launch_recurrence<16, 4, 4, true, false>(p, stream);
    return QD_ERR_UNSUPPORTED;
}
int gla_recurrence(const RecurrenceParams& p, cudaStream_t stream) {
    if (p.dim <= 64) return launch_recurrence<16, 4, 1, false, false>(p, stream);
    if (p.dim <= 128) return launch_recurrence<32, 8, 1, false, false>(p, stream);
    if (p.dim <= 256) return launch_recurrence<32, 8, 2, false, false>(p, stream);
    return QD_ERR_UNSUPPORTED;
}

// ------------------------------------------------------------------------ per-head norm, gate
// out[t, h, :] = x / rms(x) * w * act(gate); act: 0 = SiLU, 1 = sigmoid.  A warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const float* __restrict__ x, const bf16* __restrict__ w, const T* __restrict__ gate, long long ld_gate,
                      T* __restrict__ out, int tokens, int heads, int vdim, float eps, int act) {
    chain_enter();
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (item >= (long long)tokens * heads) return;
    const long long t = item / heads;
    const int h = (int)(item % heads);
    const float* row = x + item * vdim;
    float sq = 0.f;
    for (int i = lane; i < vdim; i += 32) sq = fmaf(row[i], row[i], sq);
    const float r = 1.0f / sqrtf(warp_sum(sq) / (float)vdim + eps);
    const T* g = gate + t * ld_gate + (long long)h * vdim;
    for (int i = lane; i < vdim; i += 32) {
        const float gv = load_f(g + i);
        store_f(out + item * vdim + i, row[i] * r * ld_bf16(w + i) * (act ? sigmoid_precise(gv) : silu_precise(gv)));
    }
}

// ------------------------------------------------------------------------------- decode step
struct StepParams {
    const void* q; const void* k; const void* v;            // projections of the token
    const void* low; const bf16* up; const bf16* up_bias; int rank;      // decay logits: up [heads * dim, rank] low + bias
    const void* beta; const bf16* a_log;
    const bf16* q_taps; const bf16* k_taps; const bf16* v_taps; int taps; void* history;
    float tau;
    const void* gate_low; const bf16* gate_up; int gate_rank;            // gate_up == NULL: gate_low is the gate itself
    const bf16* norm; float eps;
    const int* position_ptr; int position;
    float* state; void* out;
    int heads, kv_heads, dim, vdim;
};

constexpr int kStepThreads = 256, kStepGroups = 8;

// dot(up[row, :rank], low) by the eight lanes of a group; every lane gets the sum
QD_DEVINL float low_rank_dot(const bf16* up, const float* low, int rank, int sub) {
    float acc = 0.f;
    if (rank % 8 == 0) {
        for (int r = sub * 8; r < rank; r += 64) {
            float w[8];
            unpack8(__ldg(reinterpret_cast<const uint4*>(up + r)), w);
#pragma unroll
            for (int i = 0; i < 8; ++i) acc = fmaf(w[i], low[r + i], acc);
        }
    } else {
        for (int r = sub; r < rank; r += 8) acc = fmaf(ld_bf16(up + r), low[r], acc);
    }
    return group_sum<8>(acc);
}

// ask for `bytes` from p on (one 128-byte line per thread and round) to be in L2 soon
QD_DEVINL void prefetch_span(const void* p, size_t bytes) {
    for (size_t at = (size_t)threadIdx.x * 128; at < bytes; at += (size_t)blockDim.x * 128)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(p) + at));
}

// One channel's convolution for a single token: up to four taps have all their inputs and weights requested at
// once, before the position (which selects the ring rows) has arrived; more taps are walked.
constexpr int kStepTaps = 4;
template <typename T> struct StepConv {
    float x, ring[kStepTaps], w[kStepTaps];
    QD_DEVINL void request(const T* fresh, const bf16* taps, const ConvSource& src, int channel) {
        x = load_f(fresh);
#pragma unroll
        for (int r = 0; r < kStepTaps; ++r) {
            ring[r] = w[r] = 0.f;
            if (src.taps <= kStepTaps && r < src.taps) {
                ring[r] = load_f(reinterpret_cast<const T*>(src.history) + (size_t)r * src.channels + channel);
                w[r] = ld_bf16(taps + src.taps - 1 - r);          // w[back]
            }
        }
    }
    QD_DEVINL float finish(const T* fresh, int position, const bf16* taps, const ConvSource& src, int channel) {
        if (src.taps > kStepTaps) return conv_at(fresh, 0, 0, position, taps, src, channel);
        float acc = 0.f;
#pragma unroll
        for (int back = kStepTaps - 1; back >= 1; --back) {
            if (back < src.taps && position >= back) {
                const int row = (position - back) % src.taps;
                float v = ring[0];
#pragma unroll
                for (int r = 1; r < kStepTaps; ++r) v = row == r ? ring[r] : v;
                acc = fmaf(v, w[back], acc);
            }
        }
        return fmaf(x, w[0], acc);
    }
};

template <typename T, bool DELTA, int KPT>
__global__ void __launch_bounds__(kStepThreads) recurrence_step_kernel(const __grid_constant__ StepParams p) {
    const int head = blockIdx.y, c0 = blockIdx.x * 32, tid = threadIdx.x, col = tid & 31, kg = tid >> 5;
    const int dim = p.dim, vdim = p.vdim, kv = head / (p.heads / p.kv_heads), kv_keys = p.kv_heads * dim;
    grid_launch_dependents();
    // the state tile (one line per key row) and the head's constant matrices are on their way while the kernel before this one ends
    if (tid < dim) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.state + ((size_t)head * dim + tid) * vdim + c0));
    prefetch_span(p.up + (size_t)head * dim * p.rank, (size_t)dim * p.rank * sizeof(bf16));
    if (p.gate_up) prefetch_span(p.gate_up + ((size_t)head * vdim + c0) * p.gate_rank, (size_t)min(32, vdim - c0) * p.gate_rank * sizeof(bf16));
    grid_dependency_wait();
    extern __shared__ float low[];                 // rank + gate_rank
    __shared__ float sq[256], sk[256], sg[256], sv[32], sgate[32], part[kStepGroups][33], norms[2][kStepGroups], squares[8];
    cg::cluster_group cluster = cg::this_cluster();
    cluster.barrier_arrive();                      // waited for before the first access to another block's memory
    const bool col_ok = c0 + col < vdim;
    float* tile = p.state + (size_t)head * dim * vdim + c0 + col;
    const T* lowv = reinterpret_cast<const T*>(p.low);
    const T* gatev = reinterpret_cast<const T*>(p.gate_low);
    for (int i = tid; i < p.rank; i += kStepThreads) low[i] = load_f(lowv + i);
    if (p.gate_up) for (int i = tid; i < p.gate_rank; i += kStepThreads) low[p.rank + i] = load_f(gatev + i);
    const T* q = reinterpret_cast<const T*>(p.q) + kv * dim;
    const T* k = reinterpret_cast<const T*>(p.k) + kv * dim;
    const T* v = reinterpret_cast<const T*>(p.v) + head * vdim + c0;
    const float scale = 1.0f / sqrtf((float)dim);
    float qv = 0.f, kvv = 0.f, beta = 0.f, rate = 0.f;
    if (DELTA) {
        const ConvSource src = {p.history, p.taps, 2 * kv_keys + p.heads * vdim};
        const int kc = kv * dim + tid, vch = head * vdim + c0 + col;
        const bf16* qt = p.q_taps + (size_t)kc * p.taps;
        const bf16* kt = p.k_taps + (size_t)kc * p.taps;
        const bf16* vt = p.v_taps + (size_t)vch * p.taps;
        const bool keyed = tid < dim, valued = kg == kStepGroups - 1 && col_ok;
        StepConv<T> cq, ck, cv;
        const int position = p.position_ptr ? *p.position_ptr : p.position;
        if (keyed) { cq.request(q + tid, qt, src, kc); ck.request(k + tid, kt, src, kv_keys + kc); }
        if (valued) cv.request(v + col, vt, src, 2 * kv_keys + vch);
        beta = sigmoid_precise(load_f(reinterpret_cast<const T*>(p.beta) + head));
        rate = expf(ld_bf16(p.a_log + head));
        T* fresh = reinterpret_cast<T*>(p.history) + (size_t)(position % p.taps) * src.channels;
        if (keyed) {
            qv = silu_precise(cq.finish(q + tid, position, qt, src, kc));
            kvv = silu_precise(ck.finish(k + tid, position, kt, src, kv_keys + kc));
        }
        if (valued) sv[col] = silu_precise(cv.finish(v + col, position, vt, src, 2 * kv_keys + vch));
        // the token's row of the ring: requested above by other blocks too, used by none of them
        if (keyed && blockIdx.x == 0 && head % (p.heads / p.kv_heads) == 0) { fresh[kc] = q[tid]; fresh[kv_keys + kc] = k[tid]; }
        if (valued) fresh[2 * kv_keys + vch] = v[col];
        const float qq = warp_sum(qv * qv), kk = warp_sum(kvv * kvv);
        if (col == 0) { norms[0][kg] = qq; norms[1][kg] = kk; }
    } else {
        if (tid < dim) { qv = load_f(q + tid) * scale; kvv = load_f(k + tid); }
        if (kg == kStepGroups - 1 && col_ok) sv[col] = load_f(v + col);
    }
    sq[tid] = qv; sk[tid] = kvv;                   // not yet unit vectors in the delta rule: their factors join the sums below
    float s[KPT];
#pragma unroll
    for (int j = 0; j < KPT; ++j) {
        const int r = j * kStepGroups + kg;
        s[j] = (r < dim && col_ok) ? tile[(size_t)r * vdim] : 0.f;
    }
    __syncthreads();
    // decay of the head's key channels, output gate of the block's columns: eight lanes per row
    const int sub = tid & 7, group = tid >> 3;
    for (int d = group; d < ((dim + 31) & ~31); d += 32) {
        const int row = head * dim + min(d, dim - 1);
        const float z = low_rank_dot(p.up + (size_t)row * p.rank, low, p.rank, sub) + ld_bf16(p.up_bias + row);
        if (sub == 0 && d < dim) sg[d] = DELTA ? delta_decay_less_one(z, rate) : gla_decay_less_one(z, 1.0f / p.tau);
    }
    {
        const int c = head * vdim + min(c0 + group, vdim - 1);
        const float gv = p.gate_up ? low_rank_dot(p.gate_up + (size_t)c * p.gate_rank, low + p.rank, p.gate_rank, sub) : load_f(gatev + c);
        if (sub == 0) sgate[group] = DELTA ? sigmoid_precise(gv) : silu_precise(gv);
    }
    float qs = 1.f, ks = 1.f;
    if (DELTA) {
        float qq = 0.f, kk = 0.f;
#pragma unroll
        for (int w = 0; w < kStepGroups; ++w) { qq += norms[0][w]; kk += norms[1][w]; }
        qs = scale / sqrtf(qq + kUnitEps);
        ks = 1.0f / sqrtf(kk + kUnitEps);
    }
    __syncthreads();

    float pred = 0.f;
#pragma unroll
    for (int j = 0; j < KPT; ++j) {
        const int r = j * kStepGroups + kg;
        if (r < dim) {
            s[j] = fmaf(s[j], sg[r], s[j]);
            if (DELTA) pred = fmaf(s[j], sk[r] * ks, pred);
        }
    }
    float u = col_ok ? sv[col] : 0.f;
    if (DELTA) {
        part[kg][col] = pred;
        __syncthreads();
        float total = 0.f;
#pragma unroll
        for (int w = 0; w < kStepGroups; ++w) total += part[w][col];
        u = beta * (u - total);
        __syncthreads();
    }
    float o = 0.f;
#pragma unroll
    for (int j = 0; j < KPT; ++j) {
        const int r = j * kStepGroups + kg;
        if (r < dim) {
            s[j] = fmaf(sk[r] * ks, u, s[j]);
            o = fmaf(s[j], sq[r] * qs, o);
            if (col_ok) tile[(size_t)r * vdim] = s[j];
        }
    }
    part[kg][col] = o;
    __syncthreads();
    cluster.barrier_wait();
    float value = 0.f;
    if (kg == 0) {
#pragma unroll
        for (int w = 0; w < kStepGroups; ++w) value += part[w][col];
        if (!col_ok) value = 0.f;
        const float mine = warp_sum(value * value);
        // this block's sum of squares into slot `rank` of every block of the head
        if (col < (int)cluster.num_blocks()) *cluster.map_shared_rank(&squares[cluster.block_rank()], col) = mine;
    }
    cluster.sync();
    if (kg == 0 && col_ok) {
        float total = 0.f;
        for (unsigned int b = 0; b < cluster.num_blocks(); ++b) total += squares[b];
        const float r = 1.0f / sqrtf(total / (float)vdim + p.eps);
        store_f(reinterpret_cast<T*>(p.out) + head * vdim + c0 + col, value * r * ld_bf16(p.norm + c0 + col) * sgate[col]);
    }
}

template <typename T, bool DELTA, int KPT>
int launch_step(const StepParams& p, cudaStream_t stream) {
    const int slices = (p.vdim + 31) / 32;
    if (slices > 8) return QD_ERR_UNSUPPORTED;
    const size_t smem = (size_t)(p.rank + p.gate_rank) * 4 + 16;
    if (!allow_smem(recurrence_step_kernel<T, DELTA, KPT>, smem)) return QD_ERR_UNSUPPORTED;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(slices, p.heads); cfg.blockDim = dim3(kStepThreads); cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = slices; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr; cfg.numAttrs = qd_chain_switch() ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, recurrence_step_kernel<T, DELTA, KPT>, p) == cudaSuccess ? QD_OK : QD_ERR_LAUNCH;
}
template <typename T, bool DELTA>
int step(const StepParams& p, cudaStream_t stream) {
    if (p.dim <= 32) return launch_step<T, DELTA, 4>(p, stream);
    if (p.dim <= 64) return launch_step<T, DELTA, 8>(p, stream);
    if (p.dim <= 128) return launch_step<T, DELTA, 16>(p, stream);
    if (p.dim <= 256) return launch_step<T, DELTA, 32>(p, stream);
    return QD_ERR_UNSUPPORTED;
}

template <typename T, bool DELTA>
int prepare(const PrepareParams& p, int tokens, cudaStream_t s) {
    if (DELTA) return launch_delta_prepare<T>(p, s);
    return qd_launch(gla_prepare_kernel<T>, dim3(tokens), dim3(256), 0, s, 1, p);
}
template <typename T>
int history(const void* q, const void* k, const void* v, long long ld, void* ring, int taps, int kv_keys, int values, int tokens,
            const int* position_ptr, int position, cudaStream_t s) {
    const int rows = tokens < taps ? tokens : taps;
    return qd_launch(conv_history_kernel<T>, dim3((2 * kv_keys + values + 255) / 256, rows), dim3(256), 0, s, 1, (const T*)q, (const T*)k,
                     (const T*)v, ld, (T*)ring, taps, kv_keys, values, tokens, position_ptr, position);
}
template <typename T>
int norm_gate(const float* x, const void* w, const void* gate, long long ld, void* out, int tokens, int heads, int vdim, float eps,
              int act, cudaStream_t s) {
    return qd_launch(head_norm_gate_kernel<T>, dim3((unsigned)(((long long)tokens * heads + 7) / 8)), dim3(256), 0, s, 1, x, (const bf16*)w,
                     (const T*)gate, ld, (T*)out, tokens, heads, vdim, eps, act);
}

}  // namespace
}  // namespace qd

extern "C" int qd_gla_prepare(const void* q, const void* k, const void* v, long long ld, const float* z, const void* z_bias,
                              float tau, float* oq, float* ok, float* og, float* ov, int tokens, int heads, int dim, int vdim,
                              int dtype, void* stream) {
    QD_CHECK_ARG(q && k && v && z && z_bias && oq && ok && og && ov && tokens > 0 && heads > 0 && dim > 0 && vdim > 0 && tau > 0.f);
    qd::PrepareParams p = {};
    p.q = q; p.k = k; p.v = v; p.ld = ld; p.z = z; p.z_bias = (const bf16*)z_bias; p.tau = tau;
    p.oq = oq; p.ok = ok; p.og = og; p.ov = ov; p.tokens = tokens; p.heads = heads; p.kv_heads = heads; p.dim = dim; p.vdim = vdim;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == QD_BF16) return qd::prepare<bf16, false>(p, tokens, s);
    if (dtype == QD_F32) return qd::prepare<float, false>(p, tokens, s);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_channel_delta_prepare(const void* q, const void* k, const void* v, const void* beta, long long ld, const float* z,
                                        const void* z_bias, const void* a_log, const void* q_taps, const void* k_taps,
                                        const void* v_taps, void* history, int taps, const int* position_ptr, int position,
                                        float* oq, float* ok, float* og, float* ov, float* obeta, float* oscales, int tokens, int heads,
                                        int kv_heads, int dim, int vdim, int dtype, void* stream) {
    QD_CHECK_ARG(q && k && v && beta && z && z_bias && a_log && q_taps && k_taps && v_taps && history && oq && ok && og && ov && obeta && oscales);
    QD_CHECK_ARG(tokens > 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0 && taps > 0 && position >= 0);
    const int kv_keys = kv_heads * dim, values = heads * vdim;
    qd::PrepareParams p = {q, k, v, ld, z, (const bf16*)z_bias, beta, (const bf16*)a_log, (const bf16*)q_taps, (const bf16*)k_taps,
                           (const bf16*)v_taps, {history, taps, 2 * kv_keys + values}, 1.f, position_ptr, position, oq, ok, og, ov,
                           obeta, oscales, tokens, heads, kv_heads, dim, vdim};
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype != QD_BF16 && dtype != QD_F32) return QD_ERR_UNSUPPORTED;
    const int rc = dtype == QD_BF16 ? qd::prepare<bf16, true>(p, tokens, s) : qd::prepare<float, true>(p, tokens, s);
    if (rc != QD_OK) return rc;
    return dtype == QD_BF16 ? qd::history<bf16>(q, k, v, ld, history, taps, kv_keys, values, tokens, position_ptr, position, s)
                            : qd::history<float>(q, k, v, ld, history, taps, kv_keys, values, tokens, position_ptr, position, s);
}

extern "C" int qd_linear_recurrence(const float* q, const float* k, const float* g, const float* v, const float* beta,
                                    const float* scales, float* state, float* out, int tokens, int heads, int kv_heads, int dim, int vdim, int delta,
                                    void* stream) {
    QD_CHECK_ARG(q && k && g && v && state && out && tokens > 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0);
    QD_CHECK_ARG(!delta || (beta && scales));
    const int vectors = dim % 4 == 0 && vdim % 4 == 0 && qd::aligned16(q) && qd::aligned16(k) && qd::aligned16(g) && qd::aligned16(v);
    const qd::RecurrenceParams p = {q, k, g, v, beta, scales, state, out, tokens, heads, kv_heads, dim, vdim, vectors};
    return delta ? qd::delta_recurrence(p, (cudaStream_t)stream) : qd::gla_recurrence(p, (cudaStream_t)stream);
}

extern "C" int qd_head_norm_gate(const float* x, const void* w, const void* gate, long long ld_gate, void* out, int tokens, int heads,
                                 int vdim, float eps, int act, int dtype, void* stream) {
    QD_CHECK_ARG(x && w && gate && out && tokens > 0 && heads > 0 && vdim > 0 && (act == 0 || act == 1));
    if (dtype == QD_BF16) return qd::norm_gate<bf16>(x, w, gate, ld_gate, out, tokens, heads, vdim, eps, act, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::norm_gate<float>(x, w, gate, ld_gate, out, tokens, heads, vdim, eps, act, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_gla_step(const void* q, const void* k, const void* v, const void* low, const void* up, const void* up_bias, int rank,
                           float tau, const void* gate, const void* norm, float eps, float* state, void* out, int heads, int dim,
                           int vdim, int dtype, void* stream) {
    QD_CHECK_ARG(q && k && v && low && up && up_bias && gate && norm && state && out && rank > 0 && heads > 0 && dim > 0 && vdim > 0 && tau > 0.f);
    qd::StepParams p = {};
    p.q = q; p.k = k; p.v = v; p.low = low; p.up = (const bf16*)up; p.up_bias = (const bf16*)up_bias; p.rank = rank; p.tau = tau;
    p.gate_low = gate; p.norm = (const bf16*)norm; p.eps = eps; p.state = state; p.out = out;
    p.heads = heads; p.kv_heads = heads; p.dim = dim; p.vdim = vdim; p.taps = 1;
    if (dtype == QD_BF16) return qd::step<bf16, false>(p, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::step<float, false>(p, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_channel_delta_step(const void* q, const void* k, const void* v, const void* beta, const void* low, const void* up,
                                     const void* up_bias, int rank, const void* a_log, const void* q_taps, const void* k_taps,
                                     const void* v_taps, void* history, int taps, const int* position_ptr, int position,
                                     const void* gate_low, const void* gate_up, int gate_rank, const void* norm, float eps,
                                     float* state, void* out, int heads, int kv_heads, int dim, int vdim, int dtype, void* stream) {
    QD_CHECK_ARG(q && k && v && beta && low && up && up_bias && a_log && q_taps && k_taps && v_taps && history && gate_low && gate_up && norm);
    QD_CHECK_ARG(state && out && rank > 0 && gate_rank > 0 && taps > 0 && position >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0);
    QD_CHECK_ARG(dim > 0 && vdim > 0);
    const qd::StepParams p = {q, k, v, low, (const bf16*)up, (const bf16*)up_bias, rank, beta, (const bf16*)a_log, (const bf16*)q_taps,
                              (const bf16*)k_taps, (const bf16*)v_taps, taps, history, 1.f, gate_low, (const bf16*)gate_up, gate_rank,
                              (const bf16*)norm, eps, position_ptr, position, state, out, heads, kv_heads, dim, vdim};
    if (dtype == QD_BF16) return qd::step<bf16, true>(p, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::step<float, true>(p, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}
