// The fp32 residual stream between the products.  Two styles.  Layer norms around a gated sublayer:
// embedding rows, layer norm with weight and bias, the end of a sublayer (sigmoid gate on the sublayer's
// result, its norm, the residual sum, the weighted average over the embedding output and all layer
// results so far, the norm in front of the next sublayer) in one launch.  RMS norms in front of a
// sublayer: embedding row or stream row, plus the sublayer's result, plus a vector (that of a pass over
// looped layers), and the next RMS norm of the sum in one launch (stream_norm).  One block per token; a row of the stream lives in shared memory.
// HBM-bound (a few bytes per element and operand); at one token bound by the launch and two reductions.
#include "typed.cuh"

namespace qd {
namespace {

constexpr int kMaxThreads = 512;

// mean and reciprocal deviation of the block's fp32 row (two passes)
QD_DEVINL void row_moments(const float* row, int width, float eps, float* red, float& mean, float& rstd) {
    float sum = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) sum += row[i];
    mean = block_sum(sum, red) / (float)width;
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) { const float d = row[i] - mean; sq = fmaf(d, d, sq); }
    rstd = 1.0f / sqrtf(block_sum(sq, red) / (float)width + eps);
}

// out = layer_norm(row) * w + b.  Every thread reads and writes the elements threadIdx.x, + blockDim.x, ...
template <typename TO>
QD_DEVINL void norm_out(const float* row, int width, float eps, const bf16* w, const bf16* b, TO* out, float* red) {
    float mean, rstd;
    row_moments(row, width, eps, red, mean, rstd);
    for (int i = threadIdx.x; i < width; i += blockDim.x)
        store_f(out + i, (row[i] - mean) * rstd * ld_bf16(w + i) + ld_bf16(b + i));
}

template <typename T>
__global__ void __launch_bounds__(kMaxThreads)
embed_norm_kernel(const long long* __restrict__ tokens, const bf16* __restrict__ table, int vocab, float* __restrict__ stream_out,
                  const bf16* __restrict__ w, const bf16* __restrict__ b, T* __restrict__ normed, int width, float eps) {
    chain_enter();
    extern __shared__ float row[];
    __shared__ float red[33];
    const size_t t = blockIdx.x;
    long long id = tokens[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = ld_bf16(table + (size_t)id * width + i);
        row[i] = v;
        stream_out[t * width + i] = v;
    }
    norm_out(row, width, eps, w, b, normed + t * width, red);
}

template <typename T>
__global__ void __launch_bounds__(kMaxThreads)
layer_norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ index, const bf16* __restrict__ w,
                       const bf16* __restrict__ b, T* __restrict__ out, int width, float eps) {
    chain_enter();
    extern __shared__ float row[];
    __shared__ float red[33];
    const size_t src = index ? (size_t)index[blockIdx.x] : blockIdx.x;
    for (int i = threadIdx.x; i < width; i += blockDim.x) row[i] = x[src * width + i];
    norm_out(row, width, eps, w, b, out + (size_t)blockIdx.x * width, red);
}

struct CloseParams {
    const void* y; const void* gate; long long ld_gate; const bf16* gate_bias;
    const bf16* post_w; const bf16* post_b;
    const float* x_in; float* x_out;
    // depth average over results 0 .. older (the newest is this sublayer's and is stored as results[older]);
    // older < 0: none, x_out is the residual sum
    float* results; long long result_stride; const bf16* depth; int older;
    const bf16* next_w; const bf16* next_b; void* normed;      // next_w == NULL: no norm behind it
    int width; float eps;
};

template <typename T>
__global__ void __launch_bounds__(kMaxThreads)
sublayer_close_kernel(const __grid_constant__ CloseParams p) {
    chain_enter();
    extern __shared__ float row[];
    __shared__ float red[33];
    const int width = p.width;
    const size_t t = blockIdx.x, at = t * width;
    const T* y = reinterpret_cast<const T*>(p.y) + at;
    const T* gate = reinterpret_cast<const T*>(p.gate) + t * p.ld_gate;
    for (int i = threadIdx.x; i < width; i += blockDim.x)
        row[i] = load_f(y + i) * sigmoid_precise(load_f(gate + i) + ld_bf16(p.gate_bias + i));
    float mean, rstd;
    row_moments(row, width, p.eps, red, mean, rstd);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        float v = p.x_in[at + i] + ((row[i] - mean) * rstd * ld_bf16(p.post_w + i) + ld_bf16(p.post_b + i));
        if (p.older >= 0) {
            float* result = p.results + at + i;
            result[p.older * p.result_stride] = v;
            v *= ld_bf16(p.depth + p.older);
            float other[4] = {0.f, 0.f, 0.f, 0.f};
            int j = 0;
            for (; j + 4 <= p.older; j += 4)
#pragma unroll
                for (int q = 0; q < 4; ++q) other[q] = fmaf(result[(j + q) * p.result_stride], ld_bf16(p.depth + j + q), other[q]);
            for (; j < p.older; ++j) other[0] = fmaf(result[j * p.result_stride], ld_bf16(p.depth + j), other[0]);
            v += (other[0] + other[1]) + (other[2] + other[3]);
        }
        p.x_out[at + i] = v;
        row[i] = v;
    }
    if (p.next_w) norm_out(row, width, p.eps, p.next_w, p.next_b, reinterpret_cast<T*>(p.normed) + at, red);
}

// The same for widths that split evenly: every thread keeps VPT groups of four consecutive elements in
// registers, the sums over earlier results are formed before the first reduction, and mean and deviation
// come out of ONE exchange: equal counts merge as mean = average of the means, M2 = sum of the M2 + count
// times the squared distances of the means.
QD_DEVINL void merged_moments(const float* v, int count, int width, float eps, float2* stats, float& mean, float& rstd) {
    float m = 0.f, m2 = 0.f;
    for (int i = 0; i < count; ++i) m += v[i];
    m /= (float)count;
    for (int i = 0; i < count; ++i) { const float d = v[i] - m; m2 = fmaf(d, d, m2); }
    float n = (float)count;
#pragma unroll
    for (int x = 1; x < 32; x <<= 1) {
        const float om = __shfl_xor_sync(0xffffffffu, m, x), o2 = __shfl_xor_sync(0xffffffffu, m2, x);
        const float d = om - m;
        m2 = m2 + o2 + d * d * (0.5f * n);
        m = 0.5f * (m + om);
        n *= 2.f;
    }
    const int warps = blockDim.x >> 5;
    if ((threadIdx.x & 31) == 0) stats[threadIdx.x >> 5] = make_float2(m, m2);
    __syncthreads();
    float sum = 0.f, sq = 0.f;
    for (int w = 0; w < warps; ++w) sum += stats[w].x;
    mean = sum / (float)warps;
    for (int w = 0; w < warps; ++w) { const float d = stats[w].x - mean; sq += stats[w].y + n * d * d; }
    rstd = 1.0f / sqrtf(sq / (float)width + eps);
}

template <typename T, int VPT>
__global__ void __launch_bounds__(kMaxThreads)
sublayer_close_vec_kernel(const __grid_constant__ CloseParams p) {
    chain_enter();
    __shared__ float2 stats[2][kMaxThreads / 32];
    const int width = p.width, threads = blockDim.x;
    const size_t t = blockIdx.x, at = t * width;
    const T* y = reinterpret_cast<const T*>(p.y) + at;
    const T* gate = reinterpret_cast<const T*>(p.gate) + t * p.ld_gate;
    float z[4 * VPT], x[4 * VPT], mix[4 * VPT];
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = (threadIdx.x + k * threads) * 4;
        const float4 yv = load4(y + i), gv = load4(gate + i), bv = load4(p.gate_bias + i), xv = load4(p.x_in + at + i);
        const float ya[4] = {yv.x, yv.y, yv.z, yv.w}, ga[4] = {gv.x + bv.x, gv.y + bv.y, gv.z + bv.z, gv.w + bv.w};
        const float xa[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) { z[4 * k + e] = ya[e] * sigmoid_precise(ga[e]); x[4 * k + e] = xa[e]; mix[4 * k + e] = 0.f; }
    }
    for (int j0 = 0; j0 < p.older; j0 += 4) {
        float4 r[4][VPT];
        float c[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            c[q] = j0 + q < p.older ? ld_bf16(p.depth + j0 + q) : 0.f;
            const float* result = p.results + (size_t)min(j0 + q, p.older - 1) * p.result_stride + at;
#pragma unroll
            for (int k = 0; k < VPT; ++k) r[q][k] = load4(result + (threadIdx.x + k * threads) * 4);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q)
#pragma unroll
            for (int k = 0; k < VPT; ++k) {
                mix[4 * k] = fmaf(r[q][k].x, c[q], mix[4 * k]); mix[4 * k + 1] = fmaf(r[q][k].y, c[q], mix[4 * k + 1]);
                mix[4 * k + 2] = fmaf(r[q][k].z, c[q], mix[4 * k + 2]); mix[4 * k + 3] = fmaf(r[q][k].w, c[q], mix[4 * k + 3]);
            }
    }
    float mean, rstd;
    merged_moments(z, 4 * VPT, width, p.eps, stats[0], mean, rstd);
    const float newest = p.older >= 0 ? ld_bf16(p.depth + p.older) : 1.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = (threadIdx.x + k * threads) * 4;
        const float4 wv = load4(p.post_w + i), bv = load4(p.post_b + i);
        const float wa[4] = {wv.x, wv.y, wv.z, wv.w}, ba[4] = {bv.x, bv.y, bv.z, bv.w};
        float* v = z + 4 * k;
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = x[4 * k + e] + ((v[e] - mean) * rstd * wa[e] + ba[e]);
        if (p.older >= 0) {
            store4(p.results + (size_t)p.older * p.result_stride + at + i, make_float4(v[0], v[1], v[2], v[3]));
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = fmaf(v[e], newest, mix[4 * k + e]);
        }
        store4(p.x_out + at + i, make_float4(v[0], v[1], v[2], v[3]));
    }
    if (!p.next_w) return;
    merged_moments(z, 4 * VPT, width, p.eps, stats[1], mean, rstd);
    T* normed = reinterpret_cast<T*>(p.normed) + at;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = (threadIdx.x + k * threads) * 4;
        const float4 wv = load4(p.next_w + i), bv = load4(p.next_b + i);
        const float* v = z + 4 * k;
        store4(normed + i, make_float4((v[0] - mean) * rstd * wv.x + bv.x, (v[1] - mean) * rstd * wv.y + bv.y,
                                       (v[2] - mean) * rstd * wv.z + bv.z, (v[3] - mean) * rstd * wv.w + bv.w));
    }
}

struct StreamNorm {
    const long long* tokens; const bf16* table; int vocab;      // the rows of a table ...
    const float* x_in; const int* index;                        // ... or rows of the stream (index == NULL: row r)
    const void* y; const bf16* step;                            // added where given: a row each, one vector for all
    float* x_out;                                               // where given: the sum
    const bf16* norm; float offset, eps; void* normed;          // where given: sum / rms(sum) * (offset + norm)
    int width;
};

QD_DEVINL size_t source_row(const StreamNorm& p, size_t r) {
    if (!p.table) return p.index ? (size_t)p.index[r] : r;
    const long long id = p.tokens[r];
    return (size_t)(id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id));
}

template <typename T>
__global__ void __launch_bounds__(kMaxThreads) stream_norm_kernel(const __grid_constant__ StreamNorm p) {
    chain_enter();
    extern __shared__ float row[];
    __shared__ float red[33];
    const int width = p.width;
    const size_t at = (size_t)blockIdx.x * width, src = source_row(p, blockIdx.x) * width;
    const T* y = reinterpret_cast<const T*>(p.y) + at;
    float ss = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        float v = p.table ? ld_bf16(p.table + src + i) : p.x_in[src + i];
        if (p.y) v += load_f(y + i);
        if (p.step) v += ld_bf16(p.step + i);
        if (p.x_out) p.x_out[at + i] = v;
        row[i] = v;
        ss = fmaf(v, v, ss);
    }
    if (!p.norm) return;
    const float factor = 1.0f / sqrtf(block_sum(ss, red) / (float)width + p.eps);
    T* normed = reinterpret_cast<T*>(p.normed) + at;
    for (int i = threadIdx.x; i < width; i += blockDim.x) store_f(normed + i, row[i] * factor * (p.offset + ld_bf16(p.norm + i)));
}

// The same for widths that split evenly: VPT groups of four consecutive elements per thread, in registers.
template <typename T, int VPT>
__global__ void __launch_bounds__(kMaxThreads) stream_norm_vec_kernel(const __grid_constant__ StreamNorm p) {
    chain_enter();
    __shared__ float red[33];
    const int width = p.width, threads = blockDim.x;
    const size_t at = (size_t)blockIdx.x * width, src = source_row(p, blockIdx.x) * width;
    const T* y = reinterpret_cast<const T*>(p.y) + at;
    float4 v[VPT];
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = (threadIdx.x + k * threads) * 4;
        v[k] = p.table ? load4(p.table + src + i) : load4(p.x_in + src + i);
    }
    if (p.y)
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const float4 a = load4(y + (threadIdx.x + k * threads) * 4);
            v[k].x += a.x; v[k].y += a.y; v[k].z += a.z; v[k].w += a.w;
        }
    if (p.step)
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const float4 a = load4(p.step + (threadIdx.x + k * threads) * 4);
            v[k].x += a.x; v[k].y += a.y; v[k].z += a.z; v[k].w += a.w;
        }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        if (p.x_out) store4(p.x_out + at + (threadIdx.x + k * threads) * 4, v[k]);
        ss = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, fmaf(v[k].z, v[k].z, fmaf(v[k].w, v[k].w, ss))));
    }
    if (!p.norm) return;
    const float factor = 1.0f / sqrtf(block_sum(ss, red) / (float)width + p.eps);
    T* normed = reinterpret_cast<T*>(p.normed) + at;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = (threadIdx.x + k * threads) * 4;
        const float4 w = load4(p.norm + i);
        store4(normed + i, make_float4(v[k].x * factor * (p.offset + w.x), v[k].y * factor * (p.offset + w.y),
                                       v[k].z * factor * (p.offset + w.z), v[k].w * factor * (p.offset + w.w)));
    }
}

int row_threads(int width) {
    int threads = (width / 4 + 31) / 32 * 32;
    return threads < 64 ? 64 : (threads > kMaxThreads ? kMaxThreads : threads);
}

template <typename T>
int embed_norm(const void* tokens, const void* table, int vocab, float* x, const void* w, const void* b, void* normed,
               int count, int width, float eps, cudaStream_t s) {
    const size_t smem = (size_t)width * 4;
    if (!allow_smem(embed_norm_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(embed_norm_kernel<T>, dim3(count), dim3(row_threads(width)), smem, s, 1, (const long long*)tokens,
                     (const bf16*)table, vocab, x, (const bf16*)w, (const bf16*)b, (T*)normed, width, eps);
}
template <typename T>
int norm_rows(const float* x, const int* index, const void* w, const void* b, void* out, int rows, int width, float eps, cudaStream_t s) {
    const size_t smem = (size_t)width * 4;
    if (!allow_smem(layer_norm_rows_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(layer_norm_rows_kernel<T>, dim3(rows), dim3(row_threads(width)), smem, s, 1, x, index, (const bf16*)w,
                     (const bf16*)b, (T*)out, width, eps);
}
template <typename T>
int close(const CloseParams& p, int tokens, cudaStream_t s) {
    // groups of four per thread: few tokens want many threads, many tokens more work per thread
    const int quads = p.width / 4;
    const auto fits = [&](int vpt) { return quads % (32 * vpt) == 0 && quads / vpt <= kMaxThreads; };
    const auto at16 = [](const void* a) { return aligned16(a); };
    const bool vectors = p.width % 4 == 0 && p.ld_gate % 8 == 0 && p.result_stride % 4 == 0 && at16(p.y) && at16(p.gate) && at16(p.gate_bias) &&
                         at16(p.post_w) && at16(p.post_b) && at16(p.x_in) && at16(p.x_out) && at16(p.results) && at16(p.next_w) &&
                         at16(p.next_b) && at16(p.normed);
    if (vectors) {
        if (fits(1) && (tokens < 64 || quads <= 256)) return qd_launch(sublayer_close_vec_kernel<T, 1>, dim3(tokens), dim3(quads), 0, s, 1, p);
        if (fits(2)) return qd_launch(sublayer_close_vec_kernel<T, 2>, dim3(tokens), dim3(quads / 2), 0, s, 1, p);
        if (fits(4)) return qd_launch(sublayer_close_vec_kernel<T, 4>, dim3(tokens), dim3(quads / 4), 0, s, 1, p);
        if (fits(1)) return qd_launch(sublayer_close_vec_kernel<T, 1>, dim3(tokens), dim3(quads), 0, s, 1, p);
    }
    const size_t smem = (size_t)p.width * 4;
    if (!allow_smem(sublayer_close_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(sublayer_close_kernel<T>, dim3(tokens), dim3(row_threads(p.width)), smem, s, 1, p);
}

template <typename T>
int stream_norm(const StreamNorm& p, int rows, cudaStream_t s) {
    const int quads = p.width / 4;
    const auto fits = [&](int vpt) { return quads % (32 * vpt) == 0 && quads / vpt <= kMaxThreads; };
    if (p.width % 4 == 0 && aligned16(p.table) && aligned16(p.x_in) && aligned16(p.y) && aligned16(p.step) && aligned16(p.x_out) &&
        aligned16(p.norm) && aligned16(p.normed)) {
        if (fits(1) && (rows < 64 || quads <= 256)) return qd_launch(stream_norm_vec_kernel<T, 1>, dim3(rows), dim3(quads), 0, s, 1, p);
        if (fits(2)) return qd_launch(stream_norm_vec_kernel<T, 2>, dim3(rows), dim3(quads / 2), 0, s, 1, p);
        if (fits(4)) return qd_launch(stream_norm_vec_kernel<T, 4>, dim3(rows), dim3(quads / 4), 0, s, 1, p);
        if (fits(1)) return qd_launch(stream_norm_vec_kernel<T, 1>, dim3(rows), dim3(quads), 0, s, 1, p);
    }
    const size_t smem = (size_t)p.width * 4;
    if (!allow_smem(stream_norm_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(stream_norm_kernel<T>, dim3(rows), dim3(row_threads(p.width)), smem, s, 1, p);
}

}  // namespace
}  // namespace qd

extern "C" int qd_embed_norm(const void* tokens, const void* table, int vocab, float* x, const void* norm_w, const void* norm_b,
                             void* normed, int count, int width, float eps, int dtype, void* stream) {
    QD_CHECK_ARG(tokens && table && x && norm_w && norm_b && normed && vocab > 0 && count > 0 && width > 0);
    if (dtype == QD_BF16) return qd::embed_norm<bf16>(tokens, table, vocab, x, norm_w, norm_b, normed, count, width, eps, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::embed_norm<float>(tokens, table, vocab, x, norm_w, norm_b, normed, count, width, eps, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_layer_norm_rows(const float* x, const int* index, const void* w, const void* b, void* out, int rows, int width,
                                  float eps, int dtype, void* stream) {
    QD_CHECK_ARG(x && w && b && out && rows > 0 && width > 0);
    if (dtype == QD_BF16) return qd::norm_rows<bf16>(x, index, w, b, out, rows, width, eps, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::norm_rows<float>(x, index, w, b, out, rows, width, eps, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_sublayer_close(const void* y, const void* gate, long long ld_gate, const void* gate_bias, const void* post_w,
                                 const void* post_b, const float* x_in, float* x_out, float* results, long long result_stride,
                                 const void* depth, int older, const void* next_w, const void* next_b, void* normed, int tokens,
                                 int width, float eps, int dtype, void* stream) {
    QD_CHECK_ARG(y && gate && gate_bias && post_w && post_b && x_in && x_out && tokens > 0 && width > 0 && ld_gate >= width);
    QD_CHECK_ARG(older < 0 || (results && depth));
    QD_CHECK_ARG(!next_w || (next_b && normed));
    const qd::CloseParams p = {y, gate, ld_gate, (const bf16*)gate_bias, (const bf16*)post_w, (const bf16*)post_b, x_in, x_out,
                               results, result_stride, (const bf16*)depth, older, (const bf16*)next_w, (const bf16*)next_b, normed,
                               width, eps};
    if (dtype == QD_BF16) return qd::close<bf16>(p, tokens, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::close<float>(p, tokens, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_stream_norm(const void* tokens, const void* table, int vocab, const float* x_in, const int* index, const void* y,
                              const void* step, float* x_out, const void* norm, float norm_offset, void* normed, int rows, int width,
                              float eps, int dtype, void* stream) {
    QD_CHECK_ARG((table ? tokens && vocab > 0 : x_in != nullptr) && rows > 0 && width > 0 && (x_out || norm) && (!norm || normed));
    const qd::StreamNorm p = {(const long long*)tokens, (const bf16*)table, vocab, x_in, index, y, (const bf16*)step, x_out,
                              (const bf16*)norm, norm_offset, eps, normed, width};
    if (dtype == QD_BF16) return qd::stream_norm<bf16>(p, rows, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::stream_norm<float>(p, rows, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}
