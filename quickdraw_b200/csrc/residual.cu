// The fp32 residual stream between the products: embedding rows, layer norm with weight and bias, the
// end of a sublayer (sigmoid gate on the sublayer's result, its norm, the residual sum, the weighted
// average over the embedding output and all layer results so far, the norm in front of the next
// sublayer) in one launch.  One block per token; a row of the stream lives in shared memory.
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
    const size_t smem = (size_t)p.width * 4;
    if (!allow_smem(sublayer_close_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(sublayer_close_kernel<T>, dim3(tokens), dim3(row_threads(p.width)), smem, s, 1, p);
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
