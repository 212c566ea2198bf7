// Latent attention: queries through a normed latent, keys and values expanded per head from one normed
// latent per token, plus key columns with rotary positions (pairs i, i + rot / 2) that all heads share.  The
// cache keeps the latent and the rotated columns only, one row of `ld_cache` elements per position:
// [latent | zeros | rotated columns at rot_column | zeros], position p in row p mod capacity.
//
// Prompt chunks: latent_prepare_kernel (norm of the query latent, cache row) and rotate_half_kernel (queries in
// place); the visible rows are expanded by an ordinary product and attended by the grouped-query kernels.
//
// One token works on the latents themselves, since q . (W_uk c) = (W_uk^T q) . c and sum_j p_j W_uv c_j =
// W_uv sum_j p_j c_j.  Three launches:
//   latent_absorb_kernel   W_uk^T q per head (weights requested before the wait for the preceding kernel),
//                          rotation, the token's cache row
//   latent_mma_kernel      blocks = (split of the span, 16 heads): all heads read the same rows, so 16 heads are
//                          one m16n8k16 row block; queries and probabilities as two bf16 pieces, fp32 sums.
//                          latent_rows_kernel covers fp32 and rows that do not fit.
//   latent_values_kernel   merge of the splits, W_uv per head, output gate
#include "softmax_attention.cuh"

namespace qd {
namespace {

typedef qd_latent_args Latent;
constexpr int kTile = 32, kThreads = 256, kWarps = kThreads / 32;
constexpr int kMaxSplits = 64;

QD_DEVINL int position_of(const Latent& p) { return p.position_ptr ? *p.position_ptr : p.position; }
QD_DEVINL const bf16* weights(const void* p) { return reinterpret_cast<const bf16*>(p); }
__host__ __device__ constexpr int value_columns(int kv_rank) { return (kv_rank + 3) & ~3; }      // of a partial sum

// positions lo .. position in `active` splits of `per`
struct Splits { int lo, per, active; };
QD_DEVINL Splits split_plan(const Latent& p, int position) {
    Splits s;
    s.lo = max(0, position - p.span + 1);
    const int n = position - s.lo + 1;
    s.per = ((n + p.splits - 1) / p.splits + kTile - 1) / kTile * kTile;
    s.active = (n + s.per - 1) / s.per;
    return s;
}

// the cache row of one token from its projection row, by a whole block; trig: cosines, sines
template <typename T>
QD_DEVINL void write_row(const Latent& p, const T* dkv, int position, const float* trig, float* red) {
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.kv_rank; i += blockDim.x) { const float x = load_f(dkv + i); ss = fmaf(x, x, ss); }
    const float factor = 1.0f / sqrtf(block_sum(ss, red) / (float)p.kv_rank + p.eps);
    T* row = reinterpret_cast<T*>(p.cache) + (size_t)(position % p.capacity) * p.ld_cache;
    const int half = p.rot / 2;
    for (int i = threadIdx.x; i < (int)p.ld_cache; i += blockDim.x) {
        const int r = i - p.rot_column;
        float v = 0.f;
        if (i < p.kv_rank) v = load_f(dkv + i) * factor * ld_bf16(weights(p.dkv_norm) + i);
        else if (r >= 0 && r < p.rot) {
            const T* x = dkv + p.kv_rank;
            v = r < half ? fmaf(load_f(x + r), trig[r], -load_f(x + r + half) * trig[half + r])
                         : fmaf(load_f(x + r), trig[r - half], load_f(x + r - half) * trig[r]);
        }
        store_f(row + i, v);
    }
}
QD_DEVINL void fill_trig(const float* freq, int half, int position, float* trig) {
    for (int i = threadIdx.x; i < half; i += blockDim.x) rotation(position, freq[i], freq[half + i], trig[i], trig[half + i]);
}

// --------------------------------------------------------------------------------- prompt chunks
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_prepare_kernel(const __grid_constant__ Latent p) {
    chain_enter();
    extern __shared__ float trig[];
    __shared__ float red[33];
    const int t = blockIdx.x, position = position_of(p) + t;
    fill_trig(p.freq, p.rot / 2, position, trig);
    const T* dq = reinterpret_cast<const T*>(p.dq) + (long long)t * p.ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.q_rank; i += kThreads) { const float x = load_f(dq + i); ss = fmaf(x, x, ss); }
    const float factor = 1.0f / sqrtf(block_sum(ss, red) / (float)p.q_rank + p.eps);
    T* out = reinterpret_cast<T*>(p.q_latent) + (size_t)t * p.q_rank;
    for (int i = threadIdx.x; i < p.q_rank; i += kThreads) store_f(out + i, load_f(dq + i) * factor * ld_bf16(weights(p.dq_norm) + i));
    write_row(p, reinterpret_cast<const T*>(p.dkv) + (long long)t * p.ld, position, trig, red);
}

// x [tokens, heads, dim]: the last `rot` columns of every head, in place
template <typename T>
__global__ void __launch_bounds__(kThreads)
rotate_half_kernel(T* __restrict__ x, const float* __restrict__ freq, const int* position_ptr, int position, int heads, int dim, int rot) {
    chain_enter();
    extern __shared__ float trig[];
    const int half = rot / 2, t = blockIdx.x;
    fill_trig(freq, half, (position_ptr ? *position_ptr : position) + t, trig);
    __syncthreads();
    T* row = x + (size_t)t * heads * dim + dim - rot;
    for (int i = threadIdx.x; i < heads * half; i += kThreads) {
        T* pair = row + (size_t)(i / half) * dim + i % half;
        const float u = load_f(pair), v = load_f(pair + half), c = trig[i % half], s = trig[half + i % half];
        store_f(pair, fmaf(u, c, -v * s));
        store_f(pair + half, fmaf(v, c, u * s));
    }
}

// ------------------------------------------------------------------------- one token: queries
constexpr int kColumns = 64, kRowGroups = kThreads / 8, kAhead = 8;

// grid (column blocks of 64, heads + 1); the last row of blocks writes the cache row
template <typename T, bool VEC>
__global__ void __launch_bounds__(kThreads) latent_absorb_kernel(const __grid_constant__ Latent p) {
    extern __shared__ float trig[];
    __shared__ float red[33];
    __shared__ float sums[kWarps][kColumns];
    const int tid = threadIdx.x, h = blockIdx.y, c0 = blockIdx.x * kColumns, half = p.rot / 2;
    const int piece = tid & 7, group = tid >> 3, column = c0 + piece * 8;
    const bf16* uk = weights(p.uk) + (size_t)(h < p.heads ? h : 0) * p.dim * p.kv_rank;
    uint4 ahead[kAhead];
    const bool mine = h < p.heads && column < p.kv_rank;
    grid_launch_dependents();
    if (VEC) {
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const int d = group + i * kRowGroups;
            ahead[i] = mine && d < p.dim ? __ldg(reinterpret_cast<const uint4*>(uk + (size_t)d * p.kv_rank + column)) : make_uint4(0u, 0u, 0u, 0u);
        }
    }
    grid_dependency_wait();
    const int position = position_of(p);
    if (h == p.heads) {
        if (blockIdx.x) return;
        fill_trig(p.freq, half, position, trig);
        write_row(p, reinterpret_cast<const T*>(p.dkv), position, trig, red);
        return;
    }
    const T* q = reinterpret_cast<const T*>(p.q) + (size_t)h * (p.dim + p.rot);
    float* out = p.absorbed + (size_t)h * p.ld_cache;
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
    if (VEC) {
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const int d = group + i * kRowGroups;
            const float x = d < p.dim ? load_f(q + d) : 0.f;
            float w[8];
            unpack8(ahead[i], w);
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[e] = fmaf(x, w[e], acc[e]);
        }
    }
    if (mine)
        for (int d = group + (VEC ? kAhead * kRowGroups : 0); d < p.dim; d += kRowGroups) {
            const float x = load_f(q + d);
            const bf16* w = uk + (size_t)d * p.kv_rank + column;
#pragma unroll
            for (int e = 0; e < 8; ++e)
                if (column + e < p.kv_rank) acc[e] = fmaf(x, ld_bf16(w + e), acc[e]);
        }
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 8);
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 16);
        if ((tid & 31) < 8) sums[tid >> 5][piece * 8 + e] = acc[e];
    }
    if (blockIdx.x == 0) fill_trig(p.freq, half, position, trig);
    __syncthreads();
    if (tid < kColumns && c0 + tid < p.kv_rank) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) v += sums[w][tid];
        out[c0 + tid] = v;
    }
    if (blockIdx.x) return;
    for (int i = tid; i < (int)p.ld_cache - p.kv_rank; i += kThreads) {       // rotated columns, and zeros around them
        const int c = p.kv_rank + i, r = c - p.rot_column;
        float v = 0.f;
        if (r >= 0 && r < p.rot) {
            const T* x = q + p.dim;
            v = r < half ? fmaf(load_f(x + r), trig[r], -load_f(x + r + half) * trig[half + r])
                         : fmaf(load_f(x + r), trig[r - half], load_f(x + r - half) * trig[r]);
        }
        out[c] = v;
    }
}

// ----------------------------------------------------------------------- one token: attention
// partial results of a split: (maximum, denominator) [head][split], then sums [head][split][value_columns]
QD_DEVINL float2* split_stats(const Latent& p) { return reinterpret_cast<float2*>(p.partial); }
__host__ __device__ constexpr size_t stats_floats(int heads, int splits) { return (2 * (size_t)heads * splits + 3) / 4 * 4; }
QD_DEVINL float* split_sums(const Latent& p, int h, int split) {
    return p.partial + stats_floats(p.heads, p.splits) + ((size_t)h * p.splits + split) * value_columns(p.kv_rank);
}

constexpr int kPRow = kTile + 8;
size_t mma_smem(int row) {
    return sizeof(bf16) * ((2 * 16 + 2 * kTile) * (size_t)(row + 8) + 2 * 16 * kPRow) + sizeof(float) * (kWarps * 16 * (kTile + 1) + 3 * 16);
}

// ld_cache a multiple of sixteen; G: groups of sixteen value columns per warp
template <int G>
__global__ void __launch_bounds__(kThreads) latent_mma_kernel(const __grid_constant__ Latent p) {
    chain_enter();
    const int position = position_of(p);
    const Splits plan = split_plan(p, position);
    const int split = blockIdx.x;
    if (split >= plan.active) return;
    extern __shared__ __align__(16) bf16 tiles[];
    const int row = (int)p.ld_cache, krow = row + 8, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h0 = blockIdx.y * 16;
    bf16* q_hi = tiles;
    bf16* q_lo = q_hi + 16 * krow;
    bf16* ks = q_lo + 16 * krow;                             // two tiles
    bf16* p_hi = ks + 2 * kTile * krow;
    bf16* p_lo = p_hi + 16 * kPRow;
    float* part = reinterpret_cast<float*>(p_lo + 16 * kPRow);       // [warp][head][key], a warp's share of the columns
    float* stat = part + kWarps * 16 * (kTile + 1);          // maximum, denominator, rescaling factor [16] each
    const int first = plan.lo + split * plan.per, end = min(first + plan.per, position + 1), pieces = row / 8;
    const bf16* cache = weights(p.cache);
    auto stage = [&](int j0) {
        bf16* dst = ks + (((j0 - first) / kTile) & 1) * kTile * krow;
        for (int r = warp; r < kTile; r += kWarps) {
            const int j = j0 + r;
            const bool ok = j < end;
            const bf16* src = cache + (size_t)(ok ? j % p.capacity : 0) * row;
            for (int i = lane; i < pieces; i += 32) copy16_or_zero(dst + r * krow + i * 8, src + i * 8, ok);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(first);
    for (int i = tid; i < 16 * (row / 2); i += kThreads) {
        const int h = i / (row / 2), c = i % (row / 2) * 2;
        const float2 v = h0 + h < p.heads ? *reinterpret_cast<const float2*>(p.absorbed + (size_t)(h0 + h) * row + c) : make_float2(0.f, 0.f);
        const uint32_t hi = pack_pair(v.x, v.y);
        *reinterpret_cast<uint32_t*>(q_hi + h * krow + c) = hi;
        *reinterpret_cast<uint32_t*>(q_lo + h * krow + c) = pack_pair(v.x - __uint_as_float(hi << 16), v.y - __uint_as_float(hi & 0xffff0000u));
    }
    if (tid < 16) { stat[tid] = -INFINITY; stat[16 + tid] = 0.f; }

    float o[G][2][4];
#pragma unroll
    for (int g = 0; g < G; ++g)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) o[g][n][c] = 0.f;
    const int qa = (lane & 15) * krow + (lane >> 4) * 8;
    const int kb = ((lane & 7) + ((lane >> 4) << 3)) * krow + ((lane >> 3) & 1) * 8;
    const int groups = (p.kv_rank + 15) / 16;
    for (int j0 = first; j0 < end; j0 += kTile) {
        if (j0 + kTile < end) { stage(j0 + kTile); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const bf16* kt = ks + (((j0 - first) / kTile) & 1) * kTile * krow;
        float s[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[n][c] = 0.f;
        for (int k = warp; k < row / 16; k += kWarps) {
            uint32_t hi[4], lo[4];
            ldmatrix4(hi, q_hi + qa + k * 16);
            ldmatrix4(lo, q_lo + qa + k * 16);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                uint32_t b[4];
                ldmatrix4(b, kt + n * 16 * krow + kb + k * 16);
                mma_16816(s[2 * n], hi, b[0], b[1]);
                mma_16816(s[2 * n + 1], hi, b[2], b[3]);
                mma_16816(s[2 * n], lo, b[0], b[1]);
                mma_16816(s[2 * n + 1], lo, b[2], b[3]);
            }
        }
        float* mine = part + warp * 16 * (kTile + 1) + (lane >> 2) * (kTile + 1) + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) mine[(c >> 1) * 8 * (kTile + 1) + n * 8 + (c & 1)] = s[n][c];
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int h = warp * 2 + i;
            float score = 0.f;
#pragma unroll
            for (int w = 0; w < kWarps; ++w) score += part[(w * 16 + h) * (kTile + 1) + lane];
            score = j0 + lane < end ? score * p.scale : -INFINITY;
            const float m = stat[h], top = fmaxf(m, warp_max(score));       // the first key of a tile is always inside
            const float e = expf(score - top), sum = warp_sum(e);
            const bf16 hi = __float2bfloat16_rn(e);
            p_hi[h * kPRow + lane] = hi;
            p_lo[h * kPRow + lane] = __float2bfloat16_rn(e - __bfloat162float(hi));
            if (lane == 0) {
                const float keep = expf(m - top);
                stat[h] = top;
                stat[16 + h] = stat[16 + h] * keep + sum;
                stat[32 + h] = keep;
            }
        }
        __syncthreads();
        const float keep[2] = {stat[32 + (lane >> 2)], stat[32 + (lane >> 2) + 8]};
        uint32_t hi[2][4], lo[2][4];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            ldmatrix4(hi[k], p_hi + (lane & 15) * kPRow + (lane >> 4) * 8 + k * 16);
            ldmatrix4(lo[k], p_lo + (lane & 15) * kPRow + (lane >> 4) * 8 + k * 16);
        }
#pragma unroll
        for (int g = 0; g < G; ++g) {
            const int column = (warp + g * kWarps) * 16;
            if (warp + g * kWarps >= groups) break;
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int c = 0; c < 4; ++c) o[g][n][c] *= keep[c >> 1];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                uint32_t b[4];
                ldmatrix4_t(b, kt + (k * 16 + (lane & 15)) * krow + (lane >> 4) * 8 + column);
                mma_16816(o[g][0], hi[k], b[0], b[1]);
                mma_16816(o[g][1], hi[k], b[2], b[3]);
                mma_16816(o[g][0], lo[k], b[0], b[1]);
                mma_16816(o[g][1], lo[k], b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int h = h0 + (lane >> 2) + i * 8;
        if (h >= p.heads) continue;
        float* sums = split_sums(p, h, split);
#pragma unroll
        for (int g = 0; g < G; ++g)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const int column = (warp + g * kWarps) * 16 + n * 8 + (lane & 3) * 2;
                if (column < p.kv_rank) sums[column] = o[g][n][2 * i];
                if (column + 1 < p.kv_rank) sums[column + 1] = o[g][n][2 * i + 1];
            }
    }
    if (tid < 16 && h0 + tid < p.heads) split_stats(p)[(size_t)(h0 + tid) * p.splits + split] = make_float2(stat[tid], stat[16 + tid]);
}

// any activation type and row: block = (split, head)
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_rows_kernel(const __grid_constant__ Latent p) {
    chain_enter();
    const int position = position_of(p);
    const Splits plan = split_plan(p, position);
    const int split = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (split >= plan.active) return;
    extern __shared__ float q[];                             // query, then running sums
    __shared__ float weight[kTile], stat[3];
    const int row = (int)p.ld_cache;
    float* acc = q + row;
    for (int i = tid; i < row; i += kThreads) q[i] = p.absorbed[(size_t)h * row + i];
    for (int i = tid; i < p.kv_rank; i += kThreads) acc[i] = 0.f;
    if (tid == 0) { stat[0] = -INFINITY; stat[1] = 0.f; }
    __syncthreads();
    const int first = plan.lo + split * plan.per, end = min(first + plan.per, position + 1);
    const T* cache = reinterpret_cast<const T*>(p.cache);
    for (int j0 = first; j0 < end; j0 += kTile) {
        const int count = min(kTile, end - j0);
        for (int r = warp; r < kTile; r += kWarps) {
            float dot = 0.f;
            if (r < count) {
                const T* k = cache + (size_t)((j0 + r) % p.capacity) * row;
                for (int i = lane; i < row; i += 32) dot = fmaf(q[i], load_f(k + i), dot);
            }
            dot = warp_sum(dot);
            if (lane == 0) weight[r] = r < count ? dot * p.scale : -INFINITY;
        }
        __syncthreads();
        if (warp == 0) {
            const float score = weight[lane], m = stat[0], top = fmaxf(m, warp_max(score)), e = expf(score - top), sum = warp_sum(e);
            weight[lane] = e;
            if (lane == 0) {
                const float keep = expf(m - top);
                stat[0] = top;
                stat[1] = stat[1] * keep + sum;
                stat[2] = keep;
            }
        }
        __syncthreads();
        for (int i = tid; i < p.kv_rank; i += kThreads) {
            float a = acc[i] * stat[2];
            for (int r = 0; r < count; ++r) a = fmaf(weight[r], load_f(cache + (size_t)((j0 + r) % p.capacity) * row + i), a);
            acc[i] = a;
        }
        __syncthreads();
    }
    float* sums = split_sums(p, h, split);
    for (int i = tid; i < p.kv_rank; i += kThreads) sums[i] = acc[i];
    if (tid == 0) split_stats(p)[(size_t)h * p.splits + split] = make_float2(stat[0], stat[1]);
}

// -------------------------------------------------------------------------- one token: values
constexpr int kValueRows = 4, kValuePieces = 2;              // per warp; 16-byte pieces of a row requested ahead, per lane

// grid (blocks of 32 value columns of a head, heads)
template <typename T, bool VEC>
__global__ void __launch_bounds__(kThreads) latent_values_kernel(const __grid_constant__ Latent p) {
    extern __shared__ __align__(16) float lat[];             // [groups][value_columns]
    __shared__ float factor[kMaxSplits];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
    const int v0 = blockIdx.x * kWarps * kValueRows + warp * kValueRows;
    const bf16* uv = weights(p.uv) + ((size_t)h * p.vdim + v0) * p.kv_rank;
    uint4 ahead[kValueRows][kValuePieces];
    grid_launch_dependents();
    if (VEC) {
#pragma unroll
        for (int r = 0; r < kValueRows; ++r)
#pragma unroll
            for (int i = 0; i < kValuePieces; ++i) {
                const int c = (i * 32 + lane) * 8;
                ahead[r][i] = v0 + r < p.vdim && c < p.kv_rank ? __ldg(reinterpret_cast<const uint4*>(uv + (size_t)r * p.kv_rank + c))
                                                               : make_uint4(0u, 0u, 0u, 0u);
            }
    }
    grid_dependency_wait();
    const Splits plan = split_plan(p, position_of(p));
    if (warp == 0) {
        float2 s[2];
#pragma unroll
        for (int i = 0; i < 2; ++i)
            s[i] = i * 32 + lane < plan.active ? __ldcg(split_stats(p) + (size_t)h * p.splits + i * 32 + lane) : make_float2(-INFINITY, 0.f);
        const float top = warp_max(fmaxf(s[0].x, s[1].x)), a = expf(s[0].x - top), b = expf(s[1].x - top);
        const float total = warp_sum(fmaf(a, s[0].y, b * s[1].y));
        factor[lane] = a / total;
        factor[32 + lane] = b / total;
    }
    __syncthreads();
    const int columns = value_columns(p.kv_rank), quads = columns / 4;
    const int groups = max(1, min(8, kThreads / quads));
    for (int i = tid; i < quads * groups; i += kThreads) {
        const int c = i % quads * 4, group = i / quads;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int s = group; s < plan.active; s += groups) {
            const float4 x = __ldcg(reinterpret_cast<const float4*>(split_sums(p, h, s) + c));
            const float f = factor[s];
            a.x = fmaf(x.x, f, a.x); a.y = fmaf(x.y, f, a.y); a.z = fmaf(x.z, f, a.z); a.w = fmaf(x.w, f, a.w);
        }
        *reinterpret_cast<float4*>(lat + group * columns + c) = a;
    }
    __syncthreads();
    if (groups > 1) {
        for (int c = tid; c < p.kv_rank; c += kThreads) {
            float v = lat[c];
            for (int g = 1; g < groups; ++g) v += lat[g * columns + c];
            lat[c] = v;
        }
        __syncthreads();
    }
    float acc[kValueRows];
#pragma unroll
    for (int r = 0; r < kValueRows; ++r) acc[r] = 0.f;
    int done = 0;
    if (VEC) {
#pragma unroll
        for (int i = 0; i < kValuePieces; ++i) {
            const int c = (i * 32 + lane) * 8;
            if (c >= p.kv_rank) break;
            const float4 a = *reinterpret_cast<const float4*>(lat + c), b = *reinterpret_cast<const float4*>(lat + c + 4);
#pragma unroll
            for (int r = 0; r < kValueRows; ++r) {
                float w[8];
                unpack8(ahead[r][i], w);
                acc[r] = fmaf(w[0], a.x, fmaf(w[1], a.y, fmaf(w[2], a.z, fmaf(w[3], a.w, acc[r]))));
                acc[r] = fmaf(w[4], b.x, fmaf(w[5], b.y, fmaf(w[6], b.z, fmaf(w[7], b.w, acc[r]))));
            }
        }
        done = kValuePieces * 256;
    }
    for (int c = done + lane; c < p.kv_rank; c += 32) {
        const float a = lat[c];
#pragma unroll
        for (int r = 0; r < kValueRows; ++r)
            if (v0 + r < p.vdim) acc[r] = fmaf(ld_bf16(uv + (size_t)r * p.kv_rank + c), a, acc[r]);
    }
#pragma unroll
    for (int r = 0; r < kValueRows; ++r) {
        const float v = warp_sum(acc[r]);
        if (lane != 0 || v0 + r >= p.vdim) continue;
        const int at = h * p.vdim + v0 + r;
        const float gate = p.gate ? sigmoid_precise(load_f(reinterpret_cast<const T*>(p.gate) + at)) : 1.f;
        store_f(reinterpret_cast<T*>(p.out) + at, v * gate);
    }
}

// ----------------------------------------------------------------------------------- host side
template <typename T>
int prepare(const Latent& p, cudaStream_t s) {
    const size_t smem = sizeof(float) * (p.rot + 1);
    if (!allow_smem(latent_prepare_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(latent_prepare_kernel<T>, dim3(p.tokens), dim3(kThreads), smem, s, 1, p);
}

template <typename T>
int rotate(void* x, const float* freq, const int* position_ptr, int position, int tokens, int heads, int dim, int rot, cudaStream_t s) {
    const size_t smem = sizeof(float) * (rot + 1);
    if (!allow_smem(rotate_half_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(rotate_half_kernel<T>, dim3(tokens), dim3(kThreads), smem, s, 1, (T*)x, freq, position_ptr, position, heads, dim, rot);
}

template <int G>
int launch_mma(const Latent& p, cudaStream_t s) {
    const size_t smem = mma_smem((int)p.ld_cache);
    if (!allow_smem(latent_mma_kernel<G>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(latent_mma_kernel<G>, dim3(p.splits, (p.heads + 15) / 16), dim3(kThreads), smem, s, 1, p);
}

template <typename T, bool VEC>
int absorb(const Latent& p, cudaStream_t s) {
    const size_t smem = sizeof(float) * (p.rot + 1);
    if (!allow_smem(latent_absorb_kernel<T, VEC>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(latent_absorb_kernel<T, VEC>, dim3((p.kv_rank + kColumns - 1) / kColumns, p.heads + 1), dim3(kThreads), smem, s, 2, p);
}

template <typename T, bool VEC>
int values(const Latent& p, cudaStream_t s) {
    const int columns = value_columns(p.kv_rank), quads = columns / 4;
    const int groups = kThreads / quads > 8 ? 8 : (kThreads / quads < 1 ? 1 : kThreads / quads);
    const size_t smem = sizeof(float) * (size_t)groups * columns;
    if (!allow_smem(latent_values_kernel<T, VEC>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(latent_values_kernel<T, VEC>, dim3((p.vdim + kWarps * kValueRows - 1) / (kWarps * kValueRows), p.heads), dim3(kThreads), smem, s,
                     2, p);
}

template <typename T>
int step(const Latent& p, cudaStream_t s) {
    const bool vec = p.kv_rank % 8 == 0 && aligned16(p.uk) && aligned16(p.uv);
    int rc = vec ? absorb<T, true>(p, s) : absorb<T, false>(p, s);
    if (rc != QD_OK) return rc;
    if (sizeof(T) == 2 && p.ld_cache % 16 == 0 && aligned16(p.cache) && p.kv_rank <= 1024 && mma_smem((int)p.ld_cache) <= kMaxSmem) {
        if (p.kv_rank <= 128) rc = launch_mma<1>(p, s);
        else if (p.kv_rank <= 256) rc = launch_mma<2>(p, s);
        else if (p.kv_rank <= 512) rc = launch_mma<4>(p, s);
        else rc = launch_mma<8>(p, s);
    } else {
        const size_t smem = sizeof(float) * (size_t)(p.ld_cache + p.kv_rank);
        if (!allow_smem(latent_rows_kernel<T>, smem)) return QD_ERR_UNSUPPORTED;
        rc = qd_launch(latent_rows_kernel<T>, dim3(p.splits, p.heads), dim3(kThreads), smem, s, 1, p);
    }
    if (rc != QD_OK) return rc;
    return vec ? values<T, true>(p, s) : values<T, false>(p, s);
}

bool valid(const Latent& a) {
    return a.dkv && a.dkv_norm && a.cache && a.rot >= 0 && a.rot % 2 == 0 && (a.rot == 0 || a.freq) && a.kv_rank > 0 &&
           a.rot_column >= a.kv_rank && a.ld_cache >= a.rot_column + a.rot && a.capacity > 0 && a.position >= 0;
}

}  // namespace
}  // namespace qd

extern "C" int qd_latent_prepare(const qd_latent_args* args, void* stream) {
    QD_CHECK_ARG(args && qd::valid(*args) && args->dq && args->dq_norm && args->q_latent && args->q_rank > 0 && args->tokens > 0);
    // rows of one chunk must not fall on one another
    if (args->tokens > args->capacity) return QD_ERR_ARG;
    if (args->dtype == QD_BF16) return qd::prepare<bf16>(*args, (cudaStream_t)stream);
    if (args->dtype == QD_F32) return qd::prepare<float>(*args, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_rotate_half(void* x, const float* freq, const int* position_ptr, int position, int tokens, int heads, int dim, int rot,
                              int dtype, void* stream) {
    QD_CHECK_ARG(x && freq && tokens > 0 && heads > 0 && rot > 0 && rot % 2 == 0 && rot <= dim && position >= 0);
    if (dtype == QD_BF16) return qd::rotate<bf16>(x, freq, position_ptr, position, tokens, heads, dim, rot, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::rotate<float>(x, freq, position_ptr, position, tokens, heads, dim, rot, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" long long qd_latent_step_floats(int heads, int kv_rank, int splits) {
    return (long long)qd::stats_floats(heads, splits) + (long long)heads * splits * qd::value_columns(kv_rank);
}

extern "C" int qd_latent_step(const qd_latent_args* args, void* stream) {
    QD_CHECK_ARG(args && qd::valid(*args) && args->q && args->uk && args->uv && args->absorbed && args->partial && args->out);
    QD_CHECK_ARG(args->heads > 0 && args->dim > 0 && args->vdim > 0 && args->span > 0 && args->span <= args->capacity);
    QD_CHECK_ARG(args->splits > 0 && args->splits <= qd::kMaxSplits && qd::aligned16(args->partial) && ((uintptr_t)args->absorbed & 7u) == 0);
    if (args->dtype == QD_BF16) return qd::step<bf16>(*args, (cudaStream_t)stream);
    if (args->dtype == QD_F32) return qd::step<float>(*args, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}
