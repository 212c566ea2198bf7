// Grouped-query softmax attention over a bounded span of positions, with what a design may put around it:
//   mask     the last `span` positions, or the positions of the same chunk of `span` positions from 0
//   scores   scaled; minus a slope per head times the distance
//   sink     none, a learned score per head, or a score of zero, in the softmax's denominator only
//   q and k  RMS norm over the whole projection or per head, interleaved rotary positions
//   result   times one sigmoid gate per head or per value column
// The visible keys and values live in a ring of `capacity` rows (position p in row p mod capacity), so a
// sequence's cache does not grow with its length.  Keys may end in columns that all heads share (k_shared).
//
// Prompt chunks: attn_prepare_kernel (norm, rotation, ring rows) and attn_flash_kernel (mma.sync m16n8k16;
// 64 or 128 packed (token, head of the group) rows per block, key tiles of 64 through two cp.async buffers,
// only the tiles a row of the block can see; probabilities as two bf16 pieces).  attn_rows_kernel covers fp32
// and shapes without 16-byte rows.  Decode: attn_step_kernel, one launch: norm and rotation in every
// block, blocks = (key/value head, split of the span), the last block of a head merges.
#include "softmax_attention.cuh"

namespace qd {
namespace {

// normalised, rotated element d of the head whose elements start at `first` of a projection row
template <typename T>
QD_DEVINL float rotated(const T* row, const bf16* w, int norm, float rms, int first, int d, int rot, const float* cosine, const float* sine) {
    if (norm == QD_NORM_ROW) w += first;
    const auto at = [&](int e) { return norm == QD_NORM_NONE ? load_f(row + first + e) : load_f(row + first + e) * rms * ld_bf16(w + e); };
    const float x = at(d);
    if (d >= rot) return x;
    const int i = d >> 1;
    const float other = at(d ^ 1);
    return (d & 1) ? fmaf(x, cosine[i], other * sine[i]) : fmaf(x, cosine[i], -other * sine[i]);
}

typedef qd_attention_args AttnParams;
QD_DEVINL const bf16* as_bf16(const void* p) { return reinterpret_cast<const bf16*>(p); }
// lowest position that `position` sees
__host__ __device__ __forceinline__ int lowest_key(const AttnParams& p, int position) {
    if (p.mask == QD_MASK_CHUNK) return position - position % p.span;
    return position - p.span + 1 > 0 ? position - p.span + 1 : 0;
}

template <typename T>
__global__ void __launch_bounds__(256) attn_prepare_kernel(const __grid_constant__ AttnParams p) {
    chain_enter();
    extern __shared__ float trig[];                    // cosines, sines, head factors
    __shared__ float red[33];
    const int t = blockIdx.x, tid = threadIdx.x, half = p.rot / 2;
    const int position = (p.position_ptr ? *p.position_ptr : p.position) + t;
    const int qn = p.heads * p.dim, kn = p.kv_heads * p.dim, vn = p.kv_heads * p.vdim;
    const T* q = reinterpret_cast<const T*>(p.q) + (long long)t * p.ld;
    const T* k = reinterpret_cast<const T*>(p.k) + (long long)t * p.ld;
    const T* v = reinterpret_cast<const T*>(p.v) + (long long)t * p.ld;
    for (int i = tid; i < half; i += 256) rotation(position, p.freq[i], p.freq[half + i], trig[i], trig[half + i]);
    float* head_rms = trig + p.rot;                    // of the query heads, then of the key heads
    float qr = 1.f, kr = 1.f;
    if (p.norm == QD_NORM_ROW) {
        float qq = 0.f, kk = 0.f;
        for (int i = tid; i < qn; i += 256) { const float x = load_f(q + i); qq = fmaf(x, x, qq); }
        for (int i = tid; i < kn; i += 256) { const float x = load_f(k + i); kk = fmaf(x, x, kk); }
        qr = 1.0f / sqrtf(block_sum(qq, red) / (float)qn + p.eps);
        kr = 1.0f / sqrtf(block_sum(kk, red) / (float)kn + p.eps);
    } else if (p.norm == QD_NORM_HEAD) {
        for (int h = tid >> 5; h < p.heads + p.kv_heads; h += 8) {
            const T* row = h < p.heads ? q + h * p.dim : k + (h - p.heads) * p.dim;
            float ss = 0.f;
            for (int d = tid & 31; d < p.dim; d += 32) { const float x = load_f(row + d); ss = fmaf(x, x, ss); }
            ss = warp_sum(ss);
            if ((tid & 31) == 0) head_rms[h] = 1.0f / sqrtf(ss / (float)p.dim + p.eps);
        }
    }
    __syncthreads();
    const size_t slot = position % p.capacity;
    T* ring_k = reinterpret_cast<T*>(p.k_cache) + slot * p.ld_k;
    T* ring_v = reinterpret_cast<T*>(p.v_cache) + slot * p.ld_v;
    T* q_out = reinterpret_cast<T*>(p.q_rows) + (size_t)t * qn;
    const bool heads = p.norm == QD_NORM_HEAD;
    for (int i = tid; i < qn; i += 256) {
        const int h = i / p.dim;
        store_f(q_out + i, rotated(q, as_bf16(p.q_norm), p.norm, heads ? head_rms[h] : qr, h * p.dim, i - h * p.dim, p.rot, trig, trig + half));
    }
    for (int i = tid; i < kn; i += 256) {
        const int h = i / p.dim;
        store_f(ring_k + i, rotated(k, as_bf16(p.k_norm), p.norm, heads ? head_rms[p.heads + h] : kr, h * p.dim, i - h * p.dim, p.rot, trig,
                                    trig + half));
    }
    for (int i = tid; i < vn; i += 256) ring_v[i] = v[i];
}

// The same for rows of four-element pieces: a warp per head, no divisions by the head size.
template <typename T>
__global__ void __launch_bounds__(256) attn_prepare_vec_kernel(const __grid_constant__ AttnParams p) {
    chain_enter();
    extern __shared__ float trig[];                    // cosines, sines
    __shared__ float red[33];
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, half = p.rot / 2;
    const int position = (p.position_ptr ? *p.position_ptr : p.position) + t;
    const int qn = p.heads * p.dim, kn = p.kv_heads * p.dim, vn = p.kv_heads * p.vdim;
    const T* q = reinterpret_cast<const T*>(p.q) + (long long)t * p.ld;
    const T* k = reinterpret_cast<const T*>(p.k) + (long long)t * p.ld;
    const T* v = reinterpret_cast<const T*>(p.v) + (long long)t * p.ld;
    for (int i = tid; i < half; i += 256) rotation(position, p.freq[i], p.freq[half + i], trig[i], trig[half + i]);
    const auto squares = [](const float4& x, float sum) { return fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, sum)))); };
    float qr = 1.f, kr = 1.f;
    if (p.norm == QD_NORM_ROW) {
        float qq = 0.f, kk = 0.f;
        for (int i = tid * 4; i < qn; i += 1024) qq = squares(load4(q + i), qq);
        for (int i = tid * 4; i < kn; i += 1024) kk = squares(load4(k + i), kk);
        qr = 1.0f / sqrtf(block_sum(qq, red) / (float)qn + p.eps);
        kr = 1.0f / sqrtf(block_sum(kk, red) / (float)kn + p.eps);
    }
    __syncthreads();
    const size_t slot = position % p.capacity;
    T* ring_k = reinterpret_cast<T*>(p.k_cache) + slot * p.ld_k;
    T* ring_v = reinterpret_cast<T*>(p.v_cache) + slot * p.ld_v;
    T* q_out = reinterpret_cast<T*>(p.q_rows) + (size_t)t * qn;
    for (int h = tid >> 5; h < p.heads + p.kv_heads; h += 8) {
        const bool query = h < p.heads;
        const int at = (query ? h : h - p.heads) * p.dim;
        const T* src = (query ? q : k) + at;
        T* dst = (query ? q_out : ring_k) + at;
        const bf16* w = as_bf16(query ? p.q_norm : p.k_norm) + (p.norm == QD_NORM_ROW ? at : 0);
        float r = query ? qr : kr;
        if (p.norm == QD_NORM_HEAD) {
            float ss = 0.f;
            for (int d = lane * 4; d < p.dim; d += 128) ss = squares(load4(src + d), ss);
            r = 1.0f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
        }
        for (int d = lane * 4; d < p.dim; d += 128) {
            float4 x = load4(src + d);
            if (p.norm != QD_NORM_NONE) {
                const float4 g = load4(w + d);
                x.x *= r * g.x; x.y *= r * g.y; x.z *= r * g.z; x.w *= r * g.w;
            }
            if (d < p.rot) {
                const int i = d >> 1;
                x = make_float4(fmaf(x.x, trig[i], -x.y * trig[half + i]), fmaf(x.y, trig[i], x.x * trig[half + i]),
                                fmaf(x.z, trig[i + 1], -x.w * trig[half + i + 1]), fmaf(x.w, trig[i + 1], x.z * trig[half + i + 1]));
            }
            store4(dst + d, x);
        }
    }
    for (int i = tid * 4; i < vn; i += 1024) store4(ring_v + i, load4(v + i));
}

// ----------------------------------------------------------------------------- any type, any shape
constexpr int kRowsPerLane = 8;                        // value columns per lane: 256 per block column

template <typename T>
QD_DEVINL void add_dot(const T* q, const T* k, int n, float (&dot)[4]) {
    int d = 0;
    for (; d + 4 <= n; d += 4)
#pragma unroll
        for (int i = 0; i < 4; ++i) dot[i] = fmaf(load_f(q + d + i), load_f(k + d + i), dot[i]);
    for (; d < n; ++d) dot[0] = fmaf(load_f(q + d), load_f(k + d), dot[0]);
}

template <typename T>
__global__ void __launch_bounds__(256) attn_rows_kernel(const __grid_constant__ AttnParams p) {
    chain_enter();
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31, c0 = blockIdx.y * 32 * kRowsPerLane + lane;
    if (item >= (long long)p.tokens * p.heads) return;
    const int t = (int)(item / p.heads), h = (int)(item % p.heads), g = h / (p.heads / p.kv_heads);
    const int position = (p.position_ptr ? *p.position_ptr : p.position) + t, lo = lowest_key(p, position);
    const T* q = reinterpret_cast<const T*>(p.q_rows) + item * (p.dim + p.shared_dim);
    const T* kc = reinterpret_cast<const T*>(p.k_cache) + g * p.dim;
    const T* vc = reinterpret_cast<const T*>(p.v_cache) + g * p.vdim;
    const T* common = reinterpret_cast<const T*>(p.k_shared);
    const float slope = p.slopes ? p.slopes[h] : 0.f;
    // the sink is the first term of the running softmax
    float m = -INFINITY, l = 0.f, acc[kRowsPerLane];
    if (p.sink_kind != QD_SINK_NONE) { m = p.sink_kind == QD_SINK_LEARNED ? ld_bf16(as_bf16(p.sink) + h) : 0.f; l = 1.f; }
#pragma unroll
    for (int c = 0; c < kRowsPerLane; ++c) acc[c] = 0.f;
    for (int j0 = lo; j0 <= position; j0 += 32) {
        const int j = j0 + lane;
        float score = -INFINITY;
        if (j <= position) {
            const size_t slot = j % p.capacity;
            float dot[4] = {0.f, 0.f, 0.f, 0.f};
            add_dot(q, kc + slot * p.ld_k, p.dim, dot);
            if (p.shared_dim) add_dot(q + p.dim, common + slot * p.ld_shared, p.shared_dim, dot);
            score = ((dot[0] + dot[1]) + (dot[2] + dot[3])) * p.scale - slope * (float)(position - j);
        }
        const float top = fmaxf(m, warp_max(score)), keep = expf(m - top), w = j <= position ? expf(score - top) : 0.f;
        l = l * keep + warp_sum(w);
        m = top;
#pragma unroll
        for (int c = 0; c < kRowsPerLane; ++c) acc[c] *= keep;
        const int count = min(32, position - j0 + 1);
        for (int i = 0; i < count; ++i) {
            const float wi = __shfl_sync(0xffffffffu, w, i);
            const T* v = vc + (size_t)((j0 + i) % p.capacity) * p.ld_v;
#pragma unroll
            for (int c = 0; c < kRowsPerLane; ++c)
                if (c0 + c * 32 < p.vdim) acc[c] = fmaf(wi, load_f(v + c0 + c * 32), acc[c]);
        }
    }
    const T* gate = reinterpret_cast<const T*>(p.gate) + (long long)t * p.ld_gate;
    const float f = (p.gate_kind == QD_GATE_HEAD ? sigmoid_precise(load_f(gate + h)) : 1.f) / l;
    T* out = reinterpret_cast<T*>(p.out) + item * p.vdim;
#pragma unroll
    for (int c = 0; c < kRowsPerLane; ++c) {
        const int column = c0 + c * 32;
        if (column >= p.vdim) continue;
        const float g2 = p.gate_kind == QD_GATE_VALUE ? sigmoid_precise(load_f(gate + h * p.vdim + column)) : 1.f;
        store_f(out + column, acc[c] * f * g2);
    }
}

// ------------------------------------------------------------------------------- tensor cores
constexpr int kFlashKeys = 64;
template <int DV> size_t flash_smem(const qd_attention_args& p, int warps) {
    const int krow = ((p.dim + p.shared_dim + 15) & ~15) + 8;
    return sizeof(bf16) * ((size_t)(warps * 16 + 2 * kFlashKeys) * krow + 2ull * kFlashKeys * (DV + 8));
}

// dim, shared_dim, vdim and the row strides multiples of eight, vdim <= DV (a multiple of sixteen).  Shared rows are padded to an odd
// number of 16-byte pieces: the eight rows an ldmatrix phase touches fall into different banks.
template <int DV, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) attn_flash_kernel(const __grid_constant__ AttnParams p) {
    chain_enter();
    extern __shared__ __align__(16) bf16 tiles[];
    constexpr int kVRow = DV + 8, kFlashRows = WARPS * 16, kFlashThreads = WARPS * 32;
    const int qdim = p.dim + p.shared_dim, dk = (qdim + 15) & ~15, krow = dk + 8;
    bf16* qs = tiles;
    bf16* ks = qs + kFlashRows * krow;
    bf16* vs = ks + 2 * kFlashKeys * krow;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int share = p.heads / p.kv_heads, g = blockIdx.y, total = p.tokens * share;
    const int r0 = blockIdx.x * kFlashRows;
    const int base = p.position_ptr ? *p.position_ptr : p.position;
    const int pos_first = base + r0 / share, pos_last = base + (min(r0 + kFlashRows, total) - 1) / share;
    const int key_first = lowest_key(p, pos_first);
    const int ntiles = (pos_last - key_first) / kFlashKeys + 1;
    const bf16* kc = as_bf16(p.k_cache) + g * p.dim;
    const bf16* vc = as_bf16(p.v_cache) + g * p.vdim;
    const bf16* common = as_bf16(p.k_shared);
    const bf16* q = as_bf16(p.q_rows);

    // padding columns stay zero
    const int all = (kFlashRows + 2 * kFlashKeys) * krow + 2 * kFlashKeys * kVRow;
    for (int i = tid; i < all / 8; i += kFlashThreads) reinterpret_cast<uint4*>(tiles)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    const int kp = p.dim / 8, qp = qdim / 8, vp = p.vdim / 8;          // 16-byte pieces
    for (int r = warp; r < kFlashRows; r += WARPS) {
        const int row = r0 + r;
        const bool ok = row < total;
        const bf16* src = q + (ok ? ((size_t)(row / share) * p.heads + g * share + row % share) * qdim : 0);
        for (int piece = lane; piece < qp; piece += 32) copy16_or_zero(qs + r * krow + piece * 8, src + piece * 8, ok);
    }
    const int slot_first = key_first % p.capacity;
    auto stage = [&](int tile) {
        const int j0 = key_first + tile * kFlashKeys;
        bf16* kd = ks + (tile & 1) * kFlashKeys * krow;
        bf16* vd = vs + (tile & 1) * kFlashKeys * kVRow;
        for (int r = warp; r < kFlashKeys; r += WARPS) {          // a warp per row
            const int j = j0 + r;
            const bool ok = j <= pos_last;
            int slot = ok ? slot_first + (j - key_first) : 0;
            if (slot >= p.capacity) slot -= p.capacity;           // what a block sees fits the ring
            const bf16* own = kc + slot * p.ld_k;
            const bf16* shared_row = common + slot * p.ld_shared - p.dim;
            const bf16* value = vc + slot * p.ld_v;
            for (int piece = lane; piece < qp + vp; piece += 32) {
                if (piece < kp) copy16_or_zero(kd + r * krow + piece * 8, own + piece * 8, ok);
                else if (piece < qp) copy16_or_zero(kd + r * krow + piece * 8, shared_row + piece * 8, ok);
                else copy16_or_zero(vd + r * kVRow + (piece - qp) * 8, value + (piece - qp) * 8, ok);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0);

    float o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) o[n][c] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const int row_of[2] = {r0 + warp * 16 + (lane >> 2), r0 + warp * 16 + (lane >> 2) + 8};
    const int pos_of[2] = {base + row_of[0] / share, base + row_of[1] / share};
    const int lo_of[2] = {lowest_key(p, pos_of[0]), lowest_key(p, pos_of[1])}, lo_last = lowest_key(p, pos_last);
    const float scale = p.scale * kLog2e;
    float slope[2] = {0.f, 0.f};
    if (p.slopes)
#pragma unroll
        for (int i = 0; i < 2; ++i) slope[i] = p.slopes[g * share + row_of[i] % share] * kLog2e;
    // ldmatrix addresses: lane -> (row within 16, 8-column half)
    const bf16* qa = qs + (warp * 16 + (lane & 15)) * krow + (lane >> 4) * 8;
    const int kb = ((lane & 7) + ((lane >> 4) << 3)) * krow + ((lane >> 3) & 1) * 8;
    const int vb = (lane & 15) * kVRow + (lane >> 4) * 8;

    for (int tile = 0; tile < ntiles; ++tile) {
        if (tile + 1 < ntiles) { stage(tile + 1); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const bf16* kt = ks + (tile & 1) * kFlashKeys * krow;
        const bf16* vt = vs + (tile & 1) * kFlashKeys * kVRow;
        const int j0 = key_first + tile * kFlashKeys;
        float s[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[n][c] = 0.f;
        for (int d = 0; d < dk; d += 16) {
            uint32_t a[4];
            ldmatrix4(a, qa + d);
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                uint32_t b[4];
                ldmatrix4(b, kt + n * 16 * krow + kb + d);
                mma_16816(s[2 * n], a, b[0], b[1]);
                mma_16816(s[2 * n + 1], a, b[2], b[3]);
            }
        }
        // every key of the tile visible to every row: no masking
        const bool inside = j0 + kFlashKeys - 1 <= pos_first && j0 >= lo_last;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int j = j0 + n * 8 + (lane & 3) * 2 + (c & 1), pos = pos_of[c >> 1];
                s[n][c] = (inside || (j <= pos && j >= lo_of[c >> 1])) ? fmaf(s[n][c], scale, slope[c >> 1] * (float)(j - pos)) : -INFINITY;
                mx[c >> 1] = fmaxf(mx[c >> 1], s[n][c]);
            }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
            const float top = fmaxf(m[i], mx[i]);
            const float keep = top == -INFINITY ? 1.f : exp2f(m[i] - top);
            m[i] = top;
            l[i] *= keep;
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) { o[n][2 * i] *= keep; o[n][2 * i + 1] *= keep; }
        }
        const float sub[2] = {m[0] == -INFINITY ? 0.f : m[0], m[1] == -INFINITY ? 0.f : m[1]};
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                s[n][c] = exp2f(s[n][c] - sub[c >> 1]);
                l[c >> 1] += s[n][c];
            }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float p0 = s[2 * kk + (x >> 1)][(x & 1) * 2], p1 = s[2 * kk + (x >> 1)][(x & 1) * 2 + 1];
                hi[x] = pack_pair(p0, p1);
                lo[x] = pack_pair(p0 - __uint_as_float(hi[x] << 16), p1 - __uint_as_float(hi[x] & 0xffff0000u));
            }
#pragma unroll
            for (int n = 0; n < DV / 16; ++n) {
                uint32_t b[4];
                ldmatrix4_t(b, vt + kk * 16 * kVRow + vb + n * 16);
                mma_16816(o[2 * n], hi, b[0], b[1]);
                mma_16816(o[2 * n + 1], hi, b[2], b[3]);
                mma_16816(o[2 * n], lo, b[0], b[1]);
                mma_16816(o[2 * n + 1], lo, b[2], b[3]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        if (row_of[i] >= total) continue;
        const int t = row_of[i] / share, h = g * share + row_of[i] % share;
        const bf16* gate = as_bf16(p.gate) + (long long)t * p.ld_gate;
        float f = 1.f / l[i];
        if (p.sink_kind != QD_SINK_NONE) {
            const float sink = p.sink_kind == QD_SINK_LEARNED ? ld_bf16(as_bf16(p.sink) + h) * kLog2e : 0.f;
            const float top = fmaxf(m[i], sink), keep = exp2f(m[i] - top);
            f = keep / (l[i] * keep + exp2f(sink - top));
        }
        if (p.gate_kind == QD_GATE_HEAD) f *= sigmoid_precise(ld_bf16(gate + h));
        bf16* out = reinterpret_cast<bf16*>(p.out) + ((size_t)t * p.heads + h) * p.vdim + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n)
            if (n * 8 < p.vdim) {
                float a = o[n][2 * i] * f, b = o[n][2 * i + 1] * f;
                if (p.gate_kind == QD_GATE_VALUE) {
                    const bf16* z = gate + h * p.vdim + (lane & 3) * 2 + n * 8;
                    a *= sigmoid_precise(ld_bf16(z));
                    b *= sigmoid_precise(ld_bf16(z + 1));
                }
                *reinterpret_cast<uint32_t*>(out + n * 8) = pack_pair(a, b);
            }
    }
}

// ------------------------------------------------------------------------------------- decode
constexpr int kStepKeys = 64, kStepThreads = 256;

struct AttnStep { AttnParams a; int buffers; };      // buffers: key tiles in shared memory, 1 or 2
__host__ __device__ constexpr size_t step_stats_floats(int heads, int splits) { return (2 * (size_t)heads * splits + 3) / 4 * 4; }

// Elements of a shared row of n elements: 16-byte pieces, an odd number of them (rows read side by side
// then start in different banks).
template <typename T> __host__ __device__ constexpr int step_row(int n) {
    const int e = 16 / (int)sizeof(T), pieces = (n + e - 1) / e;
    return (pieces | 1) * e;
}

// dots of two query heads (fp32 rows) with one key row; n a multiple of a 16-byte piece where `pieces`
template <typename T>
QD_DEVINL void dot_rows2(const float* q0, const float* q1, const T* k, int n, bool pieces, float& d0, float& d1) {
    float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
    if (pieces) {
        constexpr int E = 16 / (int)sizeof(T);
#pragma unroll 2
        for (int d = 0; d < n; d += E) {
            float kv[8];
            if (sizeof(T) == 2) unpack8(*reinterpret_cast<const uint4*>(k + d), kv);
            else { const float4 x = *reinterpret_cast<const float4*>(k + d); kv[0] = x.x; kv[1] = x.y; kv[2] = x.z; kv[3] = x.w; }
#pragma unroll
            for (int i = 0; i < E; i += 4) {
                const float4 x = load4(q0 + d + i), y = load4(q1 + d + i);
                a[0] = fmaf(x.x, kv[i], a[0]); a[1] = fmaf(x.y, kv[i + 1], a[1]); a[2] = fmaf(x.z, kv[i + 2], a[2]); a[3] = fmaf(x.w, kv[i + 3], a[3]);
                b[0] = fmaf(y.x, kv[i], b[0]); b[1] = fmaf(y.y, kv[i + 1], b[1]); b[2] = fmaf(y.z, kv[i + 2], b[2]); b[3] = fmaf(y.w, kv[i + 3], b[3]);
            }
        }
    } else {
        for (int d = 0; d < n; ++d) {
            const float kv = load_f(k + d);
            a[d & 3] = fmaf(q0[d], kv, a[d & 3]);
            b[d & 3] = fmaf(q1[d], kv, b[d & 3]);
        }
    }
    d0 = (a[0] + a[1]) + (a[2] + a[3]);
    d1 = (b[0] + b[1]) + (b[2] + b[3]);
}

// shared memory of attn_step_kernel
template <typename T>
static size_t step_smem(int share, int dim, int vdim, int rot, int buffers) {
    const int dp = step_row<float>(dim), vp = step_row<float>(vdim);
    return sizeof(float) * ((size_t)share * dp + (size_t)share * vp + share * (kStepKeys + 4)) +
           sizeof(T) * (size_t)(buffers * kStepKeys) * (step_row<T>(dim) + step_row<T>(vdim)) + sizeof(float) * (rot + 4);
}

template <typename T>
__global__ void __launch_bounds__(kStepThreads) attn_step_kernel(const __grid_constant__ AttnStep sp) {
    chain_enter();
    const AttnParams& p = sp.a;
    extern __shared__ __align__(16) float shared[];
    __shared__ float red[33];
    __shared__ bool last;
    const int share = p.heads / p.kv_heads, g = blockIdx.x, split = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dim = p.dim, vdim = p.vdim, dp = step_row<float>(dim), vp = step_row<float>(vdim), half = p.rot / 2;
    const int krow = step_row<T>(dim), vrow = step_row<T>(vdim);
    float* qs = shared;                                   // [share][dp]
    float* acc = qs + share * dp;                         // [share][vp]
    float* score = acc + share * vp;                      // [share][kStepKeys]
    float* stat = score + share * kStepKeys;              // maximum, denominator, rescaling factor per head (four floats)
    T* ks = reinterpret_cast<T*>(stat + share * 4);       // buffers of [kStepKeys][krow]
    T* vs = ks + sp.buffers * kStepKeys * krow;           // buffers of [kStepKeys][vrow]
    float* trig = reinterpret_cast<float*>(vs + sp.buffers * kStepKeys * vrow);
    const int position = p.position_ptr ? *p.position_ptr : p.position, lo = lowest_key(p, position), n = position - lo + 1;
    const int per = max((n + p.splits - 1) / p.splits, 32), active = (n + per - 1) / per;
    if (split >= active) return;
    const int first = lo + split * per, end = min(first + per, position + 1);
    const int qn = p.heads * dim, kn = p.kv_heads * dim;
    T* kc = reinterpret_cast<T*>(p.k_cache) + g * dim;
    T* vc = reinterpret_cast<T*>(p.v_cache) + g * vdim;

    // a warp per cache row; the token's own row is not in the ring yet
    constexpr int E = 16 / (int)sizeof(T);
    const bool pieces = dim % E == 0 && vdim % E == 0 && p.ld_k % E == 0 && p.ld_v % E == 0;
    auto stage = [&](int j0) {
        const int buf = ((j0 - first) / kStepKeys) & (sp.buffers - 1), count = min(kStepKeys, end - j0);
        T* kd = ks + buf * kStepKeys * krow;
        T* vd = vs + buf * kStepKeys * vrow;
        for (int r = warp; r < count; r += kStepThreads / 32) {
            const int j = j0 + r;
            if (j == position) continue;
            const T* krow_of = kc + (size_t)(j % p.capacity) * p.ld_k;
            const T* vrow_of = vc + (size_t)(j % p.capacity) * p.ld_v;
            if (pieces) {
                const int kp = dim / E, all = kp + vdim / E;
                for (int i = lane; i < all; i += 32) {
                    if (i < kp) copy16_or_zero(kd + r * krow + i * E, krow_of + i * E, true);
                    else copy16_or_zero(vd + r * vrow + (i - kp) * E, vrow_of + (i - kp) * E, true);
                }
            } else {
                for (int d = lane; d < dim; d += 32) kd[r * krow + d] = krow_of[d];
                for (int d = lane; d < vdim; d += 32) vd[r * vrow + d] = vrow_of[d];
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(first);

    const T* q = reinterpret_cast<const T*>(p.q);
    const T* k = reinterpret_cast<const T*>(p.k);
    const T* v = reinterpret_cast<const T*>(p.v) + g * vdim;
    for (int i = tid; i < half; i += kStepThreads) rotation(position, p.freq[i], p.freq[half + i], trig[i], trig[half + i]);
    float qr = 1.f, kr = 1.f;
    if (p.norm == QD_NORM_ROW) {
        float qq = 0.f, kk = 0.f;
        for (int i = tid; i < qn; i += kStepThreads) { const float x = load_f(q + i); qq = fmaf(x, x, qq); }
        for (int i = tid; i < kn; i += kStepThreads) { const float x = load_f(k + i); kk = fmaf(x, x, kk); }
        qr = 1.0f / sqrtf(block_sum(qq, red) / (float)qn + p.eps);
        kr = 1.0f / sqrtf(block_sum(kk, red) / (float)kn + p.eps);
    } else {
        if (p.norm == QD_NORM_HEAD && end == position + 1) {
            float kk = 0.f;
            for (int d = tid; d < dim; d += kStepThreads) { const float x = load_f(k + g * dim + d); kk = fmaf(x, x, kk); }
            kr = 1.0f / sqrtf(block_sum(kk, red) / (float)dim + p.eps);
        }
        __syncthreads();                                  // the rotation table
    }
    for (int h = warp; h < share; h += kStepThreads / 32) {
        const int at = (g * share + h) * dim;
        float r = qr;
        if (p.norm == QD_NORM_HEAD) {
            float qq = 0.f;
            for (int d = lane; d < dim; d += 32) { const float x = load_f(q + at + d); qq = fmaf(x, x, qq); }
            r = 1.0f / sqrtf(warp_sum(qq) / (float)dim + p.eps);
        }
        for (int d = lane; d < dim; d += 32) qs[h * dp + d] = as_type<T>(rotated(q, as_bf16(p.q_norm), p.norm, r, at, d, p.rot, trig, trig + half));
    }
    for (int i = tid; i < share * vp; i += kStepThreads) acc[i] = 0.f;
    for (int i = tid; i < share; i += kStepThreads) { stat[i * 4] = -INFINITY; stat[i * 4 + 1] = 0.f; }
    if (end == position + 1) {                            // this split holds the token itself: into its tile and into the ring
        const size_t slot = position % p.capacity;
        const int r = (position - first) % kStepKeys, buf = ((position - first) / kStepKeys) & (sp.buffers - 1);
        T* kd = ks + (size_t)(buf * kStepKeys + r) * krow;
        T* vd = vs + (size_t)(buf * kStepKeys + r) * vrow;
        for (int d = tid; d < dim; d += kStepThreads) {
            store_f(kc + slot * p.ld_k + d, rotated(k, as_bf16(p.k_norm), p.norm, kr, g * dim, d, p.rot, trig, trig + half));
            if (position - first < kStepKeys * sp.buffers) kd[d] = kc[slot * p.ld_k + d];
        }
        for (int d = tid; d < vdim; d += kStepThreads) {
            vc[slot * p.ld_v + d] = v[d];
            if (position - first < kStepKeys * sp.buffers) vd[d] = v[d];
        }
    }

    const bool quads = (vdim & 3) == 0;
    for (int j0 = first; j0 < end; j0 += kStepKeys) {
        const int buf = ((j0 - first) / kStepKeys) & (sp.buffers - 1), count = min(kStepKeys, end - j0);
        T* kt = ks + buf * kStepKeys * krow;
        T* vt = vs + buf * kStepKeys * vrow;
        if (sp.buffers == 2 && j0 + kStepKeys < end) { stage(j0 + kStepKeys); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        if (position < j0 + kStepKeys && position >= j0 && position - first >= kStepKeys * sp.buffers) {      // its buffer was busy before
            const size_t slot = position % p.capacity;
            const int r = position - j0;
            for (int d = tid; d < dim; d += kStepThreads) kt[r * krow + d] = kc[slot * p.ld_k + d];
            for (int d = tid; d < vdim; d += kStepThreads) vt[r * vrow + d] = v[d];
        }
        __syncthreads();
        {       // a thread's key against two heads at a time
            constexpr int kGroups = kStepThreads / kStepKeys;
            const int r = tid % kStepKeys;
            for (int h = tid / kStepKeys; h < share; h += 2 * kGroups) {
                const int h2 = min(h + kGroups, share - 1);
                float d0 = -INFINITY, d1 = -INFINITY;
                if (r < count) {
                    dot_rows2(qs + h * dp, qs + h2 * dp, kt + r * krow, dim, pieces, d0, d1);
                    d0 *= p.scale;
                    d1 *= p.scale;
                    if (p.slopes) {
                        const float distance = (float)(position - j0 - r);
                        d0 = fmaf(-p.slopes[g * share + h], distance, d0);
                        d1 = fmaf(-p.slopes[g * share + h2], distance, d1);
                    }
                }
                score[h * kStepKeys + r] = d0;
                if (h + kGroups < share) score[h2 * kStepKeys + r] = d1;
            }
        }
        __syncthreads();
        for (int h = warp; h < share; h += kStepThreads / 32) {
            float* row = score + h * kStepKeys;
            const float a = row[lane], b = row[lane + 32];
            const float m = stat[h * 4], top = fmaxf(m, warp_max(fmaxf(a, b)));
            const float wa = expf(a - top), wb = expf(b - top);
            const float sum = warp_sum(wa + wb);
            row[lane] = wa;
            row[lane + 32] = wb;
            __syncwarp();
            if (lane == 0) {
                const float keep = expf(m - top);
                stat[h * 4] = top;
                stat[h * 4 + 1] = stat[h * 4 + 1] * keep + sum;
                stat[h * 4 + 2] = keep;
            }
        }
        __syncthreads();
        if (quads) {
            for (int i = tid; i < share * (vdim / 4); i += kStepThreads) {
                const int h = i / (vdim / 4), c = i % (vdim / 4) * 4;
                const float keep = stat[h * 4 + 2];
                float4 a = load4(acc + h * vp + c);
                a.x *= keep; a.y *= keep; a.z *= keep; a.w *= keep;
                const float* w = score + h * kStepKeys;
#pragma unroll 8
                for (int r = 0; r < count; ++r) {
                    const float4 v4 = load4(vt + r * vrow + c);
                    a.x = fmaf(w[r], v4.x, a.x); a.y = fmaf(w[r], v4.y, a.y); a.z = fmaf(w[r], v4.z, a.z); a.w = fmaf(w[r], v4.w, a.w);
                }
                store4(acc + h * vp + c, a);
            }
        } else {
            for (int i = tid; i < share * vdim; i += kStepThreads) {
                const int h = i / vdim, c = i % vdim;
                float a = acc[h * vp + c] * stat[h * 4 + 2];
                const float* w = score + h * kStepKeys;
                for (int r = 0; r < count; ++r) a = fmaf(w[r], load_f(vt + r * vrow + c), a);
                acc[h * vp + c] = a;
            }
        }
        __syncthreads();
        if (sp.buffers == 1 && j0 + kStepKeys < end) stage(j0 + kStepKeys);
    }

    // partial results: (maximum, denominator) [head][split], then sums [head][split][vdim]; the last split of this
    // key/value head to arrive merges them
    float2* stats = reinterpret_cast<float2*>(p.partial) + (size_t)g * share * p.splits;
    float* sums = p.partial + step_stats_floats(p.heads, p.splits) + (size_t)g * share * p.splits * vdim;
    for (int i = tid; i < share * vdim; i += kStepThreads) {
        const int h = i / vdim, c = i % vdim;
        sums[((size_t)h * p.splits + split) * vdim + c] = acc[h * vp + c];
    }
    for (int h = tid; h < share; h += kStepThreads) stats[h * p.splits + split] = make_float2(stat[h * 4], stat[h * 4 + 1]);
    __threadfence();
    __syncthreads();
    if (tid == 0) last = atomicAdd(p.counters + g, 1u) == (unsigned)active - 1u;
    __syncthreads();
    if (!last) return;
    __threadfence();
    if (tid == 0) p.counters[g] = 0u;
    // factor of every split (sink, denominator and gate included) into the score rows, then the weighted sums
    for (int h = warp; h < share; h += kStepThreads / 32) {
        const int head = g * share + h;
        const float sink = p.sink_kind == QD_SINK_NONE ? -INFINITY : (p.sink_kind == QD_SINK_LEARNED ? ld_bf16(as_bf16(p.sink) + head) : 0.f);
        float2 mine[kStepKeys / 32];
        float top = sink, sum = 0.f;
#pragma unroll
        for (int i = 0; i < kStepKeys / 32; ++i) {
            const int s = i * 32 + lane;
            mine[i] = s < active ? __ldcg(stats + h * p.splits + s) : make_float2(-INFINITY, 0.f);
            top = fmaxf(top, mine[i].x);
        }
        top = warp_max(top);
#pragma unroll
        for (int i = 0; i < kStepKeys / 32; ++i) { mine[i].x = expf(mine[i].x - top); sum = fmaf(mine[i].y, mine[i].x, sum); }
        const float gate_of = p.gate_kind == QD_GATE_HEAD ? sigmoid_precise(load_f(reinterpret_cast<const T*>(p.gate) + head)) : 1.f;
        const float f = gate_of / (warp_sum(sum) + expf(sink - top));
#pragma unroll
        for (int i = 0; i < kStepKeys / 32; ++i) score[h * kStepKeys + i * 32 + lane] = mine[i].x * f;
    }
    __syncthreads();
    T* out = reinterpret_cast<T*>(p.out) + (size_t)g * share * vdim;
    const T* gate = reinterpret_cast<const T*>(p.gate) + (size_t)g * share * vdim;
    const auto value_gate = [&](int i) { return p.gate_kind == QD_GATE_VALUE ? sigmoid_precise(load_f(gate + i)) : 1.f; };
    if (quads) {
        for (int i = tid; i < share * (vdim / 4); i += kStepThreads) {
            const int h = i / (vdim / 4), c = i % (vdim / 4) * 4;
            const float* rows = sums + (size_t)h * p.splits * vdim + c;
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
            for (int s = 0; s < active; ++s) {
                const float4 x = __ldcg(reinterpret_cast<const float4*>(rows + (size_t)s * vdim));
                const float f = score[h * kStepKeys + s];
                o.x = fmaf(x.x, f, o.x); o.y = fmaf(x.y, f, o.y); o.z = fmaf(x.z, f, o.z); o.w = fmaf(x.w, f, o.w);
            }
            const int i0 = h * vdim + c;
            o.x *= value_gate(i0); o.y *= value_gate(i0 + 1); o.z *= value_gate(i0 + 2); o.w *= value_gate(i0 + 3);
            store4(out + i0, o);
        }
    } else {
        for (int i = tid; i < share * vdim; i += kStepThreads) {
            const int h = i / vdim, c = i % vdim;
            float o = 0.f;
            for (int s = 0; s < active; ++s) o = fmaf(__ldcg(sums + ((size_t)h * p.splits + s) * vdim + c), score[h * kStepKeys + s], o);
            store_f(out + h * vdim + c, o * value_gate(h * vdim + c));
        }
    }
}

template <int DV, int WARPS>
int launch_flash_rows(const AttnParams& p, long long rows, cudaStream_t s) {
    const dim3 grid((unsigned)((rows + WARPS * 16 - 1) / (WARPS * 16)), p.kv_heads);
    const size_t smem = flash_smem<DV>(p, WARPS);
    if (!allow_smem(attn_flash_kernel<DV, WARPS>, smem)) return QD_ERR_UNSUPPORTED;
    return qd_launch(attn_flash_kernel<DV, WARPS>, grid, dim3(WARPS * 32), smem, s, 1, p);
}
template <int DV>
int launch_flash(const AttnParams& p, cudaStream_t s) {
    const long long rows = (long long)p.tokens * (p.heads / p.kv_heads);
    // 128 rows share a key tile once such blocks fill the GPU
    if (rows * p.kv_heads >= 128ll * device_sms() && flash_smem<DV>(p, 8) <= kMaxSmem) return launch_flash_rows<DV, 8>(p, rows, s);
    return launch_flash_rows<DV, 4>(p, rows, s);
}
template <typename T>
int chunk(const AttnParams& p, cudaStream_t s) {
    if (p.q) {
        const size_t shared = (size_t)(p.rot + p.heads + p.kv_heads + 1) * 4;
        if (!allow_smem(attn_prepare_kernel<T>, shared)) return QD_ERR_UNSUPPORTED;
        const bool quads = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.rot % 4 == 0 && p.ld % 4 == 0 && p.ld_k % 4 == 0 && p.ld_v % 4 == 0 && aligned16(p.q) &&
                           aligned16(p.k) && aligned16(p.v) && aligned16(p.q_norm) && aligned16(p.k_norm) && aligned16(p.k_cache) &&
                           aligned16(p.v_cache) && aligned16(p.q_rows);
        const int rc = quads ? qd_launch(attn_prepare_vec_kernel<T>, dim3(p.tokens), dim3(256), (size_t)(p.rot + 1) * 4, s, 1, p)
                             : qd_launch(attn_prepare_kernel<T>, dim3(p.tokens), dim3(256), shared, s, 1, p);
        if (rc != QD_OK) return rc;
    }
    const bool rows16 = sizeof(T) == 2 && p.dim % 8 == 0 && p.vdim % 8 == 0 && p.shared_dim % 8 == 0 && p.ld_k % 8 == 0 && p.ld_v % 8 == 0 &&
                        p.ld_shared % 8 == 0 && aligned16(p.q_rows) && aligned16(p.k_cache) && aligned16(p.v_cache) && aligned16(p.k_shared) &&
                        ((uintptr_t)p.out & 3u) == 0;
    if (rows16 && p.vdim <= 256 && flash_smem<256>(p, 4) <= kMaxSmem) {
        if (p.vdim <= 32) return launch_flash<32>(p, s);
        if (p.vdim <= 64) return launch_flash<64>(p, s);
        if (p.vdim <= 96) return launch_flash<96>(p, s);
        if (p.vdim <= 128) return launch_flash<128>(p, s);
        if (p.vdim <= 192) return launch_flash<192>(p, s);
        return launch_flash<256>(p, s);
    }
    const dim3 grid((unsigned)(((long long)p.tokens * p.heads + 7) / 8), (p.vdim + 32 * kRowsPerLane - 1) / (32 * kRowsPerLane));
    return qd_launch(attn_rows_kernel<T>, grid, dim3(256), 0, s, 1, p);
}
template <typename T>
int step(const AttnParams& a, cudaStream_t s) {
    AttnStep sp = {a, 2};
    const auto smem = [&] { return step_smem<T>(a.heads / a.kv_heads, a.dim, a.vdim, a.rot, sp.buffers); };
    if (smem() > 220 * 1024) sp.buffers = 1;
    if (smem() > kMaxSmem) return a.q_rows ? chunk<T>(a, s) : QD_ERR_UNSUPPORTED;      // very many heads to a key row
    if (!allow_smem(attn_step_kernel<T>, smem())) return QD_ERR_UNSUPPORTED;
    return qd_launch(attn_step_kernel<T>, dim3(a.kv_heads, a.splits), dim3(kStepThreads), smem(), s, 1, sp);
}

bool valid(const AttnParams& a) {
    const bool caches = a.k_cache && a.v_cache && a.out && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0 &&
                        a.span > 0 && a.position >= 0 && a.capacity > 0 && a.shared_dim >= 0 && (a.shared_dim == 0 || a.k_shared) &&
                        a.ld_k >= (long long)a.kv_heads * a.dim && a.ld_v >= (long long)a.kv_heads * a.vdim && a.ld_shared >= a.shared_dim;
    const bool extras = (a.sink_kind != QD_SINK_LEARNED || a.sink) && (a.gate_kind == QD_GATE_NONE || a.gate) &&
                        (a.mask == QD_MASK_WINDOW || a.mask == QD_MASK_CHUNK);
    if (!a.q) return caches && extras;
    return caches && extras && a.k && a.v && a.shared_dim == 0 && (a.norm == QD_NORM_NONE || (a.q_norm && a.k_norm)) && a.rot >= 0 && a.rot % 2 == 0 &&
           a.rot <= a.dim && (a.rot == 0 || (a.freq && a.dim % 2 == 0));
}

}  // namespace
}  // namespace qd

extern "C" int qd_attention(const qd_attention_args* args, void* stream) {
    QD_CHECK_ARG(args && qd::valid(*args) && args->tokens > 0 && args->q_rows);
    const qd_attention_args& a = *args;
    // a chunk's own rows must not push out rows that its first token still sees
    if ((long long)a.tokens + a.span - 1 > a.capacity && (a.position_ptr || (long long)a.position + a.tokens > a.capacity)) return QD_ERR_ARG;
    if (a.dtype == QD_BF16) return qd::chunk<bf16>(a, (cudaStream_t)stream);
    if (a.dtype == QD_F32) return qd::chunk<float>(a, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" long long qd_attention_step_floats(int heads, int vdim, int splits) {
    return (long long)qd::step_stats_floats(heads, splits) + (long long)heads * splits * vdim;
}

extern "C" int qd_attention_step(const qd_attention_args* args, void* stream) {
    QD_CHECK_ARG(args && qd::valid(*args) && args->q && args->partial && args->counters && args->capacity >= args->span);
    QD_CHECK_ARG(args->splits > 0 && args->splits <= qd::kStepKeys && qd::aligned16(args->partial));
    if (args->dtype == QD_BF16) return qd::step<bf16>(*args, (cudaStream_t)stream);
    if (args->dtype == QD_F32) return qd::step<float>(*args, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}
