// Sliding-window attention with a learned sink per head in the softmax's denominator, RMS norm over the
// whole query / key projection, interleaved rotary positions, and one sigmoid output gate per head.
// The window's keys and values live in a ring of `capacity` rows (position p in row p mod capacity), so a
// sequence's cache does not grow with its length.
//
// Prompt chunks: attn_prepare_kernel (norm, rotation, ring rows) and attn_flash_kernel (mma.sync m16n8k16;
// 64 or 128 packed (token, head of the group) rows per block, key tiles of 64 through two cp.async buffers,
// only the tiles a row of the block can see; probabilities as two bf16 pieces).  attn_rows_kernel covers fp32
// and shapes without 16-byte rows.  Decode: attn_step_kernel, one launch: norm and rotation in every
// block, blocks = (key/value head, split of the window), the last block of a head merges.
#include "typed.cuh"

namespace qd {
namespace {

// Angle of a pair in fp32: position * (f_hi + f_lo) with the product's rounding error carried along, so
// that the rotation is that of the exact angle to fp32 rounding at any position.
QD_DEVINL void rotation(int position, float f_hi, float f_lo, float& c, float& s) {
    const float a = (float)position * f_hi;
    const float err = fmaf((float)position, f_hi, -a) + (float)position * f_lo;
    float c0, s0;
    sincosf(a, &s0, &c0);
    c = fmaf(-err, s0, c0);
    s = fmaf(err, c0, s0);
}

// normalised, rotated element e (within its head: d) of a projection row
template <typename T>
QD_DEVINL float rotated(const T* row, const bf16* w, float rms, int e, int d, int rot, const float* cosine, const float* sine) {
    const float x = load_f(row + e) * rms * ld_bf16(w + e);
    if (d >= rot) return x;
    const int i = d >> 1;
    const float other = load_f(row + (e ^ 1) + 0) * rms * ld_bf16(w + (e ^ 1));
    return (d & 1) ? fmaf(x, cosine[i], other * sine[i]) : fmaf(x, cosine[i], -other * sine[i]);
}

struct AttnParams {
    const void* q; const void* k; const void* v; const void* gate; long long ld;      // projection rows
    const bf16* q_norm; const bf16* k_norm; const float* freq; int rot;               // freq: [2][rot / 2], high and low parts
    const bf16* sink; float scale, eps;
    void* k_cache; void* v_cache; int capacity, window;
    const int* position_ptr; int position;
    void* q_out; void* out;
    int tokens, heads, kv_heads, dim, vdim;
};

template <typename T>
__global__ void __launch_bounds__(256) attn_prepare_kernel(const __grid_constant__ AttnParams p) {
    chain_enter();
    extern __shared__ float trig[];                    // cosines, sines
    __shared__ float red[33];
    const int t = blockIdx.x, tid = threadIdx.x, half = p.rot / 2;
    const int position = (p.position_ptr ? *p.position_ptr : p.position) + t;
    const int qn = p.heads * p.dim, kn = p.kv_heads * p.dim, vn = p.kv_heads * p.vdim;
    const T* q = reinterpret_cast<const T*>(p.q) + (long long)t * p.ld;
    const T* k = reinterpret_cast<const T*>(p.k) + (long long)t * p.ld;
    const T* v = reinterpret_cast<const T*>(p.v) + (long long)t * p.ld;
    for (int i = tid; i < half; i += 256) rotation(position, p.freq[i], p.freq[half + i], trig[i], trig[half + i]);
    float qq = 0.f, kk = 0.f;
    for (int i = tid; i < qn; i += 256) { const float x = load_f(q + i); qq = fmaf(x, x, qq); }
    for (int i = tid; i < kn; i += 256) { const float x = load_f(k + i); kk = fmaf(x, x, kk); }
    const float qr = 1.0f / sqrtf(block_sum(qq, red) / (float)qn + p.eps), kr = 1.0f / sqrtf(block_sum(kk, red) / (float)kn + p.eps);
    const size_t slot = position % p.capacity;
    T* ring_k = reinterpret_cast<T*>(p.k_cache) + slot * kn;
    T* ring_v = reinterpret_cast<T*>(p.v_cache) + slot * vn;
    T* q_out = reinterpret_cast<T*>(p.q_out) + (size_t)t * qn;
    for (int i = tid; i < qn; i += 256) store_f(q_out + i, rotated(q, p.q_norm, qr, i, i % p.dim, p.rot, trig, trig + half));
    for (int i = tid; i < kn; i += 256) store_f(ring_k + i, rotated(k, p.k_norm, kr, i, i % p.dim, p.rot, trig, trig + half));
    for (int i = tid; i < vn; i += 256) ring_v[i] = v[i];
}

// ----------------------------------------------------------------------------- any type, any shape
constexpr int kRowsPerLane = 8;                        // value columns per lane: vdim <= 256

template <typename T>
__global__ void __launch_bounds__(256) attn_rows_kernel(const __grid_constant__ AttnParams p) {
    chain_enter();
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (item >= (long long)p.tokens * p.heads) return;
    const int t = (int)(item / p.heads), h = (int)(item % p.heads), g = h / (p.heads / p.kv_heads);
    const int position = (p.position_ptr ? *p.position_ptr : p.position) + t, lo = max(0, position - p.window + 1);
    const T* q = reinterpret_cast<const T*>(p.q_out) + item * p.dim;
    const T* kc = reinterpret_cast<const T*>(p.k_cache);
    const T* vc = reinterpret_cast<const T*>(p.v_cache);
    const float sink = ld_bf16(p.sink + h);
    float m = sink, l = 1.f, acc[kRowsPerLane];        // the sink is the first term of the running softmax
#pragma unroll
    for (int c = 0; c < kRowsPerLane; ++c) acc[c] = 0.f;
    for (int j0 = lo; j0 <= position; j0 += 32) {
        const int j = j0 + lane;
        float score = -INFINITY;
        if (j <= position) {
            const T* k = kc + ((size_t)(j % p.capacity) * p.kv_heads + g) * p.dim;
            float dot[4] = {0.f, 0.f, 0.f, 0.f};
            int d = 0;
            for (; d + 4 <= p.dim; d += 4)
#pragma unroll
                for (int i = 0; i < 4; ++i) dot[i] = fmaf(load_f(q + d + i), load_f(k + d + i), dot[i]);
            for (; d < p.dim; ++d) dot[0] = fmaf(load_f(q + d), load_f(k + d), dot[0]);
            score = ((dot[0] + dot[1]) + (dot[2] + dot[3])) * p.scale;
        }
        const float top = fmaxf(m, warp_max(score)), keep = expf(m - top), w = j <= position ? expf(score - top) : 0.f;
        l = l * keep + warp_sum(w);
        m = top;
#pragma unroll
        for (int c = 0; c < kRowsPerLane; ++c) acc[c] *= keep;
        const int count = min(32, position - j0 + 1);
        for (int i = 0; i < count; ++i) {
            const float wi = __shfl_sync(0xffffffffu, w, i);
            const T* v = vc + ((size_t)((j0 + i) % p.capacity) * p.kv_heads + g) * p.vdim;
#pragma unroll
            for (int c = 0; c < kRowsPerLane; ++c)
                if (c * 32 + lane < p.vdim) acc[c] = fmaf(wi, load_f(v + c * 32 + lane), acc[c]);
        }
    }
    const float gate = sigmoid_precise(load_f(reinterpret_cast<const T*>(p.gate) + (long long)t * p.ld + h)) / l;
    T* out = reinterpret_cast<T*>(p.out) + item * p.vdim;
#pragma unroll
    for (int c = 0; c < kRowsPerLane; ++c)
        if (c * 32 + lane < p.vdim) store_f(out + c * 32 + lane, acc[c] * gate);
}

// ------------------------------------------------------------------------------- tensor cores
constexpr int kFlashKeys = 64;
constexpr float kLog2e = 1.4426950408889634f;

QD_DEVINL void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
QD_DEVINL void ldmatrix4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
QD_DEVINL void ldmatrix4_t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
QD_DEVINL void copy16_or_zero(void* dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
QD_DEVINL uint32_t pack_pair(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}

// dim, vdim multiples of eight, vdim <= DV (a multiple of sixteen).  Shared rows are padded to an odd
// number of 16-byte pieces: the eight rows an ldmatrix phase touches fall into different banks.
template <int DV, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) attn_flash_kernel(const __grid_constant__ AttnParams p) {
    chain_enter();
    extern __shared__ __align__(16) bf16 tiles[];
    constexpr int kVRow = DV + 8, kFlashRows = WARPS * 16, kFlashThreads = WARPS * 32;
    const int dk = (p.dim + 15) & ~15, krow = dk + 8;
    bf16* qs = tiles;
    bf16* ks = qs + kFlashRows * krow;
    bf16* vs = ks + 2 * kFlashKeys * krow;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int share = p.heads / p.kv_heads, g = blockIdx.y, total = p.tokens * share;
    const int r0 = blockIdx.x * kFlashRows;
    const int base = p.position_ptr ? *p.position_ptr : p.position;
    const int pos_first = base + r0 / share, pos_last = base + (min(r0 + kFlashRows, total) - 1) / share;
    const int key_first = max(0, pos_first - p.window + 1);
    const int ntiles = (pos_last - key_first) / kFlashKeys + 1;
    const bf16* kc = reinterpret_cast<const bf16*>(p.k_cache);
    const bf16* vc = reinterpret_cast<const bf16*>(p.v_cache);
    const bf16* q = reinterpret_cast<const bf16*>(p.q_out);

    // padding columns stay zero
    const int all = (kFlashRows + 2 * kFlashKeys) * krow + 2 * kFlashKeys * kVRow;
    for (int i = tid; i < all / 8; i += kFlashThreads) reinterpret_cast<uint4*>(tiles)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
    const int kp = p.dim / 8, vp = p.vdim / 8;
    for (int i = tid; i < kFlashRows * kp; i += kFlashThreads) {
        const int r = i / kp, piece = i % kp, row = r0 + r;
        const bool ok = row < total;
        const size_t src = ok ? ((size_t)(row / share) * p.heads + g * share + row % share) * p.dim + piece * 8 : 0;
        copy16_or_zero(qs + r * krow + piece * 8, q + src, ok);
    }
    auto stage = [&](int tile) {
        const int j0 = key_first + tile * kFlashKeys;
        bf16* kd = ks + (tile & 1) * kFlashKeys * krow;
        bf16* vd = vs + (tile & 1) * kFlashKeys * kVRow;
        for (int i = tid; i < kFlashKeys * (kp + vp); i += kFlashThreads) {
            const int r = i / (kp + vp), piece = i % (kp + vp), j = j0 + r;
            const bool ok = j <= pos_last;
            const size_t row = ok ? (size_t)(j % p.capacity) * p.kv_heads + g : 0;
            if (piece < kp) copy16_or_zero(kd + r * krow + piece * 8, kc + row * p.dim + piece * 8, ok);
            else copy16_or_zero(vd + r * kVRow + (piece - kp) * 8, vc + row * p.vdim + (piece - kp) * 8, ok);
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
    const float scale = p.scale * kLog2e;
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
        const bool inside = j0 + kFlashKeys - 1 <= pos_first && j0 > pos_last - p.window;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int j = j0 + n * 8 + (lane & 3) * 2 + (c & 1), pos = pos_of[c >> 1];
                s[n][c] = (inside || (j <= pos && j > pos - p.window)) ? s[n][c] * scale : -INFINITY;
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
        const float sink = ld_bf16(p.sink + h) * kLog2e, top = fmaxf(m[i], sink), keep = exp2f(m[i] - top);
        const float gate = sigmoid_precise(ld_bf16(reinterpret_cast<const bf16*>(p.gate) + (long long)t * p.ld + h));
        const float f = keep / (l[i] * keep + exp2f(sink - top)) * gate;
        bf16* out = reinterpret_cast<bf16*>(p.out) + ((size_t)t * p.heads + h) * p.vdim + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n)
            if (n * 8 < p.vdim) *reinterpret_cast<uint32_t*>(out + n * 8) = pack_pair(o[n][2 * i] * f, o[n][2 * i + 1] * f);
    }
}

// ------------------------------------------------------------------------------------- decode
constexpr int kStepKeys = 64, kStepThreads = 256;

struct AttnStep { AttnParams a; float* partial; unsigned int* counters; int splits, buffers; };      // buffers: key tiles in shared memory, 1 or 2
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
    const int position = p.position_ptr ? *p.position_ptr : p.position, lo = max(0, position - p.window + 1), n = position - lo + 1;
    const int per = max((n + sp.splits - 1) / sp.splits, 32), active = (n + per - 1) / per;
    if (split >= active) return;
    const int first = lo + split * per, end = min(first + per, position + 1);
    const int qn = p.heads * dim, kn = p.kv_heads * dim, vn = p.kv_heads * vdim;
    T* kc = reinterpret_cast<T*>(p.k_cache);
    T* vc = reinterpret_cast<T*>(p.v_cache);

    // a warp per cache row; the token's own row is not in the ring yet
    constexpr int E = 16 / (int)sizeof(T);
    const bool pieces = dim % E == 0 && vdim % E == 0;
    auto stage = [&](int j0) {
        const int buf = ((j0 - first) / kStepKeys) & (sp.buffers - 1), count = min(kStepKeys, end - j0);
        T* kd = ks + buf * kStepKeys * krow;
        T* vd = vs + buf * kStepKeys * vrow;
        for (int r = warp; r < count; r += kStepThreads / 32) {
            const int j = j0 + r;
            if (j == position) continue;
            const size_t row = (size_t)(j % p.capacity) * p.kv_heads + g;
            if (pieces) {
                const int kp = dim / E, all = kp + vdim / E;
                for (int i = lane; i < all; i += 32) {
                    if (i < kp) copy16_or_zero(kd + r * krow + i * E, kc + row * dim + i * E, true);
                    else copy16_or_zero(vd + r * vrow + (i - kp) * E, vc + row * vdim + (i - kp) * E, true);
                }
            } else {
                for (int d = lane; d < dim; d += 32) kd[r * krow + d] = kc[row * dim + d];
                for (int d = lane; d < vdim; d += 32) vd[r * vrow + d] = vc[row * vdim + d];
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(first);

    const T* q = reinterpret_cast<const T*>(p.q);
    const T* k = reinterpret_cast<const T*>(p.k);
    const T* v = reinterpret_cast<const T*>(p.v) + g * vdim;
    for (int i = tid; i < half; i += kStepThreads) rotation(position, p.freq[i], p.freq[half + i], trig[i], trig[half + i]);
    float qq = 0.f, kk = 0.f;
    for (int i = tid; i < qn; i += kStepThreads) { const float x = load_f(q + i); qq = fmaf(x, x, qq); }
    for (int i = tid; i < kn; i += kStepThreads) { const float x = load_f(k + i); kk = fmaf(x, x, kk); }
    const float qr = 1.0f / sqrtf(block_sum(qq, red) / (float)qn + p.eps), kr = 1.0f / sqrtf(block_sum(kk, red) / (float)kn + p.eps);
    for (int h = warp; h < share; h += kStepThreads / 32)
        for (int d = lane; d < dim; d += 32)
            qs[h * dp + d] = as_type<T>(rotated(q, p.q_norm, qr, (g * share + h) * dim + d, d, p.rot, trig, trig + half));
    for (int i = tid; i < share * vp; i += kStepThreads) acc[i] = 0.f;
    for (int i = tid; i < share; i += kStepThreads) { stat[i * 4] = -INFINITY; stat[i * 4 + 1] = 0.f; }
    if (end == position + 1) {                            // this split holds the token itself: into its tile and into the ring
        const size_t slot = position % p.capacity;
        const int r = (position - first) % kStepKeys, buf = ((position - first) / kStepKeys) & (sp.buffers - 1);
        T* kd = ks + (size_t)(buf * kStepKeys + r) * krow;
        T* vd = vs + (size_t)(buf * kStepKeys + r) * vrow;
        for (int d = tid; d < dim; d += kStepThreads) {
            store_f(kc + slot * kn + g * dim + d, rotated(k, p.k_norm, kr, g * dim + d, d, p.rot, trig, trig + half));
            if (position - first < kStepKeys * sp.buffers) kd[d] = kc[slot * kn + g * dim + d];
        }
        for (int d = tid; d < vdim; d += kStepThreads) {
            vc[slot * vn + g * vdim + d] = v[d];
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
            for (int d = tid; d < dim; d += kStepThreads) kt[r * krow + d] = kc[slot * kn + g * dim + d];
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
    float2* stats = reinterpret_cast<float2*>(sp.partial) + (size_t)g * share * sp.splits;
    float* sums = sp.partial + step_stats_floats(p.heads, sp.splits) + (size_t)g * share * sp.splits * vdim;
    for (int i = tid; i < share * vdim; i += kStepThreads) {
        const int h = i / vdim, c = i % vdim;
        sums[((size_t)h * sp.splits + split) * vdim + c] = acc[h * vp + c];
    }
    for (int h = tid; h < share; h += kStepThreads) stats[h * sp.splits + split] = make_float2(stat[h * 4], stat[h * 4 + 1]);
    __threadfence();
    __syncthreads();
    if (tid == 0) last = atomicAdd(sp.counters + g, 1u) == (unsigned)active - 1u;
    __syncthreads();
    if (!last) return;
    __threadfence();
    if (tid == 0) sp.counters[g] = 0u;
    // factor of every split (sink, denominator and gate included) into the score rows, then the weighted sums
    for (int h = warp; h < share; h += kStepThreads / 32) {
        const int head = g * share + h;
        const float sink = ld_bf16(p.sink + head);
        float2 mine[kStepKeys / 32];
        float top = sink, sum = 0.f;
#pragma unroll
        for (int i = 0; i < kStepKeys / 32; ++i) {
            const int s = i * 32 + lane;
            mine[i] = s < active ? __ldcg(stats + h * sp.splits + s) : make_float2(-INFINITY, 0.f);
            top = fmaxf(top, mine[i].x);
        }
        top = warp_max(top);
#pragma unroll
        for (int i = 0; i < kStepKeys / 32; ++i) { mine[i].x = expf(mine[i].x - top); sum = fmaf(mine[i].y, mine[i].x, sum); }
        const float f = sigmoid_precise(load_f(reinterpret_cast<const T*>(p.gate) + head)) / (warp_sum(sum) + expf(sink - top));
#pragma unroll
        for (int i = 0; i < kStepKeys / 32; ++i) score[h * kStepKeys + i * 32 + lane] = mine[i].x * f;
    }
    __syncthreads();
    T* out = reinterpret_cast<T*>(p.out) + (size_t)g * share * vdim;
    if (quads) {
        for (int i = tid; i < share * (vdim / 4); i += kStepThreads) {
            const int h = i / (vdim / 4), c = i % (vdim / 4) * 4;
            const float* rows = sums + (size_t)h * sp.splits * vdim + c;
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
            for (int s = 0; s < active; ++s) {
                const float4 x = __ldcg(reinterpret_cast<const float4*>(rows + (size_t)s * vdim));
                const float f = score[h * kStepKeys + s];
                o.x = fmaf(x.x, f, o.x); o.y = fmaf(x.y, f, o.y); o.z = fmaf(x.z, f, o.z); o.w = fmaf(x.w, f, o.w);
            }
            store4(out + h * vdim + c, o);
        }
    } else {
        for (int i = tid; i < share * vdim; i += kStepThreads) {
            const int h = i / vdim, c = i % vdim;
            float o = 0.f;
            for (int s = 0; s < active; ++s) o = fmaf(__ldcg(sums + ((size_t)h * sp.splits + s) * vdim + c), score[h * kStepKeys + s], o);
            store_f(out + h * vdim + c, o);
        }
    }
}

template <int DV, int WARPS>
int launch_flash_rows(const AttnParams& p, long long rows, cudaStream_t s) {
    const int krow = ((p.dim + 15) & ~15) + 8;
    const size_t smem = sizeof(bf16) * ((size_t)(WARPS * 16 + 2 * kFlashKeys) * krow + 2ull * kFlashKeys * (DV + 8));
    if (!allow_smem(attn_flash_kernel<DV, WARPS>, smem)) return QD_ERR_UNSUPPORTED;
    const dim3 grid((unsigned)((rows + WARPS * 16 - 1) / (WARPS * 16)), p.kv_heads);
    return qd_launch(attn_flash_kernel<DV, WARPS>, grid, dim3(WARPS * 32), smem, s, 1, p);
}
template <int DV>
int launch_flash(const AttnParams& p, cudaStream_t s) {
    const long long rows = (long long)p.tokens * (p.heads / p.kv_heads);
    // 128 rows share a key tile once such blocks fill the GPU
    if (rows * p.kv_heads >= 128ll * device_sms()) return launch_flash_rows<DV, 8>(p, rows, s);
    return launch_flash_rows<DV, 4>(p, rows, s);
}
template <typename T>
int chunk(const AttnParams& p, cudaStream_t s) {
    const size_t trig = (size_t)(p.rot + 1) * 4;
    if (!allow_smem(attn_prepare_kernel<T>, trig)) return QD_ERR_UNSUPPORTED;
    const int rc = qd_launch(attn_prepare_kernel<T>, dim3(p.tokens), dim3(256), trig, s, 1, p);
    if (rc != QD_OK) return rc;
    const bool rows16 = sizeof(T) == 2 && p.dim % 8 == 0 && p.vdim % 8 == 0 && aligned16(p.q_out) && aligned16(p.k_cache) && aligned16(p.v_cache);
    if (rows16 && p.dim <= 256 && p.vdim <= 256 && ((uintptr_t)p.out & 3u) == 0) {
        if (p.vdim <= 32) return launch_flash<32>(p, s);
        if (p.vdim <= 64) return launch_flash<64>(p, s);
        if (p.vdim <= 96) return launch_flash<96>(p, s);
        if (p.vdim <= 128) return launch_flash<128>(p, s);
        if (p.vdim <= 192) return launch_flash<192>(p, s);
        return launch_flash<256>(p, s);
    }
    if (p.vdim > 32 * kRowsPerLane) return QD_ERR_UNSUPPORTED;
    return qd_launch(attn_rows_kernel<T>, dim3((unsigned)(((long long)p.tokens * p.heads + 7) / 8)), dim3(256), 0, s, 1, p);
}
template <typename T>
int step(AttnStep sp, cudaStream_t s) {
    const auto smem = [&] { return step_smem<T>(sp.a.heads / sp.a.kv_heads, sp.a.dim, sp.a.vdim, sp.a.rot, sp.buffers); };
    sp.buffers = 2;
    if (smem() > 220 * 1024) sp.buffers = 1;
    if (!allow_smem(attn_step_kernel<T>, smem())) return QD_ERR_UNSUPPORTED;
    return qd_launch(attn_step_kernel<T>, dim3(sp.a.kv_heads, sp.splits), dim3(kStepThreads), smem(), s, 1, sp);
}

}  // namespace
}  // namespace qd

#define QD_ATTN_ARGS_OK(tokens_ok)                                                                                         \
    QD_CHECK_ARG(q && k && v && gate && q_norm && k_norm && sink && k_cache && v_cache && out && (tokens_ok));             \
    QD_CHECK_ARG(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0 && window > 0 && position >= 0); \
    QD_CHECK_ARG(rot >= 0 && rot % 2 == 0 && rot <= dim && (rot == 0 || (freq && dim % 2 == 0)) && capacity >= window)

extern "C" int qd_window_attention(const void* q, const void* k, const void* v, const void* gate, long long ld, const void* q_norm,
                                   const void* k_norm, const float* freq, int rot, const void* sink, float scale, float eps,
                                   void* k_cache, void* v_cache, int capacity, int window, const int* position_ptr, int position,
                                   void* q_scratch, void* out, int tokens, int heads, int kv_heads, int dim, int vdim, int dtype,
                                   void* stream) {
    QD_ATTN_ARGS_OK(tokens > 0 && q_scratch);
    // a chunk's own rows must not push out rows that its first token still sees
    if (tokens + window - 1 > capacity && (position_ptr || position + tokens > capacity)) return QD_ERR_ARG;
    const qd::AttnParams p = {q, k, v, gate, ld, (const bf16*)q_norm, (const bf16*)k_norm, freq, rot, (const bf16*)sink, scale, eps,
                              k_cache, v_cache, capacity, window, position_ptr, position, q_scratch, out, tokens, heads, kv_heads,
                              dim, vdim};
    if (dtype == QD_BF16) return qd::chunk<bf16>(p, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::chunk<float>(p, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}

extern "C" long long qd_window_attention_step_floats(int heads, int vdim, int splits) {
    return (long long)qd::step_stats_floats(heads, splits) + (long long)heads * splits * vdim;
}

extern "C" int qd_window_attention_step(const void* q, const void* k, const void* v, const void* gate, const void* q_norm,
                                        const void* k_norm, const float* freq, int rot, const void* sink, float scale, float eps,
                                        void* k_cache, void* v_cache, int capacity, int window, const int* position_ptr, int position,
                                        float* partial, unsigned int* counters, int splits, void* out, int heads, int kv_heads,
                                        int dim, int vdim, int dtype, void* stream) {
    QD_ATTN_ARGS_OK(partial && counters && splits > 0 && splits <= qd::kStepKeys && qd::aligned16(partial));
    const qd::AttnStep sp = {{q, k, v, gate, 0, (const bf16*)q_norm, (const bf16*)k_norm, freq, rot, (const bf16*)sink, scale, eps, k_cache,
                              v_cache, capacity, window, position_ptr, position, nullptr, out, 1, heads, kv_heads, dim, vdim},
                             partial, counters, splits, 2};
    if (dtype == QD_BF16) return qd::step<bf16>(sp, (cudaStream_t)stream);
    if (dtype == QD_F32) return qd::step<float>(sp, (cudaStream_t)stream);
    return QD_ERR_UNSUPPORTED;
}
