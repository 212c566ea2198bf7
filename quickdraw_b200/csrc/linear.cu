// Products with bf16 weights: y[t, n] = sum_k x[t, k] w[n, k], fp32 accumulation.  What may follow in the
// same launch: a bias, the exact GELU on the leading columns (the up projection of a feed-forward whose
// launch also carries other rows), a gated linear unit over neighbouring weight rows, the addition to
// what y already holds (a residual stream).  What may precede it for few token rows: the RMS norm of x.
// Three forms behind one entry point:
//   linear_umma_kernel  many token rows, bf16 x: tcgen05.mma kind::f16, both operands by tiled TMA
//                       (128-byte swizzle), accumulators in tensor memory.  Tensor-bound.
//   linear_rows_kernel  up to eight token rows: a warp streams whole weight rows (16-byte loads, the
//                       first inputs of each row - up to 4096 - requested before the wait for the
//                       preceding kernel), the token rows in shared memory as fp32.  HBM-bound.
//   linear_tile_kernel  any shape and alignment, and fp32 x with many rows: 64 x 64 tiles on the FMA pipe.
#include <cuda.h>

#include "typed.cuh"

namespace qd {
namespace {

// What follows the sums.  glu: weight rows 2i and 2i + 1 are a gate and its linear partner, y[i] = relu(gate) * partner.
struct Finish { const float* bias; int gelu_cols; int glu; int add; };
// RMS norm of x in front of the product: x / rms(x) * (offset + weight); weight == NULL: none.
struct InputNorm { const bf16* weight; float offset, eps; };

QD_DEVINL float finished(const Finish& f, float v, int n) {
    if (f.bias) v += f.bias[n];
    return n < f.gelu_cols ? gelu_erf(v) : v;
}
template <typename T> QD_DEVINL void put(T* y, float v, bool add) { store_f(y, add ? load_f(y) + v : v); }

// ------------------------------------------------------------------------------ few token rows
// Inputs staged at a time.  One weight row per warp (few rows: one or two blocks per SM): up to sixteen 16-byte
// pieces per lane in flight; two rows per warp: eight, and more blocks.
constexpr int rows_chunk(int R, int NR) { return NR == 2 ? 1024 : (R <= 2 ? 4096 : (R == 4 ? 2048 : 1024)); }

template <typename TX, typename TY, int R, int NR>
__global__ void __launch_bounds__(256)
linear_rows_kernel(const TX* __restrict__ x, long long ldx, const bf16* __restrict__ w, TY* __restrict__ y,
                   long long ldy, int tokens, int rows, int width, const Finish f, const InputNorm norm) {
    constexpr int kRowsChunk = rows_chunk(R, NR);
    __shared__ __align__(16) float xs[R][kRowsChunk];
    __shared__ float squares[R][8];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n0 = (blockIdx.x * 8 + warp) * NR;
    constexpr int kPieces = kRowsChunk / 256;
    uint4 wv[NR][kPieces];
    auto fetch = [&](int k0) {
#pragma unroll
        for (int r = 0; r < NR; ++r)
#pragma unroll
            for (int i = 0; i < kPieces; ++i) {
                const int k = k0 + (i * 32 + lane) * 8;
                wv[r][i] = (n0 + r < rows && k < width) ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)(n0 + r) * width + k))
                                                        : make_uint4(0u, 0u, 0u, 0u);
            }
    };
    grid_launch_dependents();
    fetch(0);
    grid_dependency_wait();
    float acc[NR][R];
#pragma unroll
    for (int r = 0; r < NR; ++r)
#pragma unroll
        for (int t = 0; t < R; ++t) acc[r][t] = 0.f;
    float ss[R];                         // of this thread's inputs, for the norm
#pragma unroll
    for (int t = 0; t < R; ++t) ss[t] = 0.f;
    for (int k0 = 0; k0 < width; k0 += kRowsChunk) {
        if (k0) __syncthreads();
#pragma unroll
        for (int t = 0; t < R; ++t)
            for (int k = threadIdx.x * 4; k < kRowsChunk; k += 1024) {
                const bool ok = t < tokens && k0 + k < width;
                float4 v = ok ? load4(x + t * ldx + k0 + k) : make_float4(0.f, 0.f, 0.f, 0.f);
                if (norm.weight && ok) {
                    const float4 g = load4(norm.weight + k0 + k);
                    ss[t] = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss[t]))));
                    v.x *= norm.offset + g.x; v.y *= norm.offset + g.y; v.z *= norm.offset + g.z; v.w *= norm.offset + g.w;
                }
                *reinterpret_cast<float4*>(&xs[t][k]) = v;
            }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kPieces; ++i) {
            const int k = (i * 32 + lane) * 8;
            float wf[NR][8];
#pragma unroll
            for (int r = 0; r < NR; ++r) unpack8(wv[r][i], wf[r]);
#pragma unroll
            for (int t = 0; t < R; ++t) {
                const float4 a = *reinterpret_cast<const float4*>(&xs[t][k]), b = *reinterpret_cast<const float4*>(&xs[t][k + 4]);
#pragma unroll
                for (int r = 0; r < NR; ++r) {
                    float s = acc[r][t];
                    s = fmaf(wf[r][0], a.x, s); s = fmaf(wf[r][1], a.y, s); s = fmaf(wf[r][2], a.z, s); s = fmaf(wf[r][3], a.w, s);
                    s = fmaf(wf[r][4], b.x, s); s = fmaf(wf[r][5], b.y, s); s = fmaf(wf[r][6], b.z, s); s = fmaf(wf[r][7], b.w, s);
                    acc[r][t] = s;
                }
            }
        }
        if (k0 + kRowsChunk < width) fetch(k0 + kRowsChunk);
    }
    if (norm.weight) {                   // the same factor for every row: applied to the sums
#pragma unroll
        for (int t = 0; t < R; ++t) {
            const float part = warp_sum(ss[t]);
            if (lane == 0) squares[t][warp] = part;
        }
        __syncthreads();
#pragma unroll
        for (int t = 0; t < R; ++t) {
            float total = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) total += squares[t][i];
            const float factor = 1.0f / sqrtf(total / (float)width + norm.eps);
#pragma unroll
            for (int r = 0; r < NR; ++r) acc[r][t] *= factor;
        }
    }
#pragma unroll
    for (int t = 0; t < R; ++t) {
        float v[NR];
#pragma unroll
        for (int r = 0; r < NR; ++r) v[r] = warp_sum(acc[r][t]);
        if (lane != 0 || t >= tokens) continue;
        if (NR == 2 && f.glu) {
            if (n0 < rows) put(y + t * ldy + n0 / 2, fmaxf(finished(f, v[0], n0), 0.f) * finished(f, v[NR - 1], n0 + 1), f.add);
        } else {
#pragma unroll
            for (int r = 0; r < NR; ++r)
                if (n0 + r < rows) put(y + t * ldy + n0 + r, finished(f, v[r], n0 + r), f.add);
        }
    }
}

// ---------------------------------------------------------------------------------- any shape
constexpr int kTileT = 64, kTileR = 64, kTileStep = 16;

template <typename TX, typename TY>
__global__ void __launch_bounds__(256)
linear_tile_kernel(const TX* __restrict__ x, long long ldx, const bf16* __restrict__ w, TY* __restrict__ y,
                   long long ldy, int tokens, int rows, int width, const Finish f) {
    chain_enter();
    __shared__ __align__(16) float xs[kTileStep][kTileT + 4], ws[kTileStep][kTileR + 4];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int n0 = blockIdx.x * kTileR, t0 = blockIdx.y * kTileT;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < width; k0 += kTileStep) {
        for (int i = tid; i < kTileStep * kTileT; i += 256) {
            const int k = i & (kTileStep - 1), r = i / kTileStep;
            const bool ok = k0 + k < width;
            xs[k][r] = (ok && t0 + r < tokens) ? load_f(x + (t0 + r) * ldx + k0 + k) : 0.f;
            ws[k][r] = (ok && n0 + r < rows) ? ld_bf16(w + (size_t)(n0 + r) * width + k0 + k) : 0.f;
        }
        __syncthreads();
        float part[4][4] = {};           // summed per step: the rounding error grows with the steps, not with the inputs
#pragma unroll
        for (int k = 0; k < kTileStep; ++k) {
            const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]), b = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) part[i][j] = fmaf(av[i], bv[j], part[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (t >= tokens || n >= rows) continue;
            if (!f.glu) put(y + t * ldy + n, finished(f, acc[i][j], n), f.add);
            else if (!(j & 1)) put(y + t * ldy + n / 2, fmaxf(finished(f, acc[i][j], n), 0.f) * finished(f, acc[i][j | 1], n + 1), f.add);
        }
}

// ------------------------------------------------------------------------------- tensor cores
constexpr int kStepK = 64;                     // inputs per stage: one 128-byte swizzled row

// Tile of HALVES x 128 tokens by TN weight rows; warp 0 issues the TMA loads, warp 1 the MMAs, four warps
// per token half read the accumulators back (a warp may read the tensor-memory lanes 32 (warp mod 4) ..).
template <int HALVES, int TN> struct UmmaTile {
    static constexpr int kABytes = HALVES * 128 * 128, kBBytes = TN * 128, kStageBytes = kABytes + kBBytes;
    static constexpr int kStages = HALVES == 2 ? 3 : (TN == 256 ? 4 : 3);
    static constexpr int kCols = HALVES * TN;
    static constexpr int kThreads = 64 + HALVES * 128;
    static constexpr int kBlocksPerSm = (HALVES == 1 && TN <= 128) ? 2 : 1;
    static constexpr size_t kSmem = (size_t)kStages * kStageBytes + (2 * kStages + 1) * 8 + 16 + 1024;
};

QD_DEVINL uint64_t desc_sw128(uint32_t addr) {      // K-major, 128-byte swizzle, 1024 bytes between groups of eight rows
    return (uint64_t)((addr >> 4) & 0x3fffu) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
QD_DEVINL void tma_tile(void* dst, const CUtensorMap* map, int c0, int c1, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 ::"r"(smem_u32(dst)), "l"(map), "r"(c0), "r"(c1), "r"(smem_u32(bar)) : "memory");
}
QD_DEVINL void umma_f16(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
                 ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}
QD_DEVINL void umma_commit_to(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}
QD_DEVINL void tmem_ld32(uint32_t addr, uint32_t (&v)[32]) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x32.b32 "
                 "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
                 "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
                 : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
                   "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]),
                   "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
                   "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
                 : "r"(addr) : "memory");
    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}

struct LinearParams { void* y; long long ldy; int tokens, rows, width; Finish f; unsigned int* status; };

template <typename TY, int HALVES, int TN>
__global__ void __launch_bounds__(UmmaTile<HALVES, TN>::kThreads, UmmaTile<HALVES, TN>::kBlocksPerSm)
linear_umma_kernel(const __grid_constant__ LinearParams p, const __grid_constant__ CUtensorMap xmap,
                   const __grid_constant__ CUtensorMap wmap) {
    chain_enter();
    using Tile = UmmaTile<HALVES, TN>;
    constexpr int kStages = Tile::kStages;
    // fp32 accumulator (bits [4,6) = 1), bf16 A and B (bits [7,10), [10,13) = 1), K-major, N >> 3 at 17, M >> 4 at 24
    constexpr uint32_t kDesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TN >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + kStages * Tile::kStageBytes);
    uint64_t* empty = full + kStages;
    uint64_t* done = empty + kStages;
    uint32_t* slot = reinterpret_cast<uint32_t*>(done + 1);
    volatile int* failed = reinterpret_cast<volatile int*>(slot + 1);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int t0 = blockIdx.x * HALVES * 128, n0 = blockIdx.y * TN;
    const int steps = (p.width + kStepK - 1) / kStepK;
    __shared__ __align__(16) float bias[TN];
    if (p.f.bias)
        for (int i = tid; i < TN; i += Tile::kThreads) bias[i] = n0 + i < p.rows ? p.f.bias[n0 + i] : 0.f;
    const int halves = (HALVES == 2 && p.tokens - t0 > 128) ? 2 : 1;       // a half without tokens is not multiplied

    if (tid == 0) {
        for (int s = 0; s < kStages; ++s) { mbar_init(full + s, 1); mbar_init(empty + s, 1); }
        mbar_init(done, 1);
        mbar_fence_init();
        *failed = 0;
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(slot)), "r"(Tile::kCols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *slot;

    if (warp == 0) {
        if (lane == 0) {
            int issued = 0;
            bool ok = true;
            for (; issued < steps; ++issued) {
                const int st = issued % kStages;
                if (issued >= kStages) ok = mbar_wait(empty + st, ((issued / kStages) - 1) & 1, p.status);
                if (!ok) break;
                uint8_t* a = smem + st * Tile::kStageBytes;
                mbar_expect_tx(full + st, Tile::kStageBytes);
                tma_tile(a, &xmap, issued * kStepK, t0, full + st);
                tma_tile(a + Tile::kABytes, &wmap, issued * kStepK, n0, full + st);
            }
            if (!ok)            // leave no copy in flight behind
                for (int s = issued > kStages ? issued - kStages : 0; s < issued; ++s)
                    mbar_wait(full + s % kStages, (s / kStages) & 1, p.status);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            bool ok = true;
            for (int s = 0; s < steps; ++s) {
                const int st = s % kStages;
                ok = mbar_wait(full + st, (s / kStages) & 1, p.status);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t a = smem_u32(smem + st * Tile::kStageBytes), b = a + Tile::kABytes;
#pragma unroll 1
                for (int h = 0; h < halves; ++h)
#pragma unroll
                    for (int j = 0; j < kStepK / 16; ++j)
                        umma_f16(tmem + h * TN, desc_sw128(a + h * 128 * 128 + j * 32), desc_sw128(b + j * 32), kDesc, (s | j) ? 1u : 0u);
                umma_commit_to(empty + st);
            }
            if (ok) umma_commit_to(done);
            else *failed = 1;
        }
    } else {
        const int half = (warp - 2) >> 2, quadrant = warp & 3;
        const bool ok = mbar_wait(done, 0, p.status) && !*failed;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (ok && half < halves) {
            const int t = t0 + half * 128 + quadrant * 32 + lane;
            TY* row = reinterpret_cast<TY*>(p.y) + (long long)t * p.ldy;
#pragma unroll 1
            for (int c = 0; c < TN; c += 32) {
                if (n0 + c >= p.rows) break;
                uint32_t v[32];
                tmem_ld32(tmem + ((uint32_t)(quadrant * 32) << 16) + half * TN + c, v);
                const bool gelu = n0 + c < p.f.gelu_cols;
                if (t < p.tokens) {
#pragma unroll
                    for (int j = 0; j < 32; j += 8) {
                        const int n = n0 + c + j;
                        if (n < p.rows) {                // rows is a multiple of eight
                            float f[8];
#pragma unroll
                            for (int q = 0; q < 8; ++q) f[q] = __uint_as_float(v[j + q]);
                            if (p.f.bias) {
                                const float4 a = load4(bias + c + j), b = load4(bias + c + j + 4);
                                f[0] += a.x; f[1] += a.y; f[2] += a.z; f[3] += a.w; f[4] += b.x; f[5] += b.y; f[6] += b.z; f[7] += b.w;
                            }
                            if (gelu) {
#pragma unroll
                                for (int q = 0; q < 8; ++q)
                                    if (n + q < p.f.gelu_cols) f[q] = gelu_erf(f[q]);
                            }
                            if (p.f.glu) {
                                store4(row + n / 2, make_float4(fmaxf(f[0], 0.f) * f[1], fmaxf(f[2], 0.f) * f[3], fmaxf(f[4], 0.f) * f[5],
                                                                fmaxf(f[6], 0.f) * f[7]));
                                continue;
                            }
                            if (p.f.add) {
                                const float4 a = load4(row + n), b = load4(row + n + 4);
                                f[0] += a.x; f[1] += a.y; f[2] += a.z; f[3] += a.w; f[4] += b.x; f[5] += b.y; f[6] += b.z; f[7] += b.w;
                            }
                            store4(row + n, make_float4(f[0], f[1], f[2], f[3]));
                            store4(row + n + 4, make_float4(f[4], f[5], f[6], f[7]));
                        }
                    }
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1)
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(Tile::kCols) : "memory");
}

typedef CUresult (*EncodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiled encode_fn() {
    static EncodeTiled fn = [] {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult result;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &result) != cudaSuccess ||
            result != cudaDriverEntryPointSuccess)
            ptr = nullptr;
        return reinterpret_cast<EncodeTiled>(ptr);
    }();
    return fn;
}
// bf16 [rows, width] with `ld` elements between rows; box = 64 inputs x box_rows; what lies outside reads as zero.
int tile_map(CUtensorMap* map, const void* base, long long rows, long long width, long long ld, int box_rows) {
    EncodeTiled encode = encode_fn();
    if (!encode) return QD_ERR_UNSUPPORTED;
    const cuuint64_t dims[2] = {(cuuint64_t)width, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * sizeof(bf16)};
    const cuuint32_t box[2] = {(cuuint32_t)kStepK, (cuuint32_t)box_rows};
    const cuuint32_t elem[2] = {1, 1};
    return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, elem,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? QD_OK : QD_ERR_LAUNCH;
}

template <typename TY, int HALVES, int TN>
int launch_umma(const void* x, long long ldx, const void* w, const LinearParams& p, cudaStream_t stream) {
    using Tile = UmmaTile<HALVES, TN>;
    if (!allow_smem(linear_umma_kernel<TY, HALVES, TN>, Tile::kSmem)) return QD_ERR_LAUNCH;
    alignas(64) CUtensorMap xmap = {}, wmap = {};
    int rc = tile_map(&xmap, x, p.tokens, p.width, ldx, HALVES * 128);
    if (rc == QD_OK) rc = tile_map(&wmap, w, p.rows, p.width, p.width, TN);
    if (rc != QD_OK) return rc;
    const dim3 grid((p.tokens + HALVES * 128 - 1) / (HALVES * 128), (p.rows + TN - 1) / TN);
    return qd_launch(linear_umma_kernel<TY, HALVES, TN>, grid, dim3(Tile::kThreads), Tile::kSmem, stream, 1, p, xmap, wmap);
}

template <typename TY>
int umma_dispatch(const void* x, long long ldx, const void* w, const LinearParams& p, cudaStream_t stream) {
    const long long sms = device_sms();
    const auto tiles = [&](int tm, int tn) { return (long long)((p.tokens + tm - 1) / tm) * ((p.rows + tn - 1) / tn); };
    // the largest tile that still gives most SMs one (a larger tile reads each operand fewer times)
    if (tiles(256, 256) * 4 >= sms * 3) return launch_umma<TY, 2, 256>(x, ldx, w, p, stream);
    if (tiles(128, 256) * 4 >= sms * 3) return launch_umma<TY, 1, 256>(x, ldx, w, p, stream);
    if (tiles(128, 128) * 4 >= sms * 3) return launch_umma<TY, 1, 128>(x, ldx, w, p, stream);
    return launch_umma<TY, 1, 64>(x, ldx, w, p, stream);
}

template <typename TX, typename TY, int R>
int launch_rows(const void* x, long long ldx, const void* w, void* y, long long ldy, int tokens, int rows, int width,
                const Finish& f, const InputNorm& norm, cudaStream_t stream) {
    // two weight rows per warp once that still gives every SM a few blocks, and where pairs of rows belong together
    if (f.glu || rows >= device_sms() * 32)
        return qd_launch(linear_rows_kernel<TX, TY, R, 2>, dim3((rows + 15) / 16), dim3(256), 0, stream, 2,
                         (const TX*)x, ldx, (const bf16*)w, (TY*)y, ldy, tokens, rows, width, f, norm);
    return qd_launch(linear_rows_kernel<TX, TY, R, 1>, dim3((rows + 7) / 8), dim3(256), 0, stream, 2,
                     (const TX*)x, ldx, (const bf16*)w, (TY*)y, ldy, tokens, rows, width, f, norm);
}

template <typename TX, typename TY>
int dispatch(const void* x, long long ldx, const void* w, void* y, long long ldy, int tokens, int rows, int width,
             const Finish& f, const InputNorm& norm, unsigned int* status, cudaStream_t stream) {
    const bool vectors = width % 8 == 0 && ldx % 8 == 0 && aligned16(x) && aligned16(w);
    if (vectors && tokens <= 8 && (!norm.weight || ((uintptr_t)norm.weight & 7u) == 0)) {
        if (tokens == 1) return launch_rows<TX, TY, 1>(x, ldx, w, y, ldy, tokens, rows, width, f, norm, stream);
        if (tokens == 2) return launch_rows<TX, TY, 2>(x, ldx, w, y, ldy, tokens, rows, width, f, norm, stream);
        if (tokens <= 4) return launch_rows<TX, TY, 4>(x, ldx, w, y, ldy, tokens, rows, width, f, norm, stream);
        return launch_rows<TX, TY, 8>(x, ldx, w, y, ldy, tokens, rows, width, f, norm, stream);
    }
    if (norm.weight) return QD_ERR_UNSUPPORTED;
    if (sizeof(TX) == 2 && vectors && rows % 8 == 0 && ldy % 8 == 0 && aligned16(y)) {
        const LinearParams p = {y, ldy, tokens, rows, width, f, status};
        return umma_dispatch<TY>(x, ldx, w, p, stream);
    }
    const dim3 grid((rows + kTileR - 1) / kTileR, (tokens + kTileT - 1) / kTileT);
    return qd_launch(linear_tile_kernel<TX, TY>, grid, dim3(256), 0, stream, 1, (const TX*)x, ldx, (const bf16*)w, (TY*)y,
                     ldy, tokens, rows, width, f);
}

// ---------------------------------------------------------------------------- greedy choice
// Index of the largest of `count` fp32 logits (lowest index among equals) as int64.  A block reduces a
// slice to one 64-bit key (order-preserving bits of the value, complement of the index); the last block
// to finish reduces the keys and clears the counter for the next launch.
QD_DEVINL unsigned long long choice_key(float v, int i) {
    uint32_t b = __float_as_uint(v);
    b = (b & 0x80000000u) ? ~b : (b | 0x80000000u);
    return ((unsigned long long)b << 32) | (0xffffffffu - (uint32_t)i);
}
QD_DEVINL unsigned long long warp_max_key(unsigned long long k) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const unsigned long long other = __shfl_xor_sync(0xffffffffu, k, o);
        k = other > k ? other : k;
    }
    return k;
}
__global__ void __launch_bounds__(256)
greedy_kernel(const float* __restrict__ logits, int count, unsigned long long* keys, unsigned int* counter, long long* token) {
    chain_enter();
    __shared__ unsigned long long best[8];
    __shared__ bool last;
    const int tid = threadIdx.x;
    auto block_best = [&](unsigned long long k) {
        k = warp_max_key(k);
        __syncthreads();
        if ((tid & 31) == 0) best[tid >> 5] = k;
        __syncthreads();
        for (int i = 0; i < 8; ++i) k = best[i] > k ? best[i] : k;
        return k;
    };
    unsigned long long k = 0;
    for (int i = blockIdx.x * 256 + tid; i < count; i += gridDim.x * 256) {
        const unsigned long long c = choice_key(logits[i], i);
        k = c > k ? c : k;
    }
    k = block_best(k);
    if (tid == 0) {
        keys[blockIdx.x] = k;
        __threadfence();
        last = atomicAdd(counter, 1u) == gridDim.x - 1;
    }
    __syncthreads();
    if (!last) return;
    __threadfence();
    k = 0;
    for (int i = tid; i < gridDim.x; i += 256) {
        const unsigned long long c = *reinterpret_cast<volatile unsigned long long*>(keys + i);
        k = c > k ? c : k;
    }
    k = block_best(k);
    if (tid == 0) { *token = (long long)(0xffffffffu - (uint32_t)k); *counter = 0u; }
}

int launch_greedy(int blocks, const float* logits, int count, unsigned long long* keys, unsigned int* counter, long long* token,
                  cudaStream_t s) {
    return qd_launch(greedy_kernel, dim3(blocks), dim3(256), 0, s, 1, logits, count, keys, counter, token);
}

}  // namespace
}  // namespace qd

extern "C" int qd_linear(const void* x, long long ldx, int x_dtype, const void* w, void* y, long long ldy, int y_dtype,
                         int tokens, int rows, int width, int gelu_cols, int glu, const float* bias, int add, const void* norm,
                         float norm_offset, float eps, unsigned int* status, void* stream) {
    QD_CHECK_ARG(x && w && y && tokens > 0 && rows > 0 && width > 0 && ldx >= width && gelu_cols >= 0);
    QD_CHECK_ARG(ldy >= (glu ? rows / 2 : rows) && (!glu || (rows % 2 == 0 && gelu_cols == 0 && !add)));
    const qd::Finish f = {bias, gelu_cols, glu, add};
    const qd::InputNorm n = {(const bf16*)norm, norm_offset, eps};
    cudaStream_t s = (cudaStream_t)stream;
    if (x_dtype == QD_BF16 && y_dtype == QD_BF16) return qd::dispatch<bf16, bf16>(x, ldx, w, y, ldy, tokens, rows, width, f, n, status, s);
    if (x_dtype == QD_BF16 && y_dtype == QD_F32) return qd::dispatch<bf16, float>(x, ldx, w, y, ldy, tokens, rows, width, f, n, status, s);
    if (x_dtype == QD_F32 && y_dtype == QD_F32) return qd::dispatch<float, float>(x, ldx, w, y, ldy, tokens, rows, width, f, n, status, s);
    if (x_dtype == QD_F32 && y_dtype == QD_BF16) return qd::dispatch<float, bf16>(x, ldx, w, y, ldy, tokens, rows, width, f, n, status, s);
    return QD_ERR_UNSUPPORTED;
}

extern "C" int qd_greedy(const float* logits, int count, void* keys, unsigned int* counter, void* token, void* stream) {
    QD_CHECK_ARG(logits && keys && counter && token && count > 0);
    int blocks = (count + 1023) / 1024;
    if (blocks > QD_GREEDY_BLOCKS) blocks = QD_GREEDY_BLOCKS;
    return qd::launch_greedy(blocks, logits, count, (unsigned long long*)keys, counter, (long long*)token, (cudaStream_t)stream);
}
