// Activation types of the bf16-weight kernels: every kernel exists for bf16 activations and for
// fp32 activations (dtype codes QD_BF16 / QD_F32); weights are bf16 in both.
#pragma once
#include "common.cuh"
#include "../../include/quickdraw_b200_hybrid.h"

namespace qd {

template <typename T> QD_DEVINL float load_f(const T* p);
template <> QD_DEVINL float load_f<float>(const float* p) { return *p; }
template <> QD_DEVINL float load_f<bf16>(const bf16* p) { return __bfloat162float(*p); }
template <typename T> QD_DEVINL void store_f(T* p, float v);
template <> QD_DEVINL void store_f<float>(float* p, float v) { *p = v; }
template <> QD_DEVINL void store_f<bf16>(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
template <typename T> QD_DEVINL float as_type(float v);      // v rounded to the activation type
template <> QD_DEVINL float as_type<float>(float v) { return v; }
template <> QD_DEVINL float as_type<bf16>(float v) { return round_bf16(v); }

// four consecutive elements (pointer aligned to four elements)
QD_DEVINL float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
QD_DEVINL float4 load4(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u),
                       __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
QD_DEVINL void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
QD_DEVINL void store4(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&lo);
    u.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
}
// eight bf16 of a 16-byte word as floats
QD_DEVINL void unpack8(const uint4& u, float (&v)[8]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}

QD_DEVINL float gelu_erf(float v) { return 0.5f * v * (1.0f + erff(v * 0.7071067811865476f)); }

// Sum over a block of up to 1024 threads, the same bits in every thread.  `red`: 33 floats of shared memory.
QD_DEVINL float block_sum(float v, float* red) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();                       // the previous use of `red` is over
    if (lane == 0) red[warp] = v;
    __syncthreads();
    if (warp == 0) {
        v = warp_sum(lane < warps ? red[lane] : 0.f);
        if (lane == 0) red[32] = v;
    }
    __syncthreads();
    return red[32];
}

static inline int device_sms() {
    int dev = 0, sms = 0;
    if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    return sms > 0 ? sms : 148;
}
// Raise a kernel's dynamic shared memory limit (a few hundred nanoseconds; launches above 48 KB only).
template <typename... KArgs>
static inline bool allow_smem(void (*kernel)(KArgs...), size_t bytes) {
    if (bytes <= 48 * 1024) return true;
    return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) == cudaSuccess;
}
static inline bool aligned16(const void* p) { return ((uintptr_t)p & 15u) == 0; }

}  // namespace qd
