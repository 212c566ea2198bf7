// What the softmax attention kernels of the bf16-weight models share: rotary angles, warp-level matrix
// products and the copies that feed them.
#pragma once
#include "typed.cuh"

namespace qd {

constexpr float kLog2e = 1.4426950408889634f;
constexpr size_t kMaxSmem = 227 * 1024;

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

}  // namespace qd
