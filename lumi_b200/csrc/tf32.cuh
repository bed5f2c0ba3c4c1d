// Products of fp32 operands on the tensor cores as two tf32 terms each (three MMAs, about fp32 accuracy), for the chunked recurrences.
#pragma once
#include "internal.h"

namespace lumi {

struct Tf2 { uint32_t hi, lo; };
__device__ __forceinline__ Tf2 split_tf32(float x) {
    Tf2 r;
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r.hi) : "f"(x));
    r.lo = __float_as_uint(x - __uint_as_float(r.hi));
    return r;
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
struct FragA { Tf2 v[4]; };
struct FragB { Tf2 v[2]; };
// A[m][k] = p[m * ld + k] at (m, k) of the fragment's corner
__device__ __forceinline__ FragA frag_a(const float* p, int ld, int g, int tq) {
    FragA f;
    f.v[0] = split_tf32(p[g * ld + tq]); f.v[1] = split_tf32(p[(g + 8) * ld + tq]);
    f.v[2] = split_tf32(p[g * ld + tq + 4]); f.v[3] = split_tf32(p[(g + 8) * ld + tq + 4]);
    return f;
}
// B[k][n] = p[k * ld + n]
__device__ __forceinline__ FragB frag_b(const float* p, int ld, int g, int tq) {
    FragB f;
    f.v[0] = split_tf32(p[tq * ld + g]); f.v[1] = split_tf32(p[(tq + 4) * ld + g]);
    return f;
}
__device__ __forceinline__ void mma3(float (&d)[4], const FragA& a, const FragB& b) {
    mma_tf32(d, a.v[0].lo, a.v[1].lo, a.v[2].lo, a.v[3].lo, b.v[0].hi, b.v[1].hi);
    mma_tf32(d, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b.v[0].lo, b.v[1].lo);
    mma_tf32(d, a.v[0].hi, a.v[1].hi, a.v[2].hi, a.v[3].hi, b.v[0].hi, b.v[1].hi);
}
__device__ __forceinline__ void cp16(float* dst, const float* src, bool ok) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    const int bytes = ok ? 16 : 0;                        // 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}

}  // namespace lumi
