// Pieces of the mma.sync kernels that work on bfloat16 tiles in shared memory: fragment loads, the product, a swizzle that
// keeps them free of bank conflicts, and 32-bit numbers as three bfloat16 terms.
//
// A float x is h + m + l exactly, 8 significant bits each.  A product of a float with a bfloat16 number is then three exact
// products; one of two floats is six (hh, hm, mh, mm, hl, lh: what is left out is below 2^-24 of it), all summed in 32-bit.
#pragma once
#include "common.cuh"

namespace gbmma {

__device__ __forceinline__ void ldsm4(unsigned (&r)[4], const void* p) {
    const unsigned a = unsigned(__cvta_generic_to_shared(p));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4_trans(unsigned (&r)[4], const void* p) {
    const unsigned a = unsigned(__cvta_generic_to_shared(p));
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
// c += A B for one 16 x 16 fragment of A and 8 columns of B
__device__ __forceinline__ void mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 x 16 of A times 32 columns of B (b and b2: 16 columns each), A and B of three terms: the six products, smallest first,
// every one of them for all four accumulators before the next, so that an accumulator's products do not follow one
// another at once
__device__ __forceinline__ void mma6(float (&c0)[4], float (&c1)[4], float (&c2)[4], float (&c3)[4], const unsigned (&a)[3][4],
                                     const unsigned (&b)[3][4], const unsigned (&b2)[3][4]) {
    constexpr int TA[6] = {0, 2, 1, 0, 1, 0}, TB[6] = {2, 0, 1, 1, 0, 0};
#pragma unroll
    for (int e = 0; e < 6; ++e) {
        mma(c0, a[TA[e]], b[TB[e]][0], b[TB[e]][1]);
        mma(c1, a[TA[e]], b[TB[e]][2], b[TB[e]][3]);
        mma(c2, a[TA[e]], b2[TB[e]][0], b2[TB[e]][1]);
        mma(c3, a[TA[e]], b2[TB[e]][2], b2[TB[e]][3]);
    }
}
// the same for a B of one term: three products
__device__ __forceinline__ void mma3(float (&c0)[4], float (&c1)[4], float (&c2)[4], float (&c3)[4], const unsigned (&a)[3][4],
                                     const unsigned (&b)[4], const unsigned (&b2)[4]) {
#pragma unroll
    for (int e = 2; e >= 0; --e) {
        mma(c0, a[e], b[0], b[1]);
        mma(c1, a[e], b[2], b[3]);
        mma(c2, a[e], b2[0], b2[1]);
        mma(c3, a[e], b2[2], b2[3]);
    }
}
__device__ __forceinline__ unsigned pack2(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned*>(&v);
}
// two neighbouring numbers as three packed terms
__device__ __forceinline__ void split3(float x, float y, unsigned& h, unsigned& m, unsigned& l) {
    h = pack2(x, y);
    const float2 hf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&h));
    const float x1 = x - hf.x, y1 = y - hf.y;
    m = pack2(x1, y1);
    const float2 mf = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&m));
    l = pack2(x1 - mf.x, y1 - mf.y);
}
// Entry offset of (row, 16-byte chunk) in a tile of N-wide rows: chunks are exchanged within groups of eight (N a multiple
// of 64) or of four (N an odd multiple of 32: rows then start half a bank line apart).
template <int N> __device__ __forceinline__ int swz(int row, int chunk) {
    static_assert(N % 32 == 0, "rows of a multiple of 32 entries");
    if (N % 64) return row * N + ((chunk ^ ((row >> 1) & 3)) << 3);
    return row * N + (((chunk & ~7) | ((chunk ^ row) & 7)) << 3);
}

}  // namespace gbmma
