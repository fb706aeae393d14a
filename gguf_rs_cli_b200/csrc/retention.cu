// Retention: linear attention with one fixed decay per head and no denominator,
//   S <- decay_h S + k' v^T;   o = S^T q'
// per head, S [D, Dv] in 32-bit per sequence, q' the rotated query, k' the rotated key times a constant.  This is the walk of
// linear_walk.h with the decay the same for all key channels and tokens: the preparation turns q and k by the token's
// position (32-bit angles, products and sums) and writes the walk's rows.
#include <math.h>

#include "common.cuh"
#include "linear_walk.h"

namespace {

struct RetPrepParams {
    const void *q, *k, *v;          // q, k [T, H*D], v [T, H*Dv]: column slices of one buffer with rows ld apart
    const int* pos;
    const float* inv_freq;          // [rot / 2] or null
    const float* decay;             // [H]
    LinearWalkRows rows;
    long long ld;
    int dtype, rot, pairing, H, D, Dv;
    float k_scale;
};

// One warp per (token, head).
__global__ void __launch_bounds__(128) retention_prep_kernel(const RetPrepParams p) {
    const int t = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (h >= p.H) return;
    const int D = p.D, DA = p.rows.DA, VA = p.rows.VA;
    float* o = p.rows.qkg + (size_t(t) * p.H + h) * 3 * DA;
    const size_t row = size_t(t) * p.ld + size_t(h) * D;
    const int half = p.inv_freq ? p.rot / 2 : 0;
    const float pos = float(p.pos[t]);
    for (int i = lane; i < half; i += 32) {
        const int d0 = p.pairing ? 2 * i : i, d1 = p.pairing ? 2 * i + 1 : i + half;
        float sn, cs, y0, y1;
        sincosf(pos * p.inv_freq[i], &sn, &cs);
        gb_rotate(gb_load(p.q, p.dtype, row + d0), gb_load(p.q, p.dtype, row + d1), cs, sn, y0, y1);
        o[d0] = y0;
        o[d1] = y1;
        gb_rotate(gb_load(p.k, p.dtype, row + d0), gb_load(p.k, p.dtype, row + d1), cs, sn, y0, y1);
        o[DA + d0] = y0 * p.k_scale;
        o[DA + d1] = y1 * p.k_scale;
    }
    for (int d = 2 * half + lane; d < DA; d += 32) {
        o[d] = d < D ? gb_load(p.q, p.dtype, row + d) : 0.f;
        o[DA + d] = d < D ? gb_load(p.k, p.dtype, row + d) * p.k_scale : 0.f;
    }
    const float g = p.decay[h];
    for (int d = lane; d < DA; d += 32) o[2 * DA + d] = d < D ? g : 0.f;
    float* vo = p.rows.vf + (size_t(t) * p.H + h) * VA;
    for (int d = lane; d < VA; d += 32) vo[d] = d < p.Dv ? gb_load(p.v, p.dtype, size_t(t) * p.ld + size_t(h) * p.Dv + d) : 0.f;
}

}  // namespace

// q, k [T, H*D] and v [T, H*Dv]: column slices of one buffer with rows ld apart; pos [T]; inv_freq [rot / 2] or null: no
// rotation (pairing 0: entries (i, i + rot/2), 1: (2i, 2i+1)); decay [H]; state [slots, H, D, Dv] float32, read and renewed;
// out float32 [T, H*Dv].  scratch: gb_linear_walk_scratch_floats(T, H, D, Dv).
GB_API int gb_retention(const void* q, const void* k, const void* v, int dtype, long long ld, const int* pos, const float* inv_freq,
                        int rot, int pairing, float k_scale, const float* decay, float* state, float* out, long long ldo,
                        const int* cu, const int* slots, const int* qlens, int T, int B, int H, int D, int Dv, float* scratch,
                        int max_qlen, float* seg_scratch, cudaStream_t stream) {
    GB_REQUIRE(gb_is_dtype(dtype), "gb_retention: bad dtype");
    GB_REQUIRE(H > 0 && D > 0 && D <= 2048 && Dv > 0 && (H + 3) / 4 <= 65535,
               "gb_retention: bad sizes heads=%d dim=%d vdim=%d (dim up to 2048)", H, D, Dv);
    GB_REQUIRE(!inv_freq || (rot > 0 && rot % 2 == 0 && rot <= D), "gb_retention: %d of %d entries cannot be rotated", rot, D);
    GB_REQUIRE(scratch && (reinterpret_cast<uintptr_t>(scratch) & 15) == 0, "gb_retention: scratch missing or misaligned");
    if (B == 0 || T == 0) return 0;
    RetPrepParams pp;
    pp.rows = gb_linear_walk_rows(scratch, T, H, D, Dv, false);
    pp.q = q; pp.k = k; pp.v = v; pp.pos = pos; pp.inv_freq = inv_freq; pp.decay = decay; pp.ld = ld; pp.dtype = dtype;
    pp.rot = rot; pp.pairing = pairing; pp.H = H; pp.D = D; pp.Dv = Dv; pp.k_scale = k_scale;
    retention_prep_kernel<<<dim3(T, (H + 3) / 4), 128, 0, stream>>>(pp);
    GB_LAUNCH_OK("gb_retention (prepare)");
    return gb_linear_walk_launch(pp.rows, false, state, out, ldo, cu, slots, qlens, B, H, D, Dv, max_qlen, seg_scratch, stream,
                                 "gb_retention");
}
