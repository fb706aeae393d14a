// Layer norm with a weight and no bias, LN(v) = (v - mean v) / sqrt(mean((v - mean v)^2) + eps) * w, for layers that
// norm the sum of what they read and what a sublayer gives:
//   v = alpha * x[t,:] + y[t,:] + sum_r weights[t,r] * z[row(t,r),:]          (y and the routed rows z each optional)
//   x[t,:] = LN(v), xb[t,:] = bfloat16(LN(v)), h[t,:] = LN(v)                 (each optional)
// row(t,r) is t * top + r, or place_of[t * top + r] when the rows z lie in another order; the sum runs in the order of
// the choices.  All in 32-bit: the mean first, then the squared deviations from it.
//
// One block per row.  Rows of up to 16,384 entries that start on 16 bytes stay in registers between the passes; other
// rows lie in shared memory.
#include "common.cuh"

namespace {

struct LnParams {
    float* x;                  // [T, E] contiguous
    const void* y;             // [T, E] rows ldy apart, or null
    const float* z;            // routed rows [T * top, E] contiguous, or null
    const float* weights;      // [T, top]
    const int* place_of;       // [T * top] or null
    const int* rows;           // row numbers to gather, or null: all
    const void* w;
    void* h;
    __nv_bfloat16* xb;
    long long ldy;
    float alpha, eps;
    int y_dtype, w_dtype, h_dtype, top, E, write_x;
};

// sum over the block; `slot` names one of two arrays of partial sums, so that two sums in a row need no barrier between
__device__ __forceinline__ float ln_block_sum(float v, float* red) {
    v = gb_warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
    for (int k = 0; k < int(blockDim.x >> 5); ++k) tot += red[k];
    return tot;
}

// NV pieces of four entries per thread: piece k of thread i starts at entry 4 * (i + k * blockDim.x)
template <int NV>
__global__ void __launch_bounds__(NV < 4 ? 1024 : 512) layernorm_vec_kernel(const LnParams p) {
    __shared__ float red1[32], red2[32];
    const int E = p.E;
    float4 v[NV];
    constexpr bool EARLY = NV <= 2;        // the weights do not depend on the kernel before this one; with many pieces their
    float4 wv[EARLY ? NV : 1];             // registers would cost resident blocks
    if (EARLY) {
#pragma unroll
        for (int k = 0; k < (EARLY ? NV : 1); ++k) {
            const int i = 4 * (threadIdx.x + k * blockDim.x);
            wv[k] = i < E ? gb_load4(p.w, p.w_dtype, i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int t = p.rows ? p.rows[blockIdx.x] : int(blockIdx.x);
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < E) {
            v[k] = *reinterpret_cast<const float4*>(p.x + size_t(t) * E + i);
            v[k].x *= p.alpha; v[k].y *= p.alpha; v[k].z *= p.alpha; v[k].w *= p.alpha;
            if (p.y) {
                const float4 y = gb_load4(p.y, p.y_dtype, size_t(t) * p.ldy + i);
                v[k].x += y.x; v[k].y += y.y; v[k].z += y.z; v[k].w += y.w;
            }
        }
    }
    if (p.z) {
        for (int r = 0; r < p.top; ++r) {
            const int pair = t * p.top + r;
            const float wr = p.weights[pair];
            const float* zr = p.z + size_t(p.place_of ? p.place_of[pair] : pair) * E;
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int i = 4 * (threadIdx.x + k * blockDim.x);
                if (i < E) {
                    const float4 y = *reinterpret_cast<const float4*>(zr + i);
                    v[k].x = fmaf(wr, y.x, v[k].x); v[k].y = fmaf(wr, y.y, v[k].y);
                    v[k].z = fmaf(wr, y.z, v[k].z); v[k].w = fmaf(wr, y.w, v[k].w);
                }
            }
        }
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) s += (v[k].x + v[k].y) + (v[k].z + v[k].w);
    const float mean = ln_block_sum(s, red1) / float(E);
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        if (i < E) {
            v[k].x -= mean; v[k].y -= mean; v[k].z -= mean; v[k].w -= mean;
            ss = fmaf(v[k].x, v[k].x, ss); ss = fmaf(v[k].y, v[k].y, ss);
            ss = fmaf(v[k].z, v[k].z, ss); ss = fmaf(v[k].w, v[k].w, ss);
        }
    }
    const float f = 1.f / sqrtf(ln_block_sum(ss, red2) / float(E) + p.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        if (i < E) {
            const float4 g = EARLY ? wv[EARLY ? k : 0] : gb_load4(p.w, p.w_dtype, i);
            const float4 o = make_float4(v[k].x * f * g.x, v[k].y * f * g.y, v[k].z * f * g.z, v[k].w * f * g.w);
            if (p.write_x) *reinterpret_cast<float4*>(p.x + size_t(t) * E + i) = o;
            if (p.xb) *reinterpret_cast<uint2*>(p.xb + size_t(t) * E + i) = gb_pack4(o);
            if (p.h) {
                const size_t at = size_t(blockIdx.x) * E + i;
                if (p.h_dtype == GB_F32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(p.h) + at) = o;
                else *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p.h) + at) = gb_pack4(o);
            }
        }
    }
}

__global__ void __launch_bounds__(256) layernorm_kernel(const LnParams p) {
    extern __shared__ float ln_row[];
    __shared__ float red1[32], red2[32];
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int E = p.E, t = p.rows ? p.rows[blockIdx.x] : int(blockIdx.x);
    float s = 0.f;
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
        float v = p.alpha * p.x[size_t(t) * E + i];
        if (p.y) v += gb_load(p.y, p.y_dtype, size_t(t) * p.ldy + i);
        if (p.z) {
            for (int r = 0; r < p.top; ++r) {
                const int pair = t * p.top + r;
                v = fmaf(p.weights[pair], p.z[size_t(p.place_of ? p.place_of[pair] : pair) * E + i], v);
            }
        }
        ln_row[i] = v;
        s += v;
    }
    const float mean = ln_block_sum(s, red1) / float(E);
    float ss = 0.f;
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
        const float d = ln_row[i] - mean;
        ln_row[i] = d;
        ss = fmaf(d, d, ss);
    }
    const float f = 1.f / sqrtf(ln_block_sum(ss, red2) / float(E) + p.eps);
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
        const float o = ln_row[i] * f * gb_load(p.w, p.w_dtype, i);
        if (p.write_x) p.x[size_t(t) * E + i] = o;
        if (p.xb) p.xb[size_t(t) * E + i] = __float2bfloat16_rn(o);
        if (p.h) gb_store(p.h, p.h_dtype, size_t(blockIdx.x) * E + i, o);
    }
}

}  // namespace

// x float32 [T, E] contiguous; y [T, E] rows ldy apart or null; z float32 [T * top, E] contiguous with weights [T, top] and
// place_of [T * top] (or null: the pairs' own order), or null; rows: n_rows row numbers or null (n_rows = T); w [E]; h
// [n_rows, E] contiguous, xb bfloat16 [T, E] contiguous, each or null; write_x 0: x is left as it is.
GB_API int gb_layernorm(float* x, const void* y, int y_dtype, long long ldy, const float* z, const float* weights,
                        const int* place_of, int top, float alpha, const void* w, int w_dtype, float eps, const int* rows,
                        int n_rows, int E, void* h, int h_dtype, void* xb, int write_x, cudaStream_t stream) {
    GB_REQUIRE(x && w && gb_is_dtype(w_dtype) && eps > 0.f && E > 0 && n_rows >= 0, "gb_layernorm: bad arguments");
    GB_REQUIRE((!y || gb_is_dtype(y_dtype)) && (!h || gb_is_dtype(h_dtype)), "gb_layernorm: bad dtype");
    GB_REQUIRE(!z || (weights && top > 0), "gb_layernorm: routed rows need weights");
    GB_REQUIRE(size_t(E) * 4 <= 200 * 1024, "gb_layernorm: rows of %d entries do not fit shared memory", E);
    if (n_rows == 0) return 0;
    GB_REQUIRE(h || xb || write_x, "gb_layernorm: nowhere to put the result");
    LnParams p;
    p.x = x; p.y = y; p.z = z; p.weights = weights; p.place_of = place_of; p.rows = rows; p.w = w; p.h = h;
    p.xb = (__nv_bfloat16*)xb; p.ldy = ldy; p.alpha = alpha; p.eps = eps; p.y_dtype = y_dtype; p.w_dtype = w_dtype;
    p.h_dtype = h_dtype; p.top = top; p.E = E; p.write_x = write_x;
    const bool vec = E % 4 == 0 && E <= 16384 && gb_aligned(x, 16) && gb_aligned(w, w_dtype == GB_F32 ? 16 : 8) &&
                     (!y || (ldy % 4 == 0 && gb_aligned(y, y_dtype == GB_F32 ? 16 : 8))) && (!z || gb_aligned(z, 16)) &&
                     (!h || gb_aligned(h, h_dtype == GB_F32 ? 16 : 8)) && (!xb || gb_aligned(xb, 8));
    if (vec) {
        const int pieces = E / 4;
        // few rows: few pieces per thread, which shortens a row's way through the block; many rows: four pieces per thread,
        // so that all rows of a step are under way at once (2,048 rows of 2,048: 22 us with one piece)
        const int nv = pieces > 2048 ? 8 : n_rows >= 256 || pieces > 1024 ? 4 : pieces > 512 ? 2 : 1;
        const int threads = ((pieces + nv - 1) / nv + 31) / 32 * 32;
        if (nv == 1) gb_launch(layernorm_vec_kernel<1>, dim3(n_rows), dim3(threads), 0, stream, p);
        else if (nv == 2) gb_launch(layernorm_vec_kernel<2>, dim3(n_rows), dim3(threads), 0, stream, p);
        else if (nv == 4) gb_launch(layernorm_vec_kernel<4>, dim3(n_rows), dim3(threads), 0, stream, p);
        else gb_launch(layernorm_vec_kernel<8>, dim3(n_rows), dim3(threads), 0, stream, p);
    } else {
        const size_t smem = size_t(E) * 4;
        if (smem > 48 * 1024 &&
            cudaFuncSetAttribute(layernorm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)) != cudaSuccess)
            return gb_fail("gb_layernorm: cannot get %zu bytes of shared memory", smem);
        gb_launch(layernorm_kernel, dim3(n_rows), dim3(256), smem, stream, p);
    }
    GB_LAUNCH_OK("gb_layernorm");
    return 0;
}

// out[t,:] = in[t,:] / sqrt(mean(in[t,:]^2) + eps) * w: the norm of a low-rank row between two projections.  One warp per
// row, four rows per block; the row is read twice, the second time from cache.
__global__ void __launch_bounds__(128) rms_rows_kernel(const void* __restrict__ in, int in_dtype, long long ldi, int T, int C,
                                                       const void* __restrict__ w, int w_dtype, float eps, void* __restrict__ out,
                                                       int out_dtype, long long ldo, int vec) {
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= T) return;
    float ss = 0.f;
    if (vec) {
        for (int i = 4 * lane; i < C; i += 128) {
            const float4 v = gb_load4(in, in_dtype, size_t(t) * ldi + i);
            ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
        }
    } else {
        for (int i = lane; i < C; i += 32) {
            const float v = gb_load(in, in_dtype, size_t(t) * ldi + i);
            ss = fmaf(v, v, ss);
        }
    }
    const float f = 1.f / sqrtf(gb_warp_sum(ss) / float(C) + eps);
    if (vec) {
        for (int i = 4 * lane; i < C; i += 128) {
            const float4 v = gb_load4(in, in_dtype, size_t(t) * ldi + i), g = gb_load4(w, w_dtype, i);
            const float4 o = make_float4(v.x * f * g.x, v.y * f * g.y, v.z * f * g.z, v.w * f * g.w);
            if (out_dtype == GB_F32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(out) + size_t(t) * ldo + i) = o;
            else *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(out) + size_t(t) * ldo + i) = gb_pack4(o);
        }
    } else {
        for (int i = lane; i < C; i += 32)
            gb_store(out, out_dtype, size_t(t) * ldo + i, gb_load(in, in_dtype, size_t(t) * ldi + i) * f * gb_load(w, w_dtype, i));
    }
}

GB_API int gb_rms_rows(const void* in, int in_dtype, long long ldi, int T, int C, const void* w, int w_dtype, float eps, void* out,
                       int out_dtype, long long ldo, cudaStream_t stream) {
    GB_REQUIRE(gb_is_dtype(in_dtype) && gb_is_dtype(w_dtype) && gb_is_dtype(out_dtype), "gb_rms_rows: bad dtype");
    GB_REQUIRE(in && w && out && T >= 0 && C > 0 && eps > 0.f && ldi >= C && ldo >= C, "gb_rms_rows: bad sizes T=%d C=%d", T, C);
    if (T == 0) return 0;
    const bool vec = C % 4 == 0 && ldi % 4 == 0 && ldo % 4 == 0 && gb_aligned(in, in_dtype == GB_F32 ? 16 : 8) &&
                     gb_aligned(w, w_dtype == GB_F32 ? 16 : 8) && gb_aligned(out, out_dtype == GB_F32 ? 16 : 8);
    gb_launch(rms_rows_kernel, dim3((T + 3) / 4), dim3(128), 0, stream, in, in_dtype, ldi, T, C, w, w_dtype, eps, out, out_dtype, ldo, int(vec));
    GB_LAUNCH_OK("gb_rms_rows");
    return 0;
}
