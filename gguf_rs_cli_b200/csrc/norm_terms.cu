// RMS norm of the residual stream with a waiting term that is not a plain row: for each output row r (source row
// s = rows ? rows[r] : r)
//   u = gate[s] * y[s,:] + sum_k weights[s,k] * z[row(s,k),:]      (y, its gate and the routed rows z each optional)
//   v = x[s,:] + scale * u                                         (written back to x when write_x)
//   out[r,:] = v / sqrt(mean(v^2) + eps) * w
// row(s,k) is s * top + k, or place_of[s * top + k] when the rows z lie in another order; the sum runs in the order of the
// choices.  It serves layers whose sublayers' results enter the stream with a constant factor, and mixtures of experts
// whose weighted sum (with a shared expert that a number per token gates) then costs no kernel of its own.  All in 32-bit.
//
// One block per row.  Rows of up to 16,384 entries that start on 16 bytes stay in registers between the passes; other
// rows lie in shared memory.
#include "common.cuh"

namespace {

struct NtParams {
    float* x;                  // [T, E] contiguous
    const void* y;             // [T, E] rows ldy apart, or null
    const float* gate;         // [T] or null
    const float* z;            // [T * top, E] contiguous, or null
    const float* weights;      // [T, top]
    const int* place_of;       // [T * top] or null
    const int* rows;
    const void* w;
    void* out;
    long long ldy;
    float scale, eps;
    int y_dtype, w_dtype, out_dtype, top, E, write_x;
};

__device__ __forceinline__ float nt_block_sum(float v, float* red) {
    v = gb_warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
    for (int k = 0; k < int(blockDim.x >> 5); ++k) tot += red[k];
    return tot;
}

// NV pieces of four entries per thread: piece k of thread i starts at entry 4 * (i + k * blockDim.x)
template <int NV>
__global__ void __launch_bounds__(NV < 4 ? 1024 : 512) add_rmsnorm_terms_vec_kernel(const NtParams p) {
    __shared__ float red[32];
    const int E = p.E;
    constexpr bool EARLY = NV <= 2;        // the weights do not depend on the kernel before this one
    float4 wv[EARLY ? NV : 1];
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
    const float gt = p.gate ? p.gate[t] : 1.f;
    float4 v[NV], u[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        v[k] = u[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < E) {
            v[k] = *reinterpret_cast<const float4*>(p.x + size_t(t) * E + i);
            if (p.y) {
                const float4 y = gb_load4(p.y, p.y_dtype, size_t(t) * p.ldy + i);
                u[k] = make_float4(gt * y.x, gt * y.y, gt * y.z, gt * y.w);
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
                    u[k].x = fmaf(wr, y.x, u[k].x); u[k].y = fmaf(wr, y.y, u[k].y);
                    u[k].z = fmaf(wr, y.z, u[k].z); u[k].w = fmaf(wr, y.w, u[k].w);
                }
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        v[k].x = fmaf(p.scale, u[k].x, v[k].x); v[k].y = fmaf(p.scale, u[k].y, v[k].y);
        v[k].z = fmaf(p.scale, u[k].z, v[k].z); v[k].w = fmaf(p.scale, u[k].w, v[k].w);
        ss = fmaf(v[k].x, v[k].x, ss); ss = fmaf(v[k].y, v[k].y, ss); ss = fmaf(v[k].z, v[k].z, ss); ss = fmaf(v[k].w, v[k].w, ss);
    }
    const float rms = sqrtf(nt_block_sum(ss, red) / float(E) + p.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        if (i < E) {
            if (p.write_x) *reinterpret_cast<float4*>(p.x + size_t(t) * E + i) = v[k];
            const float4 g = EARLY ? wv[EARLY ? k : 0] : gb_load4(p.w, p.w_dtype, i);
            const float4 o = make_float4(v[k].x / rms * g.x, v[k].y / rms * g.y, v[k].z / rms * g.z, v[k].w / rms * g.w);
            const size_t at = size_t(blockIdx.x) * E + i;
            if (p.out_dtype == GB_F32) *reinterpret_cast<float4*>(reinterpret_cast<float*>(p.out) + at) = o;
            else *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p.out) + at) = gb_pack4(o);
        }
    }
}

__global__ void __launch_bounds__(256) add_rmsnorm_terms_kernel(const NtParams p) {
    extern __shared__ float nt_row[];
    __shared__ float red[32];
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int E = p.E, t = p.rows ? p.rows[blockIdx.x] : int(blockIdx.x);
    const float gt = p.gate ? p.gate[t] : 1.f;
    float ss = 0.f;
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
        float u = p.y ? gt * gb_load(p.y, p.y_dtype, size_t(t) * p.ldy + i) : 0.f;
        if (p.z) {
            for (int r = 0; r < p.top; ++r) {
                const int pair = t * p.top + r;
                u = fmaf(p.weights[pair], p.z[size_t(p.place_of ? p.place_of[pair] : pair) * E + i], u);
            }
        }
        const float v = fmaf(p.scale, u, p.x[size_t(t) * E + i]);
        nt_row[i] = v;
        if (p.write_x) p.x[size_t(t) * E + i] = v;
        ss = fmaf(v, v, ss);
    }
    const float rms = sqrtf(nt_block_sum(ss, red) / float(E) + p.eps);
    for (int i = threadIdx.x; i < E; i += blockDim.x)
        gb_store(p.out, p.out_dtype, size_t(blockIdx.x) * E + i, nt_row[i] / rms * gb_load(p.w, p.w_dtype, i));
}

__global__ void __launch_bounds__(256) scale_rows_kernel(float* __restrict__ x, const float* __restrict__ f, int E, long long total) {
    const long long i = blockIdx.x * 256LL + threadIdx.x;
    if (i < total) x[i] *= f[i / E];
}

}  // namespace

// x float32 [T, E] contiguous; y [T, E] rows ldy apart or null, gate float32 [T] or null (1); z float32 [T * top, E] contiguous
// with weights [T, top] and place_of [T * top] (or null: the pairs' own order), or null; w [E]; rows: n_rows row numbers
// or null (n_rows = T); out [n_rows, E] contiguous; write_x 0: x is left as it is.
GB_API int gb_add_rmsnorm_terms(float* x, const void* y, int y_dtype, long long ldy, const float* gate, const float* z,
                                const float* weights, const int* place_of, int top, float scale, const void* w, int w_dtype,
                                float eps, const int* rows, int n_rows, int E, void* out, int out_dtype, int write_x,
                                cudaStream_t stream) {
    if (n_rows == 0) return 0;
    GB_REQUIRE(x && w && out && gb_is_dtype(w_dtype) && gb_is_dtype(out_dtype) && eps > 0.f && E > 0 && n_rows >= 0,
               "gb_add_rmsnorm_terms: bad arguments");
    GB_REQUIRE(!y || gb_is_dtype(y_dtype), "gb_add_rmsnorm_terms: bad dtype");
    GB_REQUIRE(!z || (weights && top > 0), "gb_add_rmsnorm_terms: routed rows need weights");
    GB_REQUIRE(!rows || !write_x, "gb_add_rmsnorm_terms: chosen rows leave x as it is");
    GB_REQUIRE(size_t(E) * 4 <= 200 * 1024, "gb_add_rmsnorm_terms: rows of %d entries do not fit shared memory", E);
    NtParams p;
    p.x = x; p.y = y; p.gate = gate; p.z = z; p.weights = weights; p.place_of = place_of; p.rows = rows; p.w = w; p.out = out;
    p.ldy = ldy; p.scale = scale; p.eps = eps; p.y_dtype = y_dtype; p.w_dtype = w_dtype; p.out_dtype = out_dtype; p.top = top;
    p.E = E; p.write_x = write_x;
    const bool vec = E % 4 == 0 && E <= 16384 && gb_aligned(x, 16) && gb_aligned(w, w_dtype == GB_F32 ? 16 : 8) &&
                     (!y || (ldy % 4 == 0 && gb_aligned(y, y_dtype == GB_F32 ? 16 : 8))) && (!z || gb_aligned(z, 16)) &&
                     gb_aligned(out, out_dtype == GB_F32 ? 16 : 8);
    if (vec) {
        // few rows: few pieces per thread, which shortens a row's way through the block; many rows: more of them under way
        const int pieces = E / 4;
        const int nv = pieces > 2048 ? 8 : n_rows >= 256 || pieces > 1024 ? 4 : pieces > 512 ? 2 : 1;
        const int threads = ((pieces + nv - 1) / nv + 31) / 32 * 32;
        if (nv == 1) gb_launch(add_rmsnorm_terms_vec_kernel<1>, dim3(n_rows), dim3(threads), 0, stream, p);
        else if (nv == 2) gb_launch(add_rmsnorm_terms_vec_kernel<2>, dim3(n_rows), dim3(threads), 0, stream, p);
        else if (nv == 4) gb_launch(add_rmsnorm_terms_vec_kernel<4>, dim3(n_rows), dim3(threads), 0, stream, p);
        else gb_launch(add_rmsnorm_terms_vec_kernel<8>, dim3(n_rows), dim3(threads), 0, stream, p);
    } else {
        const size_t smem = size_t(E) * 4;
        if (smem > 48 * 1024 &&
            cudaFuncSetAttribute(add_rmsnorm_terms_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)) != cudaSuccess)
            return gb_fail("gb_add_rmsnorm_terms: cannot get %zu bytes of shared memory", smem);
        gb_launch(add_rmsnorm_terms_kernel, dim3(n_rows), dim3(256), smem, stream, p);
    }
    GB_LAUNCH_OK("gb_add_rmsnorm_terms");
    return 0;
}

// x float32 [T, E] contiguous: row t times f[t].
GB_API int gb_scale_rows(float* x, const float* f, int T, int E, cudaStream_t stream) {
    GB_REQUIRE(x && f && T >= 0 && E > 0, "gb_scale_rows: bad arguments");
    if (T == 0) return 0;
    const long long total = (long long)T * E;
    scale_rows_kernel<<<unsigned((total + 255) / 256), 256, 0, stream>>>(x, f, E, total);
    GB_LAUNCH_OK("gb_scale_rows");
    return 0;
}
