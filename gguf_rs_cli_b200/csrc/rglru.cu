// The real-gated linear recurrent unit: per channel c, with u the convolved input and z the gates' products,
//   r = sigmoid(z_r + b_r);  i = sigmoid(z_i + b_i);  log a = -rate_c r  (rate = 8 softplus(lam), the caller's)
//   S <- a S + sqrt(1 - a^2) i u;   out = S gelu_tanh(y)
// S is one 32-bit number per channel and sequence, carried from step to step; gates, decays with their logarithms and
// exponentials and the state are 32-bit.  1 - a^2 is taken as -expm1(2 log a), which keeps its digits where a is near 1.
//
// One thread per channel walks a sequence's tokens.  Long prompts: the sequence is cut into segments that run side by
// side.  A first pass walks every segment from zero and keeps what it ends with and the sum of its log a; since a
// stretch of tokens multiplies the state by exp(sum of log a), the state in front of each segment follows by a short walk
// over the segments; the second pass then walks every segment from its true state and writes the results.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int RG_THREADS = 64;
constexpr int RG_SEGMENT = 64;          // tokens per segment of a long prompt
constexpr int RG_SEGMENT_FROM = 128;    // a sequence of more new tokens than this is cut
constexpr int RG_AHEAD = 4;             // tokens whose rows are on their way while one is worked on

struct RgParams {
    const void *u, *y;            // [T, W]
    const float* z;               // [T, 2W]: per block of n channels its n columns of r, then its n of i
    const float *b_r, *b_i, *rate;
    float* state;                 // [slots, W]
    void* out;
    float* seg;                   // [B, segments, 2, W]: end state, then sum of log a; after the carry: state in front
    long long ldu, ldy, ldz, ldo;
    const int *cu, *slots, *qlens;
    int dtype, out_dtype, W, n, mode, max_segments;
};

__device__ __forceinline__ float rg_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }

// mode 0: whole sequences; 1: segments from zero, keeping end state and sum of log a; 2: segments from their true state
__global__ void __launch_bounds__(RG_THREADS) rglru_scan_kernel(const RgParams p) {
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int b = blockIdx.y, c = blockIdx.x * RG_THREADS + threadIdx.x;
    const int slot = p.slots[b];
    if (slot < 0 || c >= p.W) return;
    int first = p.cu[b], n_tok = p.qlens[b];
    float* rec = nullptr;
    if (p.mode) {
        const int seg = blockIdx.z;
        if (seg * RG_SEGMENT >= n_tok) return;
        first += seg * RG_SEGMENT;
        n_tok = min(RG_SEGMENT, n_tok - seg * RG_SEGMENT);
        rec = p.seg + (size_t(b) * p.max_segments + seg) * 2 * p.W + c;
    }
    const int zr = (c / p.n) * 2 * p.n + c % p.n, zi = zr + p.n;
    const float br = p.b_r[c], bi = p.b_i[c], rate = p.rate[c];
    float S = p.mode == 0 ? p.state[size_t(slot) * p.W + c] : p.mode == 2 ? rec[0] : 0.f, total = 0.f;
    for (int t0 = 0; t0 < n_tok; t0 += RG_AHEAD) {
        float zrv[RG_AHEAD], ziv[RG_AHEAD], uv[RG_AHEAD], yv[RG_AHEAD];
#pragma unroll
        for (int j = 0; j < RG_AHEAD; ++j) {
            zrv[j] = ziv[j] = uv[j] = yv[j] = 0.f;
            if (t0 + j < n_tok) {
                const size_t t = size_t(first + t0 + j);
                zrv[j] = p.z[t * p.ldz + zr];
                ziv[j] = p.z[t * p.ldz + zi];
                uv[j] = gb_load(p.u, p.dtype, t * p.ldu + c);
                if (p.mode != 1) yv[j] = gb_load(p.y, p.dtype, t * p.ldy + c);
            }
        }
#pragma unroll
        for (int j = 0; j < RG_AHEAD; ++j) {
            if (t0 + j >= n_tok) break;
            const float log_a = -rate * rg_sigmoid(zrv[j] + br);
            S = fmaf(expf(log_a), S, sqrtf(-expm1f(2.f * log_a)) * (rg_sigmoid(ziv[j] + bi) * uv[j]));
            if (p.mode == 1) total += log_a;
            else gb_store(p.out, p.out_dtype, size_t(first + t0 + j) * p.ldo + c, S * gb_gate_act(yv[j], GB_ACT_GELU_TANH));
        }
    }
    if (p.mode == 0) p.state[size_t(slot) * p.W + c] = S;
    else if (p.mode == 1) { rec[0] = S; rec[p.W] = total; }
}

// From the segments' own end states to the states in front of them, in place, and the sequence's new state.
__global__ void __launch_bounds__(RG_THREADS) rglru_carry_kernel(float* __restrict__ state, float* __restrict__ seg,
                                                                 const int* __restrict__ slots, const int* __restrict__ qlens,
                                                                 int W, int max_segments) {
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int b = blockIdx.y, c = blockIdx.x * RG_THREADS + threadIdx.x;
    const int slot = slots[b], n = qlens[b];
    if (slot < 0 || n <= 0 || c >= W) return;
    float S = state[size_t(slot) * W + c];
    const int segs = (n + RG_SEGMENT - 1) / RG_SEGMENT;
    for (int s = 0; s < segs; ++s) {
        float* rec = seg + (size_t(b) * max_segments + s) * 2 * W + c;
        const float local = rec[0], a = expf(rec[W]);
        rec[0] = S;
        S = fmaf(a, S, local);
    }
    state[size_t(slot) * W + c] = S;
}

}  // namespace

// Floats of scratch for the segments of a step whose longest sequence brings max_qlen tokens (0: walked whole).
GB_API long long gb_rglru_segment_floats(int B, int max_qlen, int W) {
    if (max_qlen <= RG_SEGMENT_FROM) return 0;
    return (long long)B * ((max_qlen + RG_SEGMENT - 1) / RG_SEGMENT) * 2 * W;
}

// u [T, W] rows ldu apart, y [T, W] rows ldy apart (one dtype); z float32 [T, 2W] rows ldz apart; b_r, b_i, rate [W];
// state [slots, W] float32, read and renewed; out [T, W] rows ldo apart.
GB_API int gb_rglru(const void* u, const void* y, int dtype, long long ldu, const float* z, long long ldy, long long ldz, const float* b_r,
                    const float* b_i, const float* rate, float* state, void* out, int out_dtype, long long ldo, const int* cu,
                    const int* slots, const int* qlens, int T, int B, int W, int blocks, int max_qlen, float* seg,
                    cudaStream_t stream) {
    GB_REQUIRE(gb_is_dtype(dtype) && gb_is_dtype(out_dtype), "gb_rglru: bad dtype");
    GB_REQUIRE(W > 0 && blocks > 0 && W % blocks == 0, "gb_rglru: %d channels do not form %d equal blocks", W, blocks);
    GB_REQUIRE(B <= 65535, "gb_rglru: too many sequences (%d)", B);
    if (T == 0 || B == 0) return 0;
    RgParams p;
    p.u = u; p.y = y; p.z = z; p.b_r = b_r; p.b_i = b_i; p.rate = rate; p.state = state; p.out = out; p.seg = seg;
    p.ldu = ldu; p.ldy = ldy; p.ldz = ldz; p.ldo = ldo; p.cu = cu; p.slots = slots; p.qlens = qlens; p.dtype = dtype;
    p.out_dtype = out_dtype; p.W = W; p.n = W / blocks; p.mode = 0; p.max_segments = 1;
    const dim3 grid((W + RG_THREADS - 1) / RG_THREADS, B);
    if (max_qlen <= RG_SEGMENT_FROM || !seg) {
        gb_launch(rglru_scan_kernel, grid, dim3(RG_THREADS), 0, stream, p);
        GB_LAUNCH_OK("gb_rglru");
        return 0;
    }
    p.max_segments = (max_qlen + RG_SEGMENT - 1) / RG_SEGMENT;
    GB_REQUIRE(p.max_segments <= 65535, "gb_rglru: %d tokens of one sequence are too many for one step", max_qlen);
    p.mode = 1;
    gb_launch(rglru_scan_kernel, dim3(grid.x, B, p.max_segments), dim3(RG_THREADS), 0, stream, p);
    GB_LAUNCH_OK("gb_rglru (segments)");
    gb_launch(rglru_carry_kernel, grid, dim3(RG_THREADS), 0, stream, state, seg, slots, qlens, W, p.max_segments);
    GB_LAUNCH_OK("gb_rglru (carry)");
    p.mode = 2;
    gb_launch(rglru_scan_kernel, dim3(grid.x, B, p.max_segments), dim3(RG_THREADS), 0, stream, p);
    GB_LAUNCH_OK("gb_rglru");
    return 0;
}
