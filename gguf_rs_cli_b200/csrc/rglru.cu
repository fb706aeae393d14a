// The real-gated linear recurrent unit: per channel c, with u the convolved input and z the gates' products,
//   r = sigmoid(z_r + b_r);  i = sigmoid(z_i + b_i);  log a = -rate_c r  (rate = 8 softplus(lam), the caller's)
//   S <- a S + sqrt(1 - a^2) i u;   out = S gelu_tanh(y)
// S is one 32-bit number per channel and sequence, carried from step to step; gates, decays with their logarithms and
// exponentials and the state are 32-bit.  Where a is near 1 its rounding to 32 bits would be the same error at every token
// of a long memory; so a enters as a - 1 = expm1(log a): S <- S + ((a - 1) S + input), 1 - a^2 = -(a - 1)(2 + (a - 1)), and
// products of decays are exponentials of sums of log a.
//
// One thread per channel walks a sequence's tokens.  Long prompts: the sequence is cut into segments that run side by
// side.  A first pass walks every segment from zero and keeps what it ends with and the sum of its log a; since a
// stretch of tokens multiplies the state by exp(sum of log a), the state in front of each segment follows by a short walk
// over the segments; the second pass then walks every segment from its true state and writes the results.  Prompts in
// bfloat16 and single tokens have kernels of their own that make the gates' products as well.
#include <math.h>

#include "common.cuh"
#include "mma_tiles.cuh"

namespace {

constexpr int RG_THREADS = 64;
constexpr int RG_SEGMENT = 64;          // tokens per segment of a prompt that brings more than that
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
// sqrt(1 - a^2) times v, from a - 1
__device__ __forceinline__ float rg_input(float am1, float v) { return sqrtf(-am1 * (2.f + am1)) * v; }

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
            const float am1 = expm1f(log_a);
            S += fmaf(am1, S, rg_input(am1, rg_sigmoid(ziv[j] + bi) * uv[j]));
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
    constexpr int AHEAD = 16;                 // segments whose records are on their way together
    for (int s0 = 0; s0 < segs; s0 += AHEAD) {
        float* rec = seg + (size_t(b) * max_segments + s0) * 2 * W + c;
        float local[AHEAD], total[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            local[j] = s0 + j < segs ? rec[size_t(j) * 2 * W] : 0.f;
            total[j] = s0 + j < segs ? rec[size_t(j) * 2 * W + W] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (s0 + j >= segs) break;
            rec[size_t(j) * 2 * W] = S;
            S += fmaf(expm1f(total[j]), S, local[j]);
        }
    }
    state[size_t(slot) * W + c] = S;
}

// ------------------------------------------------------------------------------------------------ prompts, gates and walk in one
// A block takes a segment of 64 tokens and 64 channels of one of the gates' blocks: the gates' products on mma.sync (the
// segment's rows of u against the r rows and the i rows of its channels; a thread then holds both of a channel's gates for
// its tokens), decays and inputs from the 32-bit sums, and the walk over the segment, one thread per channel.  Sequences of
// one segment are finished there (mode 0).  Else (mode 1) the walk starts from zero and leaves, for every token and channel,
// its state and what a state in front of the segment is multiplied by until there; with the states in front of the segments
// (rglru_carry_kernel) rglru_finish_kernel then adds up and applies the other branch, entry by entry.
constexpr int RF_TOK = RG_SEGMENT, RF_CH = 64, RF_K = 64, RF_THREADS = 256;

struct RfParams {
    const __nv_bfloat16 *u, *y, *gates;      // gates [blocks, 2n, n]: a block's r rows, then its i rows
    const float *b_r, *b_i, *rate;
    float *state, *seg;
    float* local;                            // [T, 2, W]: states of walks from zero, factors of the states in front
    __nv_bfloat16* out;
    long long ldu, ldy, ldo;
    const int *cu, *slots, *qlens;
    int W, n, slices, mode, max_segments;
};

__device__ __forceinline__ float rf_sigmoid(float v) { return __fdividef(1.f, 1.f + exp2f(-1.4426950408889634f * v)); }

__device__ __forceinline__ void rf_cp16(void* dst, const void* src, bool valid) {
    const unsigned d = unsigned(__cvta_generic_to_shared(dst));
    const int bytes = valid ? 16 : 0;                       // 0 source bytes: zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}

__global__ void __launch_bounds__(RF_THREADS) rglru_fused_kernel(const RfParams p) {
    using namespace gbmma;
    extern __shared__ __align__(128) unsigned char rf_smem[];
    constexpr int STAGE = (RF_TOK + 2 * RF_CH) * RF_K;      // entries of one stage: u [64][64], then r and i rows [128][64]
    __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(rf_smem);
    float* as = reinterpret_cast<float*>(rf_smem);          // [64][64] a - 1 (then states), over the stages
    float* bs = as + RF_TOK * RF_CH;                        // [64][64] inputs
    float* ls = bs + RF_TOK * RF_CH;                        // [64][64] log a, then their running sums
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int blk = blockIdx.x / p.slices, c0 = (blockIdx.x % p.slices) * RF_CH;       // the gates' block, first channel in it
    const int b = blockIdx.z, seg = blockIdx.y;
    const int slot = p.slots[b], n_tok = min(RF_TOK, p.qlens[b] - seg * RF_TOK);
    if (slot < 0 || n_tok <= 0) return;
    const int t0 = p.cu[b] + seg * RF_TOK, n = p.n, nch = min(RF_CH, n - c0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const __nv_bfloat16* ublk = p.u + size_t(t0) * p.ldu + size_t(blk) * n;
    const __nv_bfloat16* gblk = p.gates + size_t(blk) * 2 * n * n;
    auto load_stage = [&](int k0, int st) {
        __nv_bfloat16* us = stages + st * STAGE;
        for (int i = tid; i < (RF_TOK + 2 * RF_CH) * (RF_K / 8); i += RF_THREADS) {
            const int r = i >> 3, c = i & 7, k = k0 + 8 * c;
            if (r < RF_TOK) {
                const bool ok = r < n_tok && k < n;
                rf_cp16(us + swz<RF_K>(r, c), ok ? ublk + size_t(r) * p.ldu + k : ublk, ok);
            } else {
                const int rr = r - RF_TOK, ch = rr & (RF_CH - 1);
                const bool ok = ch < nch && k < n;
                rf_cp16(us + RF_TOK * RF_K + swz<RF_K>(rr, c), ok ? gblk + size_t((rr < RF_CH ? 0 : n) + c0 + ch) * n + k : gblk, ok);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int tw = warp & 3, cw = warp >> 2;                // 16 tokens, 32 channels of this warp
    float acc[8][4];                                        // channels 8j of r (j < 4), then of i
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const int steps = (n + RF_K - 1) / RF_K;
    load_stage(0, 0);
    for (int s = 0; s < steps; ++s) {
        if (s + 1 < steps) load_stage((s + 1) * RF_K, (s + 1) & 1);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const __nv_bfloat16* us = stages + (s & 1) * STAGE;
        const __nv_bfloat16* ws = us + RF_TOK * RF_K;
#pragma unroll
        for (int kk = 0; kk < RF_K / 16; ++kk) {
            unsigned a[4];
            ldsm4(a, us + swz<RF_K>(tw * 16 + (lane & 15), 2 * kk + (lane >> 4)));
#pragma unroll
            for (int j2 = 0; j2 < 4; ++j2) {                // 16 rows at a time: two of r, two of i
                unsigned w[4];
                const int r0 = (j2 >> 1) * RF_CH + cw * 32 + (j2 & 1) * 16;
                ldsm4(w, ws + swz<RF_K>(r0 + (lane & 7) + ((lane >> 4) << 3), 2 * kk + ((lane >> 3) & 1)));
                mma(acc[2 * j2], a, w[0], w[1]);
                mma(acc[2 * j2 + 1], a, w[2], w[3]);
            }
        }
        __syncthreads();
    }
    // ---- decays and inputs; the stages are free
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int cl = cw * 32 + 8 * j + 2 * (lane & 3);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int tl = tw * 16 + (lane >> 2) + (e >> 1) * 8, ch = cl + (e & 1);
            float av = 0.f, bv = 0.f, lv = 0.f;
            if (tl < n_tok && ch < nch) {
                const int c = blk * n + c0 + ch;
                lv = -p.rate[c] * rf_sigmoid(acc[j][e] + p.b_r[c]);
                av = expm1f(lv);
                bv = rg_input(av, rf_sigmoid(acc[j + 4][e] + p.b_i[c]) * __bfloat162float(ublk[size_t(tl) * p.ldu + c0 + ch]));
            }
            as[tl * RF_CH + ch] = av;
            bs[tl * RF_CH + ch] = bv;
            ls[tl * RF_CH + ch] = lv;
        }
    }
    __syncthreads();
    if (tid < nch) {
        const int c = blk * n + c0 + tid;
        float S = p.mode == 0 ? p.state[size_t(slot) * p.W + c] : 0.f, total = 0.f;
#pragma unroll 8
        for (int t = 0; t < n_tok; ++t) {
            S += fmaf(as[t * RF_CH + tid], S, bs[t * RF_CH + tid]);
            as[t * RF_CH + tid] = S;
            total += ls[t * RF_CH + tid];
            ls[t * RF_CH + tid] = total;
        }
        if (p.mode == 0) {
            p.state[size_t(slot) * p.W + c] = S;
        } else {
            float* rec = p.seg + (size_t(b) * p.max_segments + seg) * 2 * p.W + c;
            rec[0] = S;
            rec[p.W] = total;
        }
    }
    __syncthreads();
    for (int i = tid; i < n_tok * (RF_CH / 2); i += RF_THREADS) {
        const int tl = i / (RF_CH / 2), ch = 2 * (i % (RF_CH / 2));
        if (ch >= nch) continue;                            // n is even: pairs are whole
        const size_t col = size_t(blk) * n + c0 + ch;
        const float2 S = *reinterpret_cast<const float2*>(as + tl * RF_CH + ch);
        if (p.mode == 0) {
            const float2 yv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p.y + size_t(t0 + tl) * p.ldy + col));
            *reinterpret_cast<__nv_bfloat162*>(p.out + size_t(t0 + tl) * p.ldo + col) =
                __floats2bfloat162_rn(S.x * gb_gate_act(yv.x, GB_ACT_GELU_TANH), S.y * gb_gate_act(yv.y, GB_ACT_GELU_TANH));
        } else {
            const float2 l = *reinterpret_cast<const float2*>(ls + tl * RF_CH + ch);
            float* o = p.local + size_t(t0 + tl) * 2 * p.W + col;
            *reinterpret_cast<float2*>(o) = S;
            *reinterpret_cast<float2*>(o + p.W) = make_float2(expf(l.x), expf(l.y));
        }
    }
}

// out = (local state + factor * state in front of the token's segment) * gelu_tanh(y), four channels per thread.
__global__ void __launch_bounds__(128) rglru_finish_kernel(const RfParams p, const int* __restrict__ seq_of) {
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int t = blockIdx.x, c = 4 * (blockIdx.y * 128 + threadIdx.x);
    const int b = seq_of[t];
    if (c >= p.W || b < 0 || p.slots[b] < 0) return;
    const int seg = (t - p.cu[b]) / RF_TOK;
    const float4 S0 = *reinterpret_cast<const float4*>(p.seg + (size_t(b) * p.max_segments + seg) * 2 * p.W + c);
    const float* l = p.local + size_t(t) * 2 * p.W + c;
    const float4 s = *reinterpret_cast<const float4*>(l), f = *reinterpret_cast<const float4*>(l + p.W);
    const float4 y = gb_load4(p.y, GB_BF16, size_t(t) * p.ldy + c);
    *reinterpret_cast<uint2*>(p.out + size_t(t) * p.ldo + c) = gb_pack4(make_float4(
        fmaf(f.x, S0.x, s.x) * gb_gate_act(y.x, GB_ACT_GELU_TANH), fmaf(f.y, S0.y, s.y) * gb_gate_act(y.y, GB_ACT_GELU_TANH),
        fmaf(f.z, S0.z, s.z) * gb_gate_act(y.z, GB_ACT_GELU_TANH), fmaf(f.w, S0.w, s.w) * gb_gate_act(y.w, GB_ACT_GELU_TANH)));
}

// ------------------------------------------------------------------------------------------------ single tokens
// Every token is a sequence's own: the gates' products and the update in one kernel.  A block takes 8 tokens and 16 channels
// of one of the gates' blocks; lane l of every warp sums channel l's r (l < 16) or channel l - 16's i over the warp's share of
// the inputs, the warps' shares are added in warp order (their number follows from the block's size alone).
constexpr int RS_TOK = 8, RS_CH = 16;

struct RsParams {
    const void *u, *y;
    const void* gates;                       // [blocks, n (in), 2n (out)]
    const float *b_r, *b_i, *rate;
    float* state;
    void* out;
    long long ldu, ldy, ldo;
    const int *seq_of, *slots;
    int dtype, out_dtype, T, W, n;
};

template <typename TW, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) rglru_step_kernel(const RsParams p) {
    extern __shared__ float rs_sm[];                        // [8][n] rows of u, then [WARPS][8][32] partial sums
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int n = p.n, t0 = blockIdx.x * RS_TOK, blk = blockIdx.y, c0 = blockIdx.z * RS_CH;
    const int nt = min(RS_TOK, p.T - t0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* part = rs_sm + RS_TOK * n;
    for (int idx = threadIdx.x; idx < RS_TOK * n; idx += WARPS * 32) {
        const int tt = idx / n, i = idx - tt * n;
        rs_sm[idx] = tt < nt ? gb_load(p.u, p.dtype, size_t(t0 + tt) * p.ldu + size_t(blk) * n + i) : 0.f;
    }
    __syncthreads();
    float acc[RS_TOK];
#pragma unroll
    for (int tt = 0; tt < RS_TOK; ++tt) acc[tt] = 0.f;
    const int ch = c0 + (lane & 15), per = (n + WARPS - 1) / WARPS, i0 = warp * per, i1 = min(n, i0 + per);
    if (ch < n) {
        const TW* wp = reinterpret_cast<const TW*>(p.gates) + size_t(blk) * n * 2 * n + (lane >> 4) * n + ch;
#pragma unroll 8
        for (int i = i0; i < i1; ++i) {
            const float wv = gb_to_float(wp[size_t(i) * 2 * n]);
#pragma unroll
            for (int tt = 0; tt < RS_TOK; ++tt) acc[tt] = fmaf(rs_sm[tt * n + i], wv, acc[tt]);
        }
    }
#pragma unroll
    for (int tt = 0; tt < RS_TOK; ++tt) part[(warp * RS_TOK + tt) * 32 + lane] = acc[tt];
    __syncthreads();
    for (int idx = threadIdx.x; idx < nt * RS_CH; idx += WARPS * 32) {
        const int tt = idx / RS_CH, cl = idx - tt * RS_CH;
        if (c0 + cl >= n) continue;
        const int t = t0 + tt, b = p.seq_of[t], slot = b < 0 ? -1 : p.slots[b];
        if (slot < 0) continue;
        float zr = 0.f, zi = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
            zr += part[(w * RS_TOK + tt) * 32 + cl];
            zi += part[(w * RS_TOK + tt) * 32 + 16 + cl];
        }
        const int c = blk * n + c0 + cl;
        const float log_a = -p.rate[c] * rg_sigmoid(zr + p.b_r[c]);
        float* sp = p.state + size_t(slot) * p.W + c;
        const float am1 = expm1f(log_a), S0 = *sp;
        const float S = S0 + fmaf(am1, S0, rg_input(am1, rg_sigmoid(zi + p.b_i[c]) * rs_sm[tt * n + c0 + cl]));
        *sp = S;
        gb_store(p.out, p.out_dtype, size_t(t) * p.ldo + c, S * gb_gate_act(gb_load(p.y, p.dtype, size_t(t) * p.ldy + c), GB_ACT_GELU_TANH));
    }
}

}  // namespace

// Floats of scratch for the segments of a step whose longest sequence brings max_qlen tokens (0: walked whole).
GB_API long long gb_rglru_segment_floats(int B, int max_qlen, int W) {
    if (max_qlen <= RG_SEGMENT) return 0;
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
    if (max_qlen <= RG_SEGMENT || !seg) {
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

// Whether the fused kernel of prompts takes these blocks: bfloat16, n channels per block a multiple of 8.
GB_API int gb_rglru_fused_supported(int dtype, int n) { return dtype == GB_BF16 && n > 0 && n % 8 == 0; }

// Prompts, with the gates' products in the same kernels: u, y [T, W] bfloat16; gates [blocks, 2n, n] bfloat16 (n = W / blocks);
// the rest as gb_rglru.  seg: gb_rglru_segment_floats,
// local: 2 T W floats, both needed where a sequence brings more than 64 tokens.  One launch for steps of at most 64 tokens a sequence, else three.
GB_API int gb_rglru_fused(const void* u, long long ldu, const void* y, long long ldy, const void* gates, const float* b_r,
                          const float* b_i, const float* rate, float* state, void* out, long long ldo, const int* cu,
                          const int* slots, const int* qlens, const int* seq_of, int T, int B, int W, int blocks, int max_qlen, float* seg,
                          float* local, cudaStream_t stream) {
    GB_REQUIRE(W > 0 && blocks > 0 && W % blocks == 0 && gb_rglru_fused_supported(GB_BF16, W / blocks),
               "gb_rglru_fused: %d channels in %d blocks (of a multiple of 8 channels)", W, blocks);
    GB_REQUIRE(ldu % 8 == 0 && gb_aligned(u, 16) && gb_aligned(gates, 16) && ldy % 4 == 0 && ldo % 4 == 0 && gb_aligned(y, 8) && gb_aligned(out, 8) &&
               gb_aligned(seg, 16) && gb_aligned(local, 16),
               "gb_rglru_fused: misaligned operands");
    if (B == 0 || max_qlen <= 0) return 0;
    RfParams p;
    p.u = (const __nv_bfloat16*)u; p.y = (const __nv_bfloat16*)y; p.gates = (const __nv_bfloat16*)gates; p.b_r = b_r; p.b_i = b_i;
    p.rate = rate; p.state = state; p.seg = nullptr; p.local = nullptr; p.out = (__nv_bfloat16*)out; p.ldu = ldu; p.ldy = ldy; p.ldo = ldo; p.cu = cu;
    p.slots = slots; p.qlens = qlens; p.W = W; p.n = W / blocks; p.slices = (p.n + RF_CH - 1) / RF_CH; p.mode = 0;
    p.max_segments = (max_qlen + RF_TOK - 1) / RF_TOK;
    GB_REQUIRE(B <= 65535 && p.max_segments <= 65535, "gb_rglru_fused: %d sequences of up to %d tokens are too many for one step", B, max_qlen);
    constexpr int SMEM = 2 * (RF_TOK + 2 * RF_CH) * RF_K * 2;
    static_assert(SMEM >= 3 * RF_TOK * RF_CH * 4 && SMEM <= 48 * 1024, "the walk's arrays lie over the stages");
    const dim3 grid(blocks * p.slices, p.max_segments, B);
    if (p.max_segments == 1) {
        gb_launch(rglru_fused_kernel, grid, dim3(RF_THREADS), SMEM, stream, p);
        GB_LAUNCH_OK("gb_rglru_fused");
        return 0;
    }
    GB_REQUIRE(seg && local, "gb_rglru_fused: segments need scratch");
    p.seg = seg;
    p.local = local;
    p.mode = 1;
    gb_launch(rglru_fused_kernel, grid, dim3(RF_THREADS), SMEM, stream, p);
    GB_LAUNCH_OK("gb_rglru_fused (segments)");
    gb_launch(rglru_carry_kernel, dim3((W + RG_THREADS - 1) / RG_THREADS, B), dim3(RG_THREADS), 0, stream, state, seg, slots, qlens, W, p.max_segments);
    GB_LAUNCH_OK("gb_rglru_fused (carry)");
    gb_launch(rglru_finish_kernel, dim3(T, (W / 4 + 127) / 128), dim3(128), 0, stream, p, seq_of);
    GB_LAUNCH_OK("gb_rglru_fused");
    return 0;
}

// Single tokens (every sequence brings one), with the gates' products: gates [blocks, n (in), 2n (out)] of w_dtype, a block's r
// columns in front of its i columns; seq_of [T].
GB_API int gb_rglru_step(const void* u, const void* y, int dtype, long long ldu, long long ldy, const void* gates, int w_dtype,
                         const float* b_r, const float* b_i, const float* rate, float* state, void* out, int out_dtype, long long ldo,
                         const int* seq_of, const int* slots, int T, int W, int blocks, cudaStream_t stream) {
    GB_REQUIRE(gb_is_dtype(dtype) && gb_is_dtype(w_dtype) && gb_is_dtype(out_dtype), "gb_rglru_step: bad dtype");
    GB_REQUIRE(W > 0 && blocks > 0 && blocks <= 65535 && W % blocks == 0, "gb_rglru_step: %d channels do not form %d equal blocks", W, blocks);
    if (T == 0) return 0;
    RsParams p;
    p.u = u; p.y = y; p.gates = gates; p.b_r = b_r; p.b_i = b_i; p.rate = rate; p.state = state; p.out = out; p.ldu = ldu; p.ldy = ldy;
    p.ldo = ldo; p.seq_of = seq_of; p.slots = slots; p.dtype = dtype; p.out_dtype = out_dtype; p.T = T; p.W = W; p.n = W / blocks;
    const bool many = p.n >= 64;
    const size_t smem = (size_t(RS_TOK) * p.n + size_t(many ? 8 : 2) * RS_TOK * 32) * sizeof(float);
    GB_REQUIRE(smem <= 48 * 1024, "gb_rglru_step: blocks of %d channels exceed 1280", p.n);
    const dim3 grid((T + RS_TOK - 1) / RS_TOK, blocks, (p.n + RS_CH - 1) / RS_CH);
#define RS_LAUNCH(TW)                                                                                         \
    do {                                                                                                      \
        if (many) gb_launch(rglru_step_kernel<TW, 8>, grid, dim3(256), smem, stream, p);                      \
        else gb_launch(rglru_step_kernel<TW, 2>, grid, dim3(64), smem, stream, p);                            \
    } while (0)
    if (w_dtype == GB_F32) RS_LAUNCH(float);
    else RS_LAUNCH(__nv_bfloat16);
#undef RS_LAUNCH
    GB_LAUNCH_OK("gb_rglru_step");
    return 0;
}
