// Retention: linear attention with one fixed decay per head and no denominator,
//   S <- decay_h S + k' v^T;   o = S^T q'
// per head, S [D, Dv] in 32-bit per sequence, q' the rotated query, k' the rotated key times a constant; what is read out is
// brought to unit root mean square per head and gated.  Three ways, by the step: prompts in bfloat16 as matrix products over
// chunks, single tokens in one pass over S, and for everything else (the 32-bit mode, other head sizes) the walk of
// linear_walk.h with the decay the same for all key channels and tokens, whose preparation turns q and k by the token's
// position (32-bit angles, products and sums) and writes the walk's rows.
#include <math.h>

#include "common.cuh"
#include "linear_walk.h"
#include "mma_tiles.cuh"

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

// ------------------------------------------------------------------------------------------------ prompts, in chunks
// Because the decay is one constant per head, a stretch of n tokens in front of which the state is S0 gives
//   o_i = g^(i+1) S0^T q'_i + sum_(j <= i) g^(i-j) (q'_i . k'_j) v_j      (i, j counted from the stretch's start)
//   S1  = g^n S0 + sum_j g^(n-1-j) k'_j v_j^T
// so that all of it is matrix products but a short recurrence over the stretches (segments of RC_SEG tokens):
//   1. retention_state_kernel: every segment's own sum of k' v^T, one block per (segment, head);
//   2. retention_carry_kernel: the states in front of the segments and the sequence's new state, entry by entry;
//   3. retention_out_kernel: the results of 64 tokens per (block, head), with the read-out's norm, the SiLU gate and the
//      result's factor.
// q', k' and S are 32-bit numbers: on the tensor cores they are three bfloat16 terms each (mma_tiles.cuh), v is bfloat16.
constexpr int RC_SEG = 128, RC_TILE = 64;

struct RetChunkParams {
    const __nv_bfloat16 *q, *k, *v, *gate;      // [T, H*N] column slices; q, k, v rows ld apart, gate rows ldg apart
    const float2* angles;                       // [T, half] (cosine, sine), or null: no rotation
    const float* log2_decay;                    // [H]
    float* state;                               // [slots, H, N, N]
    float* seg;                                 // [B * n_seg, H, N, N]
    __nv_bfloat16* out;                         // [T, H*N] rows ldo apart
    const int *cu, *slots, *qlens;
    long long ld, ldg, ldo;
    int H, half, pairing, n_seg;
    float k_scale, eps, out_scale;
};

__device__ __forceinline__ void rc_unpack(const uint4& raw, float (&x)[8]) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h[e]);
        x[2 * e] = f.x;
        x[2 * e + 1] = f.y;
    }
}
// eight numbers as three planes of bfloat16 terms, `plane` entries apart
__device__ __forceinline__ void rc_store_terms(const float (&x)[8], __nv_bfloat16* at, int plane) {
    using namespace gbmma;
    uint4 h, m, l;
    split3(x[0], x[1], h.x, m.x, l.x);
    split3(x[2], x[3], h.y, m.y, l.y);
    split3(x[4], x[5], h.z, m.z, l.z);
    split3(x[6], x[7], h.w, m.w, l.w);
    *reinterpret_cast<uint4*>(at) = h;
    *reinterpret_cast<uint4*>(at + plane) = m;
    *reinterpret_cast<uint4*>(at + 2 * plane) = l;
}

// 64 rows of q or k: rotated, row r times factor * 2^(row_log2 * (last - r)), as three planes of bfloat16 terms; rows from
// n (at least 1) on are zero.  AHEAD pieces of eight entries per thread are on their way together (rows behind the last
// read the last, so that no load waits for a branch).
template <int N, int THREADS, int AHEAD>
__device__ __forceinline__ void rc_load_rotated(const RetChunkParams& p, const __nv_bfloat16* src, int t0, int n, float factor,
                                                float row_log2, int last, __nv_bfloat16* planes) {
    constexpr int CH = N / 8, ITEMS = RC_TILE * CH;
    const bool halves = !p.pairing && p.half > 0 && (p.half & 7) == 0;      // whole pieces are turned with whole pieces
    for (int base = threadIdx.x; base < ITEMS; base += THREADS * AHEAD) {
        uint4 own[AHEAD], oth[AHEAD];
        float4 ang[AHEAD][4];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int idx = min(base + u * THREADS, ITEMS - 1), r = min(idx / CH, n - 1), d = 8 * (idx % CH);
            const __nv_bfloat16* row = src + size_t(t0 + r) * p.ld;
            own[u] = __ldg(reinterpret_cast<const uint4*>(row + d));
            if (halves) {
                const bool turned = d < 2 * p.half, first = d < p.half;
                oth[u] = __ldg(reinterpret_cast<const uint4*>(row + (!turned ? d : first ? d + p.half : d - p.half)));
                const float4* a = reinterpret_cast<const float4*>(p.angles + size_t(t0 + r) * p.half + (!turned ? 0 : first ? d : d - p.half));
#pragma unroll
                for (int e = 0; e < 4; ++e) ang[u][e] = __ldg(a + e);
            }
        }
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int idx = base + u * THREADS;
            if (idx >= ITEMS) break;
            const int r = idx / CH, c = idx - r * CH, d = 8 * c;
            float x[8];
            rc_unpack(own[u], x);
            if (halves) {
                if (d < 2 * p.half) {
                    const bool first = d < p.half;
                    float o[8];
                    rc_unpack(oth[u], o);
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        const float4 a = ang[u][e >> 1];
                        const float cs = (e & 1) ? a.z : a.x, sn = (e & 1) ? a.w : a.y;
                        float y0, y1;
                        gb_rotate(first ? x[e] : o[e], first ? o[e] : x[e], cs, sn, y0, y1);
                        x[e] = first ? y0 : y1;
                    }
                }
            } else if (r < n) {
                const __nv_bfloat16* row = src + size_t(t0 + r) * p.ld;
                const float2* a = p.angles + size_t(t0 + r) * p.half;
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const int dd = d + e;
                    if (dd < 2 * p.half) {
                        const bool first = p.pairing ? (dd & 1) == 0 : dd < p.half;
                        const float2 cs = a[p.pairing ? dd >> 1 : first ? dd : dd - p.half];
                        const float other = __bfloat162float(row[p.pairing ? dd ^ 1 : first ? dd + p.half : dd - p.half]);
                        float y0, y1;
                        gb_rotate(first ? x[e] : other, first ? other : x[e], cs.x, cs.y, y0, y1);
                        x[e] = first ? y0 : y1;
                    }
                }
            }
            const float f = r >= n ? 0.f : row_log2 != 0.f ? factor * exp2f(row_log2 * float(last - r)) : factor;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = r < n ? x[e] * f : 0.f;
            rc_store_terms(x, planes + gbmma::swz<N>(r, c), RC_TILE * N);
        }
    }
}

template <int N, int THREADS>
__device__ __forceinline__ void rc_load_values(const RetChunkParams& p, const __nv_bfloat16* src, int t0, int n, __nv_bfloat16* vt) {
    constexpr int CH = N / 8, ITEMS = RC_TILE * CH;
#pragma unroll
    for (int base = 0; base < ITEMS; base += THREADS) {
        const int idx = base + threadIdx.x;
        if (ITEMS % THREADS && idx >= ITEMS) break;
        const int r = idx / CH, c = idx - r * CH;
        uint4 raw = __ldg(reinterpret_cast<const uint4*>(src + size_t(t0 + min(r, n - 1)) * p.ld + 8 * c));
        if (r >= n) raw = make_uint4(0u, 0u, 0u, 0u);
        *reinterpret_cast<uint4*>(vt + gbmma::swz<N>(r, c)) = raw;
    }
}

// seg[b * n_seg + s, h] = sum_j g^(n-1-j) k'_j v_j^T over the segment's n tokens.  N / 16 warps, 16 key channels each.
template <int N>
__global__ void __launch_bounds__(2 * N, 2) retention_state_kernel(const RetChunkParams p) {
    using namespace gbmma;
    extern __shared__ __align__(128) unsigned char rc_smem[];
    __nv_bfloat16* kp = reinterpret_cast<__nv_bfloat16*>(rc_smem);          // [3][64][N]
    __nv_bfloat16* vt = kp + 3 * RC_TILE * N;                               // [64][N]
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int b = blockIdx.x / p.n_seg, s = blockIdx.x % p.n_seg, h = blockIdx.y;
    const int n = min(RC_SEG, p.qlens[b] - s * RC_SEG);
    if (p.slots[b] < 0 || n <= 0) return;
    const int t0 = p.cu[b] + s * RC_SEG, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float lg = p.log2_decay[h];
    float acc[N / 8][4];
#pragma unroll
    for (int i = 0; i < N / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int j0 = 0; j0 < n; j0 += RC_TILE) {
        const int nb = min(RC_TILE, n - j0);
        __syncthreads();
        rc_load_rotated<N, 2 * N, 1>(p, p.k + size_t(h) * N, t0 + j0, nb, p.k_scale, lg, n - 1 - j0, kp);
        rc_load_values<N, 2 * N>(p, p.v + size_t(h) * N, t0 + j0, nb, vt);
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < RC_TILE / 16; ++kk) {
            unsigned a[3][4];
#pragma unroll
            for (int e = 0; e < 3; ++e)       // tokens are the inner dimension: a transposed load turns [token][channel]
                ldsm4_trans(a[e], kp + e * RC_TILE * N + swz<N>(kk * 16 + (lane & 7) + ((lane >> 4) << 3), 2 * warp + ((lane >> 3) & 1)));
#pragma unroll
            for (int i4 = 0; i4 < N / 32; ++i4) {
                unsigned bv[4], bw[4];
                ldsm4_trans(bv, vt + swz<N>(kk * 16 + (lane & 15), 4 * i4 + (lane >> 4)));
                ldsm4_trans(bw, vt + swz<N>(kk * 16 + (lane & 15), 4 * i4 + 2 + (lane >> 4)));
                mma3(acc[4 * i4], acc[4 * i4 + 1], acc[4 * i4 + 2], acc[4 * i4 + 3], a, bv, bw);
            }
        }
    }
    float* o = p.seg + (size_t(blockIdx.x) * p.H + h) * size_t(N) * N + size_t(16 * warp + (lane >> 2)) * N + 2 * (lane & 3);
#pragma unroll
    for (int i = 0; i < N / 8; ++i) {
        *reinterpret_cast<float2*>(o + 8 * i) = make_float2(acc[i][0], acc[i][1]);
        *reinterpret_cast<float2*>(o + 8 * N + 8 * i) = make_float2(acc[i][2], acc[i][3]);
    }
}

// S_0 = state; S_(s+1) = g^(n_s) S_s + seg_s; seg_s <- S_s; state <- the last.  One thread per four entries.
__global__ void __launch_bounds__(128) retention_carry_kernel(float4* __restrict__ state, float4* __restrict__ seg,
                                                              const float* __restrict__ log2_decay, const int* __restrict__ slots,
                                                              const int* __restrict__ qlens, int H, int entries4, int n_seg) {
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int b = blockIdx.x, h = blockIdx.y, e = blockIdx.z * blockDim.x + threadIdx.x;
    const int slot = slots[b], n = qlens[b];
    if (slot < 0 || n <= 0 || e >= entries4) return;
    const float lg = log2_decay[h];
    float4* sp = state + (size_t(slot) * H + h) * entries4 + e;
    float4 S = *sp;
    const int segs = (n + RC_SEG - 1) / RC_SEG;
    const size_t stride = size_t(H) * entries4;
    float4* row = seg + (size_t(b) * n_seg * H + h) * entries4 + e;
    constexpr int AHEAD = 8;                  // segments whose sums are on their way together
    for (int s0 = 0; s0 < segs; s0 += AHEAD) {
        float4 local[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
            if (s0 + j < segs) local[j] = row[size_t(s0 + j) * stride];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (s0 + j >= segs) break;
            row[size_t(s0 + j) * stride] = S;
            const float g = exp2f(lg * float(min(RC_SEG, n - (s0 + j) * RC_SEG)));
            S = make_float4(fmaf(g, S.x, local[j].x), fmaf(g, S.y, local[j].y), fmaf(g, S.z, local[j].z), fmaf(g, S.w, local[j].w));
        }
    }
    *sp = S;
}

// 64 queries of one head.  A warp has 16 of them and, where the head's size is a multiple of 64, half of the value columns
// (two warps share their queries): it then makes the scores of half of the keys, and the weights go through shared memory.
template <int N> struct RcOut {
    static constexpr int HALVES = N % 64 == 0 ? 2 : 1, THREADS = 128 * HALVES, COLS = N / HALVES, KEYS = RC_TILE / HALVES;
};

template <int N>
__global__ void __launch_bounds__(RcOut<N>::THREADS, 2) retention_out_kernel(const RetChunkParams p) {
    using namespace gbmma;
    using L = RcOut<N>;
    extern __shared__ __align__(128) unsigned char rc_smem[];
    __shared__ float ss_part[L::HALVES][RC_TILE];
    __nv_bfloat16* qp = reinterpret_cast<__nv_bfloat16*>(rc_smem);          // [3][64][N]
    __nv_bfloat16* kp = qp + 3 * RC_TILE * N;                               // slices of S; then keys [3][64][N]
    __nv_bfloat16* vt = kp + 3 * RC_TILE * (N > RC_TILE ? N : RC_TILE);     // [64][N]
    __nv_bfloat16* wp = kp;                                                 // weights [3][64][64], over the keys when those are used up
    gb_grid_launch_dependents();
    gb_grid_wait();
    constexpr int TILES = RC_SEG / RC_TILE;
    const int unit = blockIdx.x / TILES, tile = TILES - 1 - blockIdx.x % TILES, h = blockIdx.y;
    const int b = unit / p.n_seg, s = unit % p.n_seg;
    const int n = min(RC_SEG, p.qlens[b] - s * RC_SEG);                     // tokens of the segment
    const int q0 = tile * RC_TILE;
    if (p.slots[b] < 0 || q0 >= n) return;
    const int t0 = p.cu[b] + s * RC_SEG, rows = min(RC_TILE, n - q0);
    const int warp = (threadIdx.x >> 5) & 3, half = threadIdx.x >> 7, lane = threadIdx.x & 31, col0 = half * L::COLS;
    const float lg = p.log2_decay[h];
    // ---- q' S0, 32 rows of S0 at a time, the next rows on their way meanwhile
    const float* S0 = p.seg + (size_t(unit) * p.H + h) * size_t(N) * N;
    constexpr int PIECES = 32 * (N / 8) / L::THREADS;                       // pieces of eight entries per thread
    float4 next[PIECES][2];
    auto fetch = [&](int d0) {
#pragma unroll
        for (int u = 0; u < PIECES; ++u) {
            const int idx = u * L::THREADS + threadIdx.x, r = idx / (N / 8), c = idx - r * (N / 8);
            const float4* src = reinterpret_cast<const float4*>(S0 + size_t(d0 + r) * N + 8 * c);
            next[u][0] = __ldg(src);
            next[u][1] = __ldg(src + 1);
        }
    };
    fetch(0);
    rc_load_rotated<N, L::THREADS, 2>(p, p.q + size_t(h) * N, t0 + q0, rows, 1.f, 0.f, 0, qp);
    float acc[L::COLS / 8][4];
#pragma unroll
    for (int i = 0; i < L::COLS / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int d0 = 0; d0 < N; d0 += 32) {
#pragma unroll
        for (int u = 0; u < PIECES; ++u) {
            const int idx = u * L::THREADS + threadIdx.x, r = idx / (N / 8), c = idx - r * (N / 8);
            const float x[8] = {next[u][0].x, next[u][0].y, next[u][0].z, next[u][0].w, next[u][1].x, next[u][1].y, next[u][1].z, next[u][1].w};
            rc_store_terms(x, kp + swz<N>(r, c), 32 * N);
        }
        if (d0 + 32 < N) fetch(d0 + 32);
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
            unsigned a[3][4];
#pragma unroll
            for (int e = 0; e < 3; ++e) ldsm4(a[e], qp + e * RC_TILE * N + swz<N>(warp * 16 + (lane & 15), d0 / 8 + 2 * kk + (lane >> 4)));
#pragma unroll
            for (int i4 = 0; i4 < L::COLS / 32; ++i4) {
                unsigned bs[3][4], bt[3][4];
                const int c = col0 / 8 + 4 * i4 + (lane >> 4);
#pragma unroll
                for (int e = 0; e < 3; ++e) {
                    ldsm4_trans(bs[e], kp + e * 32 * N + swz<N>(kk * 16 + (lane & 15), c));
                    ldsm4_trans(bt[e], kp + e * 32 * N + swz<N>(kk * 16 + (lane & 15), c + 2));
                }
                mma6(acc[4 * i4], acc[4 * i4 + 1], acc[4 * i4 + 2], acc[4 * i4 + 3], a, bs, bt);
            }
        }
        __syncthreads();
    }
    const int r0 = warp * 16 + (lane >> 2), i0 = q0 + r0, i1 = i0 + 8;      // this thread's two queries: in the tile, in the segment
    const float g0 = exp2f(lg * float(i0 + 1)), g1 = exp2f(lg * float(i1 + 1));
#pragma unroll
    for (int i = 0; i < L::COLS / 8; ++i) { acc[i][0] *= g0; acc[i][1] *= g0; acc[i][2] *= g1; acc[i][3] *= g1; }
    // ---- the segment's own keys up to each query
    for (int j0 = 0; j0 <= q0; j0 += RC_TILE) {
        const int nb = min(RC_TILE, n - j0);
        rc_load_rotated<N, L::THREADS, 2>(p, p.k + size_t(h) * N, t0 + j0, nb, p.k_scale, 0.f, 0, kp);
        rc_load_values<N, L::THREADS>(p, p.v + size_t(h) * N, t0 + j0, nb, vt);
        __syncthreads();
        float w[L::KEYS / 8][4];
#pragma unroll
        for (int j = 0; j < L::KEYS / 8; ++j) w[j][0] = w[j][1] = w[j][2] = w[j][3] = 0.f;
#pragma unroll 2
        for (int kk = 0; kk < N / 16; ++kk) {
            unsigned a[3][4];
#pragma unroll
            for (int e = 0; e < 3; ++e) ldsm4(a[e], qp + e * RC_TILE * N + swz<N>(warp * 16 + (lane & 15), 2 * kk + (lane >> 4)));
#pragma unroll
            for (int j4 = 0; j4 < L::KEYS / 32; ++j4) {
                unsigned bk[3][4], bl[3][4];
                const int r = half * L::KEYS + j4 * 32 + (lane & 7) + ((lane >> 4) << 3), c = 2 * kk + ((lane >> 3) & 1);
#pragma unroll
                for (int e = 0; e < 3; ++e) {
                    ldsm4(bk[e], kp + e * RC_TILE * N + swz<N>(r, c));
                    ldsm4(bl[e], kp + e * RC_TILE * N + swz<N>(r + 16, c));
                }
                mma6(w[4 * j4], w[4 * j4 + 1], w[4 * j4 + 2], w[4 * j4 + 3], a, bk, bl);
            }
        }
        __syncthreads();                                                    // the keys are used up
#pragma unroll
        for (int j = 0; j < L::KEYS / 8; ++j) {
            const int jl = half * L::KEYS + 8 * j + 2 * (lane & 3), ja = j0 + jl;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int dist = (e < 2 ? i0 : i1) - ja - (e & 1);
                w[j][e] = dist >= 0 ? w[j][e] * exp2f(lg * float(dist)) : 0.f;
            }
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                unsigned th, tm, tl;
                split3(w[j][2 * rr], w[j][2 * rr + 1], th, tm, tl);
                __nv_bfloat16* at = wp + swz<RC_TILE>(r0 + 8 * rr, jl >> 3) + (jl & 7);
                *reinterpret_cast<unsigned*>(at) = th;
                *reinterpret_cast<unsigned*>(at + RC_TILE * RC_TILE) = tm;
                *reinterpret_cast<unsigned*>(at + 2 * RC_TILE * RC_TILE) = tl;
            }
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < RC_TILE / 16; ++kk) {
            unsigned a[3][4];
#pragma unroll
            for (int e = 0; e < 3; ++e) ldsm4(a[e], wp + e * RC_TILE * RC_TILE + swz<RC_TILE>(warp * 16 + (lane & 15), 2 * kk + (lane >> 4)));
#pragma unroll
            for (int i4 = 0; i4 < L::COLS / 32; ++i4) {
                unsigned bv[4], bw[4];
                const int c = col0 / 8 + 4 * i4 + (lane >> 4);
                ldsm4_trans(bv, vt + swz<N>(kk * 16 + (lane & 15), c));
                ldsm4_trans(bw, vt + swz<N>(kk * 16 + (lane & 15), c + 2));
                mma3(acc[4 * i4], acc[4 * i4 + 1], acc[4 * i4 + 2], acc[4 * i4 + 3], a, bv, bw);
            }
        }
        __syncthreads();
    }
    // ---- unit root mean square per row, gate, factor
    float ss0 = 0.f, ss1 = 0.f;
#pragma unroll
    for (int i = 0; i < L::COLS / 8; ++i) {
        ss0 = fmaf(acc[i][0], acc[i][0], ss0); ss0 = fmaf(acc[i][1], acc[i][1], ss0);
        ss1 = fmaf(acc[i][2], acc[i][2], ss1); ss1 = fmaf(acc[i][3], acc[i][3], ss1);
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) { ss0 += __shfl_xor_sync(0xffffffffu, ss0, o); ss1 += __shfl_xor_sync(0xffffffffu, ss1, o); }
    if (L::HALVES > 1) {
        if ((lane & 3) == 0) { ss_part[half][r0] = ss0; ss_part[half][r0 + 8] = ss1; }
        __syncthreads();
        ss0 = ss_part[0][r0] + ss_part[L::HALVES - 1][r0];
        ss1 = ss_part[0][r0 + 8] + ss_part[L::HALVES - 1][r0 + 8];
    }
    const float f0 = p.out_scale / sqrtf(ss0 / float(N) + p.eps), f1 = p.out_scale / sqrtf(ss1 / float(N) + p.eps);
    const size_t col = size_t(h) * N + col0 + 2 * (lane & 3);
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
        const int r = rr ? i1 : i0;
        if (r >= n) continue;
        const __nv_bfloat16* gr = p.gate + size_t(t0 + r) * p.ldg + col;
        __nv_bfloat16* orow = p.out + size_t(t0 + r) * p.ldo + col;
        const float f = rr ? f1 : f0;
#pragma unroll
        for (int i = 0; i < L::COLS / 8; ++i) {
            const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gr + 8 * i));
            *reinterpret_cast<__nv_bfloat162*>(orow + 8 * i) =
                __floats2bfloat162_rn(acc[i][2 * rr] * f * (z.x / (1.f + expf(-z.x))), acc[i][2 * rr + 1] * f * (z.y / (1.f + expf(-z.y))));
        }
    }
}

// Cosine and sine of every token's position times every frequency, for all heads and layers of a step.
__global__ void __launch_bounds__(128) rotary_angles_kernel(const int* __restrict__ pos, const float* __restrict__ inv_freq, int half,
                                                            float2* __restrict__ angles) {
    gb_grid_launch_dependents();
    gb_grid_wait();
    const float p = float(pos[blockIdx.x]);
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf(p * inv_freq[i], &sn, &cs);
        angles[size_t(blockIdx.x) * half + i] = make_float2(cs, sn);
    }
}

// ------------------------------------------------------------------------------------------------ single tokens
// One block per (sequence, head): rotation, update of S, read-out, its norm, gate and factor in one pass over S.  V entries
// per access; a group of threads covers the columns of a row, the groups take rows in turn, and the groups' sums are added
// in order.
struct RetStepParams {
    const void *q, *k, *v, *gate;
    const int *pos, *cu, *slots;
    const float *inv_freq, *decay;
    float* state;
    void* out;
    long long ld, ldg, ldo;
    int dtype, out_dtype, rot, pairing, H, D, Dv;
    float k_scale, eps, out_scale;
};

template <int V>
__global__ void __launch_bounds__(256) retention_step_kernel(const RetStepParams p) {
    extern __shared__ __align__(16) float rs_sm[];
    __shared__ float red[8];
    gb_grid_launch_dependents();
    gb_grid_wait();
    const int b = blockIdx.x, h = blockIdx.y, slot = p.slots[b];
    if (slot < 0) return;
    const int D = p.D, Dv = p.Dv, DA = (D + 3) / 4 * 4, VA = (Dv + 3) / 4 * 4;
    float *qs = rs_sm, *ks = qs + DA, *vs = ks + DA, *os = vs + VA, *part = os + VA;
    const size_t t = size_t(p.cu[b]);
    const size_t row = t * p.ld + size_t(h) * D;
    const int half = p.inv_freq ? p.rot / 2 : 0;
    for (int i = threadIdx.x; i < half; i += 256) {
        const int d0 = p.pairing ? 2 * i : i, d1 = p.pairing ? 2 * i + 1 : i + half;
        float sn, cs, y0, y1;
        sincosf(float(p.pos[t]) * p.inv_freq[i], &sn, &cs);
        gb_rotate(gb_load(p.q, p.dtype, row + d0), gb_load(p.q, p.dtype, row + d1), cs, sn, y0, y1);
        qs[d0] = y0;
        qs[d1] = y1;
        gb_rotate(gb_load(p.k, p.dtype, row + d0), gb_load(p.k, p.dtype, row + d1), cs, sn, y0, y1);
        ks[d0] = y0 * p.k_scale;
        ks[d1] = y1 * p.k_scale;
    }
    for (int d = 2 * half + threadIdx.x; d < D; d += 256) {
        qs[d] = gb_load(p.q, p.dtype, row + d);
        ks[d] = gb_load(p.k, p.dtype, row + d) * p.k_scale;
    }
    for (int d = threadIdx.x; d < Dv; d += 256) vs[d] = gb_load(p.v, p.dtype, t * p.ld + size_t(h) * Dv + d);
    const float g = p.decay[h];
    float* S = p.state + (size_t(slot) * p.H + h) * size_t(D) * Dv;
    const int C = Dv / V, CC = min(C, 256), RG = 256 / CC;
    const int grp = threadIdx.x / CC, lane_c = threadIdx.x - grp * CC;
    __syncthreads();
    for (int c0 = 0; c0 < C; c0 += CC) {
        const int c = c0 + lane_c;
        float acc[V];
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = 0.f;
        if (grp < RG && c < C) {
            float vv[V];
#pragma unroll
            for (int e = 0; e < V; ++e) vv[e] = vs[c * V + e];
            constexpr int AHEAD = 8;
            for (int i0 = grp; i0 < D; i0 += RG * AHEAD) {
                float s[AHEAD][V];
#pragma unroll
                for (int a = 0; a < AHEAD; ++a) {
                    const int i = i0 + a * RG;
                    if (i < D) {
                        if (V == 4) *reinterpret_cast<float4*>(s[a]) = *reinterpret_cast<const float4*>(S + size_t(i) * Dv + c * V);
                        else s[a][0] = S[size_t(i) * Dv + c];
                    }
                }
#pragma unroll
                for (int a = 0; a < AHEAD; ++a) {
                    const int i = i0 + a * RG;
                    if (i < D) {
                        const float kv = ks[i], qv = qs[i];
#pragma unroll
                        for (int e = 0; e < V; ++e) {
                            s[a][e] = fmaf(kv, vv[e], s[a][e] * g);
                            acc[e] = fmaf(s[a][e], qv, acc[e]);
                        }
                        if (V == 4) *reinterpret_cast<float4*>(S + size_t(i) * Dv + c * V) = *reinterpret_cast<const float4*>(s[a]);
                        else S[size_t(i) * Dv + c] = s[a][0];
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) part[(grp * CC + lane_c) * V + e] = acc[e];
        }
        __syncthreads();
        for (int i = threadIdx.x; i < CC * V && c0 * V + i < Dv; i += 256) {
            float o = part[i];
            for (int r = 1; r < RG; ++r) o += part[r * CC * V + i];
            os[c0 * V + i] = o;
        }
        __syncthreads();
    }
    float ss = 0.f;
    for (int d = threadIdx.x; d < Dv; d += 256) ss = fmaf(os[d], os[d], ss);
    ss = gb_warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) tot += red[w];
    const float f = p.out_scale / sqrtf(tot / float(Dv) + p.eps);
    for (int d = threadIdx.x; d < Dv; d += 256) {
        const float z = gb_load(p.gate, p.dtype, t * p.ldg + size_t(h) * Dv + d);
        gb_store(p.out, p.out_dtype, t * p.ldo + size_t(h) * Dv + d, os[d] * f * (z / (1.f + expf(-z))));
    }
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

// angles float [T, half, 2]: cosine and sine of pos[t] * inv_freq[i].
GB_API int gb_rotary_angles(const int* pos, const float* inv_freq, int T, int half, float* angles, cudaStream_t stream) {
    GB_REQUIRE(pos && inv_freq && angles && half > 0, "gb_rotary_angles: arguments missing");
    if (T == 0) return 0;
    gb_launch(rotary_angles_kernel, dim3(T), dim3(128), 0, stream, pos, inv_freq, half, (float2*)angles);
    GB_LAUNCH_OK("gb_rotary_angles");
    return 0;
}

// Whether the chunked kernels take these heads: bfloat16, keys and values of one size of 32, 64, 96 or 128 entries.
GB_API int gb_retention_chunks_supported(int dtype, int D, int Dv) {
    return dtype == GB_BF16 && D == Dv && (D == 32 || D == 64 || D == 96 || D == 128);
}

GB_API long long gb_retention_chunk_floats(int B, int max_qlen, int H, int D, int Dv) {
    return (long long)B * ((max_qlen + RC_SEG - 1) / RC_SEG) * H * D * Dv;
}

template <int N> static int retention_chunks_launch(const RetChunkParams& p, int B, cudaStream_t stream) {
    constexpr int SMEM_STATE = (3 * RC_TILE * N + RC_TILE * N) * 2, SMEM_OUT = (4 * RC_TILE * N + 3 * RC_TILE * (N > RC_TILE ? N : RC_TILE)) * 2;
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(retention_state_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_STATE) != cudaSuccess ||
            cudaFuncSetAttribute(retention_out_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_OUT) != cudaSuccess)
            return gb_fail("gb_retention_chunks: cannot get %d bytes of shared memory", SMEM_OUT);
        configured = true;
    }
    gb_launch(retention_state_kernel<N>, dim3(B * p.n_seg, p.H), dim3(2 * N), SMEM_STATE, stream, p);
    GB_LAUNCH_OK("gb_retention_chunks (states)");
    constexpr int E4 = N * N / 4;
    gb_launch(retention_carry_kernel, dim3(B, p.H, (E4 + 127) / 128), dim3(128), 0, stream, (float4*)p.state, (float4*)p.seg, p.log2_decay,
              p.slots, p.qlens, p.H, E4, p.n_seg);
    GB_LAUNCH_OK("gb_retention_chunks (carry)");
    gb_launch(retention_out_kernel<N>, dim3(B * p.n_seg * (RC_SEG / RC_TILE), p.H), dim3(RcOut<N>::THREADS), SMEM_OUT, stream, p);
    GB_LAUNCH_OK("gb_retention_chunks");
    return 0;
}

// Steps of many tokens: q, k, v [T, H*D] bfloat16 with rows ld apart, gate [T, H*D] with rows ldg apart, angles float
// [T, half, 2] (half 0: no rotation), log2_decay [H] (decays in (0, 1]); state [slots, H, D, D], read and renewed; seg:
// gb_retention_chunk_floats; out [T, H*D] bfloat16 = o / rms(o) * silu(gate) * out_scale.  Three launches.
GB_API int gb_retention_chunks(const void* q, const void* k, const void* v, long long ld, const void* gate, long long ldg,
                               const float* angles, int half, int pairing, float k_scale, const float* log2_decay, float* state,
                               float* seg, void* out, long long ldo, float eps, float out_scale, const int* cu, const int* slots,
                               const int* qlens, int B, int H, int D, int max_qlen, cudaStream_t stream) {
    GB_REQUIRE(gb_retention_chunks_supported(GB_BF16, D, D), "gb_retention_chunks: heads of %d entries are not 32, 64, 96 or 128", D);
    GB_REQUIRE(H > 0 && H <= 65535 && half >= 0 && 2 * half <= D && (half == 0 || angles) && seg && eps > 0.f, "gb_retention_chunks: bad arguments");
    GB_REQUIRE(ld % 8 == 0 && gb_aligned(q, 16) && gb_aligned(k, 16) && gb_aligned(v, 16) && ldg % 2 == 0 && ldo % 2 == 0 &&
               gb_aligned(gate, 4) && gb_aligned(out, 4) && gb_aligned(state, 16) && gb_aligned(seg, 16), "gb_retention_chunks: misaligned operands");
    if (B == 0 || max_qlen <= 0) return 0;
    RetChunkParams p;
    p.q = (const __nv_bfloat16*)q; p.k = (const __nv_bfloat16*)k; p.v = (const __nv_bfloat16*)v; p.gate = (const __nv_bfloat16*)gate;
    p.angles = (const float2*)angles; p.log2_decay = log2_decay; p.state = state; p.seg = seg; p.out = (__nv_bfloat16*)out; p.cu = cu;
    p.slots = slots; p.qlens = qlens; p.ld = ld; p.ldg = ldg; p.ldo = ldo; p.H = H; p.half = half; p.pairing = pairing;
    p.n_seg = (max_qlen + RC_SEG - 1) / RC_SEG; p.k_scale = k_scale; p.eps = eps; p.out_scale = out_scale;
    switch (D) {
        case 32: return retention_chunks_launch<32>(p, B, stream);
        case 64: return retention_chunks_launch<64>(p, B, stream);
        case 96: return retention_chunks_launch<96>(p, B, stream);
        default: return retention_chunks_launch<128>(p, B, stream);
    }
}

// Single tokens (every sequence brings one): any sizes and dtype; out as gb_retention_chunks.
GB_API int gb_retention_step(const void* q, const void* k, const void* v, int dtype, long long ld, const void* gate, long long ldg,
                             const int* pos, const float* inv_freq, int rot, int pairing, float k_scale, const float* decay,
                             float* state, void* out, int out_dtype, long long ldo, float eps, float out_scale, const int* cu,
                             const int* slots, int B, int H, int D, int Dv, cudaStream_t stream) {
    GB_REQUIRE(gb_is_dtype(dtype) && gb_is_dtype(out_dtype), "gb_retention_step: bad dtype");
    GB_REQUIRE(H > 0 && H <= 65535 && D > 0 && D <= 2048 && Dv > 0 && Dv <= 2048 && eps > 0.f,
               "gb_retention_step: bad sizes heads=%d dim=%d vdim=%d (up to 2048)", H, D, Dv);
    GB_REQUIRE(!inv_freq || (rot > 0 && rot % 2 == 0 && rot <= D), "gb_retention_step: %d of %d entries cannot be rotated", rot, D);
    if (B == 0) return 0;
    RetStepParams p;
    p.q = q; p.k = k; p.v = v; p.gate = gate; p.pos = pos; p.cu = cu; p.slots = slots; p.inv_freq = inv_freq; p.decay = decay;
    p.state = state; p.out = out; p.ld = ld; p.ldg = ldg; p.ldo = ldo; p.dtype = dtype; p.out_dtype = out_dtype; p.rot = rot;
    p.pairing = pairing; p.H = H; p.D = D; p.Dv = Dv; p.k_scale = k_scale; p.eps = eps; p.out_scale = out_scale;
    const bool vec = Dv % 4 == 0 && gb_aligned(state, 16);
    const int V = vec ? 4 : 1, C = Dv / V, CC = C < 256 ? C : 256, RG = 256 / CC;
    const size_t smem = (size_t(2) * ((D + 3) / 4 * 4) + size_t(2) * ((Dv + 3) / 4 * 4) + size_t(RG) * CC * V) * sizeof(float);
    if (vec) gb_launch(retention_step_kernel<4>, dim3(B, H), dim3(256), smem, stream, p);
    else gb_launch(retention_step_kernel<1>, dim3(B, H), dim3(256), smem, stream, p);
    GB_LAUNCH_OK("gb_retention_step");
    return 0;
}
