// Mixture of experts (dc_moe_ffn): clamped gated ones, or the square of relu between two matrices, behind a sigmoid router whose
// choices are limited to groups of experts, or a softmax router whose chosen scores are divided by their sum.
//
// Steps of up to DC_MAX_T tokens: k_moe_norm_route norms the residual and routes it (one cluster per token), k_moe_up_mma
// streams the gate and up rows of the chosen experts, k_moe_down_mma streams their down rows, every distinct expert once,
// and adds the sum over experts to the residual.  Hidden values carry the routing weight already, so the down products
// of a token are one long sum.  Larger steps (k_moe_norm_route_tile) sort the assignments by expert (k_moe_order), gather
// the input rows and run grouped tensor-core products (linear_tc.cu); f32 models use k_moe_f32 instead.  The rows of a
// token are then added up by the norm that follows (norm_act.cu).
#include <algorithm>

#include "dc_common.cuh"
#include "dc_launch.cuh"
#include "dc_stack.h"
#include "dc_stack.cuh"

using namespace dc;

namespace {

// ---------------------------------------------------------------- choices
struct RouteParams {
    int experts, top, groups, keep;
    float scale;
    bool softmax;
    const float* correction;     // or null
    int32_t* ids;
    float* weights;
};

__device__ __forceinline__ uint32_t ordered(float f) {      // order-preserving, never 0 for a number
    const uint32_t u = __float_as_uint(f);
    return f != f ? 1u : (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}

// One warp: the choices of a token.  score (softmax: the logits), correction: shared memory; PER: experts of a lane.  Equal scores:
// the lower index first.
template <int PER>
__device__ __forceinline__ void choose(const RouteParams& p, const float* score, const float* correction, int t, int lane) {
    uint32_t c[PER];             // choice of expert lane + 32 j; 0: not available
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int e = lane + 32 * j;
        c[j] = e < p.experts ? ordered(score[e] + correction[e]) : 0u;
    }
    if (p.keep < p.groups) {
        int share = 32;          // lanes of a group
        while (share * p.groups > 32) share >>= 1;
        const int n = p.experts / p.groups, g = lane / share;
        float a = -INFINITY, b = -INFINITY;                 // the group's two best
        if (g < p.groups)
            for (int i = lane % share; i < n; i += share) {
                const float v = score[g * n + i] + correction[g * n + i];
                b = fmaxf(b, fminf(a, v)), a = fmaxf(a, v);
            }
        for (int o = share >> 1; o > 0; o >>= 1) {
            const float oa = __shfl_xor_sync(0xffffffffu, a, o), ob = __shfl_xor_sync(0xffffffffu, b, o);
            b = fmaxf(fmaxf(b, ob), fminf(a, oa)), a = fmaxf(a, oa);
        }
        uint32_t key = g < p.groups && lane % share == 0 ? ordered(n > 1 ? a + b : a) : 0u, kept = 0u;
        for (int k = 0; k < p.keep; ++k) {
            const uint32_t best = __reduce_max_sync(0xffffffffu, key);
            const int at = __ffs(__ballot_sync(0xffffffffu, key == best)) - 1;
            kept |= 1u << (at / share);
            if (lane == at) key = 0u;
        }
#pragma unroll
        for (int j = 0; j < PER; ++j)
            if (lane + 32 * j < p.experts && !(kept >> ((lane + 32 * j) / n) & 1)) c[j] = 0u;
    }
    int id = 0;                  // lane k: the k-th choice
    for (int k = 0; k < p.top; ++k) {
        uint32_t best = 0u;
#pragma unroll
        for (int j = 0; j < PER; ++j) best = max(best, c[j]);
        best = __reduce_max_sync(0xffffffffu, best);
        int e = p.experts;
#pragma unroll
        for (int j = PER - 1; j >= 0; --j)
            if (c[j] == best && lane + 32 * j < p.experts) e = lane + 32 * j;
        e = min(__reduce_min_sync(0xffffffffu, e), p.experts - 1);
#pragma unroll
        for (int j = 0; j < PER; ++j)
            if (lane + 32 * j == e) c[j] = 0u;
        if (lane == k) id = e;
    }
    float w = score[id];
    if (p.softmax) {
        float m = -INFINITY, sum = 0.0f;
        for (int e = lane; e < p.experts; e += 32) m = fmaxf(m, score[e]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        for (int e = lane; e < p.experts; e += 32) sum += expf(score[e] - m);
        w = expf(w - m) / warp_sum(sum);
        w /= warp_sum(lane < p.top ? w : 0.0f) + 1e-20f;
    }
    if (lane < p.top) {
        p.ids[(size_t)t * p.top + lane] = id;
        p.weights[(size_t)t * p.top + lane] = w * p.scale;
    }
}

// A warp per token.
template <int PER>
__global__ void __launch_bounds__(128) k_moe_route(const RouteParams p, const float* __restrict__ logits, int ldl, int T) {
    __shared__ float score[4][32 * PER], correction[32 * PER];
    pdl_launch_dependents();
    for (int e = threadIdx.x; e < p.experts; e += 128) correction[e] = p.correction ? p.correction[e] : 0.0f;
    __syncthreads();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp;
    if (t >= T) return;
    for (int e = lane; e < p.experts; e += 32) {
        const float z = logits[(size_t)t * ldl + e];
        score[warp][e] = p.softmax ? z : sigmoid(z);
    }
    __syncwarp();
    choose<PER>(p, score[warp], correction, t, lane);
}

// ---------------------------------------------------------------- norm and choices together
struct NormRouteParams {
    RouteParams r;
    dc_hyper hy;             // S > 0: where the row comes from
    const float *x, *w;
    const __nv_bfloat16* router;
    int ldw, H, ld;
    float eps;
    float* out;
    __nv_bfloat16* outb;
};

constexpr int NR_CTAS = 8, NR_WARPS = 8, NR_AHEAD = 4;

// A cluster per token: every CTA norms the row and takes its share of the experts, the first one chooses.  S: streams at most
// (0: the row is x).
template <int PER, int S>
__global__ void __launch_bounds__(NR_WARPS * 32) k_moe_norm_route(const NormRouteParams p) {
    extern __shared__ __align__(16) float h[];              // the normed row, padded with zeros to a multiple of 256
    __shared__ float red[33], score[32 * PER], correction[32 * PER], coef[S ? S * (S + 2) : 1];
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");       // waited for ahead of the first remote store
    pdl_launch_dependents();
    const int rank = blockIdx.x % NR_CTAS, t = blockIdx.x / NR_CTAS, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int per = (p.r.experts + NR_CTAS - 1) / NR_CTAS, e0 = rank * per, e1 = min(p.r.experts, e0 + per);
    const int K8 = p.ld;         // rows of the matrix are padded with zeros beyond the width
    auto fetch = [&](int e, int i) {
        const int k = 8 * lane + 256 * i;
        return e < e1 && k < K8 ? __ldg(reinterpret_cast<const uint4*>(p.router + (size_t)e * p.ldw + k)) : make_uint4(0, 0, 0, 0);
    };
    uint4 ahead[NR_AHEAD];
#pragma unroll
    for (int i = 0; i < NR_AHEAD; ++i) ahead[i] = fetch(e0 + warp, i);
    for (int e = e0 + warp; e < e1; e += NR_WARPS)          // the rest comes from L2
        for (int k = 64 * lane; k < K8; k += 64 * 32) prefetch_l2(p.router + (size_t)e * p.ldw + k);
    if (rank == 0)
        for (int e = tid; e < p.r.experts; e += NR_WARPS * 32) correction[e] = p.r.correction ? p.r.correction[e] : 0.0f;
    if constexpr (S > 0) {
        if (tid < S * (S + 2)) coef[tid] = hyper_coefficient<S>(p.hy, tid);
        __syncthreads();
    }
    pdl_wait();
    const int n4 = p.ld / 4;
    const float4* x4 = reinterpret_cast<const float4*>(p.x + (size_t)t * p.ld);
    float ss = 0.0f;
    for (int i = tid; i < n4; i += NR_WARPS * 32) {
        float4 v;
        if constexpr (S > 0) {
            float4 streams[S];
            hyper_load<S>(p.hy, t, i, p.ld, streams);
            v = hyper_mix<S>(p.hy, coef, t, i, p.ld, streams, reinterpret_cast<const float4*>(p.hy.y + (size_t)t * p.ld)[i], i % NR_CTAS == rank);
        } else {
            v = x4[i];
        }
        reinterpret_cast<float4*>(h)[i] = v;
        ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.H + p.eps);
    for (int i = tid; i < (p.ld + 255) / 256 * 64; i += NR_WARPS * 32) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n4) {
            const float4 a = reinterpret_cast<float4*>(h)[i], w = reinterpret_cast<const float4*>(p.w)[i];
            v = make_float4(a.x * inv * w.x, a.y * inv * w.y, a.z * inv * w.z, a.w * inv * w.w);
            if (i % NR_CTAS == rank) {
                const size_t at = (size_t)t * p.ld / 4 + i;
                if (p.outb) reinterpret_cast<uint2*>(p.outb)[at] = make_uint2(pack_bf2(v.x, v.y), pack_bf2(v.z, v.w));
                else reinterpret_cast<float4*>(p.out)[at] = v;
            }
        }
        reinterpret_cast<float4*>(h)[i] = v;
    }
    __syncthreads();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    for (int e = e0 + warp; e < e1; e += NR_WARPS) {
        float a = 0.0f;
        for (int i0 = 0; 256 * i0 < K8; i0 += NR_AHEAD) {
            uint4 c[NR_AHEAD];
#pragma unroll
            for (int i = 0; i < NR_AHEAD; ++i) {
                c[i] = ahead[i];
                const bool more = 256 * (i0 + NR_AHEAD) < K8;
                ahead[i] = more ? fetch(e, i0 + NR_AHEAD + i) : fetch(e + NR_WARPS, i);
            }
#pragma unroll
            for (int i = 0; i < NR_AHEAD; ++i) {
                const int k = 8 * lane + 256 * (i0 + i);
                if (256 * (i0 + i) >= K8) break;
                float f[8];
                unpack16(c[i], f, __nv_bfloat16());
                const float4 u = *reinterpret_cast<const float4*>(h + k), v = *reinterpret_cast<const float4*>(h + k + 4);
                a = fmaf(f[0], u.x, fmaf(f[1], u.y, fmaf(f[2], u.z, fmaf(f[3], u.w, a))));
                a = fmaf(f[4], v.x, fmaf(f[5], v.y, fmaf(f[6], v.z, fmaf(f[7], v.w, a))));
            }
        }
        a = warp_sum(a);
        if (!p.r.softmax) a = sigmoid(a);
        if (lane == 0) {
            uint32_t to;
            asm("mapa.shared::cluster.u32 %0, %1, 0;" : "=r"(to) : "r"(smem_u32(score + e)));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(to), "f"(a) : "memory");
        }
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (rank == 0 && warp == 0) choose<PER>(p.r, score, correction, t, lane);
}

// Prompts of bf16 models: sixteen tokens per CTA, a warp norms each; the router product takes the rounded rows (tensor cores,
// f32 sums), sixteen experts and a share of the columns per warp; then a warp chooses for each token.  Without NORM the rounded rows
// are there already.
constexpr int NT_WARPS = 16, NT_AHEAD = 4;
struct TileSizes {
    int tiles, shares, ldh;      // expert tiles, column shares, pitch of a normed row in shared memory
    size_t part, score, bytes;   // offsets
    __host__ __device__ static TileSizes of(int experts, int ld) {
        TileSizes z;
        z.tiles = (experts + 15) / 16;
        z.shares = z.tiles < NT_WARPS ? NT_WARPS / z.tiles : 1;
        z.ldh = (ld + 63) / 64 * 64 + 32;
        z.part = (size_t)16 * z.ldh * 2;
        z.score = z.part + (size_t)z.shares * z.tiles * 16 * 17 * 4;
        z.bytes = z.score + (size_t)16 * z.tiles * 16 * 4;
        return z;
    }
};

template <int PER, bool NORM>
__global__ void __launch_bounds__(NT_WARPS * 32) k_moe_norm_route_tile(const NormRouteParams p, int rows, int T) {
    extern __shared__ __align__(16) uint8_t sm[];
    __shared__ float correction[32 * PER];
    const TileSizes z = TileSizes::of(p.r.experts, p.ld);
    __nv_bfloat16* h = reinterpret_cast<__nv_bfloat16*>(sm);            // [16][ldh]
    float* part = reinterpret_cast<float*>(sm + z.part);                // [shares][experts][17]
    float* score = reinterpret_cast<float*>(sm + z.score);              // [16][experts]
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3, t = blockIdx.x * 16 + warp, E = 16 * z.tiles;
    const int runs = (p.ld + 31) / 32, n4 = p.ld / 4;
    const int share = warp / z.tiles, per = (runs + z.shares - 1) / z.shares, begin = share * per, end = min(runs, begin + per);
    uint4 a[NT_AHEAD][2];
    auto fetch = [&](int j, int tile, int run) {
        const int k = 32 * run + 8 * q;
        const bool ok = run < end && k < p.ld;
        const __nv_bfloat16* w = p.router + (ok ? k : 0);
        a[j][0] = ok ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)min(16 * tile + g, rows - 1) * p.ldw)) : make_uint4(0, 0, 0, 0);
        a[j][1] = ok ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)min(16 * tile + 8 + g, rows - 1) * p.ldw)) : make_uint4(0, 0, 0, 0);
    };
    const bool working = share < z.shares;
    if (working)
#pragma unroll
        for (int j = 0; j < NT_AHEAD; ++j) fetch(j, warp % z.tiles, begin + j);
    for (int e = tid; e < p.r.experts; e += NT_WARPS * 32) correction[e] = p.r.correction ? p.r.correction[e] : 0.0f;
    pdl_wait();
    if constexpr (!NORM) {
        const uint4* from = reinterpret_cast<const uint4*>(p.outb + (size_t)min(t, T - 1) * p.ld);
        uint4* to = reinterpret_cast<uint4*>(h + warp * z.ldh);
#pragma unroll 8
        for (int i = lane; i < (z.ldh - 32) / 8; i += 32) to[i] = i < p.ld / 8 ? from[i] : make_uint4(0, 0, 0, 0);
    } else {
        const float4* x4 = reinterpret_cast<const float4*>(p.x + (size_t)min(t, T - 1) * p.ld);
        const float4* w4 = reinterpret_cast<const float4*>(p.w);
        uint2* to = reinterpret_cast<uint2*>(h + warp * z.ldh);
        constexpr int KEEP = 16;             // groups of four that a lane holds; wider rows are read twice
        float4 x[KEEP];
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < KEEP; ++j) x[j] = lane + 32 * j < n4 ? x4[lane + 32 * j] : make_float4(0.f, 0.f, 0.f, 0.f);
        auto square = [&](const float4& v) { ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); };
#pragma unroll
        for (int j = 0; j < KEEP; ++j) square(x[j]);
#pragma unroll 8
        for (int i = lane + 32 * KEEP; i < n4; i += 32) square(x4[i]);
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.H + p.eps);
        auto put = [&](int i, const float4& v) {
            uint2 r = make_uint2(0u, 0u);
            if (i < n4) {
                const float4 w = w4[i];
                r = make_uint2(pack_bf2(v.x * inv * w.x, v.y * inv * w.y), pack_bf2(v.z * inv * w.z, v.w * inv * w.w));
                if (t < T) reinterpret_cast<uint2*>(p.outb + (size_t)t * p.ld)[i] = r;
            }
            if (i < (z.ldh - 32) / 4) to[i] = r;
        };
#pragma unroll
        for (int j = 0; j < KEEP; ++j) put(lane + 32 * j, x[j]);
#pragma unroll 8
        for (int i = lane + 32 * KEEP; i < (z.ldh - 32) / 4; i += 32) put(i, i < n4 ? x4[i] : make_float4(0.f, 0.f, 0.f, 0.f));
    }
    __syncthreads();
    for (int tile = warp % z.tiles; working && tile < z.tiles; tile += z.shares > 1 ? z.tiles : NT_WARPS) {
        float acc[2][4] = {};
        if (tile != warp % z.tiles)
#pragma unroll
            for (int j = 0; j < NT_AHEAD; ++j) fetch(j, tile, begin + j);
        for (int rb = begin; rb < end; rb += NT_AHEAD) {
#pragma unroll
            for (int j = 0; j < NT_AHEAD; ++j) {
                const int run = rb + j;
                const uint4 a0 = a[j][0], a1 = a[j][1];
                fetch(j, tile, run + NT_AHEAD);
                if (run >= end) continue;
                const uint32_t lo[4] = {a0.x, a1.x, a0.y, a1.y}, hi[4] = {a0.z, a1.z, a0.w, a1.w};
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const uint4 b = *reinterpret_cast<const uint4*>(h + (8 * i + g) * z.ldh + 32 * run + 8 * q);
                    mma_bf16(acc[i], lo, b.x, b.y);
                    mma_bf16(acc[i], hi, b.z, b.w);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) part[(size_t)(share * E + 16 * tile + g + 8 * (j >> 1)) * 17 + 8 * i + 2 * q + (j & 1)] = acc[i][j];
    }
    __syncthreads();
    for (int i = tid; i < 16 * E; i += NT_WARPS * 32) {
        const int e = i % E, tok = i / E;
        float v = 0.0f;
        for (int k = 0; k < z.shares; ++k) v += part[(size_t)(k * E + e) * 17 + tok];
        score[tok * E + e] = p.r.softmax ? v : sigmoid(v);
    }
    __syncthreads();
    if (t < T) choose<PER>(p.r, score + warp * E, correction, t, lane);
}

// ---------------------------------------------------------------- few tokens: weights streamed once
constexpr int ME_WARPS = 16;     // warps of a CTA; a CTA takes sixteen rows at a time, column order within a run of 32 as in linear.cu

// The distinct experts of a step and which of their assignments (-1: none) belongs to which token, in shared memory.
template <int NT>
struct Units {
    static constexpr int CAP = 8 * NT * DC_MOE_MAX_TOP;
    int16_t expert[CAP], asg[CAP][8 * NT];
    int first[DC_MOE_MAX_EXPERTS], n;

    __device__ __forceinline__ void clear(int T, int experts) {         // ahead of the dependency wait
        if (T == 1) return;
        for (int i = threadIdx.x; i < experts; i += ME_WARPS * 32) first[i] = 1 << 30;
        for (int i = threadIdx.x; i < CAP * 8 * NT / 2; i += ME_WARPS * 32) reinterpret_cast<uint32_t*>(&asg[0][0])[i] = 0xffffffffu;
        __syncthreads();
    }
    __device__ __forceinline__ void build(const int32_t* ids, int T, int top) {
        const int tid = threadIdx.x, lane = tid & 31, A = T * top;
        if (T == 1) {
            if (tid < A) expert[tid] = (int16_t)ids[tid], asg[tid][0] = (int16_t)tid;
            if (tid == 0) n = A;
            __syncthreads();
            return;
        }
        for (int i = tid; i < A; i += ME_WARPS * 32) atomicMin(&first[ids[i]], i);
        __syncthreads();
        if (tid < 32) {
            int count = 0;
            for (int i0 = 0; i0 < A; i0 += 32) {
                const int i = i0 + lane, e = i < A ? ids[i] : 0;
                const bool is = i < A && first[e] == i;
                const unsigned hit = __ballot_sync(0xffffffffu, is);
                const int u = count + __popc(hit & ((1u << lane) - 1));
                if (is) expert[u] = (int16_t)e;
                __syncwarp();
                if (is) first[e] = -1 - u;
                __syncwarp();
                count += __popc(hit);
            }
            if (lane == 0) n = count;
        }
        __syncthreads();
        for (int i = tid; i < A; i += ME_WARPS * 32) asg[-1 - first[ids[i]]][i / top] = (int16_t)i;
        __syncthreads();
    }
};

struct UpParams {
    const __nv_bfloat16* w;
    int K, ldw, rows, top, T, ff, experts;
    float limit;
    bool plain;
    const __nv_bfloat16* x;
    int ldx;
    const int32_t* ids;
    const float* weights;
    __nv_bfloat16* hid;
    int ldh;
};

// Gate and up rows (plain: up rows) of every distinct expert for its tokens: hidden value times routing weight.  A CTA walks over tiles of
// sixteen rows and fetches the next tile's first runs ahead of a tile's sum.
template <int NT>
__global__ void __launch_bounds__(ME_WARPS * 32, 2) k_moe_up_mma(const UpParams p) {
    constexpr int AHEAD = 2, BUFS = NT > 1 ? 1 : 2;
    __shared__ float red[BUFS][ME_WARPS][16][8 * NT + 1];
    __shared__ Units<NT> units;
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3;
    const int K8 = (p.K + 7) & ~7, runs = (p.K + 31) / 32, row_tiles = p.rows / 16;
    units.clear(p.T, p.experts);
    pdl_wait();
    units.build(p.ids, p.T, p.top);
    const int tiles = units.n * row_tiles;
    uint4 a[AHEAD][2];
    auto rows_of = [&](int tile) {          // the lane's first row and column of a tile, null: no more tiles
        const int u = tile / row_tiles;
        return tile < tiles ? p.w + ((size_t)units.expert[u] * p.rows + 16 * (tile - u * row_tiles) + g) * p.ldw + 8 * q : nullptr;
    };
    auto fetch = [&](int j, const __nv_bfloat16* w, int run) {
        const bool ok = w && run < runs && 32 * run + 8 * q < K8;
        a[j][0] = ok ? __ldg(reinterpret_cast<const uint4*>(w + 32 * run)) : make_uint4(0, 0, 0, 0);
        a[j][1] = ok ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)8 * p.ldw + 32 * run)) : make_uint4(0, 0, 0, 0);
    };
    int tile = blockIdx.x;
    const __nv_bfloat16* w = rows_of(tile);
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) fetch(j, w, warp * AHEAD + j);
    for (int buf = 0; tile < tiles; tile += gridDim.x, buf ^= BUFS - 1) {
        const int u = tile / row_tiles;
        const __nv_bfloat16* next = rows_of(tile + gridDim.x);
        const __nv_bfloat16* x[NT];
#pragma unroll
        for (int i = 0; i < NT; ++i) x[i] = units.asg[u][8 * i + g] >= 0 && 8 * i + g < p.T ? p.x + (size_t)(8 * i + g) * p.ldx : nullptr;
        float acc[NT][4];
#pragma unroll
        for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
        for (int rb = warp * AHEAD; rb < runs; rb += ME_WARPS * AHEAD) {
            const bool last = rb + ME_WARPS * AHEAD >= runs;
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                const int run = rb + j, k = 32 * run + 8 * q;
                const uint4 a0 = a[j][0], a1 = a[j][1];
                fetch(j, last ? next : w, last ? warp * AHEAD + j : run + ME_WARPS * AHEAD);
                if (run >= runs) continue;
                const uint32_t lo[4] = {a0.x, a1.x, a0.y, a1.y}, hi[4] = {a0.z, a1.z, a0.w, a1.w};
#pragma unroll
                for (int i = 0; i < NT; ++i) {
                    const uint4 b = x[i] && k < K8 ? *reinterpret_cast<const uint4*>(x[i] + k) : make_uint4(0, 0, 0, 0);
                    mma_bf16(acc[i], lo, b.x, b.y);
                    mma_bf16(acc[i], hi, b.z, b.w);
                }
            }
        }
        w = next;
        if (BUFS == 1) __syncthreads();
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) red[buf][warp][g + 8 * (j >> 1)][8 * i + 2 * q + (j & 1)] = acc[i][j];
        __syncthreads();
        const int r = tid & 15, t = tid >> 4, o = 8 * (tile - u * row_tiles) + (r >> 1);
        if (tid >= 128 * NT) continue;
        float v = 0.0f;
#pragma unroll
        for (int i = 0; i < ME_WARPS; ++i) v += red[buf][i][r][t];
        const float up = __shfl_down_sync(0xffffffffu, v, 1);
        const int as = t < p.T ? units.asg[u][t] : -1;
        if (p.plain) {
            const int row = 16 * (tile - u * row_tiles) + r;
            if (as >= 0 && row < p.ff) p.hid[(size_t)as * p.ldh + row] = __float2bfloat16_rn(relu2(v) * p.weights[as]);
        } else if (!(r & 1) && as >= 0 && o < p.ff) {
            dc_lin_epi epi;
            epi.pair_kind = DC_PAIR_CLAMPED, epi.limit = p.limit;
            p.hid[(size_t)as * p.ldh + o] = __float2bfloat16_rn(pair_value(epi, v, up) * p.weights[as]);
        }
    }
}

struct DownParams {
    const __nv_bfloat16* w;
    int K, ldw, rows, top, T, H, experts;
    const __nv_bfloat16* hid;
    int ldh;
    const int32_t* ids;
    float* x;
    int ldx;
    bool add;
};

// x[t] = or += sum over the token's assignments of W_down hid.  The distinct experts' columns are one long row: a token has
// zeros where an expert is not its own.  KS: CTAs of a cluster that share sixteen rows, each with its part of that row.
template <int NT, int KS>
__global__ void __launch_bounds__(ME_WARPS * 32, 2) k_moe_down_mma(const DownParams p) {
    constexpr int AHEAD = NT > 1 ? 2 : 3;
    __shared__ float red[ME_WARPS][16][8 * NT + 1];
    __shared__ float other[KS > 1 ? KS - 1 : 1][KS > 1 ? 128 * NT : 1];
    __shared__ Units<NT> units;
    if (KS > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3, part = blockIdx.x % KS, row0 = blockIdx.x / KS * 16;
    const int K8 = (p.K + 7) & ~7, per_expert = (p.K + 31) / 32;
    units.clear(p.T, p.experts);
    pdl_wait();
    units.build(p.ids, p.T, p.top);
    const int all = units.n * per_expert, share = (all + KS - 1) / KS, begin = part * share, end = min(all, begin + share);
    uint4 a[AHEAD][2];
    auto fetch = [&](int j, int run) {
        const int u = run / per_expert, k = 32 * (run - u * per_expert) + 8 * q;
        const bool ok = run < end && k < K8;
        const __nv_bfloat16* w = p.w + ((size_t)units.expert[ok ? u : 0] * p.rows + row0 + g) * p.ldw + (ok ? k : 0);
        a[j][0] = ok ? __ldg(reinterpret_cast<const uint4*>(w)) : make_uint4(0, 0, 0, 0);
        a[j][1] = ok ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)8 * p.ldw)) : make_uint4(0, 0, 0, 0);
    };
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) fetch(j, begin + warp * AHEAD + j);
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    for (int rb = begin + warp * AHEAD; rb < end; rb += ME_WARPS * AHEAD) {
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int run = rb + j;
            const uint4 a0 = a[j][0], a1 = a[j][1];
            fetch(j, run + ME_WARPS * AHEAD);
            if (run >= end) continue;
            const int u = run / per_expert, k = 32 * (run - u * per_expert) + 8 * q;
            const uint32_t lo[4] = {a0.x, a1.x, a0.y, a1.y}, hi[4] = {a0.z, a1.z, a0.w, a1.w};
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int t = 8 * i + g, as = t < p.T ? units.asg[u][t] : -1;
                const uint4 b = as >= 0 && k < K8 ? *reinterpret_cast<const uint4*>(p.hid + (size_t)as * p.ldh + k) : make_uint4(0, 0, 0, 0);
                mma_bf16(acc[i], lo, b.x, b.y);
                mma_bf16(acc[i], hi, b.z, b.w);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) red[warp][g + 8 * (j >> 1)][8 * i + 2 * q + (j & 1)] = acc[i][j];
    __syncthreads();
    const int r = tid & 15, t = tid >> 4, row = row0 + r;
    const bool mine = tid < 128 * NT;
    float v = 0.0f;
    if (mine)
#pragma unroll
        for (int i = 0; i < ME_WARPS; ++i) v += red[i][r][t];
    if (KS > 1) {
        asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
        if (part > 0 && mine) {
            uint32_t to;
            asm("mapa.shared::cluster.u32 %0, %1, 0;" : "=r"(to) : "r"(smem_u32(&other[part - 1][tid])));
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(to), "f"(v) : "memory");
        }
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
        asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
        if (part > 0) return;
        if (mine)
#pragma unroll
            for (int k = 0; k < KS - 1; ++k) v += other[k][tid];
    }
    if (mine && t < p.T && row < p.H) p.x[(size_t)t * p.ldx + row] = p.add ? p.x[(size_t)t * p.ldx + row] + v : v;
}

// ---------------------------------------------------------------- many tokens: assignments sorted by expert
// A CTA per expert: how many assignments go to lower experts, then its own.  A warp has a run of assignments and reads 128 of
// them at a time.
__global__ void __launch_bounds__(256) k_moe_order(const int32_t* __restrict__ ids, const float* __restrict__ weights, int A, int top, int experts,
                                                   int32_t* __restrict__ off, int32_t* src, float* __restrict__ row_w, int32_t* __restrict__ row) {
    __shared__ int s_mine[8], s_below[8];
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per = (A + 1023) / 1024 * 128, begin = min(A, warp * per), end = min(A, begin + per);
    auto four = [&](int i, int (&v)[4]) {                   // -1 beyond the run
        if (i + 4 <= end) {
            const int4 u = *reinterpret_cast<const int4*>(ids + i);
            v[0] = u.x, v[1] = u.y, v[2] = u.z, v[3] = u.w;
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) v[j] = i + j < end ? ids[i + j] : -1;
        }
    };
    constexpr int B = 8;         // loads in flight
    int mine = 0, below = 0;
    for (int i0 = begin; i0 < end; i0 += 128 * B) {
        int v[B][4];
#pragma unroll
        for (int k = 0; k < B; ++k) four(i0 + 128 * k + 4 * lane, v[k]);
#pragma unroll
        for (int k = 0; k < B; ++k)
#pragma unroll
            for (int j = 0; j < 4; ++j) mine += v[k][j] == e, below += v[k][j] >= 0 && v[k][j] < e;
    }
    mine = __reduce_add_sync(0xffffffffu, mine), below = __reduce_add_sync(0xffffffffu, below);
    if (lane == 0) s_mine[warp] = mine, s_below[warp] = below;
    __syncthreads();
    int at = 0, total = 0, own = 0;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
        at += s_below[w] + (w < warp ? s_mine[w] : 0);
        total += s_below[w], own += s_mine[w];
    }
    if (threadIdx.x == 0) {
        off[e] = total;
        if (e == experts - 1) off[experts] = A;
    }
    for (int i0 = begin; i0 < end && mine; i0 += 128 * B) {
        int v[B][4];
#pragma unroll
        for (int k = 0; k < B; ++k) four(i0 + 128 * k + 4 * lane, v[k]);
#pragma unroll
        for (int k = 0; k < B; ++k)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const unsigned hit = __ballot_sync(0xffffffffu, v[k][j] == e);
                if (v[k][j] == e) src[at + __popc(hit & ((1u << lane) - 1))] = i0 + 128 * k + 4 * lane + j;
                at += __popc(hit);
            }
    }
    __syncthreads();
    for (int r = total + threadIdx.x; r < total + own; r += 256) {       // the assignments are listed: rows side by side
        const int i = src[r];
        src[r] = i / top;
        row_w[r] = weights[i];
        row[i] = r;
    }
}

// out[r] = x[src[r]], rows of ld elements (a multiple of eight); a warp per row
__global__ void __launch_bounds__(256) k_moe_gather(const __nv_bfloat16* __restrict__ x, int ld, const int32_t* __restrict__ src, int rows,
                                                    __nv_bfloat16* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (r >= rows) return;
    const uint4* from = reinterpret_cast<const uint4*>(x + (size_t)src[r] * ld);
    uint4* to = reinterpret_cast<uint4*>(out + (size_t)r * ld);
#pragma unroll 8
    for (int i = lane; i < ld / 8; i += 32) to[i] = from[i];
}

// f32 tile product of an expert's rows: 64 weight rows x 64 sorted rows per CTA, 4 x 4 outputs per thread.
struct F32Params {
    const __nv_bfloat16* w;
    int K, ldw, experts, group_rows;
    const int32_t* off;
    const float* x;
    int ldx;
    const int32_t* src;
    dc_lin_epi e;
};

__global__ void __launch_bounds__(256) k_moe_f32(const F32Params p) {
    __shared__ float sw[16][68], sx[16][68];
    pdl_launch_dependents();
    pdl_wait();
    int tile = blockIdx.y, ex = 0, r0 = 0, r1 = 0;
    for (; ex < p.experts; ++ex) {
        r0 = p.off[ex], r1 = p.off[ex + 1];
        const int tiles = (r1 - r0 + 63) / 64;
        if (tile < tiles) break;
        tile -= tiles;
    }
    if (ex == p.experts) return;
    r0 += 64 * tile;
    const __nv_bfloat16* w = p.w + (size_t)ex * p.group_rows * p.ldw;
    const int tid = threadIdx.x, n0 = blockIdx.x * 64, tn = (tid & 15) * 4, tt = (tid >> 4) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int at = tid + i * 256, r = at >> 4, k = at & 15;
            sw[k][r] = n0 + r < p.group_rows && k0 + k < p.K ? __bfloat162float(w[(size_t)(n0 + r) * p.ldw + k0 + k]) : 0.0f;
            const int in = r0 + r < r1 ? p.src ? p.src[r0 + r] : r0 + r : -1;
            sx[k][r] = in >= 0 && k0 + k < p.K ? p.x[(size_t)in * p.ldx + k0 + k] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float4 a = *reinterpret_cast<const float4*>(&sw[k][tn]), b = *reinterpret_cast<const float4*>(&sx[k][tt]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(bv[i], av[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = r0 + tt + i;
        if (t >= r1) continue;
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
            const int n = n0 + tn + j;
            if (n >= p.e.pair0) {
                const int c = (n - p.e.pair0) >> 1;
                if (c < p.e.n_pairs) put_pair(p.e, t, c, pair_value(p.e, acc[i][j], acc[i][j + 1]) * (p.e.tok_scale ? p.e.tok_scale[t] : 1.0f));
            } else {
                if (n < p.e.n_store) put_row(p.e, t, n, acc[i][j]);
                if (n + 1 < p.e.n_store) put_row(p.e, t, n + 1, acc[i][j + 1]);
            }
        }
    }
}

RouteParams route_params(const dc_moe_ffn& f, int32_t* ids, float* weights) {
    return RouteParams{f.experts, f.top, f.groups, f.keep, f.scale, f.softmax, f.correction, ids, weights};
}

template <int NT, int KS>
int launch_down(dc_ctx* ctx, const DownParams& p) {
    const int tiles = p.rows / 16;
    const dim3 block(ME_WARPS * 32);
    if (KS > 1) return dc_launch_cluster(ctx, "k_moe_down_mma", k_moe_down_mma<NT, KS>, dim3(tiles * KS), block, 0, KS, p);
    return dc_launch(ctx, "k_moe_down_mma", k_moe_down_mma<NT, 1>, dim3(tiles), block, 0, p);
}

template <int PER>
int launch_route_tile(dc_ctx* ctx, const NormRouteParams& p, const dc_moe_ffn& f, int T, bool normed) {
    const TileSizes z = TileSizes::of(f.experts, p.ld);
    const void* k = normed ? (const void*)k_moe_norm_route_tile<PER, false> : (const void*)k_moe_norm_route_tile<PER, true>;
    const int st = dc_kernel_setup(ctx, k, (int)z.bytes, "k_moe_norm_route_tile");
    if (st != DC_B200_OK) return st;
    const dim3 grid((T + 15) / 16), block(NT_WARPS * 32);
    if (normed) return dc_launch(ctx, "k_moe_route_tile", k_moe_norm_route_tile<PER, false>, grid, block, z.bytes, p, f.router.N, T);
    return dc_launch(ctx, "k_moe_norm_route_tile", k_moe_norm_route_tile<PER, true>, grid, block, z.bytes, p, f.router.N, T);
}

}  // namespace

int dc_launch_moe_norm_route(dc_ctx* ctx, const dc_moe_ffn& f, const float* x, const dc_hyper* hy, const float* w, int T, int H, int ld, float eps, float* out,
                             __nv_bfloat16* outb, int32_t* ids, float* weights) {
    if (f.experts > DC_MOE_MAX_EXPERTS || f.groups > DC_MOE_MAX_GROUPS || ld % 8) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "moe_norm_route: bad operand");
    // prompt-sized steps bring the streams up to date in a kernel of their own: what this one reads of a row it would read twice
    if (hy && T > DC_MAX_T) {
        const int st = dc_launch_hyper_norm(ctx, *hy, w, nullptr, 0, T, H, ld, eps, out, outb);
        if (st != DC_B200_OK) return st;
    } else if (hy && (hy->streams > DC_MAX_STREAMS || hy->sum.k || !hy->y || !hy->x_out || hy->x == hy->x_out))
        return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "moe_norm_route: bad streams");
    const NormRouteParams p = {route_params(f, ids, weights), hy ? *hy : dc_hyper(), x, w, f.router.w, f.router.ld, H, ld, eps, out, outb};
    const size_t smem = (size_t)(ld + 255) / 256 * 256 * 4;
#define DC_ROUTE_S(PER, S)                                                                                                                       \
    do {                                                                                                                                         \
        const int st = dc_kernel_setup_small(ctx, (const void*)k_moe_norm_route<PER, S>, (int)smem, "k_moe_norm_route");                          \
        if (st != DC_B200_OK) return st;                                                                                                         \
        return dc_launch_cluster(ctx, "k_moe_norm_route", k_moe_norm_route<PER, S>, dim3(T * NR_CTAS), dim3(NR_WARPS * 32), smem, NR_CTAS, p);    \
    } while (0)
#define DC_ROUTE(PER)                                   \
    do {                                                \
        if (T > DC_MAX_T) return launch_route_tile<PER>(ctx, p, f, T, hy != nullptr); \
        if (!hy) DC_ROUTE_S(PER, 0);                    \
        if (hy->streams <= 2) DC_ROUTE_S(PER, 2);       \
        if (hy->streams <= 4) DC_ROUTE_S(PER, 4);       \
        DC_ROUTE_S(PER, DC_MAX_STREAMS);                \
    } while (0)
    if (f.experts <= 64) DC_ROUTE(2);
    if (f.experts <= 128) DC_ROUTE(4);
    if (f.experts <= 256) DC_ROUTE(8);
    DC_ROUTE(16);
#undef DC_ROUTE
#undef DC_ROUTE_S
}

bool dc_moe_norm_route_fits(const dc_moe_ffn& f, bool b16, int T, int ld) {
    return T <= DC_MAX_T || (b16 && TileSizes::of(f.experts, ld).bytes <= 200 * 1024);
}

int dc_launch_moe_route(dc_ctx* ctx, const dc_moe_ffn& f, const float* logits, int ldl, int T, int32_t* ids, float* weights) {
    if (f.experts > DC_MOE_MAX_EXPERTS || f.groups > DC_MOE_MAX_GROUPS) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "moe_route: bad operand");
    const dim3 grid((T + 3) / 4), block(128);
    if (f.experts <= 128) return dc_launch(ctx, "k_moe_route", k_moe_route<4>, grid, block, 0, route_params(f, ids, weights), logits, ldl, T);
    return dc_launch(ctx, "k_moe_route", k_moe_route<16>, grid, block, 0, route_params(f, ids, weights), logits, ldl, T);
}

int dc_launch_moe_order(dc_ctx* ctx, const dc_moe_ffn& f, const int32_t* ids, const float* weights, int T, int32_t* off, int32_t* src, float* row_w,
                        int32_t* row) {
    return dc_launch(ctx, "k_moe_order", k_moe_order, dim3(f.experts), dim3(256), 0, ids, weights, T * f.top, f.top, f.experts, off, src, row_w, row);
}

int dc_launch_moe_gather(dc_ctx* ctx, const __nv_bfloat16* x, int ldx, const int32_t* src, int rows, __nv_bfloat16* out) {
    return dc_launch(ctx, "k_moe_gather", k_moe_gather, dim3((rows + 7) / 8), dim3(256), 0, x, ldx, src, rows, out);
}

int dc_launch_moe_up_mma(dc_ctx* ctx, const dc_moe_ffn& f, const __nv_bfloat16* xb, int ldx, int T, const int32_t* ids, const float* weights,
                         __nv_bfloat16* hid, int ldh) {
    if (T < 1 || T > DC_MAX_T || ldx % 8) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "moe_up: bad operand");
    const UpParams p = {f.up.w, f.up.K, f.up.ld, f.up_rows, f.top, T, f.ff, f.experts, f.limit, f.plain, xb, ldx, ids, weights, hid, ldh};
    const int tiles = f.up_rows / 16 * std::min(f.experts, T * f.top), room = 2 * ctx->num_sms, rounds = (tiles + room - 1) / room;
    const dim3 grid(T == 1 ? (tiles + rounds - 1) / rounds : std::min(tiles, room)), block(ME_WARPS * 32);
    if (T <= 8) return dc_launch(ctx, "k_moe_up_mma", k_moe_up_mma<1>, grid, block, 0, p);
    return dc_launch(ctx, "k_moe_up_mma", k_moe_up_mma<2>, grid, block, 0, p);
}

int dc_launch_moe_down_mma(dc_ctx* ctx, const dc_moe_ffn& f, const __nv_bfloat16* hid, int ldh, int T, const int32_t* ids, int H, float* x, int ldx,
                             bool add) {
    if (T < 1 || T > DC_MAX_T || ldh % 8) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "moe_down: bad operand");
    const DownParams p = {f.down.w, f.down.K, f.down.ld, f.down_rows, f.top, T, H, f.experts, hid, ldh, ids, x, ldx, add};
    // fewer row tiles than SMs: the long rows are shared by a cluster
    const int tiles = f.down_rows / 16;
    if (2 * tiles <= ctx->num_sms) return T <= 8 ? launch_down<1, 4>(ctx, p) : launch_down<2, 4>(ctx, p);
    if (tiles <= ctx->num_sms) return T <= 8 ? launch_down<1, 2>(ctx, p) : launch_down<2, 2>(ctx, p);
    return T <= 8 ? launch_down<1, 1>(ctx, p) : launch_down<2, 1>(ctx, p);
}

int dc_launch_moe_f32(dc_ctx* ctx, const dc_lin& w, int experts, int group_rows, const int32_t* off, int rows, const float* x, int ldx,
                      const int32_t* src, const dc_lin_epi& epi) {
    F32Params p = {w.w, w.K, w.ld, experts, group_rows, off, x, ldx, src, epi};
    p.e.n_store = std::min(epi.n_store, std::min(group_rows, epi.pair0));
    return dc_launch(ctx, "k_moe_f32", k_moe_f32, dim3((group_rows + 63) / 64, rows / 64 + std::min(experts, rows)), dim3(256), 0, p);
}
