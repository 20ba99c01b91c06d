// Products y = W x with bf16 weights and f32 accumulation for up to sixteen tokens, and for f32 activations.
//
// k_linear_mma (bf16 activations) streams the weight rows once: a CTA takes sixteen rows at a time, its sixteen warps
// take neighbouring runs of 32 columns and feed them to m16n8k16 products.  A lane loads sixteen bytes of a row at a time;
// both operands use the same order of columns within a run, so the fragments need no shuffling.  k_linear_rows (f32
// activations, f32 models) does the same on the CUDA cores: a warp owns R rows, a lane takes runs of eight weights, the
// activations come through L1.  Weights do not depend on the kernel before, so every warp fetches its first ones
// ahead of the dependency wait.  k_linear_f32 (any number of tokens, f32 models) is a 64 x 64 shared-memory tile
// product.
//
// Epilogues (dc_lin_epi): store with bias and silu, add to the residual, one value per gate and up row pair; stored rows
// can also be folded into packed greedy picks per token.
#include <algorithm>

#include "dc_common.cuh"
#include "dc_launch.cuh"
#include "dc_stack.h"
#include "dc_stack.cuh"

namespace {

constexpr int LR_WARPS = 4;

struct RowsParams {
    const __nv_bfloat16* w;
    int N, K, ldw;
    const float* x;
    int ldx, T;
    dc_lin_epi e;
};

// TT: tokens (at most), R: rows of a warp, D: 16-byte loads per row that a lane keeps in flight.
template <int TT, int R, int D>
__global__ void __launch_bounds__(LR_WARPS * 32) k_linear_rows(const RowsParams p) {
    dc::pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row0 = (blockIdx.x * LR_WARPS + warp) * R;
    const bool live = row0 < p.N;
    const int K8 = (p.K + 7) & ~7;
    const uint4* wr[R];
#pragma unroll
    for (int r = 0; r < R; ++r) wr[r] = reinterpret_cast<const uint4*>(p.w + (size_t)min(row0 + r, p.N - 1) * p.ldw) + lane;
    uint4 nxt[D][R];
    const int k0 = lane * 8;
#pragma unroll
    for (int j = 0; j < D; ++j)
#pragma unroll
        for (int r = 0; r < R; ++r) nxt[j][r] = live && k0 + 256 * j < K8 ? __ldg(wr[r] + 32 * j) : make_uint4(0, 0, 0, 0);
    dc::pdl_wait();
    uint64_t acc2[TT][R];        // sums over even and odd k
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int r = 0; r < R; ++r) acc2[t][r] = 0;
    if (live) {
        for (int kb = k0; kb < K8; kb += 256 * D) {
#pragma unroll
            for (int j = 0; j < D; ++j) {
                const int k = kb + 256 * j;
                uint64_t wf[R][4];
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const uint4 c = nxt[j][r];
                    nxt[j][r] = k + 256 * D < K8 ? __ldg(wr[r] + (k - k0 + 256 * D) / 8) : make_uint4(0, 0, 0, 0);
                    const uint32_t u[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) wf[r][i] = dc::pair(__uint_as_float(u[i] << 16), __uint_as_float(u[i] & 0xffff0000u));
                }
                if (k >= K8) break;
#pragma unroll
                for (int t = 0; t < TT; ++t) {
                    if (TT > 1 && t >= p.T) break;
                    const float* xr = p.x + (size_t)t * p.ldx + k;
                    uint64_t xv[4];
                    if (k + 8 <= p.K) {
                        const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(xr), b = *reinterpret_cast<const ulonglong2*>(xr + 4);
                        xv[0] = a.x, xv[1] = a.y, xv[2] = b.x, xv[3] = b.y;
                    } else {
#pragma unroll
                        for (int i = 0; i < 4; ++i)
                            xv[i] = dc::pair(k + 2 * i < p.K ? xr[2 * i] : 0.0f, k + 2 * i + 1 < p.K ? xr[2 * i + 1] : 0.0f);
                    }
#pragma unroll
                    for (int r = 0; r < R; ++r)
#pragma unroll
                        for (int i = 0; i < 4; ++i) acc2[t][r] = dc::fma2(wf[r][i], xv[i], acc2[t][r]);
                }
            }
        }
    }
    float acc[TT][R];
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const float2 f = dc::unpair(acc2[t][r]);
            acc[t][r] = dc::warp_sum(f.x + f.y);
        }
    const bool pairs = row0 >= p.e.pair0;
    if (pairs) {
#pragma unroll
        for (int t = 0; t < TT; ++t)
#pragma unroll
            for (int r = 0; r < R; r += 2) {
                const int o = (row0 + r - p.e.pair0) >> 1;
                if (((t * R + r) / 2 & 31) == lane && live && t < p.T && o < p.e.n_pairs) dc::put_pair(p.e, t, o, dc::pair_value(p.e, acc[t][r], acc[t][r + 1]));
            }
    } else {
#pragma unroll
        for (int t = 0; t < TT; ++t)
#pragma unroll
            for (int r = 0; r < R; ++r)
                if (((t * R + r) & 31) == lane && live && t < p.T && row0 + r < p.e.n_store) dc::put_row(p.e, t, row0 + r, acc[t][r]);
    }
    if (!p.e.keys) return;
    // greedy pick: the first maximum wins (key = order-preserving value bits, then the complement of the row)
    __shared__ unsigned long long best[LR_WARPS][TT];
#pragma unroll
    for (int t = 0; t < TT; ++t) {
        unsigned long long k = 0ull;
#pragma unroll
        for (int r = 0; r < R; ++r)
            if (live && row0 + r < p.e.n_store) {
                const unsigned long long c = dc::argmax_key(acc[t][r], row0 + r);
                k = c > k ? c : k;
            }
        if (lane == 0) best[warp][t] = k;
    }
    __syncthreads();
    if (threadIdx.x < (unsigned)TT && (int)threadIdx.x < p.T) {
        unsigned long long k = 0ull;
        for (int w = 0; w < LR_WARPS; ++w) k = best[w][threadIdx.x] > k ? best[w][threadIdx.x] : k;
        atomicMax(p.e.keys + threadIdx.x, k);
    }
}

template <int TT, int R, int D>
int launch_rows(dc_ctx* ctx, const RowsParams& p) {
    return dc_launch(ctx, "k_linear_rows", k_linear_rows<TT, R, D>, dim3((p.N + LR_WARPS * R - 1) / (LR_WARPS * R)), dim3(LR_WARPS * 32), 0, p);
}

// ---- sixteen rows per CTA on the tensor cores
constexpr int LM_WARPS = 16, LM_CTAS = 2;       // warps of a CTA, resident CTAs per SM

struct MmaParams {
    const __nv_bfloat16* w;
    int N, K, ldw;
    const __nv_bfloat16* x;
    int ldx, T;
    dc_lin_epi e;
};

__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// NT: groups of eight tokens; AHEAD: neighbouring runs of 32 columns that a warp keeps in flight.  Column 8 q + 4 s + e of a run (q: lane % 4) is k-slot 2 q + e % 2 + 8 (e / 2) of product s.
// KS: CTAs of a cluster that share sixteen rows, each with its part of the columns; the first adds the parts up.
// With KS 1 a CTA walks over its tiles of sixteen rows and fetches the next tile's first runs ahead of a tile's sum.
template <int NT, int AHEAD, int KS>
__global__ void __launch_bounds__(LM_WARPS * 32) k_linear_mma(const MmaParams p) {
    __shared__ float red[2][LM_WARPS][16][8 * NT + 1];
    __shared__ float other[KS > 1 ? KS - 1 : 1][KS > 1 ? 128 * NT : 1];
    if (KS > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");       // waited for ahead of the first remote store
    dc::pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
    const int part = blockIdx.x % KS, tiles = (p.N + 15) / 16, K8 = (p.K + 7) & ~7;
    const int all = (p.K + 31) / 32, per = (all + KS - 1) / KS, first = part * per, runs = min(all, first + per);
    uint4 a[AHEAD][2];
    // the matrix has a multiple of eight rows
    auto fetch = [&](int j, int tile, int run) {
        const bool ok = tile < tiles && run < runs && 32 * run + 8 * q < K8;
        const uint4* w0 = reinterpret_cast<const uint4*>(p.w + (size_t)(16 * tile + g) * p.ldw) + q;
        const uint4* w1 = reinterpret_cast<const uint4*>(p.w + (size_t)min(16 * tile + 8 + g, p.N - 1) * p.ldw) + q;
        a[j][0] = ok ? __ldg(w0 + 4 * run) : make_uint4(0, 0, 0, 0);
        a[j][1] = ok ? __ldg(w1 + 4 * run) : make_uint4(0, 0, 0, 0);
    };
    int tile = blockIdx.x / KS;
    const int step = gridDim.x / KS;
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) fetch(j, tile, first + warp * AHEAD + j);
    dc::pdl_wait();
    for (int buf = 0; tile < tiles; tile += step, buf ^= 1) {
        const int row0 = 16 * tile;
        float acc[NT][4];
#pragma unroll
        for (int n = 0; n < NT; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
        for (int rb = first + warp * AHEAD; rb < runs; rb += LM_WARPS * AHEAD) {
            const bool last = KS == 1 && rb + LM_WARPS * AHEAD >= runs;
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                const int run = rb + j, k = 32 * run + 8 * q;
                const uint4 a0 = a[j][0], a1 = a[j][1];
                if (last) fetch(j, tile + step, first + warp * AHEAD + j);
                else fetch(j, tile, run + LM_WARPS * AHEAD);
                if (run >= runs) continue;
#pragma unroll
                for (int n = 0; n < NT; ++n) {
                    uint4 b = make_uint4(0, 0, 0, 0);
                    if (8 * n + g < p.T && k < K8) b = *reinterpret_cast<const uint4*>(p.x + (size_t)(8 * n + g) * p.ldx + k);
                    mma_bf16(acc[n], a0.x, a1.x, a0.y, a1.y, b.x, b.y);
                    mma_bf16(acc[n], a0.z, a1.z, a0.w, a1.w, b.z, b.w);
                }
            }
        }
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) red[buf][warp][g + 8 * (i >> 1)][8 * n + 2 * q + (i & 1)] = acc[n][i];
        __syncthreads();
        const int r = threadIdx.x & 15, t = threadIdx.x >> 4, row = row0 + r;      // one thread per (row, token), rows fastest
        const bool mine = threadIdx.x < 128 * NT;
        float v = 0.0f;
        if (mine)
#pragma unroll
            for (int w = 0; w < LM_WARPS; ++w) v += red[buf][w][r][t];
        if (KS > 1) {                // one tile a cluster
            asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
            if (part > 0 && mine) {
                uint32_t to;
                asm("mapa.shared::cluster.u32 %0, %1, 0;" : "=r"(to) : "r"(dc::smem_u32(&other[part - 1][threadIdx.x])));
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(to), "f"(v) : "memory");
            }
            asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
            asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
            if (part > 0) return;
            if (mine)
#pragma unroll
                for (int k = 0; k < KS - 1; ++k) v += other[k][threadIdx.x];
        }
        if (!mine) continue;
        if (row0 >= p.e.pair0) {
            const float up = __shfl_down_sync(0xffffffffu, v, 1);
            const int o = (row - p.e.pair0) >> 1;
            if (!(r & 1) && t < p.T && o < p.e.n_pairs) dc::put_pair(p.e, t, o, dc::pair_value(p.e, v, up));
        } else {
            const bool ok = t < p.T && row < p.e.n_store;
            if (ok) dc::put_row(p.e, t, row, v);
            if (p.e.keys) {
                unsigned long long key = ok ? dc::argmax_key(v, row) : 0ull;
#pragma unroll
                for (int o = 8; o > 0; o >>= 1) {
                    const unsigned long long best = __shfl_xor_sync(0xffffffffu, key, o);
                    key = best > key ? best : key;
                }
                if (r == 0 && t < p.T) atomicMax(p.e.keys + t, key);
            }
        }
    }
}

// ---- f32 tile product: 64 weight rows x 64 tokens per CTA, 4 x 4 outputs per thread
__global__ void __launch_bounds__(256) k_linear_f32(const RowsParams p) {
    dc::pdl_launch_dependents();
    dc::pdl_wait();
    __shared__ float sw[16][68], sx[16][68];
    const int tid = threadIdx.x, n0 = blockIdx.x * 64, t0 = blockIdx.y * 64;
    const int tn = (tid & 15) * 4, tt = (tid >> 4) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += 16) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = tid + i * 256, r = e >> 4, k = e & 15;
            sw[k][r] = n0 + r < p.N && k0 + k < p.K ? __bfloat162float(p.w[(size_t)(n0 + r) * p.ldw + k0 + k]) : 0.0f;
            sx[k][r] = t0 + r < p.T && k0 + k < p.K ? p.x[(size_t)(t0 + r) * p.ldx + k0 + k] : 0.0f;
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
        if (t0 + tt + i >= p.T) continue;
        if (n0 + tn >= p.e.pair0) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int c = (n0 + tn + j - p.e.pair0) >> 1;
                if (c < p.e.n_pairs) dc::put_pair(p.e, t0 + tt + i, c, dc::pair_value(p.e, acc[i][j], acc[i][j + 1]));
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n0 + tn + j < p.e.n_store) dc::put_row(p.e, t0 + tt + i, n0 + tn + j, acc[i][j]);
        }
    }
}

template <int NT, int AHEAD, int KS>
int launch_mma(dc_ctx* ctx, const MmaParams& p) {
    const int tiles = (p.N + 15) / 16;
    const dim3 block(LM_WARPS * 32);
    if (KS > 1) return dc_launch_cluster(ctx, "k_linear_mma", k_linear_mma<NT, AHEAD, KS>, dim3(tiles * KS), block, 0, KS, p);
    const int room = LM_CTAS * ctx->num_sms, rounds = (tiles + room - 1) / room;
    return dc_launch(ctx, "k_linear_mma", k_linear_mma<NT, AHEAD, 1>, dim3((tiles + rounds - 1) / rounds), block, 0, p);
}

dc_lin_epi clipped(const dc_lin& w, dc_lin_epi e) {
    e.n_store = std::min(e.n_store, std::min(w.N, e.pair0));
    e.n_pairs = std::max(0, std::min(e.n_pairs, (w.N - e.pair0) / 2));
    return e;
}
bool epi_ok(const dc_lin_epi& e) { return e.pair0 >= (1 << 30) || e.pair0 % DC_PAIR_ALIGN == 0; }

}  // namespace

int dc_launch_linear_mma(dc_ctx* ctx, const dc_lin& w, const __nv_bfloat16* x, int ldx, int T, const dc_lin_epi& epi) {
    if (T < 1 || T > DC_MAX_T || ((uintptr_t)x & 15) || (ldx & 7) || (w.N & 7) || !epi_ok(epi)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_mma: bad operand");
    MmaParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, clipped(w, epi)};
    // fewer tiles than SMs: long rows are shared by a cluster, short ones need more in flight per warp
    const int tiles = (w.N + 15) / 16;
    if (2 * tiles <= ctx->num_sms && w.K >= 2048) return T <= 8 ? launch_mma<1, 2, 4>(ctx, p) : launch_mma<2, 2, 4>(ctx, p);
    if (tiles <= ctx->num_sms && w.K >= 4096) return T <= 8 ? launch_mma<1, 2, 2>(ctx, p) : launch_mma<2, 2, 2>(ctx, p);
    if (tiles <= ctx->num_sms) return T <= 8 ? launch_mma<1, 4, 1>(ctx, p) : launch_mma<2, 4, 1>(ctx, p);
    return T <= 8 ? launch_mma<1, 2, 1>(ctx, p) : launch_mma<2, 2, 1>(ctx, p);
}

int dc_launch_linear_rows(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, const dc_lin_epi& epi) {
    if (T < 1 || T > DC_MAX_T || ((uintptr_t)x & 15) || (ldx & 3) || !epi_ok(epi)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_rows: bad operand");
    RowsParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, clipped(w, epi)};
    if (T <= 1) return launch_rows<1, 2, 4>(ctx, p);
    if (T <= 4) return launch_rows<4, 2, 4>(ctx, p);
    return launch_rows<16, 4, 1>(ctx, p);
}

int dc_launch_linear_f32(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, const dc_lin_epi& epi) {
    if (!epi_ok(epi)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_f32: bad operand");
    RowsParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, clipped(w, epi)};
    return dc_launch(ctx, "k_linear_f32", k_linear_f32, dim3((w.N + 63) / 64, (T + 63) / 64), dim3(256), 0, p);
}
