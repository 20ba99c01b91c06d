// Products y = W x with bf16 weights and f32 accumulation for up to sixteen tokens, and for f32 activations.
//
// k_linear_mma (bf16 activations) streams the weight rows once: a CTA owns sixteen rows, its sixteen warps
// take neighbouring runs of 32 columns and feed them to m16n8k16 products.  A lane loads sixteen bytes of a row at a time;
// both operands use the same order of columns within a run, so the fragments need no shuffling.  k_linear_rows (f32
// activations, f32 models) does the same on the CUDA cores: a warp owns R rows, a lane takes runs of eight weights, the
// activations come through L1.  Weights do not depend on the kernel before, so every warp fetches its first ones
// ahead of the dependency wait.  k_linear_f32 (any number of tokens, f32 models) is a 64 x 64 shared-memory tile
// product.
//
// Epilogues: store; or tanh-gelu of the even rows times the odd rows (gate and up rows interleaved), half as many
// outputs.  The rows kernel can also fold the greedy pick of every token into packed keys.
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
    float* out;
    int ldo;
    int n_out;                     // rows stored (pair epilogue: pairs)
    unsigned long long* keys;
};

// TT: tokens (at most), R: rows of a warp, D: 16-byte loads per row that a lane keeps in flight.
template <int TT, int R, int D, int EPI>
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
    if (EPI == DC_LIN_GELU_PAIR) {
#pragma unroll
        for (int t = 0; t < TT; ++t)
#pragma unroll
            for (int r = 0; r < R; r += 2) {
                const int o = (row0 + r) >> 1;
                if (((t * R + r) / 2 & 31) == lane && live && t < p.T && o < p.n_out)
                    p.out[(size_t)t * p.ldo + o] = dc::gelu_tanh(acc[t][r]) * acc[t][r + 1];
            }
        return;
    }
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int r = 0; r < R; ++r)
            if (((t * R + r) & 31) == lane && live && t < p.T && row0 + r < p.n_out) p.out[(size_t)t * p.ldo + row0 + r] = acc[t][r];
    if (!p.keys) return;
    // greedy pick: the first maximum wins (key = order-preserving value bits, then the complement of the row)
    __shared__ unsigned long long best[LR_WARPS][TT];
#pragma unroll
    for (int t = 0; t < TT; ++t) {
        unsigned long long k = 0ull;
#pragma unroll
        for (int r = 0; r < R; ++r)
            if (live && row0 + r < p.n_out) {
                const unsigned long long c = dc::argmax_key(acc[t][r], row0 + r);
                k = c > k ? c : k;
            }
        if (lane == 0) best[warp][t] = k;
    }
    __syncthreads();
    if (threadIdx.x < (unsigned)TT && (int)threadIdx.x < p.T) {
        unsigned long long k = 0ull;
        for (int w = 0; w < LR_WARPS; ++w) k = best[w][threadIdx.x] > k ? best[w][threadIdx.x] : k;
        atomicMax(p.keys + threadIdx.x, k);
    }
}

template <int TT, int R, int D, int EPI>
int launch_rows(dc_ctx* ctx, const RowsParams& p) {
    return dc_launch(ctx, "k_linear_rows", k_linear_rows<TT, R, D, EPI>, dim3((p.N + LR_WARPS * R - 1) / (LR_WARPS * R)), dim3(LR_WARPS * 32), 0, p);
}
template <int EPI>
int launch_rows_any(dc_ctx* ctx, const RowsParams& p) {
    if (p.T <= 1) return launch_rows<1, 2, 4, EPI>(ctx, p);
    if (p.T <= 4) return launch_rows<4, 2, 4, EPI>(ctx, p);
    return launch_rows<16, 4, 1, EPI>(ctx, p);
}

// ---- sixteen rows per CTA on the tensor cores
constexpr int LM_WARPS = 16;

struct MmaParams {
    const __nv_bfloat16* w;
    int N, K, ldw;
    const __nv_bfloat16* x;
    int ldx, T;
    float* out;
    __nv_bfloat16* outb;
    int ldo, n_out;
    unsigned long long* keys;
};

__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// NT: groups of eight tokens; AHEAD: neighbouring runs of 32 columns that a warp keeps in flight.  Column 8 q + 4 s + e of a run (q: lane % 4) is k-slot 2 q + e % 2 + 8 (e / 2) of product s.
template <int NT, int AHEAD, int EPI>
__global__ void __launch_bounds__(LM_WARPS * 32) k_linear_mma(const MmaParams p) {
    __shared__ float red[LM_WARPS][16][8 * NT + 1];
    dc::pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
    const int row0 = blockIdx.x * 16, runs = (p.K + 31) / 32, K8 = (p.K + 7) & ~7;
    // the matrix has a multiple of eight rows
    const uint4* w0 = reinterpret_cast<const uint4*>(p.w + (size_t)(row0 + g) * p.ldw) + q;
    const uint4* w1 = reinterpret_cast<const uint4*>(p.w + (size_t)min(row0 + 8 + g, p.N - 1) * p.ldw) + q;
    uint4 a[AHEAD][2];
    auto fetch = [&](int j, int run) {
        const bool ok = 32 * run + 8 * q < K8;
        a[j][0] = ok ? __ldg(w0 + 4 * run) : make_uint4(0, 0, 0, 0);
        a[j][1] = ok ? __ldg(w1 + 4 * run) : make_uint4(0, 0, 0, 0);
    };
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) fetch(j, warp * AHEAD + j);
    dc::pdl_wait();
    float acc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
    for (int rb = warp * AHEAD; rb < runs; rb += LM_WARPS * AHEAD) {
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int run = rb + j, k = 32 * run + 8 * q;
            if (run >= runs) break;
            const uint4 a0 = a[j][0], a1 = a[j][1];
            fetch(j, run + LM_WARPS * AHEAD);
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
        for (int i = 0; i < 4; ++i) red[warp][g + 8 * (i >> 1)][8 * n + 2 * q + (i & 1)] = acc[n][i];
    __syncthreads();
    if (threadIdx.x < 128 * NT) {               // one thread per (row, token), rows fastest
        const int r = threadIdx.x & 15, t = threadIdx.x >> 4, row = row0 + r;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < LM_WARPS; ++w) v += red[w][r][t];
        if (EPI == DC_LIN_GELU_PAIR) {
            const float up = __shfl_down_sync(0xffffffffu, v, 1);
            const int o = row >> 1;
            if (!(r & 1) && t < p.T && o < p.n_out) {
                const float h = dc::gelu_tanh(v) * up;
                if (p.outb) p.outb[(size_t)t * p.ldo + o] = __float2bfloat16_rn(h);
                else p.out[(size_t)t * p.ldo + o] = h;
            }
        } else {
            const bool ok = t < p.T && row < p.n_out;
            if (ok) p.out[(size_t)t * p.ldo + row] = v;
            if (p.keys) {
                unsigned long long key = ok ? dc::argmax_key(v, row) : 0ull;
#pragma unroll
                for (int o = 8; o > 0; o >>= 1) {
                    const unsigned long long other = __shfl_xor_sync(0xffffffffu, key, o);
                    key = other > key ? other : key;
                }
                if (r == 0 && t < p.T) atomicMax(p.keys + t, key);
            }
        }
    }
}

// ---- f32 tile product: 64 weight rows x 64 tokens per CTA, 4 x 4 outputs per thread
__global__ void __launch_bounds__(256) k_linear_f32(const RowsParams p, int epi) {
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
        float* o = p.out + (size_t)(t0 + tt + i) * p.ldo;
        if (epi == DC_LIN_GELU_PAIR) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int c = (n0 + tn + j) >> 1;
                if (c < p.n_out) o[c] = dc::gelu_tanh(acc[i][j]) * acc[i][j + 1];
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (n0 + tn + j < p.n_out) o[n0 + tn + j] = acc[i][j];
        }
    }
}

template <int NT, int AHEAD>
int launch_mma_any(dc_ctx* ctx, const MmaParams& p, bool gelu) {
    const dim3 grid((p.N + 15) / 16), block(LM_WARPS * 32);
    return gelu ? dc_launch(ctx, "k_linear_mma", k_linear_mma<NT, AHEAD, DC_LIN_GELU_PAIR>, grid, block, 0, p)
                : dc_launch(ctx, "k_linear_mma", k_linear_mma<NT, AHEAD, DC_LIN_STORE>, grid, block, 0, p);
}

}  // namespace

int dc_launch_linear_mma(dc_ctx* ctx, const dc_lin& w, const __nv_bfloat16* x, int ldx, int T, int epi, float* out, __nv_bfloat16* outb, int ldo,
                         unsigned long long* keys) {
    if (T < 1 || T > DC_MAX_T || ((uintptr_t)x & 15) || (ldx & 7) || (w.N & 7)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_mma: bad operand");
    const bool gelu = epi == DC_LIN_GELU_PAIR;
    MmaParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, out, outb, ldo, gelu ? w.N / 2 : w.N, keys};
    if (p.n_out > ldo) p.n_out = ldo;
    // a small matrix needs more of it in flight per warp, a large one has enough warps
    const bool small = (w.N + 15) / 16 <= 2 * ctx->num_sms;
    if (T <= 8) return small ? launch_mma_any<1, 4>(ctx, p, gelu) : launch_mma_any<1, 2>(ctx, p, gelu);
    return small ? launch_mma_any<2, 4>(ctx, p, gelu) : launch_mma_any<2, 2>(ctx, p, gelu);
}

int dc_launch_linear_rows(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, int epi, float* out, int ldo, unsigned long long* keys) {
    if (T < 1 || T > DC_MAX_T || ((uintptr_t)x & 15) || (ldx & 3)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_rows: bad operand");
    RowsParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, out, ldo, epi == DC_LIN_GELU_PAIR ? ldo : w.N, keys};
    if (p.n_out > ldo) p.n_out = ldo;
    if (epi == DC_LIN_GELU_PAIR) return launch_rows_any<DC_LIN_GELU_PAIR>(ctx, p);
    return launch_rows_any<DC_LIN_STORE>(ctx, p);
}

int dc_launch_linear_f32(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, int epi, float* out, int ldo) {
    RowsParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, out, ldo, epi == DC_LIN_GELU_PAIR ? ldo : w.N, nullptr};
    if (p.n_out > ldo) p.n_out = ldo;
    return dc_launch(ctx, "k_linear_f32", k_linear_f32, dim3((w.N + 63) / 64, (T + 63) / 64), dim3(256), 0, p, epi);
}
