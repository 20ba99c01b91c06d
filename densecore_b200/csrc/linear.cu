// Products y = W x with bf16 weights and f32 activations, f32 accumulation.
//
// k_linear_rows (up to sixteen tokens) streams the weight rows once: a warp owns R rows, its lanes take
// consecutive runs of eight weights (one 16-byte load each), the activations come through L1, which all warps of a
// CTA share.  Weights do not depend on the kernel before, so every warp fetches its first ones ahead of the
// dependency wait.  k_linear_f32 (any number of tokens, f32 models) is a 64 x 64 shared-memory tile product.
//
// Epilogues: store; or tanh-gelu of the even rows times the odd rows (gate and up rows interleaved), half as many
// outputs.  The rows kernel can also fold the greedy pick of every token into packed keys.
#include "dc_common.cuh"
#include "dc_launch.cuh"
#include "dc_stack.h"
#include "dc_stack.cuh"

namespace {

constexpr int LR_WARPS = 8;

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

__device__ __forceinline__ void unpack8(const uint4& v, float (&f)[8]) {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        f[2 * i] = __uint_as_float(u[i] << 16);
        f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
}

template <int TT, int R, int EPI>
__global__ void __launch_bounds__(LR_WARPS * 32) k_linear_rows(const RowsParams p) {
    dc::pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row0 = (blockIdx.x * LR_WARPS + warp) * R;
    const bool live = row0 < p.N;
    const int K8 = (p.K + 7) & ~7;
    const uint4* wr[R];
#pragma unroll
    for (int r = 0; r < R; ++r) wr[r] = reinterpret_cast<const uint4*>(p.w + (size_t)min(row0 + r, p.N - 1) * p.ldw);
    uint4 nxt[R];
    const int k0 = lane * 8;
#pragma unroll
    for (int r = 0; r < R; ++r) nxt[r] = live && k0 < K8 ? __ldg(wr[r] + lane) : make_uint4(0, 0, 0, 0);
    dc::pdl_wait();
    float acc[TT][R];
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int r = 0; r < R; ++r) acc[t][r] = 0.0f;
    if (live) {
        for (int k = k0; k < K8; k += 256) {
            uint4 cur[R];
#pragma unroll
            for (int r = 0; r < R; ++r) {
                cur[r] = nxt[r];
                nxt[r] = k + 256 < K8 ? __ldg(wr[r] + (k + 256) / 8) : make_uint4(0, 0, 0, 0);
            }
            float wf[R][8];
#pragma unroll
            for (int r = 0; r < R; ++r) unpack8(cur[r], wf[r]);
#pragma unroll
            for (int t = 0; t < TT; ++t) {
                if (TT > 1 && t >= p.T) break;
                const float* xr = p.x + (size_t)t * p.ldx + k;
                float xv[8];
                if (k + 8 <= p.K) {
                    const float4 a = *reinterpret_cast<const float4*>(xr), b = *reinterpret_cast<const float4*>(xr + 4);
                    xv[0] = a.x, xv[1] = a.y, xv[2] = a.z, xv[3] = a.w, xv[4] = b.x, xv[5] = b.y, xv[6] = b.z, xv[7] = b.w;
                } else {
#pragma unroll
                    for (int i = 0; i < 8; ++i) xv[i] = k + i < p.K ? xr[i] : 0.0f;
                }
#pragma unroll
                for (int r = 0; r < R; ++r)
#pragma unroll
                    for (int i = 0; i < 8; ++i) acc[t][r] = fmaf(wf[r][i], xv[i], acc[t][r]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < TT; ++t)
#pragma unroll
        for (int r = 0; r < R; ++r)
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) acc[t][r] += __shfl_xor_sync(0xffffffffu, acc[t][r], o);
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

template <int R, int EPI>
int launch_rows(dc_ctx* ctx, const RowsParams& p) {
    const dim3 grid((p.N + LR_WARPS * R - 1) / (LR_WARPS * R)), block(LR_WARPS * 32);
    if (p.T <= 1) return dc_launch(ctx, "k_linear_rows", k_linear_rows<1, R, EPI>, grid, block, 0, p);
    if (p.T <= 2) return dc_launch(ctx, "k_linear_rows", k_linear_rows<2, R, EPI>, grid, block, 0, p);
    if (p.T <= 4) return dc_launch(ctx, "k_linear_rows", k_linear_rows<4, R, EPI>, grid, block, 0, p);
    if (p.T <= 8) return dc_launch(ctx, "k_linear_rows", k_linear_rows<8, R, EPI>, grid, block, 0, p);
    return dc_launch(ctx, "k_linear_rows", k_linear_rows<16, R, EPI>, grid, block, 0, p);
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

}  // namespace

int dc_launch_linear_rows(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, int epi, float* out, int ldo, unsigned long long* keys) {
    if (T < 1 || T > DC_MAX_T || ((uintptr_t)x & 15) || (ldx & 3)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_rows: bad operand");
    RowsParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, out, ldo, epi == DC_LIN_GELU_PAIR ? ldo : w.N, keys};
    if (p.n_out > ldo) p.n_out = ldo;
    // two rows per warp until four rows still fill the machine
    const bool wide = w.N >= ctx->num_sms * LR_WARPS * 4 * 2;
    if (epi == DC_LIN_GELU_PAIR) return wide ? launch_rows<4, DC_LIN_GELU_PAIR>(ctx, p) : launch_rows<2, DC_LIN_GELU_PAIR>(ctx, p);
    return wide ? launch_rows<4, DC_LIN_STORE>(ctx, p) : launch_rows<2, DC_LIN_STORE>(ctx, p);
}

int dc_launch_linear_f32(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, int epi, float* out, int ldo) {
    RowsParams p = {w.w, w.N, w.K, w.ld, x, ldx, T, out, ldo, epi == DC_LIN_GELU_PAIR ? ldo : w.N, nullptr};
    if (p.n_out > ldo) p.n_out = ldo;
    return dc_launch(ctx, "k_linear_f32", k_linear_f32, dim3((w.N + 63) / 64, (T + 63) / 64), dim3(256), 0, p, epi);
}
