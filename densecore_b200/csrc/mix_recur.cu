// Recurrent mixers: short causal convolution, gated delta rule with one decay per key channel, generalized delta rule whose
// removed part is read from the old state, Mamba-2 state-space scan, linear attention with a constant decay per head, and
// their gated output norms.
//
// Per-sequence state (f32) lives in the cache manager's state slots: the matrix S as [head][value column][key
// channel], and the convolution's last inputs as a ring [position % taps][channel].  A sequence at position 0 starts
// from zero whatever its slot holds, so slots need no clearing when they change hands.
//
// Value columns of S never mix: a column c obeys S_c <- g S_c; u = beta (v_c - S_c . k); S_c <- S_c + u k;
// o_c = S_c . q.  A single token (decode) is done as written, by one kernel per mixer from projections to normed
// output.  Longer entries go through blocks of sixteen tokens (see "blocks of sixteen tokens" below): what a head's
// columns share is computed once per block, and k_state_scan walks the blocks with two or four columns in the registers of
// each warp.  All of it is f32 on the CUDA cores.
#include "dc_common.cuh"
#include "dc_launch.cuh"
#include "dc_stack.h"
#include "dc_stack.cuh"

#define DC_TRY(expr)                       \
    do {                                   \
        int st_ = (expr);                  \
        if (st_ != DC_B200_OK) return st_; \
    } while (0)

using namespace dc;

namespace {

constexpr int BT = 16, BROW = 20;                       // tokens of a block; pitch of a 16 x 16 factor (conflict-free rows)

// The entries' last inputs into their rings (after every kernel that read the old ones).
__global__ void __launch_bounds__(256) k_ring_update(ConvRef cr, const float* __restrict__ proj, int ldp, int off) {
    pdl_launch_dependents();
    pdl_wait();
    const int e = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    if (c >= cr.C) return;
    const int t0 = cr.starts[e], t1 = cr.starts[e + 1];
    for (int t = max(t0, t1 - cr.taps); t < t1; ++t)
        cr.ring(cr.seq_ids[t])[(size_t)(cr.positions[t] % cr.taps) * cr.C + c] = proj[(size_t)t * ldp + off + c];
}

// ---------------------------------------------------------------- delta rule: per-token inputs
struct DeltaPrep {
    ConvRef cr;
    const float* proj;
    int ldp;
    const float* conv;
    int heads, kv_heads, dim, vdim, off_q, off_k, off_v, off_b, off_a, n_low;
    float unit_eps, q_scale;
    float* act;
    int lda;
    float* small;            // [T][heads]: step sizes
    __nv_bfloat16* lowb;     // bf16 copy of the low-rank inputs (columns off_a ..)
    int ldl, T, v_items;
};

// One warp per (token, item): items are the kv heads (q and k: convolution, silu, unit length), runs of 128 value
// channels, and one for the step sizes and the low-rank columns.
__global__ void __launch_bounds__(256) k_delta_prep(DeltaPrep p) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, items = p.kv_heads + p.v_items + 1;
    const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= (long long)p.T * items) return;
    const int t = (int)(id / items), item = (int)(id % items);
    const int e = entry_of(p.cr.starts, p.cr.E, t), i = t - p.cr.starts[e], pos = p.cr.positions[t], taps = p.cr.taps;
    const float* ring = p.cr.ring(p.cr.seq_ids[t]);
    float* act = p.act + (size_t)t * p.lda;
    if (item < p.kv_heads) {
        float q[8], k[8], sq = 0.0f, sk = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int d = lane + 32 * j;
            q[j] = k[j] = 0.0f;
            if (d < p.dim) {
                const int cq = p.off_q + item * p.dim + d, ck = p.off_k + item * p.dim + d;
                q[j] = silu(conv_at(p.proj, p.ldp, ring, p.cr.C, cq, taps, p.conv + cq, p.cr.ldw, cq, t, i, pos));
                k[j] = silu(conv_at(p.proj, p.ldp, ring, p.cr.C, ck, taps, p.conv + ck, p.cr.ldw, ck, t, i, pos));
            }
            sq = fmaf(q[j], q[j], sq);
            sk = fmaf(k[j], k[j], sk);
        }
        const float iq = p.q_scale / sqrtf(warp_sum(sq) + p.unit_eps), ik = 1.0f / sqrtf(warp_sum(sk) + p.unit_eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int d = lane + 32 * j;
            q[j] *= iq;
            k[j] *= ik;
            if (d < p.dim) {
                act[p.off_q + item * p.dim + d] = q[j];
                act[p.off_k + item * p.dim + d] = k[j];
            }
        }
    } else if (item < p.kv_heads + p.v_items) {
        const int c0 = (item - p.kv_heads) * 128, V = p.heads * p.vdim;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = c0 + lane + 32 * j;
            if (c < V) {
                const int cv = p.off_v + c;
                act[cv] = silu(conv_at(p.proj, p.ldp, ring, p.cr.C, cv, taps, p.conv + cv, p.cr.ldw, cv, t, i, pos));
            }
        }
    } else {
        for (int h = lane; h < p.heads; h += 32)
            p.small[(size_t)t * p.heads + h] = sigmoid(p.proj[(size_t)t * p.ldp + p.off_b + h]);
        if (p.lowb)
            for (int c = lane; c < p.n_low; c += 32)
                p.lowb[(size_t)t * p.ldl + c] = __float2bfloat16_rn(p.proj[(size_t)t * p.ldp + p.off_a + c]);
    }
}

// Four taps: a warp takes an item through a block of up to sixteen tokens with the convolution's window in registers.
// NJ: groups of 32 key channels.
template <int NJ>
__global__ void __launch_bounds__(256) k_delta_prep4(DeltaPrep p) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, items = p.kv_heads + p.v_items, item = blockIdx.y * 8 + (threadIdx.x >> 5);
    const BlockRef br = block_at<BT>(p.cr.starts, p.cr.E, blockIdx.x);
    if (br.n <= 0) return;
    if (blockIdx.y == gridDim.y - 1) {          // the step sizes and the low-rank columns
        for (int i = threadIdx.x; i < br.n * p.heads; i += 256) {
            const int t = br.t0 + i / p.heads, h = i % p.heads;
            p.small[(size_t)t * p.heads + h] = sigmoid(p.proj[(size_t)t * p.ldp + p.off_b + h]);
        }
        if (p.lowb)
            for (int i = threadIdx.x; i < br.n * p.n_low; i += 256) {
                const int t = br.t0 + i / p.n_low, c = i % p.n_low;
                p.lowb[(size_t)t * p.ldl + c] = __float2bfloat16_rn(p.proj[(size_t)t * p.ldp + p.off_a + c]);
            }
        return;
    }
    if (item >= items) return;
    const int i0 = br.t0 - p.cr.starts[br.e], pos0 = p.cr.positions[br.t0], ldw = p.cr.ldw;
    const float* ring = p.cr.ring(p.cr.seq_ids[br.t0]);
    auto before = [&](int col, int back) {        // the input `back` tokens before the block
        if (pos0 < back) return 0.0f;
        return back <= i0 ? p.proj[(size_t)(br.t0 - back) * p.ldp + col] : ring[(size_t)((pos0 - back) % 4) * p.cr.C + col];
    };
    if (item < p.kv_heads) {
        float wq[NJ][4], wk[NJ][4], hq[NJ][3], hk[NJ][3];
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
            const int d = min(lane + 32 * j, p.dim - 1), cq = p.off_q + item * p.dim + d, ck = p.off_k + item * p.dim + d;
#pragma unroll
            for (int k = 0; k < 4; ++k) wq[j][k] = p.conv[(size_t)k * ldw + cq], wk[j][k] = p.conv[(size_t)k * ldw + ck];
#pragma unroll
            for (int k = 0; k < 3; ++k) hq[j][k] = before(cq, 3 - k), hk[j][k] = before(ck, 3 - k);
        }
        constexpr int AHEAD = NJ <= 4 ? 4 : 2;        // tokens whose inputs are in flight
        for (int ub = 0; ub < br.n; ub += AHEAD) {
            float xq[AHEAD][NJ], xk[AHEAD][NJ];
#pragma unroll
            for (int v = 0; v < AHEAD; ++v) {
                const float* row = p.proj + (size_t)(br.t0 + min(ub + v, br.n - 1)) * p.ldp + item * p.dim;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const int dc = min(lane + 32 * j, p.dim - 1);
                    xq[v][j] = row[p.off_q + dc], xk[v][j] = row[p.off_k + dc];
                }
            }
            float sq[AHEAD], sk[AHEAD];
#pragma unroll
            for (int v = 0; v < AHEAD; ++v) {
                sq[v] = sk[v] = 0.0f;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const float q = xq[v][j], k = xk[v][j];
                    xq[v][j] = silu(fmaf(wq[j][3], q, fmaf(wq[j][2], hq[j][2], fmaf(wq[j][1], hq[j][1], wq[j][0] * hq[j][0]))));
                    xk[v][j] = silu(fmaf(wk[j][3], k, fmaf(wk[j][2], hk[j][2], fmaf(wk[j][1], hk[j][1], wk[j][0] * hk[j][0]))));
                    hq[j][0] = hq[j][1], hq[j][1] = hq[j][2], hq[j][2] = q;
                    hk[j][0] = hk[j][1], hk[j][1] = hk[j][2], hk[j][2] = k;
                    if (lane + 32 * j >= p.dim) xq[v][j] = xk[v][j] = 0.0f;
                    sq[v] = fmaf(xq[v][j], xq[v][j], sq[v]);
                    sk[v] = fmaf(xk[v][j], xk[v][j], sk[v]);
                }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int v = 0; v < AHEAD; ++v) {
                    sq[v] += __shfl_xor_sync(0xffffffffu, sq[v], o);
                    sk[v] += __shfl_xor_sync(0xffffffffu, sk[v], o);
                }
#pragma unroll
            for (int v = 0; v < AHEAD; ++v) {
                const float iq = p.q_scale / sqrtf(sq[v] + p.unit_eps), ik = 1.0f / sqrtf(sk[v] + p.unit_eps);
                float* act = p.act + (size_t)(br.t0 + ub + v) * p.lda + item * p.dim;
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const int d = lane + 32 * j;
                    if (ub + v < br.n && d < p.dim) {
                        act[p.off_q + d] = xq[v][j] * iq;
                        act[p.off_k + d] = xk[v][j] * ik;
                    }
                }
            }
        }
    } else {
        const int V = p.heads * p.vdim, c0 = (item - p.kv_heads) * 128 + lane;
        float w[4][4], h[4][3];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int cv = p.off_v + min(c0 + 32 * j, V - 1);
#pragma unroll
            for (int k = 0; k < 4; ++k) w[j][k] = p.conv[(size_t)k * ldw + cv];
#pragma unroll
            for (int k = 0; k < 3; ++k) h[j][k] = before(cv, 3 - k);
        }
        for (int ub = 0; ub < br.n; ub += 8) {
            float x[8][4];
#pragma unroll
            for (int v = 0; v < 8; ++v)
#pragma unroll
                for (int j = 0; j < 4; ++j) x[v][j] = p.proj[(size_t)(br.t0 + min(ub + v, br.n - 1)) * p.ldp + p.off_v + min(c0 + 32 * j, V - 1)];
#pragma unroll
            for (int v = 0; v < 8; ++v)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float y = silu(fmaf(w[j][3], x[v][j], fmaf(w[j][2], h[j][2], fmaf(w[j][1], h[j][1], w[j][0] * h[j][0]))));
                    h[j][0] = h[j][1], h[j][1] = h[j][2], h[j][2] = x[v][j];
                    if (ub + v < br.n && c0 + 32 * j < V) p.act[(size_t)(br.t0 + ub + v) * p.lda + p.off_v + c0 + 32 * j] = y;
                }
        }
    }
}

// ---------------------------------------------------------------- blocks of sixteen tokens
// Within a block that starts from the state S0, with cumulative decays G_t (products of g over the block's tokens up
// to t) and products P_ti of g over (i, t]:
//   u_t = beta_t (v_t - S0 . (G_t k_t) - sum_{i<t} A_ti u_i),   A_ti = sum_d P_ti k_i k_t
//   o_t = S0 . (G_t q_t) + sum_{i<=t} B_ti u_i,                 B_ti = sum_d P_ti k_i q_t
//   S   = G_15 S0 + sum_i (P_15,i k_i) u_i
// Everything but S0, v, u and o is shared by a head's value columns and computed once per (block, head): the decayed
// vectors, B, and W = (I + diag(beta) A)^-1 diag(beta), so that u = W (v - S0 . G k).  Every decay factor is a
// product of g, at most 1.  The state-space scan is the same with one decay per head, no A, and u_i = dt_i x_i; linear
// attention with a constant decay is that with steps of 1.

// Sum of v[i] over the warp lands in lane i (31 shuffles for 32 sums).
__device__ __forceinline__ float transpose_sum32(float (&v)[32], int lane) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
        for (int i = 0; i < 16; ++i)
            if (i < o) {
                const bool up = lane & o;
                const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
    }
    return v[0];
}

// Floats of one (block, head) of the delta rule: G k, G q, P k (each [16][dp]), G_15 [dp], W and B [16][20].
__host__ __device__ constexpr int delta_block_floats(int dp) { return 3 * BT * dp + dp + 2 * BT * BROW; }

struct DeltaBlock {
    const float* act;
    int lda, off_q, off_k, heads, per, dim, dp;
    const float* raw;            // decay projection
    int ldr;
    const float *neg_a, *dt_bias, *small;
    int lds;
    const int32_t* starts;
    int E;
    float* out;
};

__global__ void __launch_bounds__(128) k_delta_blocks(const DeltaBlock p) {
    extern __shared__ __align__(16) float sm[];         // k, q, g: [16][dim] each
    __shared__ float sA[BT][BT + 1], sB[BT][BT], sX[BT][BT + 1], sbeta[BT];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dim = p.dim, dp = p.dp;
    const BlockRef br = block_at<BT>(p.starts, p.E, blockIdx.x);
    if (br.n <= 0) return;
    float *sk = sm, *sq = sm + BT * dim, *sg = sm + 2 * BT * dim;
    float* out = p.out + ((size_t)blockIdx.x * p.heads + h) * delta_block_floats(dp);
    if (tid < BT) sbeta[tid] = tid < br.n ? p.small[(size_t)(br.t0 + tid) * p.lds + h] : 0.0f;
    for (int d = tid; d < dp; d += 128) {
        float k[BT], q[BT], g[BT], cum = 1.0f;
        const bool in = d < dim;
        const int dc = min(d, dim - 1);
        const float na = p.neg_a[h], bias = p.dt_bias[(size_t)h * dim + dc];
#pragma unroll
        for (int t = 0; t < BT; ++t) {                  // every load before the arithmetic
            const int tc = br.t0 + min(t, br.n - 1);
            const float* a = p.act + (size_t)tc * p.lda + (h / p.per) * dim + dc;
            k[t] = a[p.off_k];
            q[t] = a[p.off_q];
            g[t] = p.raw[(size_t)tc * p.ldr + h * dim + dc];
        }
#pragma unroll
        for (int t = 0; t < BT; ++t) {
            const bool ok = in && t < br.n;
            k[t] = ok ? k[t] : 0.0f;
            q[t] = ok ? q[t] : 0.0f;
            g[t] = ok ? expf(na * softplus(g[t] + bias)) : 1.0f;
            cum *= g[t];
            out[t * dp + d] = cum * k[t];
            out[(BT + t) * dp + d] = cum * q[t];
            if (in) sk[t * dim + d] = k[t], sq[t * dim + d] = q[t], sg[t * dim + d] = g[t];
        }
        out[3 * BT * dp + d] = cum;
        float suffix = 1.0f;
#pragma unroll
        for (int t = BT - 1; t >= 0; --t) {
            out[(2 * BT + t) * dp + d] = suffix * k[t];
            suffix *= g[t];
        }
    }
    __syncthreads();
    // A and B of the key tokens i = warp, warp + 4, ...: c runs over P_ti k_i (zero before i, k_i at i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        float v[2][32];
#pragma unroll
        for (int j = 0; j < 32; ++j) v[0][j] = v[1][j] = 0.0f;
        for (int d = lane; d < dim; d += 32) {
            float c[2] = {0.0f, 0.0f};
#pragma unroll
            for (int t = 0; t < BT; ++t) {
                const float k = sk[t * dim + d], q = sq[t * dim + d], g = sg[t * dim + d];
#pragma unroll
                for (int m = 0; m < 2; ++m) {
                    c[m] = t == warp + 4 * (2 * half + m) ? k : c[m] * g;
                    v[m][t] = fmaf(c[m], k, v[m][t]);
                    v[m][BT + t] = fmaf(c[m], q, v[m][BT + t]);
                }
            }
        }
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            const int i = warp + 4 * (2 * half + m);
            const float r = transpose_sum32(v[m], lane);
            if (lane < BT) sA[lane][i] = r;             // read below the diagonal only
            else sB[lane - BT][i] = r;
        }
    }
    __syncthreads();
    if (tid < BT) {                                     // column tid of (I + diag(beta) A)^-1 diag(beta)
        float x[BT];
#pragma unroll
        for (int t = 0; t < BT; ++t) {
            float a[2] = {};
#pragma unroll
            for (int i = 0; i < t; ++i) a[i & 1] = fmaf(sA[t][i], x[i], a[i & 1]);
            x[t] = t < tid ? 0.0f : t == tid ? 1.0f : -sbeta[t] * (a[0] + a[1]);
            sX[t][tid] = x[t];
        }
    }
    __syncthreads();
    float* W = out + 3 * BT * dp + dp;
    for (int i = tid; i < BT * BT; i += 128) {
        W[i / BT * BROW + i % BT] = sX[i / BT][i % BT] * sbeta[i % BT];
        W[(BT + i / BT) * BROW + i % BT] = sB[i / BT][i % BT];
    }
}

// The generalized delta rule, S <- diag(w) S - (a u)(u^T S) + k v^T, with W_t and P_ti products of w as above, c_t = -a_t u_t:
//   z_t = u_t . S_(t-1) = d_t + sum_{i<t} (A_ti z_i + K_ti v_i),   d_t = S0 . (W_(t-1) u_t),
//   A_ti = sum_d P_(t-1,i) c_i u_t,   K_ti = sum_d P_(t-1,i) k_i u_t,   so that z = X d + M v with X = (I - A)^-1, M = X K
//   o_t = S0 . (W_t r_t) + sum_{i<=t} (C_ti z_i + B_ti v_i),   C_ti = sum_d P_ti c_i r_t,   B_ti = sum_d P_ti k_i r_t
//   S   = W_15 S0 + sum_i (P_15,i c_i z_i + P_15,i k_i v_i)
// z is eliminated: with N = C X and N' = B + C M, o = S0 . W r + N d + N' v; with D = P c X and E = P c M + P k (over the block's
// tokens), S = W_15 S0 + D d + E v.  A block leaves W_(t-1) u, W r, D, E, W_15, N and N'.
// Floats of one (block, head): W u, W r, D, E (each [16][dp]), W_15 [dp], N and N' [16][20].
__host__ __device__ constexpr int general_block_floats(int dp) { return 4 * BT * dp + dp + 2 * BT * BROW; }

// exp(-e^(-1/2) sigmoid(z))
__device__ __forceinline__ float decay_below_one(float z) { return expf(-0.6065306597126334f * sigmoid(z)); }

struct GeneralBlock {
    const float* proj;
    int ldp, off_r, off_k, off_a, heads, dim;
    const float* low;            // decay projection [T][ldd]
    int ldd;
    const float *w0, *a_bias;
    float unit_eps;
    const int32_t* starts;
    int E;
    float* out;
};

// The decays are never below 0.545, so a block's cumulative ones W_t stay above 6e-5 and their quotients keep their bits:
// P_ti = W_t / W_i.  One 32 x 32 product of the rows W_(t-1) u_t, W_t r_t with the rows c_i / W_i, k_i / W_i holds A, K, C and B.
// EPL: key channels of a lane.
template <int EPL>
__global__ void __launch_bounds__(128) k_general_blocks(const GeneralBlock p) {
    constexpr int DP = 32 * EPL, LD = DP + 4, TW = BT / 4;      // tokens of a warp
    extern __shared__ __align__(16) float sm[];                 // u, r | c, k: [16][LD] each, then the decays
    __shared__ float sA[BT][BT + 1], sK[BT][BT + 1], sC[BT][BT + 1], sB[BT][BT + 1];
    __shared__ __align__(16) float sF[2][BT][BROW];             // X, M
    pdl_launch_dependents();
    float *su = sm, *sr = su + BT * LD, *sc = sr + BT * LD, *sk = sc + BT * LD, *sw = sk + BT * LD;
    const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dim = p.dim;
    float w0[EPL], ab[EPL];
#pragma unroll
    for (int j = 0; j < EPL; ++j) {
        const int d = min(lane + 32 * j, dim - 1);
        w0[j] = p.w0[h * dim + d], ab[j] = p.a_bias[h * dim + d];
    }
    pdl_wait();
    const BlockRef br = block_at<BT>(p.starts, p.E, blockIdx.x);
    if (br.n <= 0) return;
    float* out = p.out + ((size_t)blockIdx.x * p.heads + h) * general_block_floats(DP);
    constexpr int AT = EPL <= 4 ? TW : 2;                       // tokens whose inputs are in flight
#pragma unroll
    for (int i0 = 0; i0 < TW; i0 += AT) {
        float k[AT][EPL], r[AT][EPL], a[AT][EPL], w[AT][EPL];
#pragma unroll
        for (int i = 0; i < AT; ++i) {
            const int tc = br.t0 + min(TW * warp + i0 + i, br.n - 1);
            const float *row = p.proj + (size_t)tc * p.ldp + h * dim, *low = p.low + (size_t)tc * p.ldd + h * dim;
#pragma unroll
            for (int j = 0; j < EPL; ++j) {
                const int d = min(lane + 32 * j, dim - 1);
                k[i][j] = row[p.off_k + d], r[i][j] = row[p.off_r + d], a[i][j] = row[p.off_a + d], w[i][j] = low[d];
            }
        }
#pragma unroll
        for (int i = 0; i < AT; ++i) {
            const int t = TW * warp + i0 + i;
            float ss = 0.0f;
#pragma unroll
            for (int j = 0; j < EPL; ++j) {
                if (t >= br.n || lane + 32 * j >= dim) k[i][j] = r[i][j] = 0.0f;
                ss = fmaf(k[i][j], k[i][j], ss);
            }
            const float unit = 1.0f / sqrtf(warp_sum(ss) + p.unit_eps);
#pragma unroll
            for (int j = 0; j < EPL; ++j) {
                const int at = t * LD + lane + 32 * j;
                const float u = k[i][j] * unit;
                su[at] = u, sr[at] = r[i][j], sk[at] = k[i][j];
                sc[at] = -sigmoid(a[i][j] + ab[j]) * u;
                sw[at] = t < br.n ? decay_below_one(w[i][j] + w0[j]) : 1.0f;
            }
        }
    }
    __syncthreads();
    for (int i = tid; i < 2 * DP; i += 128) {           // a channel's u and c, or its r and k
        const bool second = i >= DP;
        const int d = second ? i - DP : i;
        float *x = (second ? sr : su) + d, *y = (second ? sk : sc) + d, *to = out + (second ? BT * DP : 0) + d;
        float w[BT], cum = 1.0f;
#pragma unroll
        for (int t = 0; t < BT; ++t) w[t] = sw[t * LD + d];
#pragma unroll
        for (int t = 0; t < BT; ++t) {
            const float before = cum;
            cum *= w[t];
            const float v = x[t * LD] * (second ? cum : before);
            x[t * LD] = v;
            to[t * DP] = v;
            y[t * LD] = __fdividef(y[t * LD], cum);
        }
        if (second) out[4 * BT * DP + d] = cum;
    }
    __syncthreads();
    {
        // rows 2 ty, 2 ty + 1 of (u | r) with rows tx, tx + 8, .. of (c | k)
        const int tx = tid & 7, ty = tid >> 3;
        uint64_t acc[2][4] = {};
        const float *xa = sm + 2 * ty * LD, *ya = sc + tx * LD;
#pragma unroll 4
        for (int d = 0; d < DP; d += 4) {
            ulonglong2 x[2], y[4];
#pragma unroll
            for (int i = 0; i < 2; ++i) x[i] = *reinterpret_cast<const ulonglong2*>(xa + i * LD + d);
#pragma unroll
            for (int j = 0; j < 4; ++j) y[j] = *reinterpret_cast<const ulonglong2*>(ya + 8 * j * LD + d);
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fma2(x[i].y, y[j].y, fma2(x[i].x, y[j].x, acc[i][j]));
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float2 f = unpair(acc[i][j]);
                const int t = (2 * ty + i) % BT, s = (tx + 8 * j) % BT;
                const bool answer = 2 * ty >= BT;
                float(*to)[BT + 1] = answer ? (j < 2 ? sC : sB) : (j < 2 ? sA : sK);
                to[t][s] = s < t || (answer && s == t) ? f.x + f.y : 0.0f;
            }
    }
    __syncthreads();
    if (tid < BT) {                                     // column tid of (I - A)^-1
        float x[BT];
#pragma unroll
        for (int t = 0; t < BT; ++t) {
            float a[2] = {};
#pragma unroll
            for (int i = 0; i < t; ++i) a[i & 1] = fmaf(sA[t][i], x[i], a[i & 1]);
            x[t] = t < tid ? 0.0f : t == tid ? 1.0f : a[0] + a[1];
            sF[0][t][tid] = x[t];
        }
    }
    __syncthreads();
    float* N = out + 4 * BT * DP + DP;
    {
        const int t = tid >> 3, i = 2 * (tid & 7);      // two neighbouring elements
        float m[2] = {}, n[2] = {};
#pragma unroll
        for (int q = 0; q < BT; ++q) {
            const float x = sF[0][t][q], c = sC[t][q];
            const float2 f = *reinterpret_cast<const float2*>(&sF[0][q][i]);
            m[0] = fmaf(x, sK[q][i], m[0]), m[1] = fmaf(x, sK[q][i + 1], m[1]);
            n[0] = fmaf(c, f.x, n[0]), n[1] = fmaf(c, f.y, n[1]);
        }
        *reinterpret_cast<float2*>(&sF[1][t][i]) = make_float2(m[0], m[1]);
        *reinterpret_cast<float2*>(N + t * BROW + i) = make_float2(n[0], n[1]);
        __syncthreads();
        n[0] = sB[t][i], n[1] = sB[t][i + 1];
#pragma unroll
        for (int q = 0; q < BT; ++q) {
            const float c = sC[t][q];
            const float2 f = *reinterpret_cast<const float2*>(&sF[1][q][i]);
            n[0] = fmaf(c, f.x, n[0]), n[1] = fmaf(c, f.y, n[1]);
        }
        *reinterpret_cast<float2*>(N + (BT + t) * BROW + i) = make_float2(n[0], n[1]);
    }
    for (int i = tid; i < 2 * DP; i += 128) {           // a channel of D or of E
        const bool second = i >= DP;
        const int d = second ? i - DP : i;
        float last = 1.0f, a[BT];
#pragma unroll
        for (int t = 0; t < BT; ++t) {
            last *= sw[t * LD + d];
            a[t] = second ? sk[t * LD + d] : 0.0f;
        }
        const float (*F)[BROW] = sF[second];
#pragma unroll
        for (int t = 0; t < BT; ++t) {
            const float c = sc[t * LD + d];
#pragma unroll
            for (int j = 0; j <= t; j += 4) {           // zero above the diagonal
                const float4 f = *reinterpret_cast<const float4*>(&F[t][j]);
                a[j] = fmaf(c, f.x, a[j]), a[j + 1] = fmaf(c, f.y, a[j + 1]), a[j + 2] = fmaf(c, f.z, a[j + 2]), a[j + 3] = fmaf(c, f.w, a[j + 3]);
            }
        }
#pragma unroll
        for (int j = 0; j < BT; ++j) out[((second ? 3 : 2) * BT + j) * DP + d] = last * a[j];
    }
}

template <int EPL>
int launch_general_blocks(dc_ctx* ctx, const GeneralBlock& p, dim3 grid) {
    constexpr int bytes = 5 * BT * (32 * EPL + 4) * 4;
    DC_TRY(dc_kernel_setup(ctx, (const void*)k_general_blocks<EPL>, bytes, "k_general_blocks"));
    return dc_launch(ctx, "k_general_blocks", k_general_blocks<EPL>, grid, dim3(128), (size_t)bytes, p);
}

// Floats of one (block, head) of the state-space scan: M [16][20], cumulative decays [16], update factors [16].
constexpr int SSD_BLOCK = BT * BROW + 2 * BT;

struct SsdBlock {
    const float* act;
    int lda, off_b, off_c, heads, per, state;
    const float* small;          // [T][2 heads]: dt, decay; or null with
    const float* decay;          // [heads]: a constant decay and steps of 1
    const int32_t* starts;
    int E;
    float* out;
};

// One CTA per (block, group): M_ti = (C_t . B_i) P_ti dt_i for i <= t, for every head of the group.
__global__ void __launch_bounds__(256) k_ssd_blocks(const SsdBlock p) {
    extern __shared__ __align__(16) float sm[];         // B, C: [16][state + 1]
    __shared__ float sa[BT], sd[BT];
    pdl_launch_dependents();
    pdl_wait();
    const BlockRef br = block_at<BT>(p.starts, p.E, blockIdx.x);
    if (br.n <= 0) return;
    const int g = blockIdx.y, tid = threadIdx.x, ld = p.state + 1, t = tid / BT, i = tid % BT;
    float *sb = sm, *sc = sm + BT * ld;
    for (int j = tid; j < BT * p.state; j += 256) {
        const int tk = j / p.state, d = j - tk * p.state;
        const float* a = p.act + (size_t)(br.t0 + tk) * p.lda + g * p.state + d;
        sb[tk * ld + d] = tk < br.n ? a[p.off_b] : 0.0f;
        sc[tk * ld + d] = tk < br.n ? a[p.off_c] : 0.0f;
    }
    __syncthreads();
    float cb = 0.0f;
    if (i <= t)
        for (int d = 0; d < p.state; ++d) cb = fmaf(sc[t * ld + d], sb[i * ld + d], cb);
    for (int hh = 0; hh < p.per; ++hh) {
        const int h = g * p.per + hh;
        __syncthreads();
        if (tid < BT) {
            const float* s = p.small ? p.small + (size_t)(br.t0 + tid) * 2 * p.heads : nullptr;
            sd[tid] = tid < br.n ? (s ? s[h] : 1.0f) : 0.0f;
            sa[tid] = tid < br.n ? (s ? s[p.heads + h] : p.decay[h]) : 1.0f;
        }
        __syncthreads();
        float* out = p.out + ((size_t)blockIdx.x * p.heads + h) * SSD_BLOCK;
        float m = 0.0f;
        if (i <= t) {
            m = cb * sd[i];
            for (int j = i + 1; j <= t; ++j) m *= sa[j];
        }
        out[t * BROW + i] = m;
        if (tid < BT) {
            float c = 1.0f, u = sd[tid];
            for (int j = 0; j <= tid; ++j) c *= sa[j];
            for (int j = tid + 1; j < BT; ++j) u *= sa[j];
            out[BT * BROW + tid] = c;
            out[BT * BROW + BT + tid] = u;
        }
    }
}

// ---------------------------------------------------------------- the scan over blocks
constexpr int SC_COLS = 16;                             // value columns per CTA
enum { SCAN_SSD = 0, SCAN_DELTA = 1, SCAN_GENERAL = 2 };

struct ScanParams {
    const float* blocks;           // k_delta_blocks / k_general_blocks / k_ssd_blocks
    const float *k, *q;            // ssd: B and C of group 0
    const float* v;                // values of head 0
    int ld, heads, per, dim, vdim;
    const float* D;                // ssd: per head, or null
    float* o;
    int ldo;
    uint8_t* base;
    size_t slot_bytes, state_off;
    const int32_t *seq_ids, *positions, *starts;
    int vec;                       // ssd: B, C rows allow 16-byte copies
};

// EPL consecutive-chunk channels per lane: lane's channel i is W * lane + 32 W (i / W) + i % W.
template <int EPL>
struct Chan {
    static constexpr int W = EPL < 4 ? EPL : 4;
    static __device__ __forceinline__ int at(int lane, int i) { return W * lane + 32 * W * (i / W) + i % W; }
    static __device__ __forceinline__ void load(const float* row, int lane, float (&f)[EPL]) {
#pragma unroll
        for (int j = 0; j < EPL / W; ++j) {
            const float* r = row + W * lane + 32 * W * j;
            if (W == 4) {
                const float4 v = *reinterpret_cast<const float4*>(r);
                f[4 * j] = v.x, f[(4 * j + 1) % EPL] = v.y, f[(4 * j + 2) % EPL] = v.z, f[(4 * j + 3) % EPL] = v.w;
            } else if (W == 2) {
                const float2 v = *reinterpret_cast<const float2*>(r);
                f[2 * j] = v.x, f[(2 * j + 1) % EPL] = v.y;
            } else {
                f[j] = *r;
            }
        }
    }
};

// Dot products of the warp's NC columns (s: this lane's channels of each) with NS sets of sixteen rows of shared memory, eight
// rows in flight ahead of the arithmetic.  L = 32 / NC lanes work for a column: lane L c + j gets column c's products with rows
// j, j + L, ...
template <int EPL, int NS, int NC>
__device__ __forceinline__ void column_dots(const float* rows, int dp, const float (&s)[NC][EPL], int lane, float (&out)[NS][NC / 2]) {
    constexpr int G = EPL <= 4 ? 8 : 4, L = 32 / NC, PER = NC / 2;
    float r[NS][BT * NC], w[2][G][EPL];
#pragma unroll
    for (int t = 0; t < G; ++t) Chan<EPL>::load(rows + t * dp, lane, w[0][t]);
#pragma unroll
    for (int g = 0; g < NS * BT / G; ++g) {
        if (g + 1 < NS * BT / G) {
#pragma unroll
            for (int t = 0; t < G; ++t) Chan<EPL>::load(rows + (G * (g + 1) + t) * dp, lane, w[(g + 1) & 1][t]);
        }
#pragma unroll
        for (int u = 0; u < G; ++u) {
            const int row = G * g + u, t = row % BT;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                float& dst = r[row / BT][BT * c + PER * (t % L) + t / L];
                if (EPL == 1) {
                    dst = s[c][0] * w[g & 1][u][0];
                } else {
                    uint64_t a = 0;
#pragma unroll
                    for (int i = 0; i + 1 < EPL; i += 2) a = fma2(pair(s[c][i], s[c][i + 1]), pair(w[g & 1][u][i], w[g & 1][u][i + 1]), a);
                    const float2 f = unpair(a);
                    dst = f.x + f.y;
                }
            }
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {                           // each step halves the sums a lane carries
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < BT * NC / 2; ++i)
            if (i < PER * o) {
#pragma unroll
                for (int k = 0; k < NS; ++k) {
                    const float send = up ? r[k][i] : r[k][i + PER * o], keep = up ? r[k][i + PER * o] : r[k][i];
                    r[k][i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
            }
    }
#pragma unroll
    for (int k = 0; k < NS; ++k)
#pragma unroll
        for (int i = 0; i < PER; ++i) out[k][i] = r[k][i];
}

// EPL: key channels per lane (the key size, padded to 32 EPL).
constexpr int scan_block_floats(int kind, int dp) { return kind == SCAN_DELTA ? delta_block_floats(dp) : kind == SCAN_GENERAL ? general_block_floats(dp) : 2 * BT * dp + SSD_BLOCK; }

// Blocks in flight or at work: a block takes less time than its way from L2.
constexpr int scan_stages(int kind, int dp) {
    const int bytes = (scan_block_floats(kind, dp) + BT * SC_COLS) * 4;
    return 4 * bytes <= 160 * 1024 ? 4 : 3 * bytes <= 220 * 1024 ? 3 : 2;
}

// NC: columns of a warp.
template <int EPL, int KIND, int NC>
__global__ void __launch_bounds__(SC_COLS / NC * 32) k_state_scan(const ScanParams p) {
    constexpr bool GENERAL = KIND == SCAN_GENERAL, DELTA = KIND != SCAN_SSD;         // the delta rules' factors come whole from memory
    constexpr int DP = 32 * EPL, BLK = scan_block_floats(KIND, DP), BUF = BLK + BT * SC_COLS;
    constexpr int SC_THREADS = SC_COLS / NC * 32, LANES = 32 / NC, PER = NC / 2, STAGES = scan_stages(KIND, DP);
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(16) float s_d[SC_COLS / NC][NC][BT], s_u[SC_COLS / NC][NC][BT];
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lt = lane % LANES, lc = lane / LANES;
    const int c0 = blockIdx.x * SC_COLS, h = blockIdx.y, e = blockIdx.z, kh = h / p.per;
    const int col = c0 + warp * NC + lc;
    if (!DELTA) {
        for (int i = tid; i < STAGES * BUF; i += SC_THREADS) sm[i] = 0.0f;    // padded channels stay zero
        __syncthreads();
    }
    pdl_wait();
    const int t0 = p.starts[e], t1 = p.starts[e + 1];
    if (t0 >= t1) return;
    const int seq = p.seq_ids[t0], blocks = (t1 - t0 + BT - 1) / BT;
    const float* bsrc = p.blocks + ((size_t)block_base<BT>(p.starts, e) * p.heads + h) * (DELTA ? BLK : SSD_BLOCK);
    const size_t bstep = (size_t)p.heads * (DELTA ? BLK : SSD_BLOCK);
    float* S = reinterpret_cast<float*>(p.base + (size_t)seq * p.slot_bytes + p.state_off) + ((size_t)h * p.vdim + c0 + warp * NC) * p.dim;
    float s[NC][EPL];            // channels Chan::at of the warp's columns
    const bool fresh = p.positions[t0] == 0, live = col < p.vdim;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int i = 0; i < EPL; ++i) {
            const int d = Chan<EPL>::at(lane, i);
            s[c][i] = !fresh && c0 + warp * NC + c < p.vdim && d < p.dim ? S[(size_t)c * p.dim + d] : 0.0f;
        }

    auto load = [&](int b, int buf) {
        float* dst = sm + buf * BUF;
        const int tb = t0 + b * BT;
        const float* src = bsrc + b * bstep;
        if (DELTA) {
            for (int i = tid; i < BLK / 4; i += SC_THREADS) cp_async16z(smem_u32(dst + 4 * i), src + 4 * i, true);
        } else {
            for (int i = tid; i < SSD_BLOCK / 4; i += SC_THREADS) cp_async16z(smem_u32(dst + 2 * BT * DP + 4 * i), src + 4 * i, true);
            const int t = tid / (SC_THREADS / BT), part = tid % (SC_THREADS / BT);
            const bool ok = tb + t < t1;
#pragma unroll
            for (int a = 0; a < 2; ++a) {
                const float* row = (a ? p.k : p.q) + (size_t)kh * p.dim + (size_t)(ok ? tb + t : tb) * p.ld;
                const uint32_t to = smem_u32(dst + (a * BT + t) * DP);
                if (p.vec) {
                    for (int d = 4 * part; d < p.dim; d += SC_THREADS / BT * 4) cp_async16z(to + 4 * d, row + d, ok);
                } else {
                    for (int d = part; d < p.dim; d += SC_THREADS / BT) cp_async4z(to + 4 * d, row + d, ok);
                }
            }
        }
        for (int i = tid; i < BT * SC_COLS; i += SC_THREADS) {
            const int t = i / SC_COLS, c = c0 + i % SC_COLS;
            const bool ok = tb + t < t1 && c < p.vdim;
            cp_async4z(smem_u32(dst + BLK + i), ok ? p.v + (size_t)(tb + t) * p.ld + (size_t)h * p.vdim + c : p.v, ok);
        }
        cp_async_commit();
    };
    const float Dh = DELTA || !p.D ? 0.0f : p.D[h];
    for (int b = 0; b < STAGES - 1; ++b)
        if (b < blocks) load(b, b);
        else cp_async_commit();
    for (int b = 0; b < blocks; ++b) {
        cp_async_wait<STAGES - 2>();
        __syncthreads();         // the block has landed; every warp is done with the stage that the next load fills
        if (b + STAGES - 1 < blocks) load(b + STAGES - 1, (b + STAGES - 1) % STAGES);
        else cp_async_commit();
        const float* x = sm + b % STAGES * BUF;
        // ---- the columns against the block's (decayed) keys and queries; see column_dots for who works for whom
        float r[DELTA ? 2 : 1][PER];
        column_dots<EPL, DELTA ? 2 : 1, NC>(x, DP, s, lane, r);
        const float* rq = r[DELTA ? 1 : 0];
        float v[PER];
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            v[k] = x[BLK + (lt + LANES * k) * SC_COLS + warp * NC + lc];
            s_d[warp][lc][lt + LANES * k] = GENERAL ? r[0][k] : DELTA ? v[k] - r[0][k] : v[k];
            if (GENERAL) s_u[warp][lc][lt + LANES * k] = v[k];
        }
        __syncwarp();
        auto row_dot = [&](const float* row, const float* vals) {      // rows of W, B, M are zero above the diagonal
            float a[4] = {};
#pragma unroll
            for (int i = 0; i < BT / 4; ++i) {
                const float4 f = *reinterpret_cast<const float4*>(row + 4 * i), d = *reinterpret_cast<const float4*>(vals + 4 * i);
                a[0] = fmaf(f.x, d.x, a[0]);
                a[1] = fmaf(f.y, d.y, a[1]);
                a[2] = fmaf(f.z, d.z, a[2]);
                a[3] = fmaf(f.w, d.w, a[3]);
            }
            return (a[0] + a[1]) + (a[2] + a[3]);
        };
        const float* scal = x + (GENERAL ? 4 * BT * DP + DP : DELTA ? 3 * BT * DP + DP : 2 * BT * DP);
        float out[PER];
        if (GENERAL) {
#pragma unroll
            for (int k = 0; k < PER; ++k)
                out[k] = rq[k] + row_dot(scal + (lt + LANES * k) * BROW, s_d[warp][lc]) + row_dot(scal + (BT + lt + LANES * k) * BROW, s_u[warp][lc]);
        } else if (DELTA) {
#pragma unroll
            for (int k = 0; k < PER; ++k) s_u[warp][lc][lt + LANES * k] = row_dot(scal + (lt + LANES * k) * BROW, s_d[warp][lc]);
            __syncwarp();
#pragma unroll
            for (int k = 0; k < PER; ++k) out[k] = rq[k] + row_dot(scal + (BT + lt + LANES * k) * BROW, s_u[warp][lc]);
        } else {
            const float* cd = scal + BT * BROW;
#pragma unroll
            for (int k = 0; k < PER; ++k) {
                const int t = lt + LANES * k;
                s_u[warp][lc][t] = v[k] * cd[BT + t];
                out[k] = fmaf(cd[t], rq[k], row_dot(scal + t * BROW, s_d[warp][lc])) + Dh * v[k];
            }
            __syncwarp();
        }
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int t = t0 + b * BT + lt + LANES * k;
            if (t < t1 && live) p.o[(size_t)t * p.ldo + (size_t)h * p.vdim + col] = out[k];
        }
        // ---- the state after the block
        const float* keys = x + (DELTA ? 2 * BT * DP : BT * DP);
        {
            float g[EPL];
            if (DELTA) Chan<EPL>::load(x + (GENERAL ? 4 : 3) * BT * DP, lane, g);
#pragma unroll
            for (int c = 0; c < NC; ++c)
#pragma unroll
                for (int i = 0; i < EPL; ++i) s[c][i] *= DELTA ? g[i] : scal[BT * BROW + BT - 1];
        }
        constexpr int G = EPL <= 4 ? 8 : 4;
#pragma unroll
        for (int row = 0; row < (GENERAL ? 2 : 1) * BT; row += G) {
            const int t = row % BT;
            float (*vals)[BT] = GENERAL && row < BT ? s_d[warp] : s_u[warp];
            float w[G][EPL], u[NC][G];
#pragma unroll
            for (int g = 0; g < G; ++g) Chan<EPL>::load(keys + (row + g) * DP, lane, w[g]);
#pragma unroll
            for (int c = 0; c < NC; ++c)
#pragma unroll
                for (int g = 0; g < G; g += 4) {
                    const float4 f = *reinterpret_cast<const float4*>(&vals[c][t + g]);
                    u[c][g] = f.x, u[c][g + 1] = f.y, u[c][g + 2] = f.z, u[c][g + 3] = f.w;
                }
#pragma unroll
            for (int g = 0; g < G; ++g)
#pragma unroll
                for (int c = 0; c < NC; ++c)
#pragma unroll
                    for (int i = 0; i < EPL; ++i) s[c][i] = fmaf(w[g][i], u[c][g], s[c][i]);
        }
        __syncwarp();
    }
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int i = 0; i < EPL; ++i) {
            const int d = Chan<EPL>::at(lane, i);
            if (c0 + warp * NC + c < p.vdim && d < p.dim) S[(size_t)c * p.dim + d] = s[c][i];
        }
}

template <int EPL, int KIND, int NC>
int launch_scan_epl(dc_ctx* ctx, const ScanParams& p, int E) {
    // a few CTAs that run long: started while the many of the kernel before still leave, they would crowd on the first free SMs
    const size_t smem = (size_t)scan_stages(KIND, 32 * EPL) * (scan_block_floats(KIND, 32 * EPL) + BT * SC_COLS) * 4;
    DC_TRY(dc_kernel_setup(ctx, (const void*)k_state_scan<EPL, KIND, NC>, (int)smem, "k_state_scan"));
    return dc_launch_drained(ctx, "k_state_scan", k_state_scan<EPL, KIND, NC>, dim3((p.vdim + SC_COLS - 1) / SC_COLS, p.heads, E), dim3(SC_COLS / NC * 32), smem, p);
}
int key_pad(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
// Few columns in the whole step: the delta rules' warps, which work on more rows, take fewer of them each.
template <int EPL, int KIND>
int launch_scan_columns(dc_ctx* ctx, const ScanParams& p, int E) {
    const int ctas = (p.vdim + SC_COLS - 1) / SC_COLS * p.heads * E;
    return KIND != SCAN_SSD && ctas <= 2 * ctx->num_sms ? launch_scan_epl<EPL, KIND, 2>(ctx, p, E) : launch_scan_epl<EPL, KIND, 4>(ctx, p, E);
}
template <int KIND>
int launch_scan(dc_ctx* ctx, const ScanParams& p, int E) {
    switch (key_pad(p.dim)) {
    case 32: return launch_scan_columns<1, KIND>(ctx, p, E);
    case 64: return launch_scan_columns<2, KIND>(ctx, p, E);
    case 128: return launch_scan_columns<4, KIND>(ctx, p, E);
    default: return launch_scan_columns<8, KIND>(ctx, p, E);
    }
}

// ---------------------------------------------------------------- decode: one token per sequence
struct DeltaDecode {
    ConvRef cr;
    const float* proj;
    int ldp;
    const float* conv;
    int heads, per, dim, vdim, off_q, off_k, off_v, off_b, off_a, off_g, a_rank, g_rank;
    float unit_eps, q_scale, eps;
    const __nv_bfloat16 *a2, *g2;
    int lda2, ldg2;
    const float *neg_a, *dt_bias, *norm;
    size_t state_off;
    float* mix;
    __nv_bfloat16* mixb;         // instead of mix
    int ldm;
};

// Decode convolutions of the channels tid, tid + NT, ...: B of them at a time, every load before the arithmetic.  place(c)
// gives the channel's projection column, ring column and weight column (below zero: none, the result is 0); put(c, y)
// takes the silu of the convolution.  own(c): this CTA also puts the channel's input into the ring (a row that no tap
// of this token reads).
struct ConvPlace {
    int col, rc, wc;
};
template <int NT, int B, typename Place, typename Put, typename Own>
__device__ __forceinline__ void conv_decode(const float* row, float* ring, int C, int taps, const float* w, int ldw, const float* bias, int pos, int total,
                                            Place place, Put put, Own own) {
    for (int c0 = threadIdx.x; c0 < total; c0 += NT * B) {
        ConvPlace at[B];
        float s[B] = {}, last[B], add[B];
#pragma unroll
        for (int b = 0; b < B; ++b) {
            at[b] = place(min(c0 + NT * b, total - 1));
            last[b] = row[max(at[b].col, 0)];
            add[b] = bias ? bias[max(at[b].wc, 0)] : 0.0f;
        }
        for (int j0 = 0; j0 < taps - 1; j0 += 3) {
            float in[B][3], wj[B][3];
#pragma unroll
            for (int k = 0; k < 3; ++k) {
                const int j = min(j0 + k, taps - 2), back = taps - 1 - j;
                const bool ok = j0 + k < taps - 1 && pos >= back;
                const size_t r = (size_t)(max(pos - back, 0) % taps) * C;
#pragma unroll
                for (int b = 0; b < B; ++b) {
                    in[b][k] = ring[r + max(at[b].rc, 0)];
                    wj[b][k] = ok ? w[(size_t)j * ldw + max(at[b].wc, 0)] : 0.0f;
                }
                if (!ok) {
#pragma unroll
                    for (int b = 0; b < B; ++b) in[b][k] = 0.0f;
                }
            }
#pragma unroll
            for (int k = 0; k < 3; ++k)
#pragma unroll
                for (int b = 0; b < B; ++b) s[b] = fmaf(wj[b][k], in[b][k], s[b]);
        }
#pragma unroll
        for (int b = 0; b < B; ++b) {
            const int c = c0 + NT * b;
            if (c >= total) continue;
            if (at[b].col < 0) {
                put(c, 0.0f);
                continue;
            }
            put(c, silu(fmaf(w[(size_t)(taps - 1) * ldw + at[b].wc], last[b], s[b]) + add[b]));
            if (own(c)) ring[(size_t)(pos % taps) * C + at[b].rc] = last[b];
        }
    }
}

// out[r] = rows r < n of a bf16 matrix (padded with zeros) times x in shared memory (zero up to a multiple of 128); sixteen
// lanes a row, eight rows of a half-warp in flight
__device__ __forceinline__ void low_rank_rows(const __nv_bfloat16* w, int ldw, int n, const float* x, int rank, float* out) {
    constexpr int AHEAD = 8;
    const int lane = threadIdx.x & 31, sub = lane & 15, half = 2 * (threadIdx.x >> 5) + (lane >> 4), halves = blockDim.x >> 4;
    for (int rb = 0; rb < n; rb += AHEAD * halves) {
        float a[AHEAD] = {};
        for (int k = 8 * sub; k < rank; k += 128) {
            float xr[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) xr[i] = x[k + i];
            uint4 v[AHEAD];
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                const int r = rb + j * halves + half;
                v[j] = r < n && k < ldw ? *reinterpret_cast<const uint4*>(w + (size_t)r * ldw + k) : make_uint4(0, 0, 0, 0);
            }
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                const uint32_t u[4] = {v[j].x, v[j].y, v[j].z, v[j].w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    a[j] = fmaf(__uint_as_float(u[i] << 16), xr[2 * i], a[j]);
                    a[j] = fmaf(__uint_as_float(u[i] & 0xffff0000u), xr[2 * i + 1], a[j]);
                }
            }
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) a[j] += __shfl_xor_sync(0xffffffffu, a[j], o);
            const int r = rb + j * halves + half;
            if (sub == 0 && r < n) out[r] = a[j];
        }
    }
}

// NC columns of a head's state, lane's channels Chan<EPL>::at
template <int NC, int EPL>
__device__ __forceinline__ void load_columns(const float* S, int c0, int vdim, int dim, int lane, bool fresh, float (&s)[NC][EPL]) {
    const bool vec = (dim & 3) == 0 && EPL >= 4;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        const float* col = S + (size_t)min(c0 + c, vdim - 1) * dim;
        const bool ok = !fresh && c0 + c < vdim;
        if (vec) {
#pragma unroll
            for (int j = 0; j < EPL / 4; ++j) {
                const int d = Chan<EPL>::at(lane, 4 * j);
                const float4 v = ok && d < dim ? *reinterpret_cast<const float4*>(col + d) : make_float4(0.f, 0.f, 0.f, 0.f);
                s[c][(4 * j) % EPL] = v.x, s[c][(4 * j + 1) % EPL] = v.y, s[c][(4 * j + 2) % EPL] = v.z, s[c][(4 * j + 3) % EPL] = v.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < EPL; ++i) {
                const int d = Chan<EPL>::at(lane, i);
                s[c][i] = ok && d < dim ? col[d] : 0.0f;
            }
        }
    }
}
template <int NC, int EPL>
__device__ __forceinline__ void store_columns(float* S, int c0, int vdim, int dim, int lane, const float (&s)[NC][EPL]) {
    const bool vec = (dim & 3) == 0 && EPL >= 4;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        if (c0 + c >= vdim) continue;
        float* col = S + (size_t)(c0 + c) * dim;
        if (vec) {
#pragma unroll
            for (int j = 0; j < EPL / 4; ++j) {
                const int d = Chan<EPL>::at(lane, 4 * j);
                if (d < dim)
                    *reinterpret_cast<float4*>(col + d) =
                        make_float4(s[c][(4 * j) % EPL], s[c][(4 * j + 1) % EPL], s[c][(4 * j + 2) % EPL], s[c][(4 * j + 3) % EPL]);
            }
        } else {
#pragma unroll
            for (int i = 0; i < EPL; ++i) {
                const int d = Chan<EPL>::at(lane, i);
                if (d < dim) col[d] = s[c][i];
            }
        }
    }
}
// Sums of v[0 .. 7] over the warp; lane l gets the sum of v[l / 4].
__device__ __forceinline__ float transpose_sum8(float (&v)[8], int lane) {
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (i < o) {
                const bool up = lane & (4 * o);
                const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
                v[i] = keep + __shfl_xor_sync(0xffffffffu, send, 4 * o);
            }
    }
    v[0] += __shfl_xor_sync(0xffffffffu, v[0], 2);
    return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
}

// One CTA per (head, sequence): convolutions, unit vectors, decays and gates, the state's step, the gated norm.
template <int EPL>
__global__ void __launch_bounds__(256) k_delta_decode(const DeltaDecode p) {
    constexpr int DP = 32 * EPL, NC = 8;            // columns of a warp at a time
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[33], s_iq, s_ik;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, t = blockIdx.y, kh = h / p.per;
    const int ra = (p.a_rank + 127) & ~127, rg = (p.g_rank + 127) & ~127;
    float *sq = sm, *sk = sq + DP, *sg = sk + DP, *sa = sg + DP, *sgl = sa + ra, *sv = sgl + rg, *so = sv + p.vdim, *sgate = so + p.vdim;
    pdl_launch_dependents();
    // the gates' weights do not depend on the kernel before: on their way to L2 while this one still waits
    const char *pa = (const char*)(p.a2 + (size_t)h * p.dim * p.lda2), *pg = (const char*)(p.g2 + (size_t)h * p.vdim * p.ldg2);
    for (int i = tid * 128; i < p.dim * p.lda2 * 2; i += 256 * 128) prefetch_l2(pa + i);
    for (int i = tid * 128; i < p.vdim * p.ldg2 * 2; i += 256 * 128) prefetch_l2(pg + i);
    pdl_wait();
    const int pos = p.cr.positions[t], seq = p.cr.seq_ids[t], taps = p.cr.taps;
    float* S = reinterpret_cast<float*>(p.cr.base + (size_t)seq * p.cr.slot_bytes + p.state_off) + (size_t)h * p.vdim * p.dim;
    for (int i = tid * 32; i < p.vdim * p.dim; i += 256 * 32) prefetch_l2(S + i);
    float* ring = p.cr.ring(seq);
    const float* row = p.proj + (size_t)t * p.ldp;
    const bool first = h % p.per == 0;
    conv_decode<256, 2>(
        row, ring, p.cr.C, taps, p.conv, p.cr.ldw, nullptr, pos, 2 * DP + p.vdim,
        [&](int c) {
            const int d = c < DP ? c : c < 2 * DP ? c - DP : c - 2 * DP;
            if (c < 2 * DP && d >= p.dim) return ConvPlace{-1, -1, -1};
            const int col = c < DP ? p.off_q + kh * p.dim + d : c < 2 * DP ? p.off_k + kh * p.dim + d : p.off_v + h * p.vdim + d;
            return ConvPlace{col, col, col};
        },
        [&](int c, float v) { sm[c < 2 * DP ? c : (int)(sv - sm) + c - 2 * DP] = v; }, [&](int c) { return c >= 2 * DP || first; });
    for (int c = tid; c < ra; c += 256) sa[c] = c < p.a_rank ? row[p.off_a + c] : 0.0f;
    for (int c = tid; c < rg; c += 256) sgl[c] = c < p.g_rank ? row[p.off_g + c] : 0.0f;
    __syncthreads();
    if (warp < 2) {
        float ss = 0.0f;
        for (int d = lane; d < DP; d += 32) ss = fmaf(sm[warp * DP + d], sm[warp * DP + d], ss);
        ss = warp_sum(ss);
        if (lane == 0) (warp ? s_ik : s_iq) = (warp ? 1.0f : p.q_scale) / sqrtf(ss + p.unit_eps);
    }
    low_rank_rows(p.a2 + (size_t)h * p.dim * p.lda2, p.lda2, p.dim, sa, p.a_rank, sg);
    low_rank_rows(p.g2 + (size_t)h * p.vdim * p.ldg2, p.ldg2, p.vdim, sgl, p.g_rank, sgate);
    __syncthreads();
    for (int d = tid; d < DP; d += 256) {
        sg[d] = d < p.dim ? expf(p.neg_a[h] * softplus(sg[d] + p.dt_bias[(size_t)h * p.dim + d])) : 0.0f;
        sq[d] *= s_iq;
        sk[d] *= s_ik;
    }
    __syncthreads();
    float kr[EPL], qr[EPL], gr[EPL], kq = 0.0f;
    Chan<EPL>::load(sk, lane, kr);
    Chan<EPL>::load(sq, lane, qr);
    Chan<EPL>::load(sg, lane, gr);
#pragma unroll
    for (int i = 0; i < EPL; ++i) kq = fmaf(kr[i], qr[i], kq);
    kq = warp_sum(kq);
    const float beta = sigmoid(row[p.off_b + h]);
    for (int c0 = NC * warp; c0 < p.vdim; c0 += 8 * NC) {
        float s[NC][EPL], a[NC], b[NC];
        load_columns<NC, EPL>(S, c0, p.vdim, p.dim, lane, pos == 0, s);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            a[c] = b[c] = 0.0f;
#pragma unroll
            for (int i = 0; i < EPL; ++i) {
                s[c][i] *= gr[i];
                a[c] = fmaf(s[c][i], kr[i], a[c]);
                b[c] = fmaf(s[c][i], qr[i], b[c]);
            }
        }
        // lane l works for column l / 4
        const float ka = transpose_sum8(a, lane), qb = transpose_sum8(b, lane);
        const int mine = c0 + (lane >> 2);
        const float u = mine < p.vdim ? beta * (sv[mine] - ka) : 0.0f;
        if ((lane & 3) == 0 && mine < p.vdim) so[mine] = fmaf(kq, u, qb);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const float uc = __shfl_sync(0xffffffffu, u, 4 * c);
#pragma unroll
            for (int i = 0; i < EPL; ++i) s[c][i] = fmaf(kr[i], uc, s[c][i]);
        }
        store_columns<NC, EPL>(S, c0, p.vdim, p.dim, lane, s);
    }
    __syncthreads();
    float ss = 0.0f;
    for (int c = tid; c < p.vdim; c += 256) ss = fmaf(so[c], so[c], ss);
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.vdim + p.eps);
    for (int c = tid; c < p.vdim; c += 256) {
        const float v = so[c] * inv * p.norm[c] * sigmoid(sgate[c]);
        const size_t o = (size_t)t * p.ldm + (size_t)h * p.vdim + c;
        if (p.mixb) p.mixb[o] = __float2bfloat16_rn(v);
        else p.mix[o] = v;
    }
}

struct GeneralDecode {
    const float* proj;
    int ldp, heads, dim, rank, off_r, off_k, off_v, off_g, off_a, off_w;
    float unit_eps, eps;
    const __nv_bfloat16* w2;
    int ldw2;
    const float *w0, *a_bias, *norm;
    uint8_t* base;
    size_t slot_bytes, state_off;
    const int32_t *seq_ids, *positions;
    float* mix;
    __nv_bfloat16* mixb;         // instead of mix
    int ldm;
};

// Generalized delta rule, one CTA per (head, sequence): decays and removal rates, the state's step, the gated norm.
template <int EPL>
__global__ void __launch_bounds__(256) k_general_decode(const GeneralDecode p) {
    constexpr int DP = 32 * EPL, NC = 8;            // columns of a warp at a time
    extern __shared__ __align__(16) float sm[];     // r, k, removal rate, decay, v, gate: [DP]; answers [DP]; low-rank inputs
    __shared__ float red[33];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, t = blockIdx.y, dim = p.dim, rank = (p.rank + 127) & ~127;
    float *sr = sm, *sk = sr + DP, *sa = sk + DP, *sw = sa + DP, *sv = sw + DP, *sg = sv + DP, *so = sg + DP, *sl = so + DP;
    pdl_launch_dependents();
    // the weights do not depend on the kernel before: on their way to L2 while this one still waits
    const char* pw = (const char*)(p.w2 + (size_t)h * dim * p.ldw2);
    for (int i = tid * 128; i < dim * p.ldw2 * 2; i += 256 * 128) prefetch_l2(pw + i);
    pdl_wait();
    const int pos = p.positions[t];
    float* S = reinterpret_cast<float*>(p.base + (size_t)p.seq_ids[t] * p.slot_bytes + p.state_off) + (size_t)h * dim * dim;
    for (int i = tid * 32; i < dim * dim; i += 256 * 32) prefetch_l2(S + i);
    const float* row = p.proj + (size_t)t * p.ldp;
    for (int c = tid; c < rank; c += 256) sl[c] = c < p.rank ? tanhf(row[p.off_w + c]) : 0.0f;
    for (int i = tid; i < 5 * DP; i += 256) {
        const int part = i / DP, d = i - part * DP, off = part == 0 ? p.off_r : part == 1 ? p.off_k : part == 2 ? p.off_a : part == 3 ? p.off_v : p.off_g;
        float v = d < dim ? row[off + h * dim + d] : 0.0f;
        if (part == 2) v = d < dim ? sigmoid(v + p.a_bias[h * dim + d]) : 0.0f;
        (part < 3 ? sm + part * DP : sv + (part - 3) * DP)[d] = v;
    }
    __syncthreads();
    low_rank_rows(p.w2 + (size_t)h * dim * p.ldw2, p.ldw2, dim, sl, p.rank, sw);
    float rr[EPL], kr[EPL], ur[EPL], cr[EPL], wr[EPL], ss = 0.0f, kq = 0.0f, cq = 0.0f;
    Chan<EPL>::load(sr, lane, rr);
    Chan<EPL>::load(sk, lane, kr);
    Chan<EPL>::load(sa, lane, cr);
#pragma unroll
    for (int i = 0; i < EPL; ++i) ss = fmaf(kr[i], kr[i], ss);
    const float unit = 1.0f / sqrtf(warp_sum(ss) + p.unit_eps);
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
        ur[i] = kr[i] * unit;
        cr[i] *= -ur[i];
        kq = fmaf(kr[i], rr[i], kq);
        cq = fmaf(cr[i], rr[i], cq);
    }
    kq = warp_sum(kq);
    cq = warp_sum(cq);
    __syncthreads();
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
        const int d = Chan<EPL>::at(lane, i);
        wr[i] = d < dim ? decay_below_one(sw[d] + p.w0[h * dim + d]) : 0.0f;
        rr[i] *= wr[i];
    }
    for (int c0 = NC * warp; c0 < dim; c0 += 8 * NC) {
        float s[NC][EPL], a[NC], b[NC];
        load_columns<NC, EPL>(S, c0, dim, dim, lane, pos == 0, s);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            a[c] = b[c] = 0.0f;
#pragma unroll
            for (int i = 0; i < EPL; ++i) {
                a[c] = fmaf(s[c][i], ur[i], a[c]);
                b[c] = fmaf(s[c][i], rr[i], b[c]);
            }
        }
        // lane l works for column l / 4
        const float z = transpose_sum8(a, lane), q = transpose_sum8(b, lane);
        const int mine = c0 + (lane >> 2);
        const float v = mine < dim ? sv[mine] : 0.0f;
        if ((lane & 3) == 0 && mine < dim) so[mine] = fmaf(kq, v, fmaf(cq, z, q));
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const float zc = __shfl_sync(0xffffffffu, z, 4 * c), vc = __shfl_sync(0xffffffffu, v, 4 * c);
#pragma unroll
            for (int i = 0; i < EPL; ++i) s[c][i] = fmaf(kr[i], vc, fmaf(cr[i], zc, s[c][i] * wr[i]));
        }
        store_columns<NC, EPL>(S, c0, dim, dim, lane, s);
    }
    __syncthreads();
    float sq = 0.0f;
    for (int c = tid; c < dim; c += 256) sq = fmaf(so[c], so[c], sq);
    const float inv = 1.0f / sqrtf(block_sum(sq, red) / (float)dim + p.eps);
    for (int c = tid; c < dim; c += 256) {
        const float v = so[c] * inv * p.norm[h * dim + c] * sigmoid(sg[c]);
        const size_t o = (size_t)t * p.ldm + (size_t)h * dim + c;
        if (p.mixb) p.mixb[o] = __float2bfloat16_rn(v);
        else p.mix[o] = v;
    }
}

// tanh of n columns, to lowb or in place
__global__ void __launch_bounds__(256) k_tanh_columns(float* proj, int ldp, int n, int T, __nv_bfloat16* __restrict__ lowb, int ldl) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= (long long)T * n) return;
    const int t = (int)(i / n), c = (int)(i % n);
    const float v = tanhf(proj[(size_t)t * ldp + c]);
    if (lowb) lowb[(size_t)t * ldl + c] = __float2bfloat16_rn(v);
    else proj[(size_t)t * ldp + c] = v;
}

struct SsdDecode {
    ConvRef cr;
    const float* proj;
    int ldp;
    const float *conv, *conv_b, *dt_bias, *neg_a, *D;
    int heads, per, groups, state, vdim, off_x, off_dt, off_z;
    size_t state_off;
    float* y;                    // gated: y silu(z)
    int ldy;
};

// One CTA per (head, sequence): convolutions, the state's step, the gate (the group norm spans heads).
template <int EPL>
__global__ void __launch_bounds__(128) k_ssd_decode(const SsdDecode p) {
    constexpr int DP = 32 * EPL, NC = 8;            // columns of a warp at a time
    extern __shared__ __align__(16) float sm[];     // B, C: [DP]; x: [vdim]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, t = blockIdx.y, g = h / p.per;
    float* sx = sm + 2 * DP;
    pdl_launch_dependents();
    pdl_wait();
    const int pos = p.cr.positions[t], seq = p.cr.seq_ids[t], taps = p.cr.taps, inner = p.heads * p.vdim, GN = p.groups * p.state;
    float* S = reinterpret_cast<float*>(p.cr.base + (size_t)seq * p.cr.slot_bytes + p.state_off) + (size_t)h * p.vdim * p.state;
    for (int i = tid * 32; i < p.vdim * p.state; i += 128 * 32) prefetch_l2(S + i);
    float* ring = p.cr.ring(seq);
    const float* row = p.proj + (size_t)t * p.ldp;
    const bool first = h % p.per == 0;
    conv_decode<128, 3>(
        row, ring, p.cr.C, taps, p.conv, p.cr.ldw, p.conv_b, pos, 2 * DP + p.vdim,
        [&](int c) {
            const int d = c < DP ? c : c < 2 * DP ? c - DP : c - 2 * DP;
            if (c < 2 * DP && d >= p.state) return ConvPlace{-1, -1, -1};
            const int ch = c < DP ? inner + g * p.state + d : c < 2 * DP ? inner + GN + g * p.state + d : h * p.vdim + d;
            return ConvPlace{p.off_x + ch, ch, ch};
        },
        [&](int c, float v) { sm[c] = v; }, [&](int c) { return c >= 2 * DP || first; });
    const float dt = softplus(row[p.off_dt + h] + p.dt_bias[h]), decay = expf(p.neg_a[h] * dt), Dh = p.D[h];
    __syncthreads();
    float br[EPL], cr[EPL];
    Chan<EPL>::load(sm, lane, br);
    Chan<EPL>::load(sm + DP, lane, cr);
    for (int c0 = NC * warp; c0 < p.vdim; c0 += 4 * NC) {
        float s[NC][EPL], a[NC];
        load_columns<NC, EPL>(S, c0, p.vdim, p.state, lane, pos == 0, s);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const float u = c0 + c < p.vdim ? dt * sx[c0 + c] : 0.0f;
            a[c] = 0.0f;
#pragma unroll
            for (int i = 0; i < EPL; ++i) {
                s[c][i] = fmaf(s[c][i], decay, br[i] * u);
                a[c] = fmaf(s[c][i], cr[i], a[c]);
            }
        }
        store_columns<NC, EPL>(S, c0, p.vdim, p.state, lane, s);
        const float sum = transpose_sum8(a, lane);
        const int mine = c0 + (lane >> 2);
        if ((lane & 3) == 0 && mine < p.vdim)
            p.y[(size_t)t * p.ldy + (size_t)h * p.vdim + mine] = fmaf(Dh, sx[mine], sum) * silu(row[p.off_z + (size_t)h * p.vdim + mine]);
    }
}

// ---------------------------------------------------------------- output norms
// Four neighbouring values as f32.
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf2(v.x, v.y), pack_bf2(v.z, v.w)); }

// delta rules: one warp per (token, head): o / rms(o) * w * sigmoid(gate).  ws: pitch of the heads' weights, 0: they share them
template <typename TO>
__global__ void __launch_bounds__(256) k_head_norm_gate(const float* __restrict__ o, int ldo, const float* __restrict__ gate, int ldg,
                                                        const float* __restrict__ w, int ws, int heads, int vdim, int T, float eps,
                                                        TO* __restrict__ out, int ldm) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (id >= (long long)T * heads) return;
    const int t = (int)(id / heads), h = (int)(id % heads);
    const float* r = o + (size_t)t * ldo + (size_t)h * vdim;
    float ss = 0.0f;
    for (int c = lane; c < vdim; c += 32) ss = fmaf(r[c], r[c], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int c = lane; c < vdim; c += 32)
        store_as(out + (size_t)t * ldm + (size_t)h * vdim + c, r[c] * inv * w[h * ws + c] * sigmoid(gate[(size_t)t * ldg + (size_t)h * vdim + c]));
}

// The same for value sizes that are a power of two from 4 to 128: vdim / 4 lanes a head, each with four units of (token, head).
template <typename TO>
__global__ void __launch_bounds__(256) k_head_norm_gate4(const float* __restrict__ o, int ldo, const float* __restrict__ gate, int ldg,
                                                         const float* __restrict__ w, int ws, int heads, int vdim, int T, float eps,
                                                         TO* __restrict__ out, int ldm) {
    constexpr int U = 4;
    pdl_launch_dependents();
    pdl_wait();
    const int lanes = vdim / 4, per = 256 / lanes, c = 4 * (threadIdx.x % lanes);
    const long long id0 = (long long)blockIdx.x * per * U + threadIdx.x / lanes, all = (long long)T * heads;
    float4 v[U], g[U], f[U];
    float ss[U];
#pragma unroll
    for (int i = 0; i < U; ++i) {
        const long long id = min(id0 + per * i, all - 1);
        const int t = (int)(id / heads), h = (int)(id % heads);
        v[i] = load4(o + (size_t)t * ldo + h * vdim + c), g[i] = load4(gate + (size_t)t * ldg + h * vdim + c), f[i] = load4(w + h * ws + c);
    }
#pragma unroll
    for (int i = 0; i < U; ++i) ss[i] = (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
    for (int x = lanes >> 1; x > 0; x >>= 1)
#pragma unroll
        for (int i = 0; i < U; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], x);
#pragma unroll
    for (int i = 0; i < U; ++i) {
        const long long id = id0 + per * i;
        if (id >= all) break;
        const int t = (int)(id / heads), h = (int)(id % heads);
        const float inv = 1.0f / sqrtf(ss[i] / (float)vdim + eps);
        store4(out + (size_t)t * ldm + h * vdim + c, make_float4(v[i].x * inv * f[i].x * sigmoid(g[i].x), v[i].y * inv * f[i].y * sigmoid(g[i].y),
                                                                 v[i].z * inv * f[i].z * sigmoid(g[i].z), v[i].w * inv * f[i].w * sigmoid(g[i].w)));
    }
}

int launch_head_norm_gate(dc_ctx* ctx, const float* o, int ldo, const float* gate, int ldg, const float* w, int ws, int heads, int vdim, int T, float eps,
                          float* mix, __nv_bfloat16* mixb, int ldm) {
    const dim3 grid((unsigned)(((long long)T * heads + 7) / 8)), block(256);
    if (vdim >= 4 && vdim <= 128 && !(vdim & (vdim - 1)) && ldo % 4 == 0 && ldg % 4 == 0 && ldm % 4 == 0 && ((uintptr_t)gate & 15) == 0) {
        const int units = 4 * 256 / (vdim / 4);
        const dim3 grid4((unsigned)(((long long)T * heads + units - 1) / units));
        if (mixb) return dc_launch(ctx, "k_head_norm_gate4", k_head_norm_gate4<__nv_bfloat16>, grid4, block, 0, o, ldo, gate, ldg, w, ws, heads, vdim, T, eps, mixb, ldm);
        return dc_launch(ctx, "k_head_norm_gate4", k_head_norm_gate4<float>, grid4, block, 0, o, ldo, gate, ldg, w, ws, heads, vdim, T, eps, mix, ldm);
    }
    if (mixb) return dc_launch(ctx, "k_head_norm_gate", k_head_norm_gate<__nv_bfloat16>, grid, block, 0, o, ldo, gate, ldg, w, ws, heads, vdim, T, eps, mixb, ldm);
    return dc_launch(ctx, "k_head_norm_gate", k_head_norm_gate<float>, grid, block, 0, o, ldo, gate, ldg, w, ws, heads, vdim, T, eps, mix, ldm);
}

// ssd: one CTA per (token, norm group): y silu(z) (unless gated already), over its root mean square, times w
template <typename TO, int NT>
__global__ void __launch_bounds__(NT) k_gate_group_norm(const float* __restrict__ y, int ldy, const float* __restrict__ z, int ldz,
                                                         const float* __restrict__ w, int n, float eps, TO* __restrict__ out, int ldm) {
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.y, c0 = blockIdx.x * n;
    const float* yr = y + (size_t)t * ldy + c0;
    const float* zr = z ? z + (size_t)t * ldz + c0 : nullptr;
    constexpr int KEEP = 8;      // values per thread kept between the two passes
    float v[KEEP], ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + NT * j;
        v[j] = i < n ? (zr ? yr[i] * silu(zr[i]) : yr[i]) : 0.0f;
        ss = fmaf(v[j], v[j], ss);
    }
    for (int i = threadIdx.x + NT * KEEP; i < n; i += NT) {
        const float x = zr ? yr[i] * silu(zr[i]) : yr[i];
        ss = fmaf(x, x, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + NT * j;
        if (i < n) store_as(out + (size_t)t * ldm + c0 + i, v[j] * inv * w[c0 + i]);
    }
    for (int i = threadIdx.x + NT * KEEP; i < n; i += NT)
        store_as(out + (size_t)t * ldm + c0 + i, (zr ? yr[i] * silu(zr[i]) : yr[i]) * inv * w[c0 + i]);
}

// small groups get small CTAs: more of them are resident
template <typename TO>
int launch_group_norm(dc_ctx* ctx, const float* y, int ldy, const float* z, int ldz, const float* w, int n, int groups, int T, float eps, TO* out, int ldm) {
    const dim3 grid(groups, T);
    if (n <= 512) return dc_launch(ctx, "k_gate_group_norm", k_gate_group_norm<TO, 64>, grid, dim3(64), 0, y, ldy, z, ldz, w, n, eps, out, ldm);
    return dc_launch(ctx, "k_gate_group_norm", k_gate_group_norm<TO, 256>, grid, dim3(256), 0, y, ldy, z, ldz, w, n, eps, out, ldm);
}

// lightning: one CTA per token: y over its root mean square, times w, times sigmoid(gate).  Rows are padded to multiples of
// eight (what the padding holds does not matter); KEEP: groups of four values of a thread.
template <int KEEP, typename TZ, typename TO>
__global__ void __launch_bounds__(256) k_norm_gate(const float* __restrict__ y, int ldy, const TZ* __restrict__ gate, int ldz, const float* __restrict__ w,
                                                   int n, float eps, TO* __restrict__ out, int ldm) {
    __shared__ float red[33];
    pdl_launch_dependents();
    float4 v[KEEP], g[KEEP], wv[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = 4 * (threadIdx.x + 256 * j);
        wv[j] = i < n ? load4(w + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    const int t = blockIdx.x;
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = 4 * (threadIdx.x + 256 * j);
        v[j] = g[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n) v[j] = load4(y + (size_t)t * ldy + i), g[j] = load4(gate + (size_t)t * ldz + i);
        if (i + 1 >= n) v[j].y = 0.0f;
        if (i + 2 >= n) v[j].z = 0.0f;
        if (i + 3 >= n) v[j].w = 0.0f;
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j) ss += (v[j].x * v[j].x + v[j].y * v[j].y) + (v[j].z * v[j].z + v[j].w * v[j].w);
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = 4 * (threadIdx.x + 256 * j);
        if (i < n)
            store4(out + (size_t)t * ldm + i, make_float4(v[j].x * inv * wv[j].x * sigmoid(g[j].x), v[j].y * inv * wv[j].y * sigmoid(g[j].y),
                                                          v[j].z * inv * wv[j].z * sigmoid(g[j].z), v[j].w * inv * wv[j].w * sigmoid(g[j].w)));
    }
}
template <typename TZ, typename TO>
int launch_norm_gate(dc_ctx* ctx, const float* y, int ldy, const TZ* gate, int ldz, const float* w, int n, int T, float eps, TO* out, int ldm) {
    const dim3 grid(T), block(256);
    if (n <= 1024) return dc_launch(ctx, "k_norm_gate", k_norm_gate<1, TZ, TO>, grid, block, 0, y, ldy, gate, ldz, w, n, eps, out, ldm);
    if (n <= 2048) return dc_launch(ctx, "k_norm_gate", k_norm_gate<2, TZ, TO>, grid, block, 0, y, ldy, gate, ldz, w, n, eps, out, ldm);
    if (n <= 4096) return dc_launch(ctx, "k_norm_gate", k_norm_gate<4, TZ, TO>, grid, block, 0, y, ldy, gate, ldz, w, n, eps, out, ldm);
    if (n <= 8192) return dc_launch(ctx, "k_norm_gate", k_norm_gate<8, TZ, TO>, grid, block, 0, y, ldy, gate, ldz, w, n, eps, out, ldm);
    return dc_launch(ctx, "k_norm_gate", k_norm_gate<16, TZ, TO>, grid, block, 0, y, ldy, gate, ldz, w, n, eps, out, ldm);
}

// ---------------------------------------------------------------- linear attention with a constant decay: decode
struct LightningDecode {
    int ld, off_q, off_k, off_v, dim, vdim;
    const float* decay;
    uint8_t* base;
    size_t slot_bytes, state_off;
    const int32_t *seq_ids, *positions;
    float* y;
    int ldy;
};

// One CTA per (head, 32 value columns, sequence), eight columns a warp.
template <int EPL, typename TA>
__global__ void __launch_bounds__(128) k_lightning_decode(const TA* __restrict__ act, const LightningDecode p) {
    constexpr int NC = 8;
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.x, c0 = blockIdx.y * 32 + NC * warp, t = blockIdx.z;
    const float decay = p.decay[h];
    pdl_wait();
    if (c0 >= p.vdim) return;
    const int pos = p.positions[t], seq = p.seq_ids[t];
    float* S = reinterpret_cast<float*>(p.base + (size_t)seq * p.slot_bytes + p.state_off) + (size_t)h * p.vdim * p.dim;
    const TA* row = act + (size_t)t * p.ld;
    float s[NC][EPL], q[EPL], k[EPL], v[NC], a[NC];
    load_columns<NC, EPL>(S, c0, p.vdim, p.dim, lane, pos == 0, s);
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
        const int d = Chan<EPL>::at(lane, i);
        q[i] = d < p.dim ? load_as(row + p.off_q + (size_t)h * p.dim + d) : 0.0f;
        k[i] = d < p.dim ? load_as(row + p.off_k + (size_t)h * p.dim + d) : 0.0f;
    }
#pragma unroll
    for (int c = 0; c < NC; ++c) v[c] = load_as(row + p.off_v + (size_t)h * p.vdim + min(c0 + c, p.vdim - 1));
#pragma unroll
    for (int c = 0; c < NC; ++c) {
        a[c] = 0.0f;
#pragma unroll
        for (int i = 0; i < EPL; ++i) {
            s[c][i] = fmaf(s[c][i], decay, k[i] * v[c]);
            a[c] = fmaf(s[c][i], q[i], a[c]);
        }
    }
    store_columns<NC, EPL>(S, c0, p.vdim, p.dim, lane, s);
    const float sum = transpose_sum8(a, lane);
    const int mine = c0 + (lane >> 2);
    if ((lane & 3) == 0 && mine < p.vdim) p.y[(size_t)t * p.ldy + (size_t)h * p.vdim + mine] = sum;
}

template <typename TA>
int launch_lightning_decode(dc_ctx* ctx, const TA* act, const LightningDecode& p, int heads, int T) {
    const dim3 grid(heads, (p.vdim + 31) / 32, T), block(128);
    switch (key_pad(p.dim)) {
    case 32: return dc_launch(ctx, "k_lightning_decode", k_lightning_decode<1, TA>, grid, block, 0, act, p);
    case 64: return dc_launch(ctx, "k_lightning_decode", k_lightning_decode<2, TA>, grid, block, 0, act, p);
    case 128: return dc_launch(ctx, "k_lightning_decode", k_lightning_decode<4, TA>, grid, block, 0, act, p);
    default: return dc_launch(ctx, "k_lightning_decode", k_lightning_decode<8, TA>, grid, block, 0, act, p);
    }
}

// ---------------------------------------------------------------- ssd: per-token inputs
struct SsdPrep {
    ConvRef cr;
    const float* proj;
    int ldp, off_x, off_dt, heads, T;
    const float *conv, *conv_b, *dt_bias, *neg_a;
    float* act;
    int lda;
    float* small;            // [T][2 heads]: step, decay
};
__global__ void __launch_bounds__(256) k_ssd_prep(SsdPrep p) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
    const int e = entry_of(p.cr.starts, p.cr.E, t), i = t - p.cr.starts[e], pos = p.cr.positions[t];
    if (c < p.cr.C)
        p.act[(size_t)t * p.lda + c] = silu(conv_at(p.proj, p.ldp, p.cr.ring(p.cr.seq_ids[t]), p.cr.C, c, p.cr.taps, p.conv + c, p.cr.ldw,
                                                    p.off_x + c, t, i, pos) + p.conv_b[c]);
    if (blockIdx.x == 0)
        for (int h = threadIdx.x; h < p.heads; h += 256) {
            const float dt = softplus(p.proj[(size_t)t * p.ldp + p.off_dt + h] + p.dt_bias[h]);
            p.small[(size_t)t * 2 * p.heads + h] = dt;
            p.small[(size_t)t * 2 * p.heads + p.heads + h] = expf(p.neg_a[h] * dt);
        }
}

// Four taps: a thread takes its channel through a block of up to sixteen tokens with the window in registers.
__global__ void __launch_bounds__(256) k_ssd_prep4(SsdPrep p) {
    pdl_launch_dependents();
    pdl_wait();
    const int c = blockIdx.y * 256 + threadIdx.x;
    const BlockRef br = block_at<BT>(p.cr.starts, p.cr.E, blockIdx.x);
    if (br.n <= 0) return;
    if (c < p.cr.C) {
        const int i0 = br.t0 - p.cr.starts[br.e], pos0 = p.cr.positions[br.t0];
        const float* ring = p.cr.ring(p.cr.seq_ids[br.t0]);
        const float* in = p.proj + (size_t)br.t0 * p.ldp + p.off_x + c;
        float w[4], h[3], x[BT];
#pragma unroll
        for (int k = 0; k < 4; ++k) w[k] = p.conv[(size_t)k * p.cr.ldw + c];
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            const int back = 3 - k;
            h[k] = pos0 < back ? 0.0f : back <= i0 ? in[-(ptrdiff_t)back * p.ldp] : ring[(size_t)((pos0 - back) % 4) * p.cr.C + c];
        }
#pragma unroll
        for (int u = 0; u < BT; ++u) x[u] = u < br.n ? in[(size_t)u * p.ldp] : 0.0f;
        const float bias = p.conv_b[c];
#pragma unroll
        for (int u = 0; u < BT; ++u) {
            const float y = silu(fmaf(w[3], x[u], fmaf(w[2], h[2], fmaf(w[1], h[1], w[0] * h[0]))) + bias);
            h[0] = h[1], h[1] = h[2], h[2] = x[u];
            if (u < br.n) p.act[(size_t)(br.t0 + u) * p.lda + c] = y;
        }
    }
    if (blockIdx.y == 0)
        for (int i = threadIdx.x; i < br.n * p.heads; i += 256) {
            const int t = br.t0 + i / p.heads, h = i % p.heads;
            const float dt = softplus(p.proj[(size_t)t * p.ldp + p.off_dt + h] + p.dt_bias[h]);
            p.small[(size_t)t * 2 * p.heads + h] = dt;
            p.small[(size_t)t * 2 * p.heads + p.heads + h] = expf(p.neg_a[h] * dt);
        }
}

ConvRef conv_ref(const dc_step& st, const dc_state_ref& sr, int taps, int C) {
    return ConvRef{sr.base, sr.slot_bytes, sr.ring_off, st.seq_ids, st.positions, st.starts, st.E, taps, C, C};
}

}  // namespace

int dc_scan_blocks(int T, int E) { return T / BT + E; }
size_t dc_delta_block_floats(const dc_delta_mixer& m) { return (size_t)m.heads * delta_block_floats(key_pad(m.dim)); }
size_t dc_ssd_block_floats(const dc_ssd_mixer& m) { return (size_t)m.heads * SSD_BLOCK; }

int dc_launch_ring_update(dc_ctx* ctx, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, int off, int C, int taps) {
    return dc_launch(ctx, "k_ring_update", k_ring_update, dim3((C + 255) / 256, st.E), dim3(256), 0, conv_ref(st, sr, taps, C), proj, ldp, off);
}

int dc_launch_delta_prep(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp,
                         float* act, int lda, float* small, __nv_bfloat16* lowb, int ldl) {
    DeltaPrep p;
    const int V = m.heads * m.vdim, C = m.off_v + V;
    p.cr = conv_ref(st, sr, m.taps, C);
    p.cr.ldw = m.off_v + dc_pad8(V);
    p.proj = proj, p.ldp = ldp, p.conv = m.conv;
    p.heads = m.heads, p.kv_heads = m.kv_heads, p.dim = m.dim, p.vdim = m.vdim;
    p.off_q = m.off_q, p.off_k = m.off_k, p.off_v = m.off_v, p.off_b = m.off_b, p.off_a = m.off_a;
    p.n_low = m.off_g + m.g_rank - m.off_a;
    p.unit_eps = m.unit_eps, p.q_scale = m.q_scale;
    p.act = act, p.lda = lda, p.small = small, p.lowb = lowb, p.ldl = ldl, p.T = st.T, p.v_items = (V + 127) / 128;
    const int items = m.kv_heads + p.v_items + 1;
    if (m.taps == 4) {
        const dim3 grid(dc_scan_blocks(st.T, st.E), (items - 1 + 7) / 8 + 1);
        switch (key_pad(m.dim)) {
        case 32: DC_TRY(dc_launch(ctx, "k_delta_prep4", k_delta_prep4<1>, grid, dim3(256), 0, p)); break;
        case 64: DC_TRY(dc_launch(ctx, "k_delta_prep4", k_delta_prep4<2>, grid, dim3(256), 0, p)); break;
        case 128: DC_TRY(dc_launch(ctx, "k_delta_prep4", k_delta_prep4<4>, grid, dim3(256), 0, p)); break;
        default: DC_TRY(dc_launch(ctx, "k_delta_prep4", k_delta_prep4<8>, grid, dim3(256), 0, p));
        }
    } else {
        DC_TRY(dc_launch(ctx, "k_delta_prep", k_delta_prep, dim3((unsigned)(((long long)st.T * items + 7) / 8)), dim3(256), 0, p));
    }
    return dc_launch_ring_update(ctx, st, sr, proj, ldp, 0, C, m.taps);
}

int dc_launch_delta_scan(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* act, int lda,
                         const float* small, const float* low, int ldd, float* blk, const float* raw_g, int ldg, float eps, float* o,
                         float* mix, __nv_bfloat16* mixb, int ldm) {
    const int dp = key_pad(m.dim), nb = dc_scan_blocks(st.T, st.E);
    DeltaBlock d = {act, lda, m.off_q, m.off_k, m.heads, m.heads / m.kv_heads, m.dim, dp, low, ldd, m.neg_a, m.dt_bias, small, m.heads, st.starts, st.E, blk};
    const size_t smem = (size_t)3 * BT * m.dim * 4;
    DC_TRY(dc_kernel_setup(ctx, (const void*)k_delta_blocks, (int)smem, "k_delta_blocks"));
    DC_TRY(dc_launch(ctx, "k_delta_blocks", k_delta_blocks, dim3(nb, m.heads), dim3(128), smem, d));
    ScanParams p = {};
    p.blocks = blk, p.v = act + m.off_v;
    p.ld = lda, p.heads = m.heads, p.per = m.heads / m.kv_heads, p.dim = m.dim, p.vdim = m.vdim;
    p.o = o, p.ldo = lda;
    p.base = sr.base, p.slot_bytes = sr.slot_bytes, p.state_off = sr.state_off;
    p.seq_ids = st.seq_ids, p.positions = st.positions, p.starts = st.starts;
    DC_TRY(launch_scan<SCAN_DELTA>(ctx, p, st.E));
    return launch_head_norm_gate(ctx, o, lda, raw_g, ldg, m.norm, 0, m.heads, m.vdim, st.T, eps, mix, mixb, ldm);
}

size_t dc_general_block_floats(const dc_general_mixer& m) { return (size_t)m.heads * general_block_floats(key_pad(m.dim)); }

int dc_launch_general_tanh(dc_ctx* ctx, const dc_general_mixer& m, int T, float* proj, int ldp, __nv_bfloat16* lowb, int ldl) {
    const int n = dc_pad8(m.rank);
    return dc_launch(ctx, "k_tanh_columns", k_tanh_columns, dim3((unsigned)(((long long)T * n + 255) / 256)), dim3(256), 0, proj + m.off_w, ldp, n, T, lowb, ldl);
}

int dc_launch_general_scan(dc_ctx* ctx, const dc_general_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, const float* low,
                           int ldd, float* blk, float eps, float* o, int ldo, float* mix, __nv_bfloat16* mixb, int ldm) {
    const GeneralBlock b = {proj, ldp, m.off_r, m.off_k, m.off_a, m.heads, m.dim, low, ldd, m.w0, m.a_bias, m.unit_eps, st.starts, st.E, blk};
    const dim3 grid(dc_scan_blocks(st.T, st.E), m.heads);
    switch (key_pad(m.dim)) {
    case 32: DC_TRY(launch_general_blocks<1>(ctx, b, grid)); break;
    case 64: DC_TRY(launch_general_blocks<2>(ctx, b, grid)); break;
    case 128: DC_TRY(launch_general_blocks<4>(ctx, b, grid)); break;
    default: DC_TRY(launch_general_blocks<8>(ctx, b, grid));
    }
    ScanParams p = {};
    p.blocks = blk, p.v = proj + m.off_v;
    p.ld = ldp, p.heads = m.heads, p.per = 1, p.dim = m.dim, p.vdim = m.dim;
    p.o = o, p.ldo = ldo;
    p.base = sr.base, p.slot_bytes = sr.slot_bytes, p.state_off = sr.state_off;
    p.seq_ids = st.seq_ids, p.positions = st.positions, p.starts = st.starts;
    DC_TRY(launch_scan<SCAN_GENERAL>(ctx, p, st.E));
    return launch_head_norm_gate(ctx, o, ldo, proj + m.off_g, ldp, m.norm, m.dim, m.heads, m.dim, st.T, eps, mix, mixb, ldm);
}

int dc_launch_general_decode(dc_ctx* ctx, const dc_general_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float eps,
                             float* mix, __nv_bfloat16* mixb, int ldm) {
    const GeneralDecode p = {proj, ldp, m.heads, m.dim, m.rank, m.off_r, m.off_k, m.off_v, m.off_g, m.off_a, m.off_w, m.unit_eps, eps, m.w2.w, m.w2.ld, m.w0,
                             m.a_bias, m.norm, sr.base, sr.slot_bytes, sr.state_off, st.seq_ids, st.positions, mix, mixb, ldm};
    const int dp = key_pad(m.dim);
    const size_t smem = (size_t)(7 * dp + ((m.rank + 127) & ~127)) * 4;
    const dim3 grid(m.heads, st.T), block(256);
    if (smem > 48 * 1024) return dc_fail(ctx, DC_B200_UNSUPPORTED, "generalized delta rule: decay rank %d is too large", m.rank);
    if (dp == 32) return dc_launch(ctx, "k_general_decode", k_general_decode<1>, grid, block, smem, p);
    if (dp == 64) return dc_launch(ctx, "k_general_decode", k_general_decode<2>, grid, block, smem, p);
    if (dp == 128) return dc_launch(ctx, "k_general_decode", k_general_decode<4>, grid, block, smem, p);
    return dc_launch(ctx, "k_general_decode", k_general_decode<8>, grid, block, smem, p);
}

int dc_launch_ssd(dc_ctx* ctx, const dc_ssd_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float* act,
                  int lda, float* small, float* blk, float* y, float eps, float* mix, __nv_bfloat16* mixb, int ldm) {
    const int inner = m.heads * m.vdim, GN = m.groups * m.state, C = inner + 2 * GN;
    SsdPrep s = {conv_ref(st, sr, m.taps, C), proj, ldp, m.off_x, m.off_dt, m.heads, st.T, m.conv, m.conv_b, m.dt_bias, m.neg_a, act, lda, small};
    if (m.taps == 4) DC_TRY(dc_launch(ctx, "k_ssd_prep4", k_ssd_prep4, dim3(dc_scan_blocks(st.T, st.E), (C + 255) / 256), dim3(256), 0, s));
    else DC_TRY(dc_launch(ctx, "k_ssd_prep", k_ssd_prep, dim3((C + 255) / 256, st.T), dim3(256), 0, s));
    DC_TRY(dc_launch_ring_update(ctx, st, sr, proj, ldp, m.off_x, C, m.taps));
    SsdBlock sb = {act, lda, inner, inner + GN, m.heads, m.heads / m.groups, m.state, small, nullptr, st.starts, st.E, blk};
    DC_TRY(dc_launch(ctx, "k_ssd_blocks", k_ssd_blocks, dim3(dc_scan_blocks(st.T, st.E), m.groups), dim3(256), (size_t)2 * BT * (m.state + 1) * 4, sb));
    ScanParams p = {};
    p.blocks = blk, p.k = act + inner, p.q = act + inner + GN, p.v = act;
    p.ld = lda, p.heads = m.heads, p.per = m.heads / m.groups, p.dim = m.state, p.vdim = m.vdim;
    p.D = m.D, p.o = y, p.ldo = lda;
    p.base = sr.base, p.slot_bytes = sr.slot_bytes, p.state_off = sr.state_off;
    p.seq_ids = st.seq_ids, p.positions = st.positions, p.starts = st.starts;
    p.vec = m.state % 4 == 0 && lda % 4 == 0 && inner % 4 == 0;
    DC_TRY(launch_scan<SCAN_SSD>(ctx, p, st.E));
    const int n = inner / m.norm_groups;
    const float* z = proj + m.off_z;
    return mixb ? launch_group_norm(ctx, y, lda, z, ldp, m.norm, n, m.norm_groups, st.T, eps, mixb, ldm)
                : launch_group_norm(ctx, y, lda, z, ldp, m.norm, n, m.norm_groups, st.T, eps, mix, ldm);
}

int dc_launch_delta_decode(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float eps,
                           float* mix, __nv_bfloat16* mixb, int ldm) {
    const int V = m.heads * m.vdim;
    DeltaDecode p = {conv_ref(st, sr, m.taps, m.off_v + V), proj, ldp, m.conv, m.heads, m.heads / m.kv_heads, m.dim, m.vdim, m.off_q, m.off_k, m.off_v, m.off_b,
                     m.off_a, m.off_g, m.a_rank, m.g_rank, m.unit_eps, m.q_scale, eps, m.a2.w, m.g2.w, m.a2.ld, m.g2.ld, m.neg_a, m.dt_bias, m.norm,
                     sr.state_off, mix, mixb, ldm};
    p.cr.ldw = m.off_v + dc_pad8(V);
    const int dp = key_pad(m.dim);
    const size_t smem = (size_t)(3 * dp + ((m.a_rank + 127) & ~127) + ((m.g_rank + 127) & ~127) + 3 * m.vdim) * 4;
    const dim3 grid(m.heads, st.T), block(256);
    if (smem > 48 * 1024) return dc_fail(ctx, DC_B200_UNSUPPORTED, "delta rule: gate ranks %d and %d are too large", m.a_rank, m.g_rank);
    if (dp == 32) return dc_launch(ctx, "k_delta_decode", k_delta_decode<1>, grid, block, smem, p);
    if (dp == 64) return dc_launch(ctx, "k_delta_decode", k_delta_decode<2>, grid, block, smem, p);
    if (dp == 128) return dc_launch(ctx, "k_delta_decode", k_delta_decode<4>, grid, block, smem, p);
    return dc_launch(ctx, "k_delta_decode", k_delta_decode<8>, grid, block, smem, p);
}

int dc_launch_ssd_decode(dc_ctx* ctx, const dc_ssd_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float* y, int ldy,
                         float eps, float* mix, __nv_bfloat16* mixb, int ldm) {
    const int inner = m.heads * m.vdim, C = inner + 2 * m.groups * m.state;
    SsdDecode p = {conv_ref(st, sr, m.taps, C), proj, ldp, m.conv, m.conv_b, m.dt_bias, m.neg_a, m.D, m.heads, m.heads / m.groups, m.groups, m.state, m.vdim,
                   m.off_x, m.off_dt, m.off_z, sr.state_off, y, ldy};
    const int dp = key_pad(m.state);
    const size_t smem = (size_t)(2 * dp + m.vdim) * 4;
    const dim3 grid(m.heads, st.T), block(128);
    if (dp == 32) DC_TRY(dc_launch(ctx, "k_ssd_decode", k_ssd_decode<1>, grid, block, smem, p));
    else if (dp == 64) DC_TRY(dc_launch(ctx, "k_ssd_decode", k_ssd_decode<2>, grid, block, smem, p));
    else if (dp == 128) DC_TRY(dc_launch(ctx, "k_ssd_decode", k_ssd_decode<4>, grid, block, smem, p));
    else DC_TRY(dc_launch(ctx, "k_ssd_decode", k_ssd_decode<8>, grid, block, smem, p));
    const int n = inner / m.norm_groups;
    return mixb ? launch_group_norm(ctx, y, ldy, nullptr, 0, m.norm, n, m.norm_groups, st.T, eps, mixb, ldm)
                : launch_group_norm(ctx, y, ldy, nullptr, 0, m.norm, n, m.norm_groups, st.T, eps, mix, ldm);
}

size_t dc_lightning_block_floats(const dc_lightning_mixer& m) { return (size_t)m.heads * SSD_BLOCK; }

int dc_launch_lightning_scan(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* act, int lda,
                             float* blk, float* y, int ldy) {
    SsdBlock sb = {act, lda, m.off_k, m.off_q, m.heads, 1, m.dim, nullptr, m.decay, st.starts, st.E, blk};
    DC_TRY(dc_launch(ctx, "k_ssd_blocks", k_ssd_blocks, dim3(dc_scan_blocks(st.T, st.E), m.heads), dim3(256), (size_t)2 * BT * (m.dim + 1) * 4, sb));
    ScanParams p = {};
    p.blocks = blk, p.k = act + m.off_k, p.q = act + m.off_q, p.v = act + m.off_v;
    p.ld = lda, p.heads = m.heads, p.per = 1, p.dim = m.dim, p.vdim = m.vdim;
    p.o = y, p.ldo = ldy;
    p.base = sr.base, p.slot_bytes = sr.slot_bytes, p.state_off = sr.state_off;
    p.seq_ids = st.seq_ids, p.positions = st.positions, p.starts = st.starts;
    p.vec = m.dim % 4 == 0 && lda % 4 == 0;
    return launch_scan<SCAN_SSD>(ctx, p, st.E);
}

int dc_launch_lightning_decode(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* act,
                               const __nv_bfloat16* actb, int lda, float* y, int ldy) {
    LightningDecode p = {lda, m.off_q, m.off_k, m.off_v, m.dim, m.vdim, m.decay, sr.base, sr.slot_bytes, sr.state_off, st.seq_ids, st.positions, y, ldy};
    return actb ? launch_lightning_decode(ctx, actb, p, m.heads, st.T) : launch_lightning_decode(ctx, act, p, m.heads, st.T);
}

int dc_launch_lightning_norm(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const float* y, int ldy, const float* act,
                             const __nv_bfloat16* actb, int lda, float eps, float* mix, __nv_bfloat16* mixb, int ldm) {
    const int n = m.heads * m.vdim;
    return mixb ? launch_norm_gate(ctx, y, ldy, actb + m.off_g, lda, m.norm, n, st.T, eps, mixb, ldm)
                : launch_norm_gate(ctx, y, ldy, act + m.off_g, lda, m.norm, n, st.T, eps, mix, ldm);
}
