// Recurrent mixers: short causal convolution, gated delta rule with one decay per key channel, Mamba-2 state-space
// scan, and their gated output norms.
//
// Per-sequence state (f32) lives in the cache manager's state slots: the matrix S as [head][value column][key
// channel], and the convolution's last inputs as a ring [position % taps][channel].  A sequence at position 0 starts
// from zero whatever its slot holds, so slots need no clearing when they change hands.
//
// Value columns of S never mix: a column c obeys S_c <- g S_c; u = beta (v_c - S_c . k); S_c <- S_c + u k;
// o_c = S_c . q.  k_state_scan gives each column to eight lanes and walks an entry's tokens with the column in
// registers.  Since o_c = (g S_c) . q + (k . q) u, both dot products of a token share one reduction.  The arithmetic
// of a token does not depend on where an entry starts, so cutting a prompt changes nothing.
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

__device__ __forceinline__ int entry_of(const int32_t* starts, int E, int t) {
    int e = 0;
    while (e + 1 < E && starts[e + 1] <= t) ++e;
    return e;
}

// Convolution of one channel at token t (local index i in its entry, position pos): weights w[0 .. taps - 1], the last
// for the token itself.
__device__ __forceinline__ float conv_at(const float* __restrict__ proj, int ldp, const float* __restrict__ ring, int C, int rc, int taps,
                                         const float* __restrict__ w, int col, int t, int i, int pos) {
    float s = 0.0f;
    for (int j = 0; j < taps; ++j) {
        const int back = taps - 1 - j;
        float in = 0.0f;
        if (back <= i) in = proj[(size_t)(t - back) * ldp + col];
        else if (pos >= back) in = ring[(size_t)((pos - back) % taps) * C + rc];
        s = fmaf(w[j], in, s);
    }
    return s;
}

struct ConvRef {
    uint8_t* base;
    size_t slot_bytes, ring_off;
    const int32_t *seq_ids, *positions, *starts;
    int E, taps, C;          // C: channels of a ring row
    __device__ float* ring(int seq) const { return reinterpret_cast<float*>(base + (size_t)seq * slot_bytes + ring_off); }
};

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
    float* small;            // [T][heads + kv_heads]: beta, then k . q
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
                q[j] = silu(conv_at(p.proj, p.ldp, ring, p.cr.C, cq, taps, p.conv + (size_t)cq * taps, cq, t, i, pos));
                k[j] = silu(conv_at(p.proj, p.ldp, ring, p.cr.C, ck, taps, p.conv + (size_t)ck * taps, ck, t, i, pos));
            }
            sq = fmaf(q[j], q[j], sq);
            sk = fmaf(k[j], k[j], sk);
        }
        const float iq = p.q_scale / sqrtf(warp_sum(sq) + p.unit_eps), ik = 1.0f / sqrtf(warp_sum(sk) + p.unit_eps);
        float kq = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int d = lane + 32 * j;
            q[j] *= iq;
            k[j] *= ik;
            kq = fmaf(q[j], k[j], kq);
            if (d < p.dim) {
                act[p.off_q + item * p.dim + d] = q[j];
                act[p.off_k + item * p.dim + d] = k[j];
            }
        }
        kq = warp_sum(kq);
        if (lane == 0) p.small[(size_t)t * (p.heads + p.kv_heads) + p.heads + item] = kq;
    } else if (item < p.kv_heads + p.v_items) {
        const int c0 = (item - p.kv_heads) * 128, V = p.heads * p.vdim;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = c0 + lane + 32 * j;
            if (c < V) {
                const int cv = p.off_v + c;
                act[cv] = silu(conv_at(p.proj, p.ldp, ring, p.cr.C, cv, taps, p.conv + (size_t)cv * taps, cv, t, i, pos));
            }
        }
    } else {
        for (int h = lane; h < p.heads; h += 32)
            p.small[(size_t)t * (p.heads + p.kv_heads) + h] = sigmoid(p.proj[(size_t)t * p.ldp + p.off_b + h]);
        if (p.lowb)
            for (int c = lane; c < p.n_low; c += 32)
                p.lowb[(size_t)t * p.ldl + c] = __float2bfloat16_rn(p.proj[(size_t)t * p.ldp + p.off_a + c]);
    }
}

// decay[t][c] = exp(neg_a[head] * softplus(raw + dt_bias)), in place
__global__ void __launch_bounds__(256) k_delta_decay(float* __restrict__ raw, int ld, const float* __restrict__ neg_a,
                                                     const float* __restrict__ dt_bias, int dim, int n) {
    pdl_launch_dependents();
    pdl_wait();
    float* r = raw + (size_t)blockIdx.y * ld;
    const int c = blockIdx.x * 256 + threadIdx.x;
    if (c < n) r[c] = expf(neg_a[c / dim] * softplus(r[c] + dt_bias[c]));
}

// ---------------------------------------------------------------- the scan
constexpr int SC_TOK = 16, SC_COLS = 16, SC_THREADS = 128;   // tokens per staged chunk, columns per CTA

struct ScanParams {
    const float *k, *q, *v, *g;    // first head's columns; k and q of head h start at (h / per) * dim
    int ld, ldg;                   // pitch of k, q, v and of g
    int heads, per, dim, vdim;
    const float* small;            // delta: beta per head, then k . q per kv head;  ssd: step and decay per head
    int lds, small2;               // pitch, offset of the second set
    const float* D;                // ssd: per head
    float* o;
    int ldo;
    uint8_t* base;
    size_t slot_bytes, state_off;
    const int32_t *seq_ids, *positions, *starts;
    int vec;                       // dim and pitches allow 16-byte copies
};

__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// EPL: key channels per lane (the state's key size, padded to 8 EPL).
template <int EPL, bool DELTA>
__global__ void __launch_bounds__(SC_THREADS) k_state_scan(const ScanParams p) {
    constexpr int DP = 8 * EPL, NV = DELTA ? 3 : 2, BUF = SC_TOK * (NV * DP + SC_COLS + 2);
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7;
    const int c0 = blockIdx.x * SC_COLS, h = blockIdx.y, e = blockIdx.z, kh = h / p.per;
    const int col = c0 + warp * 4 + (lane >> 3);
    for (int i = tid; i < 2 * BUF; i += SC_THREADS) sm[i] = 0.0f;    // padded channels and columns stay zero
    __syncthreads();
    pdl_wait();
    const int t0 = p.starts[e], t1 = p.starts[e + 1];
    if (t0 >= t1) return;
    const int seq = p.seq_ids[t0];
    float* S = reinterpret_cast<float*>(p.base + (size_t)seq * p.slot_bytes + p.state_off) + ((size_t)h * p.vdim + col) * p.dim;
    float s[EPL];
    const bool fresh = p.positions[t0] == 0;
#pragma unroll
    for (int j = 0; j < EPL; ++j) {
        const int d = 4 * (l8 + 8 * (j >> 2)) + (j & 3);
        s[j] = !fresh && col < p.vdim && d < p.dim ? S[d] : 0.0f;
    }
    auto load = [&](int chunk, int buf) {
        float* b = sm + buf * BUF;
        const int tb = t0 + chunk * SC_TOK, n = min(SC_TOK, t1 - tb);
        const float* src[3] = {p.k + (size_t)kh * p.dim, p.q + (size_t)kh * p.dim, DELTA ? p.g + (size_t)h * p.dim : nullptr};
#pragma unroll
        for (int a = 0; a < NV; ++a) {
            const int ld = a == 2 ? p.ldg : p.ld;
            float* dst = b + a * SC_TOK * DP;
            if (p.vec) {
                const int d4 = p.dim >> 2;
                for (int i = tid; i < n * d4; i += SC_THREADS) {
                    const int tk = i / d4, d = (i - tk * d4) * 4;
                    cp_async16(smem_u32(dst + tk * DP + d), src[a] + (size_t)(tb + tk) * ld + d);
                }
            } else {
                for (int i = tid; i < n * p.dim; i += SC_THREADS) {
                    const int tk = i / p.dim, d = i - tk * p.dim;
                    cp_async4(smem_u32(dst + tk * DP + d), src[a] + (size_t)(tb + tk) * ld + d);
                }
            }
        }
        float* bv = b + NV * SC_TOK * DP;
        for (int i = tid; i < n * SC_COLS; i += SC_THREADS) {
            const int tk = i / SC_COLS, c = i % SC_COLS;
            if (c0 + c < p.vdim) cp_async4(smem_u32(bv + i), p.v + (size_t)(tb + tk) * p.ld + (size_t)h * p.vdim + c0 + c);
        }
        for (int i = tid; i < n * 2; i += SC_THREADS) {
            const int tk = i >> 1;
            const int off = (i & 1) ? p.small2 + (DELTA ? kh : h) : h;
            cp_async4(smem_u32(bv + SC_TOK * SC_COLS + i), p.small + (size_t)(tb + tk) * p.lds + off);
        }
        cp_async_commit();
    };
    const int chunks = (t1 - t0 + SC_TOK - 1) / SC_TOK;
    const float Dh = !DELTA ? p.D[h] : 0.0f;
    load(0, 0);
    for (int ch = 0; ch < chunks; ++ch) {
        if (ch + 1 < chunks) {
            load(ch + 1, (ch + 1) & 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const float* b = sm + (ch & 1) * BUF;
        const float* bv = b + NV * SC_TOK * DP + warp * 4 + (lane >> 3);
        const float* bs = b + NV * SC_TOK * DP + SC_TOK * SC_COLS;
        const int tb = t0 + ch * SC_TOK, n = min(SC_TOK, t1 - tb);
#pragma unroll(DELTA ? 1 : 4)
        for (int tk = 0; tk < n; ++tk) {
            const float4* kp = reinterpret_cast<const float4*>(b + tk * DP) + l8;
            const float4* qp = reinterpret_cast<const float4*>(b + (SC_TOK + tk) * DP) + l8;
            const float v = bv[tk * SC_COLS], s0 = bs[2 * tk], s1 = bs[2 * tk + 1];
            float pk[4] = {}, pq[4] = {};
            if (DELTA) {
                const float4* gp = reinterpret_cast<const float4*>(b + (2 * SC_TOK + tk) * DP) + l8;
                float kr[EPL];
#pragma unroll
                for (int j = 0; j < EPL / 4; ++j) {
                    const float4 kv = kp[8 * j], qv = qp[8 * j], gv = gp[8 * j];
                    const float kk[4] = {kv.x, kv.y, kv.z, kv.w}, qq[4] = {qv.x, qv.y, qv.z, qv.w}, gg[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        kr[4 * j + i] = kk[i];
                        s[4 * j + i] *= gg[i];
                        pk[i] = fmaf(s[4 * j + i], kk[i], pk[i]);
                        pq[i] = fmaf(s[4 * j + i], qq[i], pq[i]);
                    }
                }
                float a = (pk[0] + pk[1]) + (pk[2] + pk[3]), c = (pq[0] + pq[1]) + (pq[2] + pq[3]);
#pragma unroll
                for (int o = 4; o > 0; o >>= 1) {
                    a += __shfl_xor_sync(0xffffffffu, a, o);
                    c += __shfl_xor_sync(0xffffffffu, c, o);
                }
                const float u = s0 * (v - a);
#pragma unroll
                for (int j = 0; j < EPL; ++j) s[j] = fmaf(kr[j], u, s[j]);
                if (l8 == 0 && col < p.vdim) p.o[(size_t)(tb + tk) * p.ldo + (size_t)h * p.vdim + col] = fmaf(s1, u, c);
            } else {
                const float u = s0 * v;
#pragma unroll
                for (int j = 0; j < EPL / 4; ++j) {
                    const float4 kv = kp[8 * j], qv = qp[8 * j];
                    const float kk[4] = {kv.x, kv.y, kv.z, kv.w}, qq[4] = {qv.x, qv.y, qv.z, qv.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        s[4 * j + i] = fmaf(s[4 * j + i], s1, kk[i] * u);
                        pq[i] = fmaf(s[4 * j + i], qq[i], pq[i]);
                    }
                }
                float c = (pq[0] + pq[1]) + (pq[2] + pq[3]);
#pragma unroll
                for (int o = 4; o > 0; o >>= 1) c += __shfl_xor_sync(0xffffffffu, c, o);
                if (l8 == 0 && col < p.vdim) p.o[(size_t)(tb + tk) * p.ldo + (size_t)h * p.vdim + col] = fmaf(Dh, v, c);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < EPL; ++j) {
        const int d = 4 * (l8 + 8 * (j >> 2)) + (j & 3);
        if (col < p.vdim && d < p.dim) S[d] = s[j];
    }
}

template <int EPL, bool DELTA>
int launch_scan_epl(dc_ctx* ctx, const ScanParams& p, int E) {
    const size_t smem = (size_t)2 * SC_TOK * ((DELTA ? 3 : 2) * 8 * EPL + SC_COLS + 2) * 4;
    DC_TRY(dc_kernel_setup(ctx, (const void*)k_state_scan<EPL, DELTA>, (int)smem, "k_state_scan"));
    return dc_launch(ctx, "k_state_scan", k_state_scan<EPL, DELTA>, dim3((p.vdim + SC_COLS - 1) / SC_COLS, p.heads, E), dim3(SC_THREADS), smem, p);
}
template <bool DELTA>
int launch_scan(dc_ctx* ctx, const ScanParams& p, int E) {
    if (p.dim <= 32) return launch_scan_epl<4, DELTA>(ctx, p, E);
    if (p.dim <= 64) return launch_scan_epl<8, DELTA>(ctx, p, E);
    if (p.dim <= 128) return launch_scan_epl<16, DELTA>(ctx, p, E);
    return launch_scan_epl<32, DELTA>(ctx, p, E);
}

// ---------------------------------------------------------------- output norms
// delta: one warp per (token, head): o / rms(o) * w * sigmoid(gate)
template <typename TO>
__global__ void __launch_bounds__(256) k_head_norm_gate(const float* __restrict__ o, int ldo, const float* __restrict__ gate, int ldg,
                                                        const float* __restrict__ w, int heads, int vdim, int T, float eps,
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
        store_as(out + (size_t)t * ldm + (size_t)h * vdim + c, r[c] * inv * w[c] * sigmoid(gate[(size_t)t * ldg + (size_t)h * vdim + c]));
}

// ssd: one CTA per (token, norm group): y silu(z) (unless gated already), over its root mean square, times w
template <typename TO>
__global__ void __launch_bounds__(256) k_gate_group_norm(const float* __restrict__ y, int ldy, const float* __restrict__ z, int ldz,
                                                         const float* __restrict__ w, int n, float eps, TO* __restrict__ out, int ldm) {
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.y, c0 = blockIdx.x * n;
    const float* yr = y + (size_t)t * ldy + c0;
    const float* zr = z ? z + (size_t)t * ldz + c0 : nullptr;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += 256) {
        const float v = zr ? yr[i] * silu(zr[i]) : yr[i];
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += 256) {
        const float v = zr ? yr[i] * silu(zr[i]) : yr[i];
        store_as(out + (size_t)t * ldm + c0 + i, v * inv * w[c0 + i]);
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
        p.act[(size_t)t * p.lda + c] = silu(conv_at(p.proj, p.ldp, p.cr.ring(p.cr.seq_ids[t]), p.cr.C, c, p.cr.taps, p.conv + (size_t)c * p.cr.taps,
                                                    p.off_x + c, t, i, pos) + p.conv_b[c]);
    if (blockIdx.x == 0)
        for (int h = threadIdx.x; h < p.heads; h += 256) {
            const float dt = softplus(p.proj[(size_t)t * p.ldp + p.off_dt + h] + p.dt_bias[h]);
            p.small[(size_t)t * 2 * p.heads + h] = dt;
            p.small[(size_t)t * 2 * p.heads + p.heads + h] = expf(p.neg_a[h] * dt);
        }
}

ConvRef conv_ref(const dc_step& st, const dc_state_ref& sr, int taps, int C) {
    return ConvRef{sr.base, sr.slot_bytes, sr.ring_off, st.seq_ids, st.positions, st.starts, st.E, taps, C};
}

}  // namespace

int dc_launch_ring_update(dc_ctx* ctx, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, int off, int C, int taps) {
    return dc_launch(ctx, "k_ring_update", k_ring_update, dim3((C + 255) / 256, st.E), dim3(256), 0, conv_ref(st, sr, taps, C), proj, ldp, off);
}

int dc_launch_delta_prep(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp,
                         float* act, int lda, float* small, __nv_bfloat16* lowb, int ldl) {
    DeltaPrep p;
    const int V = m.heads * m.vdim, C = m.off_v + V;
    p.cr = conv_ref(st, sr, m.taps, C);
    p.proj = proj, p.ldp = ldp, p.conv = m.conv;
    p.heads = m.heads, p.kv_heads = m.kv_heads, p.dim = m.dim, p.vdim = m.vdim;
    p.off_q = m.off_q, p.off_k = m.off_k, p.off_v = m.off_v, p.off_b = m.off_b, p.off_a = m.off_a;
    p.n_low = m.off_g + m.g_rank - m.off_a;
    p.unit_eps = m.unit_eps, p.q_scale = m.q_scale;
    p.act = act, p.lda = lda, p.small = small, p.lowb = lowb, p.ldl = ldl, p.T = st.T, p.v_items = (V + 127) / 128;
    const long long warps = (long long)st.T * (m.kv_heads + p.v_items + 1);
    DC_TRY(dc_launch(ctx, "k_delta_prep", k_delta_prep, dim3((unsigned)((warps + 7) / 8)), dim3(256), 0, p));
    return dc_launch_ring_update(ctx, st, sr, proj, ldp, 0, C, m.taps);
}

int dc_launch_delta_scan(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* act, int lda,
                         const float* small, float* decay, int ldd, const float* raw_g, int ldg, float eps, float* o,
                         float* mix, __nv_bfloat16* mixb, int ldm) {
    const int nd = m.heads * m.dim;
    DC_TRY(dc_launch(ctx, "k_delta_decay", k_delta_decay, dim3((nd + 255) / 256, st.T), dim3(256), 0, decay, ldd, m.neg_a, m.dt_bias, m.dim, nd));
    ScanParams p = {};
    p.k = act + m.off_k, p.q = act + m.off_q, p.v = act + m.off_v, p.g = decay;
    p.ld = lda, p.ldg = ldd, p.heads = m.heads, p.per = m.heads / m.kv_heads, p.dim = m.dim, p.vdim = m.vdim;
    p.small = small, p.lds = m.heads + m.kv_heads, p.small2 = m.heads;
    p.o = o, p.ldo = lda;
    p.base = sr.base, p.slot_bytes = sr.slot_bytes, p.state_off = sr.state_off;
    p.seq_ids = st.seq_ids, p.positions = st.positions, p.starts = st.starts;
    p.vec = m.dim % 4 == 0 && lda % 4 == 0 && ldd % 4 == 0;
    DC_TRY(launch_scan<true>(ctx, p, st.E));
    const unsigned blocks = (unsigned)(((long long)st.T * m.heads + 7) / 8);
    if (mixb)
        return dc_launch(ctx, "k_head_norm_gate", k_head_norm_gate<__nv_bfloat16>, dim3(blocks), dim3(256), 0, o, lda, raw_g, ldg, m.norm, m.heads,
                         m.vdim, st.T, eps, mixb, ldm);
    return dc_launch(ctx, "k_head_norm_gate", k_head_norm_gate<float>, dim3(blocks), dim3(256), 0, o, lda, raw_g, ldg, m.norm, m.heads, m.vdim, st.T,
                     eps, mix, ldm);
}

int dc_launch_ssd(dc_ctx* ctx, const dc_ssd_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float* act,
                  int lda, float* small, float* y, float eps, float* mix, __nv_bfloat16* mixb, int ldm) {
    const int inner = m.heads * m.vdim, GN = m.groups * m.state, C = inner + 2 * GN;
    SsdPrep s = {conv_ref(st, sr, m.taps, C), proj, ldp, m.off_x, m.off_dt, m.heads, st.T, m.conv, m.conv_b, m.dt_bias, m.neg_a, act, lda, small};
    DC_TRY(dc_launch(ctx, "k_ssd_prep", k_ssd_prep, dim3((C + 255) / 256, st.T), dim3(256), 0, s));
    DC_TRY(dc_launch_ring_update(ctx, st, sr, proj, ldp, m.off_x, C, m.taps));
    ScanParams p = {};
    p.k = act + inner, p.q = act + inner + GN, p.v = act;
    p.ld = lda, p.heads = m.heads, p.per = m.heads / m.groups, p.dim = m.state, p.vdim = m.vdim;
    p.small = small, p.lds = 2 * m.heads, p.small2 = m.heads, p.D = m.D;
    p.o = y, p.ldo = lda;
    p.base = sr.base, p.slot_bytes = sr.slot_bytes, p.state_off = sr.state_off;
    p.seq_ids = st.seq_ids, p.positions = st.positions, p.starts = st.starts;
    p.vec = m.state % 4 == 0 && lda % 4 == 0 && inner % 4 == 0;
    DC_TRY(launch_scan<false>(ctx, p, st.E));
    const int n = inner / m.norm_groups;
    if (mixb)
        return dc_launch(ctx, "k_gate_group_norm", k_gate_group_norm<__nv_bfloat16>, dim3(m.norm_groups, st.T), dim3(256), 0, y, lda, proj + m.off_z, ldp,
                         m.norm, n, eps, mixb, ldm);
    return dc_launch(ctx, "k_gate_group_norm", k_gate_group_norm<float>, dim3(m.norm_groups, st.T), dim3(256), 0, y, lda, proj + m.off_z, ldp, m.norm, n,
                     eps, mix, ldm);
}
