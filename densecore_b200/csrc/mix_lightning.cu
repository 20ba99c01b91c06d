// Linear attention with one constant decay per head (S <- decay S + k v^T, o = S^T q) for entries of bf16 models: chunks of
// 64 tokens on the tensor cores, the state in f32.
//
// With a chunk's tokens t = 0 .. n - 1, the state S0 ahead of it and the head's decay a:
//   o_t = a^(t + 1) S0^T q_t + sum_{i <= t} a^(t - i) (q_t . k_i) v_i,     S = a^n S0 + sum_i a^(n - 1 - i) k_i v_i^T
// Three kernels: k_lightning_sums (the last sum of every chunk), k_lightning_carry (the states ahead of the chunks, one pass
// over them), k_lightning_out (the answers).  q, k and v are bf16; what is f32 in these equations enters the bf16 products
// as three bf16 terms that together hold its 24 bits, so nothing of it is rounded.
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

constexpr int CT = 64;              // tokens of a chunk
constexpr int TE = 64;              // value columns of a tile
constexpr int LDT = 64 + 8;         // pitch of a 64-wide bf16 tile

struct ChunkParams {
    const __nv_bfloat16* act;
    int ld, off_q, off_k, off_v, heads, dim, vdim;
    const float* decay;
    float* state;                   // [chunk][head][vdim][dim]
    uint8_t* base;
    size_t slot_bytes, state_off;
    const int32_t *seq_ids, *positions, *starts;
    int E, vec;                     // vec: rows allow 16-byte copies
    float* y;
    int ldy;
};

// CT rows x cols (a multiple of eight) of a bf16 matrix into shared memory by 128 threads, eight a row; what lies beyond n
// rows or `valid` columns is zero
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, int ldd, const __nv_bfloat16* src, int lds, int n, int valid, int cols, bool vec) {
    if (vec) {
        const int r0 = threadIdx.x >> 3, c0 = 8 * (threadIdx.x & 7);
        const uint32_t to = smem_u32(dst + r0 * ldd + c0);
        const __nv_bfloat16* from = src + (size_t)r0 * lds + c0;
        for (int c = 0; c0 + c < cols; c += 64)
#pragma unroll
            for (int i = 0; i < CT / 16; ++i) {
                const bool ok = r0 + 16 * i < n && c0 + c < valid;
                cp_async16z(to + 2 * (16 * i * ldd + c), ok ? from + (size_t)(16 * i) * lds + c : src, ok);
            }
    } else {
        for (int i = threadIdx.x; i < CT * cols; i += blockDim.x) {
            const int r = i / cols, c = i - r * cols;
            dst[r * ldd + c] = r < n && c < valid ? src[(size_t)r * lds + c] : __float2bfloat16_rn(0.0f);
        }
    }
}

// x = t[0] + t[1] + t[2] (pairs of values), each term bf16
__device__ __forceinline__ void split3(float x0, float x1, uint32_t (&t)[3]) {
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        t[i] = pack_bf2(x0, x1);
        x0 -= __uint_as_float(t[i] << 16);
        x1 -= __uint_as_float(t[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ float bf_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float bf_hi(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

// One CTA per (chunk, head, tile of 64 value columns x 64 key channels), sixteen value columns a warp.
__global__ void __launch_bounds__(128) k_lightning_sums(const ChunkParams p) {
    __shared__ __align__(16) __nv_bfloat16 sK[CT * LDT], sV[CT * LDT];
    __shared__ float sw[CT];
    pdl_launch_dependents();
    pdl_wait();
    const BlockRef br = block_at<CT>(p.starts, p.E, blockIdx.x);
    if (br.n <= 0) return;
    const int h = blockIdx.y, dt = (p.dim + 63) / 64, e0 = (blockIdx.z / dt) * TE, d0 = (blockIdx.z % dt) * 64;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3, mi = lane >> 3, r8 = lane & 7;
    const __nv_bfloat16* row = p.act + (size_t)br.t0 * p.ld;
    load_tile(sK, LDT, row + p.off_k + h * p.dim + d0, p.ld, br.n, p.dim - d0, 64, p.vec);
    load_tile(sV, LDT, row + p.off_v + h * p.vdim + e0, p.ld, br.n, p.vdim - e0, 64, p.vec);
    cp_async_commit();
    if (tid < CT) sw[tid] = tid < br.n ? powf(p.decay[h], (float)(br.n - 1 - tid)) : 0.0f;
    cp_async_wait<0>();
    __syncthreads();
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
#pragma unroll
    for (int ks = 0; ks < CT / 16; ++ks) {
        if (16 * ks >= br.n) break;
        uint32_t v[4], a[3][4];
        ldsm_x4_t(smem_u32(sV + (16 * ks + (mi >> 1) * 8 + r8) * LDT + 16 * warp + (mi & 1) * 8), v);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 w = *reinterpret_cast<const float2*>(sw + 16 * ks + (i >> 1) * 8 + 2 * q);
            uint32_t t[3];
            split3(bf_lo(v[i]) * w.x, bf_hi(v[i]) * w.y, t);
            a[0][i] = t[0], a[1][i] = t[1], a[2][i] = t[2];
        }
        uint32_t b[4][4];
#pragma unroll
        for (int np = 0; np < 4; ++np) ldsm_x4_t(smem_u32(sK + (16 * ks + (mi & 1) * 8 + r8) * LDT + 16 * np + (mi >> 1) * 8), b[np]);
#pragma unroll
        for (int i = 2; i >= 0; --i)             // products of one term are independent of each other
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                mma_bf16(acc[2 * np], a[i], b[np][0], b[np][1]);
                mma_bf16(acc[2 * np + 1], a[i], b[np][2], b[np][3]);
            }
    }
    float* out = p.state + ((size_t)blockIdx.x * p.heads + h) * p.vdim * p.dim;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int e = e0 + 16 * warp + g + 8 * half, d = d0 + 8 * nt + 2 * q;
            if (e >= p.vdim) continue;
            float* o = out + (size_t)e * p.dim + d;
            if (d + 1 < p.dim && !(p.dim & 1)) *reinterpret_cast<float2*>(o) = make_float2(acc[nt][2 * half], acc[nt][2 * half + 1]);
            else {
                if (d < p.dim) o[0] = acc[nt][2 * half];
                if (d + 1 < p.dim) o[1] = acc[nt][2 * half + 1];
            }
        }
}

// The chunks' sums become the states ahead of the chunks; the sequence's slot gets the state after the last.  One thread
// per W elements of a head's state.
template <int W>
__global__ void __launch_bounds__(256) k_lightning_carry(const ChunkParams p) {
    constexpr int AHEAD = 8;
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, e = blockIdx.z, size = p.vdim * p.dim, i0 = (blockIdx.x * 256 + threadIdx.x) * W;
    const int t0 = p.starts[e], n = p.starts[e + 1] - t0, chunks = (n + CT - 1) / CT;
    if (n <= 0 || i0 >= size) return;
    float* slot = reinterpret_cast<float*>(p.base + (size_t)p.seq_ids[t0] * p.slot_bytes + p.state_off) + (size_t)h * size + i0;
    float* u = p.state + ((size_t)block_base<CT>(p.starts, e) * p.heads + h) * size + i0;
    const size_t step = (size_t)p.heads * size;
    const float whole = powf(p.decay[h], (float)CT), rest = powf(p.decay[h], (float)(n - (chunks - 1) * CT));
    float s[W];
    auto get = [](const float* from, float (&v)[W]) {
        if (W == 4) {
            const float4 f = *reinterpret_cast<const float4*>(from);
            v[0] = f.x, v[1 % W] = f.y, v[2 % W] = f.z, v[3 % W] = f.w;
        } else {
            v[0] = *from;
        }
    };
    auto put = [](float* to, const float (&v)[W]) {
        if (W == 4) *reinterpret_cast<float4*>(to) = make_float4(v[0], v[1 % W], v[2 % W], v[3 % W]);
        else *to = v[0];
    };
    if (p.positions[t0] == 0) {
#pragma unroll
        for (int k = 0; k < W; ++k) s[k] = 0.0f;
    } else {
        get(slot, s);
    }
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float f[AHEAD][W];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) get(u + (size_t)min(c0 + j, chunks - 1) * step, f[j]);
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c0 + j >= chunks) break;
            put(u + (size_t)(c0 + j) * step, s);
            const float a = c0 + j == chunks - 1 ? rest : whole;
#pragma unroll
            for (int k = 0; k < W; ++k) s[k] = fmaf(s[k], a, f[j][k]);
        }
    }
    put(slot, s);
}

// One CTA per (chunk, head, tile of 64 value columns).  Against the state a warp has sixteen value columns and all queries,
// so that a column of the state is taken apart once; inside the chunk it has sixteen queries.  Shared memory is used twice:
// keys and values take the place of the state's columns, the answers from the state that of the queries.
struct OutSmem {
    int ldq, lds, first, second;                        // pitches; bytes of the two regions
    __host__ __device__ explicit OutSmem(int dim) {
        const int dp = (dim + 15) & ~15;
        ldq = dp + 8, lds = dp + 8;
        const int queries = CT * ldq * 2, answers = CT * (TE + 4) * 4, state = TE * lds * 4, tokens = CT * (ldq + LDT) * 2;
        first = queries > answers ? queries : answers;
        second = state > tokens ? state : tokens;
    }
};

__global__ void __launch_bounds__(128, 4) k_lightning_out(const ChunkParams p) {
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ float spow[CT + 1];
    const OutSmem L(p.dim);
    const int dp = (p.dim + 15) & ~15, LDQ = L.ldq, LDS = L.lds;
    constexpr int LDO = TE + 4;
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem);     // [CT][LDQ]
    float* sO = reinterpret_cast<float*>(smem);                     // [CT][LDO]
    float* sS = reinterpret_cast<float*>(smem + L.first);           // [TE][LDS]: columns of the state
    __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(smem + L.first);    // [CT][LDQ]
    __nv_bfloat16* sV = sK + CT * LDQ;                              // [CT][LDT]
    pdl_launch_dependents();
    pdl_wait();
    const BlockRef br = block_at<CT>(p.starts, p.E, blockIdx.x);
    if (br.n <= 0) return;
    const int h = blockIdx.y, e0 = blockIdx.z * TE, ne = min(TE, p.vdim - e0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3, mi = lane >> 3, r8 = lane & 7;
    const __nv_bfloat16* row = p.act + (size_t)br.t0 * p.ld;
    const float* S = p.state + (((size_t)blockIdx.x * p.heads + h) * p.vdim + e0) * p.dim;
    load_tile(sQ, LDQ, row + p.off_q + h * p.dim, p.ld, br.n, p.dim, dp, p.vec);
    if (p.dim % 4 == 0) {
        const int r0 = tid >> 3, c0 = 4 * (tid & 7);
        for (int c = c0; c < dp; c += 32)
#pragma unroll
            for (int i = 0; i < TE / 16; ++i) {
                const int r = r0 + 16 * i;
                const bool ok = r < ne && c < p.dim;
                cp_async16z(smem_u32(sS + r * LDS + c), ok ? S + r * p.dim + c : S, ok);
            }
    } else {
        for (int i = tid; i < TE * dp; i += 128) {
            const int r = i / dp, c = i - r * dp;
            sS[r * LDS + c] = r < ne && c < p.dim ? S[(size_t)r * p.dim + c] : 0.0f;
        }
    }
    cp_async_commit();
    if (tid <= CT) spow[tid] = powf(p.decay[h], (float)tid);
    cp_async_wait<0>();
    __syncthreads();
    // ---- S0^T q for the columns 16 warp .. + 15, all queries
    float acc[4][2][4];
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j) acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.0f;
    for (int kk = 0; kk < dp; kk += 16) {
        uint32_t b[2][2][3], a[4][4];
#pragma unroll
        for (int m = 0; m < 4; ++m) ldsm_x4(smem_u32(sQ + (16 * m + (mi & 1) * 8 + r8) * LDQ + (mi >> 1) * 8 + kk), a[m]);
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float2 f = *reinterpret_cast<const float2*>(sS + (16 * warp + 8 * j + g) * LDS + kk + 8 * i + 2 * q);
                split3(f.x, f.y, b[j][i]);
            }
#pragma unroll
        for (int i = 2; i >= 0; --i)             // products of one term are independent of each other
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                mma_bf16(acc[m][0], a[m], b[0][0][i], b[0][1][i]);
                mma_bf16(acc[m][1], a[m], b[1][0][i], b[1][1][i]);
            }
    }
    __syncthreads();
    load_tile(sK, LDQ, row + p.off_k + h * p.dim, p.ld, br.n, p.dim, dp, p.vec);
    load_tile(sV, LDT, row + p.off_v + h * p.vdim + e0, p.ld, br.n, ne, TE, p.vec);
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
    // ---- the chunk's own tokens: weights a^(t - i) (q_t . k_i) of the warp's queries, then the values
    float s[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
    const uint32_t qa = smem_u32(sQ + (16 * warp + (mi & 1) * 8 + r8) * LDQ + (mi >> 1) * 8);
    const uint32_t ka = smem_u32(sK + ((mi >> 1) * 8 + r8) * LDQ + (mi & 1) * 8);
    for (int kk = 0; kk < dp; kk += 16) {
        uint32_t a[4];
        ldsm_x4(qa + 2 * kk, a);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
            if (np > warp) break;                                   // keys after every query of the warp
            uint32_t b[4];
            ldsm_x4(ka + 2 * (16 * np * LDQ + kk), b);
            mma_bf16(s[2 * np], a, b[0], b[1]);
            mma_bf16(s[2 * np + 1], a, b[2], b[3]);
        }
    }
    __syncthreads();             // every warp is done with the queries
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int t = 16 * m + g + 8 * i;
                *reinterpret_cast<float2*>(sO + t * LDO + 16 * warp + 8 * j + 2 * q) = make_float2(acc[m][j][2 * i] * spow[t + 1], acc[m][j][2 * i + 1] * spow[t + 1]);
            }
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int back = 16 * warp + g + (j >> 1) * 8 - (8 * nt + 2 * q + (j & 1));
            s[nt][j] = back >= 0 ? s[nt][j] * spow[back] : 0.0f;
        }
    float o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
#pragma unroll
    for (int ks = 0; ks < CT / 16; ++ks) {
        if (ks > warp) break;
        uint32_t pa[3][4], b[4][4];
#pragma unroll
        for (int np = 0; np < 4; ++np) ldsm_x4_t(smem_u32(sV + (16 * ks + (mi & 1) * 8 + r8) * LDT + 16 * np + (mi >> 1) * 8), b[np]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            uint32_t t[3];
            split3(s[2 * ks + (i >> 1)][2 * (i & 1)], s[2 * ks + (i >> 1)][2 * (i & 1) + 1], t);
            pa[0][i] = t[0], pa[1][i] = t[1], pa[2][i] = t[2];
        }
#pragma unroll
        for (int i = 2; i >= 0; --i)
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                mma_bf16(o[2 * np], pa[i], b[np][0], b[np][1]);
                mma_bf16(o[2 * np + 1], pa[i], b[np][2], b[np][3]);
            }
    }
    __syncthreads();
    const bool even = !(p.vdim & 1);
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int t = 16 * warp + g + 8 * i, c = 8 * nt + 2 * q;
            if (t >= br.n || c >= ne) continue;
            const float2 f = *reinterpret_cast<const float2*>(sO + t * LDO + c);
            float* y = p.y + (size_t)(br.t0 + t) * p.ldy + (size_t)h * p.vdim + e0 + c;
            if (even) {
                *reinterpret_cast<float2*>(y) = make_float2(o[nt][2 * i] + f.x, o[nt][2 * i + 1] + f.y);
            } else {
                y[0] = o[nt][2 * i] + f.x;
                if (c + 1 < ne) y[1] = o[nt][2 * i + 1] + f.y;
            }
        }
}

}  // namespace

int dc_lightning_chunks(int T, int E) { return T / CT + E; }

int dc_launch_lightning_chunks(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const dc_state_ref& sr, const __nv_bfloat16* act,
                               int lda, float* chunk_state, float* y, int ldy) {
    ChunkParams p = {act, lda, m.off_q, m.off_k, m.off_v, m.heads, m.dim, m.vdim, m.decay, chunk_state, sr.base, sr.slot_bytes, sr.state_off, st.seq_ids,
                     st.positions, st.starts, st.E, m.dim % 8 == 0 && m.vdim % 8 == 0 && lda % 8 == 0, y, ldy};
    const int nc = dc_lightning_chunks(st.T, st.E), size = m.dim * m.vdim;
    DC_TRY(dc_launch(ctx, "k_lightning_sums", k_lightning_sums, dim3(nc, m.heads, ((m.dim + 63) / 64) * ((m.vdim + TE - 1) / TE)), dim3(128), 0, p));
    if (size % 4 == 0) DC_TRY(dc_launch(ctx, "k_lightning_carry", k_lightning_carry<4>, dim3((size / 4 + 255) / 256, m.heads, st.E), dim3(256), 0, p));
    else DC_TRY(dc_launch(ctx, "k_lightning_carry", k_lightning_carry<1>, dim3((size + 255) / 256, m.heads, st.E), dim3(256), 0, p));
    const OutSmem L(m.dim);
    const int bytes = L.first + L.second;
    DC_TRY(dc_kernel_setup(ctx, (const void*)k_lightning_out, bytes, "k_lightning_out"));
    return dc_launch(ctx, "k_lightning_out", k_lightning_out, dim3(nc, m.heads, (m.vdim + TE - 1) / TE), dim3(128), (size_t)bytes, p);
}
