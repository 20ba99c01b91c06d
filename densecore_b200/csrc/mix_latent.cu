// Attention over a compressed key/value latent (one row per token: the normed latent c and a rotated key part that
// all heads share), with an optional sliding window and an optional gate per head on the output.
//
// Decode-sized steps and f32 models use the absorbed form: a head's unrotated query is taken through its W_uk once
// (q' = W_uk^T q), scores are q' . c + q_rot . k_rot, the softmax-weighted sum of latents goes through W_uv at the
// end; the cache row is the key and the value of every head.  Prompt-sized steps of bf16 models gather the visible
// rows of each entry, expand them to per-head keys and values with one tensor-core product, and run a tiled
// attention over them.  Scores and softmax are f32 in both.
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

// ---------------------------------------------------------------- rotation, latent norm, cache write
struct PrepParams {
    float* proj;             // queries are turned in place
    int ldp, off_q, off_kv, heads, dim, rot, rank, max_pos;
    const float* norm;       // null: another layer writes the cache
    const float* cos_sin;
    float eps;
    const int32_t *seq_ids, *positions;
    CacheRef c;
};

template <typename TC>
__global__ void __launch_bounds__(256) k_latent_prep(const PrepParams p) {
    __shared__ float red[33];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int pos = min(max(p.positions[t], 0), p.max_pos - 1);
    const float* cs = p.cos_sin + (size_t)pos * p.rot;
    float* row = p.proj + (size_t)t * p.ldp;
    const int half = p.rot / 2;
    if (p.norm) {
        const float* src = row + p.off_kv;
        TC* dst = reinterpret_cast<TC*>(p.c.arena) + p.c.at(p.seq_ids[t], pos);
        float v[4], ss = 0.0f;       // kv_rank <= 1024
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = threadIdx.x + 256 * j;
            v[j] = i < p.rank ? src[i] : 0.0f;
            ss = fmaf(v[j], v[j], ss);
        }
        const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.rank + p.eps);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = threadIdx.x + 256 * j;
            if (i < p.rank) store_as(dst + i, v[j] * inv * p.norm[i]);
        }
        for (int i = threadIdx.x; i < half; i += 256) {
            const float u = src[p.rank + 2 * i], w = src[p.rank + 2 * i + 1], c = cs[2 * i], s = cs[2 * i + 1];
            store_as(dst + p.rank + 2 * i, u * c - w * s);
            store_as(dst + p.rank + 2 * i + 1, w * c + u * s);
        }
        for (int i = p.rank + p.rot + threadIdx.x; i < p.c.row; i += 256) store_as(dst + i, 0.0f);
    }
    for (int i = threadIdx.x; i < p.heads * half; i += 256) {
        const int h = i / half, j = i - h * half;
        float* q = row + p.off_q + h * (p.dim + p.rot) + p.dim + 2 * j;
        const float u = q[0], v = q[1], c = cs[2 * j], s = cs[2 * j + 1];
        q[0] = u * c - v * s;
        q[1] = v * c + u * s;
    }
}

// ---------------------------------------------------------------- absorbed form
// qa[t][h][r] = sum_d q[t][h][d] * uk[h][d][r].  CTA: one head, 128 columns, up to NT tokens; warp w takes the rows
// w, w + 8, ..., a lane four columns.  The first rows are fetched ahead of the dependency wait.
template <int NT>
__global__ void __launch_bounds__(256) k_latent_absorb(const float* __restrict__ proj, int ldp, int off_q, int heads, int dim, int rot,
                                                       const __nv_bfloat16* __restrict__ uk, int ldw, int dim_p, int rank, int T,
                                                       float* __restrict__ qa, int ldq) {
    constexpr int AHEAD = 16;
    extern __shared__ float sq[];    // [NT][dim]
    __shared__ float red[8][NT][128];
    pdl_launch_dependents();
    const int h = blockIdx.x, tb = blockIdx.z * NT, nt = min(NT, T - tb), r0 = blockIdx.y * 128, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = r0 + 4 * lane;
    const bool in = r < ldw;         // rows are padded with zeros to ldw columns
    const __nv_bfloat16* w = uk + (size_t)h * dim_p * ldw + r;
    uint2 ahead[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
        const int d = warp + 8 * i;
        ahead[i] = in && d < dim ? __ldg(reinterpret_cast<const uint2*>(w + (size_t)d * ldw)) : make_uint2(0, 0);
    }
    pdl_wait();
    for (int i = threadIdx.x; i < NT * dim; i += 256) {
        const int t = i / dim, d = i - t * dim;
        sq[i] = t < nt ? proj[(size_t)(tb + t) * ldp + off_q + h * (dim + rot) + d] : 0.0f;
    }
    __syncthreads();
    float a[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t) a[t][0] = a[t][1] = a[t][2] = a[t][3] = 0.0f;
    auto add = [&](uint2 v, int d) {
        const float f[4] = {__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u)};
#pragma unroll
        for (int t = 0; t < NT; ++t)
#pragma unroll
            for (int i = 0; i < 4; ++i) a[t][i] = fmaf(sq[t * dim + d], f[i], a[t][i]);
    };
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (warp + 8 * i < dim) add(ahead[i], warp + 8 * i);
    for (int d = warp + 8 * AHEAD; d < dim; d += 8) add(in ? __ldg(reinterpret_cast<const uint2*>(w + (size_t)d * ldw)) : make_uint2(0, 0), d);
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int i = 0; i < 4; ++i) red[warp][t][4 * lane + i] = a[t][i];
    __syncthreads();
    for (int i = threadIdx.x; i < nt * 128; i += 256) {
        const int t = i >> 7, c = i & 127;
        float v = 0.0f;
#pragma unroll
        for (int k = 0; k < 8; ++k) v += red[k][t][c];
        if (r0 + c < rank) qa[((size_t)(tb + t) * heads + h) * ldq + r0 + c] = v;
    }
}

struct AbsorbedParams {
    const float* qa;         // [T][heads][ldq]
    int ldq;
    const float* proj;
    int ldp, off_q, heads, dim, rot, rank, window, splits;
    float scale;
    const int32_t *seq_ids, *positions;
    CacheRef c;
    float *part, *part_ml;   // [T][heads][splits][rank], [T][heads][splits][2]
};

constexpr int AB_KEYS = 32, AB_HEADS = 4;

// One CTA per (key split, group of four heads, token): a warp is a head.  Scores: a lane is a key; sums: a lane owns
// the 16-byte chunks lane, lane + 32, ... of the latent (RP of them).
template <typename TC, int RP>
__global__ void __launch_bounds__(AB_HEADS * 32) k_latent_absorbed(const AbsorbedParams p) {
    constexpr int EPC = 16 / sizeof(TC);      // elements of a 16-byte chunk
    extern __shared__ __align__(16) uint8_t sm[];
    float* sq = reinterpret_cast<float*>(sm);                              // [AB_HEADS][row]
    const int row = p.c.row, ldk = row + EPC;
    TC* sk = reinterpret_cast<TC*>(sm + (size_t)AB_HEADS * row * 4);       // [AB_KEYS][ldk]
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.x, h0 = blockIdx.y * AB_HEADS, t = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = h0 + warp, pos = p.positions[t], seq = p.seq_ids[t];
    const bool live = h < p.heads;
    {                            // a warp's own query: the absorbed part, then the rotated part, zeros in the padding
        const float *qa = p.qa + ((size_t)t * p.heads + min(h, p.heads - 1)) * p.ldq;
        const float* qr = p.proj + (size_t)t * p.ldp + p.off_q + min(h, p.heads - 1) * (p.dim + p.rot) + p.dim;
#pragma unroll 8
        for (int c = lane; c < p.rank; c += 32) sq[warp * row + c] = qa[c] * p.scale;
        for (int c = p.rank + lane; c < row; c += 32) sq[warp * row + c] = c < p.rank + p.rot ? qr[c - p.rank] * p.scale : 0.0f;
    }
    const int first = first_key(pos, p.window), nk = pos - first + 1;
    const int per = ((nk + p.splits - 1) / p.splits + AB_KEYS - 1) / AB_KEYS * AB_KEYS;
    const int kb = first + s * per, ke = min(first + nk, kb + per);
    float m = -INFINITY, l = 0.0f, acc[RP][EPC];
#pragma unroll
    for (int j = 0; j < RP; ++j)
#pragma unroll
        for (int i = 0; i < EPC; ++i) acc[j][i] = 0.0f;
    const int chunks = row / EPC;
    for (int k0 = kb; k0 < ke; k0 += AB_KEYS) {
        __syncthreads();
        const TC* src[AB_KEYS / AB_HEADS];                  // a warp's keys: all rows asked for before any arrives
#pragma unroll
        for (int i = 0; i < AB_KEYS / AB_HEADS; ++i)
            src[i] = reinterpret_cast<const TC*>(p.c.arena) + p.c.at(seq, min(k0 + warp * (AB_KEYS / AB_HEADS) + i, ke - 1));
        for (int c = lane; c < chunks; c += 32)
#pragma unroll
            for (int i = 0; i < AB_KEYS / AB_HEADS; ++i)
                cp_async16z(smem_u32(sk + (warp * (AB_KEYS / AB_HEADS) + i) * ldk + c * EPC), src[i] + c * EPC, true);
        cp_async_commit();
        cp_async_wait<0>();
        __syncthreads();
        if (!live) continue;
        float part[EPC] = {};
        const float* q = sq + warp * row;
#pragma unroll 8
        for (int c = 0; c < chunks; ++c) {
            float f[EPC];
            unpack16(*reinterpret_cast<const uint4*>(sk + lane * ldk + c * EPC), f, TC());
#pragma unroll
            for (int i = 0; i < EPC; ++i) part[i] = fmaf(f[i], q[c * EPC + i], part[i]);
        }
        float sc = 0.0f;
#pragma unroll
        for (int i = 0; i < EPC; ++i) sc += part[i];
        if (k0 + lane >= ke) sc = -INFINITY;
        float mx = sc;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float mn = fmaxf(m, mx), corr = expf(m - mn), pr = expf(sc - mn);
        m = mn;
        l = l * corr + warp_sum(pr);
#pragma unroll
        for (int j = 0; j < RP; ++j)
#pragma unroll
            for (int i = 0; i < EPC; ++i) acc[j][i] *= corr;
#pragma unroll 8
        for (int kk = 0; kk < AB_KEYS; ++kk) {
            const float w = __shfl_sync(0xffffffffu, pr, kk);
#pragma unroll
            for (int j = 0; j < RP; ++j) {
                const int c = lane + 32 * j;
                float f[EPC];
                unpack16(*reinterpret_cast<const uint4*>(sk + kk * ldk + min(c, chunks - 1) * EPC), f, TC());   // beyond the latent: never stored
#pragma unroll
                for (int i = 0; i < EPC; ++i) acc[j][i] = fmaf(w, f[i], acc[j][i]);
            }
        }
    }
    if (!live) return;
    const size_t o = ((size_t)t * p.heads + h) * p.splits + s;
    if (lane == 0) {
        p.part_ml[2 * o] = m;
        p.part_ml[2 * o + 1] = l;
    }
#pragma unroll
    for (int j = 0; j < RP; ++j)
#pragma unroll
        for (int i = 0; i < EPC; ++i) {
            const int r = EPC * (lane + 32 * j) + i;
            if (r < p.rank) p.part[o * p.rank + r] = acc[j][i];
        }
}

// The same on the tensor cores for bf16 caches: sixteen heads are the rows of the products.  One CTA per (key split, sixteen
// heads, token), eight warps: a warp scores eight of a tile's 64 keys for all heads, then turns two heads' scores into
// weights, then sums NV groups of eight latent columns for all heads.  The queries are rounded to bf16, as the weights are.
constexpr int HD_KEYS = 64, HD_WARPS = 8;

template <int NV>
__global__ void __launch_bounds__(HD_WARPS * 32) k_latent_heads(const AbsorbedParams p) {
    extern __shared__ __align__(16) uint8_t sm[];
    const int row = p.c.row, dk = (row + 15) & ~15, ldk = (dk + 63) / 64 * 64 + 8;
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(sm);          // [16][ldk]
    __nv_bfloat16* sk = sq + 16 * ldk;                                 // [HD_KEYS][ldk]
    __shared__ __align__(16) __nv_bfloat16 sp[16][HD_KEYS + 8];
    __shared__ float ss[16][HD_KEYS + 1], s_corr[16];
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.x, h0 = blockIdx.y * 16, t = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pos = p.positions[t], seq = p.seq_ids[t], first = first_key(pos, p.window), nk = pos - first + 1;
    const int per = ((nk + p.splits - 1) / p.splits + 15) / 16 * 16, kb = first + s * per, ke = min(first + nk, kb + per);
    const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.c.arena);
    auto load = [&](int k0) {            // a warp's keys: all rows asked for before any arrives; zeros beyond the split
        const __nv_bfloat16* src[HD_KEYS / HD_WARPS];
#pragma unroll
        for (int i = 0; i < HD_KEYS / HD_WARPS; ++i) src[i] = cache + p.c.at(seq, max(first, min(k0 + warp * (HD_KEYS / HD_WARPS) + i, ke - 1)));
        for (int c = lane; c < dk / 8; c += 32)
#pragma unroll
            for (int i = 0; i < HD_KEYS / HD_WARPS; ++i) {
                const int key = warp * (HD_KEYS / HD_WARPS) + i;
                const bool in = k0 + key < ke && 8 * c < row;
                cp_async16z(smem_u32(sk + key * ldk + 8 * c), in ? src[i] + 8 * c : cache, in);
            }
        cp_async_commit();
    };
    if (kb < ke) load(kb);
    // a warp's two heads: the absorbed part, all loads in flight, then the rotated part, zeros in the padding
    {
        const float *qa[2], *qr[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int h = min(h0 + 2 * warp + r, p.heads - 1);
            qa[r] = p.qa + ((size_t)t * p.heads + h) * p.ldq;
            qr[r] = p.proj + (size_t)t * p.ldp + p.off_q + h * (p.dim + p.rot) + p.dim - p.rank;
        }
        const int whole = p.rank & ~3;
        float4 v[2][NV / 2];             // 64 NV columns at most
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int j = 0; j < NV / 2; ++j) {
                const int c = 4 * lane + 128 * j;
                v[r][j] = c < whole ? *reinterpret_cast<const float4*>(qa[r] + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        for (int c = whole + lane; c < dk; c += 32)
#pragma unroll
            for (int r = 0; r < 2; ++r)
                sq[(2 * warp + r) * ldk + c] = __float2bfloat16_rn((c < p.rank ? qa[r][c] : c < p.rank + p.rot ? qr[r][c] : 0.0f) * p.scale);
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int j = 0; j < NV / 2; ++j) {
                const int c = 4 * lane + 128 * j;
                if (c < whole)
                    *reinterpret_cast<uint2*>(sq + (2 * warp + r) * ldk + c) = make_uint2(pack_bf2(v[r][j].x * p.scale, v[r][j].y * p.scale),
                                                                                          pack_bf2(v[r][j].z * p.scale, v[r][j].w * p.scale));
            }
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};          // of heads 2 warp, 2 warp + 1
    float acc[NV][4];
#pragma unroll
    for (int i = 0; i < NV; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    const int mi = lane >> 3, r8 = lane & 7, g = lane >> 2, q = lane & 3;
    for (int k0 = kb; k0 < ke; k0 += HD_KEYS) {
        cp_async_wait<0>();
        __syncthreads();
        float sc[2][4] = {};
        const uint32_t qa = smem_u32(sq + ((mi & 1) * 8 + r8) * ldk + (mi >> 1) * 8), ka = smem_u32(sk + (8 * warp + r8) * ldk + mi * 8);
#pragma unroll 4
        for (int kk = 0; kk < dk; kk += 32) {          // a row of keys is padded to whole groups of 32 columns
            uint32_t a[4], b[4];
            ldsm_x4(ka + 2 * kk, b);
            ldsm_x4(qa + 2 * kk, a);
            mma_bf16(sc[0], a, b[0], b[1]);
            if (kk + 16 < dk) {
                ldsm_x4(qa + 2 * (kk + 16), a);
                mma_bf16(sc[1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) ss[g + 8 * (i >> 1)][8 * warp + 2 * q + (i & 1)] = sc[0][i] + sc[1][i];
        __syncthreads();
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int h = 2 * warp + r;
            float v[2];
#pragma unroll
            for (int j = 0; j < 2; ++j) v[j] = k0 + lane + 32 * j < ke ? ss[h][lane + 32 * j] : -INFINITY;
            float mx = fmaxf(v[0], v[1]);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m[r], mx), corr = expf(m[r] - mn), w0 = expf(v[0] - mn), w1 = expf(v[1] - mn);
            m[r] = mn;
            l[r] = l[r] * corr + warp_sum(w0 + w1);
            sp[h][lane] = __float2bfloat16_rn(w0), sp[h][lane + 32] = __float2bfloat16_rn(w1);
            if (lane == 0) s_corr[h] = corr;
        }
        __syncthreads();
        const float c0 = s_corr[g], c1 = s_corr[g + 8];
#pragma unroll
        for (int i = 0; i < NV; ++i) acc[i][0] *= c0, acc[i][1] *= c0, acc[i][2] *= c1, acc[i][3] *= c1;
#pragma unroll
        for (int ks = 0; ks < HD_KEYS / 16; ++ks) {
            uint32_t a[4];
            ldsm_x4(smem_u32(&sp[(mi & 1) * 8 + r8][16 * ks + (mi >> 1) * 8]), a);
#pragma unroll
            for (int i = 0; i < NV; i += 2) {
                const int c = 8 * (NV * warp + i);
                if (c >= p.rank) break;
                uint32_t b[4];
                ldsm_x4_t(smem_u32(sk + (16 * ks + (mi & 1) * 8 + r8) * ldk + c + (mi >> 1) * 8), b);
                mma_bf16(acc[i], a, b[0], b[1]);
                mma_bf16(acc[i + 1], a, b[2], b[3]);
            }
        }
        if (k0 + HD_KEYS < ke) {
            __syncthreads();                           // every warp is done with the tile
            load(k0 + HD_KEYS);
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int h = h0 + 2 * warp + r;
        if (lane == 0 && h < p.heads) {
            float* to = p.part_ml + 2 * (((size_t)t * p.heads + h) * p.splits + s);
            to[0] = m[r], to[1] = l[r];
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int h = h0 + g + 8 * r;
        if (h >= p.heads) continue;
        float* to = p.part + (((size_t)t * p.heads + h) * p.splits + s) * p.rank;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = 8 * (NV * warp + i) + 2 * q;
            if (p.rank % 2 == 0) {
                if (c < p.rank) *reinterpret_cast<float2*>(to + c) = make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
            } else {
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    if (c + j < p.rank) to[c + j] = acc[i][2 * r + j];
            }
        }
    }
}

int launch_heads(dc_ctx* ctx, const AbsorbedParams& p, int T) {
    const int ldk = (((p.c.row + 15) & ~15) + 63) / 64 * 64 + 8;
    const size_t smem = (size_t)(16 + HD_KEYS) * ldk * 2;
    const dim3 grid(p.splits, (p.heads + 15) / 16, T), block(HD_WARPS * 32);
#define DC_HD(NV)                                                                                                  \
    do {                                                                                                           \
        DC_TRY(dc_kernel_setup(ctx, (const void*)k_latent_heads<NV>, (int)smem, "k_latent_heads"));                \
        return dc_launch(ctx, "k_latent_heads", k_latent_heads<NV>, grid, block, smem, p);                         \
    } while (0)
    if (p.rank <= 128) DC_HD(2);
    if (p.rank <= 256) DC_HD(4);
    if (p.rank <= 512) DC_HD(8);
    DC_HD(16);
#undef DC_HD
}

// Splits of one (head, token) joined, then taken through OUT_ROWS rows of the head's W_uv and multiplied by the head's gate.
constexpr int OUT_ROWS = 64;
__global__ void __launch_bounds__(256) k_latent_out(const float* __restrict__ part, const float* __restrict__ part_ml, int heads, int splits,
                                                    int rank, const __nv_bfloat16* __restrict__ uv, int ldw, int vdim_p, int vdim,
                                                    const float* __restrict__ gate, int ldg,
                                                    float* __restrict__ mix, __nv_bfloat16* __restrict__ mixb, int ldm) {
    extern __shared__ __align__(16) float lat[];      // twice [rank padded to 8]
    __shared__ float sw[DC_MAX_SPLITS];
    pdl_launch_dependents();
    const int h = blockIdx.x, t = blockIdx.y, e0 = blockIdx.z * OUT_ROWS, e1 = min(vdim, e0 + OUT_ROWS), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const char* rows = reinterpret_cast<const char*>(uv + (size_t)(h * vdim_p + e0) * ldw);
    for (int i = threadIdx.x * 128; i < (e1 - e0) * ldw * 2; i += 256 * 128) prefetch_l2(rows + i);
    pdl_wait();
    const size_t o = ((size_t)t * heads + h) * splits;
    const float mul = gate ? sigmoid(gate[(size_t)t * ldg + h]) : 1.0f;
    if (warp == 0) join_weights(part_ml + 2 * o, splits, lane, -INFINITY, 1.0f, sw);
    __syncthreads();
    const int rank8 = (rank + 7) & ~7;
    if (rank % 4 == 0) {         // two threads share four values of a latent
        float* half = lat + rank8;
        const int n4 = rank8 / 4, share = threadIdx.x >> 7;
        for (int i = threadIdx.x & 127; i < n4; i += 128) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (4 * i < rank) {
#pragma unroll 16
                for (int s = share; s < splits; s += 2) {
                    const float4 x = *reinterpret_cast<const float4*>(part + (o + s) * rank + 4 * i);
                    v.x = fmaf(x.x, sw[s], v.x), v.y = fmaf(x.y, sw[s], v.y), v.z = fmaf(x.z, sw[s], v.z), v.w = fmaf(x.w, sw[s], v.w);
                }
            }
            reinterpret_cast<float4*>(share ? half : lat)[i] = v;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < rank8; i += 256) lat[i] += half[i];
    } else {
        for (int r = threadIdx.x; r < rank8; r += 256) {
            float v = 0.0f;
            if (r < rank) {
#pragma unroll 16
                for (int s = 0; s < splits; ++s) v = fmaf(part[(o + s) * rank + r], sw[s], v);
            }
            lat[r] = v;
        }
    }
    __syncthreads();
    constexpr int ROWS = OUT_ROWS / 8;                // of a warp, all in flight
    float a[ROWS] = {};
    for (int c = lane; c < rank8 / 8; c += 32) {
        uint4 v[ROWS];
#pragma unroll
        for (int i = 0; i < ROWS; ++i) v[i] = *reinterpret_cast<const uint4*>(uv + (size_t)(h * vdim_p + min(e0 + warp + 8 * i, e1 - 1)) * ldw + 8 * c);
#pragma unroll
        for (int i = 0; i < ROWS; ++i) {
            float f[8];
            unpack16(v[i], f, __nv_bfloat16());
#pragma unroll
            for (int j = 0; j < 8; ++j) a[i] = fmaf(f[j], lat[8 * c + j], a[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        const int e = e0 + warp + 8 * i;
        const float v = warp_sum(a[i]) * mul;
        const size_t at = (size_t)t * ldm + (size_t)h * vdim + e;
        if (lane == 0 && e < e1) {
            if (mixb) mixb[at] = __float2bfloat16_rn(v);
            else mix[at] = v;
        }
    }
}

template <typename TC>
int launch_absorbed(dc_ctx* ctx, const AbsorbedParams& p, int T) {
    const size_t smem = (size_t)AB_HEADS * p.c.row * 4 + (size_t)AB_KEYS * (p.c.row * sizeof(TC) + 16);
    const dim3 grid(p.splits, (p.heads + AB_HEADS - 1) / AB_HEADS, T), block(AB_HEADS * 32);
#define DC_AB(RP)                                                                                                     \
    do {                                                                                                              \
        DC_TRY(dc_kernel_setup(ctx, (const void*)k_latent_absorbed<TC, RP>, (int)smem, "k_latent_absorbed"));         \
        return dc_launch(ctx, "k_latent_absorbed", k_latent_absorbed<TC, RP>, grid, block, smem, p);                  \
    } while (0)
    const int rp = (p.rank * (int)sizeof(TC) + 511) / 512;
    if (rp <= 1) DC_AB(1);
    if (rp <= 2) DC_AB(2);
    if (rp <= 4) DC_AB(4);
    DC_AB(8);
#undef DC_AB
}

// ---------------------------------------------------------------- prompt form
// Row i of the gathered keys: the cached latent and rotated part of an entry's visible positions (from the first key
// that its first token sees to its last token).
__global__ void __launch_bounds__(256) k_latent_gather(CacheRef c, const int32_t* __restrict__ seq_ids, const int32_t* __restrict__ positions,
                                                       const int32_t* __restrict__ starts, const int32_t* __restrict__ key_base, int E, int n_keys,
                                                       int window, int rank, int rot, __nv_bfloat16* __restrict__ kc, int ldc,
                                                       __nv_bfloat16* __restrict__ kr, int ldr) {
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (i >= n_keys) return;
    int e = 0;
    while (e + 1 < E && key_base[e + 1] <= i) ++e;
    const int t0 = starts[e], pos = first_key(positions[t0], window) + i - key_base[e];
    const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(c.arena) + c.at(seq_ids[t0], pos);
    if (rank % 8 == 0) {
        for (int j = lane; j < rank / 8; j += 32) reinterpret_cast<uint4*>(kc + (size_t)i * ldc)[j] = reinterpret_cast<const uint4*>(src)[j];
    } else {
        for (int j = lane; j < rank; j += 32) kc[(size_t)i * ldc + j] = src[j];
    }
    for (int j = lane; j < ldr; j += 32) kr[(size_t)i * ldr + j] = j < rot ? src[rank + j] : __float2bfloat16_rn(0.0f);
}

struct PromptParams {
    const float* proj;
    int ldp, off_q, off_g, dim, rot, dim_p, vdim, vdim_p, uv_row, window;
    float scale;
    const int32_t *positions, *starts, *key_base, *tiles;    // tiles: (entry, first query of the entry) pairs
    const __nv_bfloat16* kv;
    int ldkv;
    const __nv_bfloat16* kr;
    int ldr, dq;             // dq: padded key length (dim_p + ldr, up to a multiple of 16)
    __nv_bfloat16* out;
    int ldm;
};

constexpr int PK = 64;           // keys per tile

// One CTA per (PQ queries of one entry, head), sixteen queries a warp; key and value tiles in a ring of ST stages.
// VD: value columns, padded.
template <int VD, int PQ, int ST>
__global__ void __launch_bounds__(2 * PQ) k_latent_prompt(const PromptParams p) {
    constexpr int LDV = VD + 8, NT = 2 * PQ;
    extern __shared__ __align__(16) uint8_t smem[];
    const int ldk = p.dq + 8;
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem);     // [PQ][ldk]
    __nv_bfloat16* sK = sQ + PQ * ldk;                              // [ST][PK][ldk]
    __nv_bfloat16* sV = sK + ST * PK * ldk;                         // [ST][PK][LDV]
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, head = blockIdx.y;
    const int tile0 = (int)(gridDim.x - 1 - blockIdx.x);           // later queries see more keys: they start first
    const int e = p.tiles[2 * tile0], q0 = p.tiles[2 * tile0 + 1];
    if (q0 % PQ) return;                                            // tiles are listed per DC_LATENT_QTILE queries
    const int t0 = p.starts[e], n = p.starts[e + 1] - t0, pos0 = p.positions[t0];
    const int key0 = first_key(pos0, p.window);                     // position of the entry's first gathered key
    const int first = first_key(pos0 + q0, p.window), last = pos0 + min(q0 + PQ, n) - 1;
    const int n_tiles = (last - first) / PK + 1;
    const __nv_bfloat16* kv = p.kv + (size_t)(p.key_base[e] - key0) * p.ldkv;      // indexed by position
    const __nv_bfloat16* kr = p.kr + (size_t)(p.key_base[e] - key0) * p.ldr;
    const int kc = p.dim_p / 8, rc = p.ldr / 8, pad = p.dq / 8, vc = p.vdim_p / 8;

    // eight threads per key row
    const int lrow = tid >> 3, lc = tid & 7;
    auto load = [&](int tile, int buf) {
#pragma unroll
        for (int i = 0; i < PK * 8 / NT; ++i) {
            const int key = lrow + NT / 8 * i, pos = first + tile * PK + key;
            const bool ok = pos <= last;
            const __nv_bfloat16* krow = ok ? kv + (ptrdiff_t)pos * p.ldkv : p.kv;
            const __nv_bfloat16* rrow = (ok ? kr + (ptrdiff_t)pos * p.ldr : p.kr) - kc * 8;
            const uint32_t dk = smem_u32(sK + (buf * PK + key) * ldk), dv = smem_u32(sV + (buf * PK + key) * LDV);
            for (int c = lc; c < pad; c += 8) {
                const bool in = ok && c < kc + rc;
                cp_async16z(dk + 16 * c, in ? (c < kc ? krow + head * p.dim_p : rrow) + 8 * c : p.kv, in);
            }
#pragma unroll
            for (int c0 = 0; c0 < VD / 8; c0 += 8) {
                const int c = c0 + lc;
                if (VD / 8 < 8 && c >= VD / 8) break;
                const bool in = ok && c < vc;
                cp_async16z(dv + 16 * c, in ? krow + p.uv_row + head * p.vdim_p + 8 * c : p.kv, in);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int i = 0; i < ST - 1; ++i)
        if (i < n_tiles) load(i, i);
        else cp_async_commit();
    // queries: a warp takes its own sixteen rows, many loads in flight
    {
        const float* q0p = p.proj + (size_t)(t0 + q0) * p.ldp + p.off_q + head * (p.dim + p.rot);
        const int dq = p.dq;
#pragma unroll 12
        for (int i = lane; i < 16 * dq; i += 32) {
            const int r = i / dq, c = i - r * dq, qr = 16 * warp + r;
            const int from = c < p.dim_p ? (c < p.dim ? c : -1) : c - p.dim_p < p.rot ? p.dim + c - p.dim_p : -1;
            const float v = q0p[(size_t)min(qr, n - 1 - q0) * p.ldp + max(from, 0)];
            sQ[qr * ldk + c] = __float2bfloat16_rn(q0 + qr < n && from >= 0 ? v : 0.0f);
        }
    }
    float o[VD / 8][4];
#pragma unroll
    for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m_run[2] = {-1e30f, -1e30f}, l_run[2] = {0.0f, 0.0f};
    const float sl2 = p.scale * 1.4426950408889634f;
    const int g = lane >> 2, t4 = lane & 3, mi = lane >> 3, r8 = lane & 7;
    const int qpos0 = pos0 + q0 + 16 * warp + g;
    const int window = p.window > 0 ? p.window : 0x7fffffff;

    for (int tile = 0; tile < n_tiles; ++tile) {
        const int buf = tile % ST, k0 = first + tile * PK;
        cp_async_wait<ST - 2>();
        __syncthreads();         // the tile has landed; every warp is done with the stage that the next load fills
        if (tile + ST - 1 < n_tiles) load(tile + ST - 1, (tile + ST - 1) % ST);
        else cp_async_commit();
        float s[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        const uint32_t qa = smem_u32(sQ + (16 * warp + (mi & 1) * 8 + r8) * ldk + (mi >> 1) * 8);
        const uint32_t ka = smem_u32(sK + (buf * PK + (mi >> 1) * 8 + r8) * ldk + (mi & 1) * 8);
#pragma unroll 2
        for (int kk = 0; kk < p.dq; kk += 16) {
            uint32_t a[4];
            ldsm_x4(qa + 2 * kk, a);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                uint32_t b[4];
                ldsm_x4(ka + 2 * (16 * np * ldk + kk), b);
                mma_bf16(s[2 * np], a, b[0], b[1]);
                mma_bf16(s[2 * np + 1], a, b[2], b[3]);
            }
        }
        // the warp's sixteen queries see the whole tile, or the mask decides key by key
        const int wq0 = pos0 + q0 + 16 * warp;
        if (!(k0 + PK - 1 <= wq0 && wq0 + 15 - k0 < window)) {
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int kp = k0 + 8 * nt + 2 * t4 + (j & 1), qp = qpos0 + (j >> 1) * 8;
                    if (!(kp <= qp && qp - kp < window)) s[nt][j] = -INFINITY;
                }
        }
        float mx[2] = {-1e30f, -1e30f};
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            mx[0] = fmaxf(mx[0], fmaxf(s[nt][0], s[nt][1]));
            mx[1] = fmaxf(mx[1], fmaxf(s[nt][2], s[nt][3]));
        }
        float m_new[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            m_new[h] = fmaxf(m_run[h], mx[h] * sl2);
        }
        if (__any_sync(0xffffffffu, m_new[0] > m_run[0] || m_new[1] > m_run[1])) {
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const float corr = ex2(m_run[h] - m_new[h]);
                m_run[h] = m_new[h];
                l_run[h] *= corr;
#pragma unroll
                for (int i = 0; i < VD / 8; ++i) {
                    o[i][2 * h] *= corr;
                    o[i][2 * h + 1] *= corr;
                }
            }
        }
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float w = ex2(fmaf(s[nt][j], sl2, -m_run[j >> 1]));
                s[nt][j] = w;
                l_run[j >> 1] += w;
            }
        const uint32_t va = smem_u32(sV + (buf * PK + (mi & 1) * 8 + r8) * LDV + (mi >> 1) * 8);
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            uint32_t a[4];
            a[0] = pack_bf2(s[2 * ks][0], s[2 * ks][1]);
            a[1] = pack_bf2(s[2 * ks][2], s[2 * ks][3]);
            a[2] = pack_bf2(s[2 * ks + 1][0], s[2 * ks + 1][1]);
            a[3] = pack_bf2(s[2 * ks + 1][2], s[2 * ks + 1][3]);
#pragma unroll
            for (int dp = 0; dp < VD / 16; ++dp) {
                uint32_t b[4];
                ldsm_x4_t(va + 2 * (16 * ks * LDV + 16 * dp), b);
                mma_bf16(o[2 * dp], a, b[0], b[1]);
                mma_bf16(o[2 * dp + 1], a, b[2], b[3]);
            }
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
        l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
        const int row = q0 + 16 * warp + g + 8 * h;
        if (row >= n) continue;
        const float inv = (p.off_g < 0 ? 1.0f : sigmoid(p.proj[(size_t)(t0 + row) * p.ldp + p.off_g + head])) / l_run[h];
        __nv_bfloat16* dst = p.out + (size_t)(t0 + row) * p.ldm + (size_t)head * p.vdim;
#pragma unroll
        for (int nt = 0; nt < VD / 8; ++nt)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int c = 8 * nt + 2 * t4 + j;
                if (c < p.vdim) dst[c] = __float2bfloat16_rn(o[nt][2 * h + j] * inv);
            }
    }
}

CacheRef cache_ref(const dc_latent_cache& c, int row) { return CacheRef{c.arena, c.tables, c.max_blocks, row}; }

}  // namespace

int dc_launch_latent_prep(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const dc_latent_cache& c, float* proj, int ldp, float eps,
                          int max_pos) {
    PrepParams p = {proj, ldp, m.off_q, m.off_kv, m.heads, m.dim, m.rot_dim, m.kv_rank, max_pos, m.kv_from < 0 ? m.kv_norm : nullptr,
                    m.cos_sin, eps, st.seq_ids, st.positions, cache_ref(c, m.row)};
    if (c.f32) return dc_launch(ctx, "k_latent_prep", k_latent_prep<float>, dim3(st.T), dim3(256), 0, p);
    return dc_launch(ctx, "k_latent_prep", k_latent_prep<__nv_bfloat16>, dim3(st.T), dim3(256), 0, p);
}

int dc_launch_latent_absorbed(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const dc_latent_cache& c, const float* proj, int ldp,
                              int splits, float* qa, float* part, float* part_ml, float* mix, __nv_bfloat16* mixb, int ldm) {
    const int ldq = dc_pad8(m.kv_rank), rb = (m.kv_rank + 127) / 128;
#define DC_ABSORB(NT)                                                                                                                        \
    DC_TRY(dc_launch(ctx, "k_latent_absorb", k_latent_absorb<NT>, dim3(m.heads, rb, (st.T + NT - 1) / NT), dim3(256), (size_t)NT * m.dim * 4, \
                     proj, ldp, m.off_q, m.heads, m.dim, m.rot_dim, m.ukv.w, m.ukv.ld, m.dim_p, m.kv_rank, st.T, qa, ldq))
    if (st.T == 1) DC_ABSORB(1);
    else DC_ABSORB(4);
#undef DC_ABSORB
    AbsorbedParams p = {qa, ldq, proj, ldp, m.off_q, m.heads, m.dim, m.rot_dim, m.kv_rank, m.window, splits, m.scale, st.seq_ids, st.positions,
                        cache_ref(c, m.row), part, part_ml};
    DC_TRY(c.f32 ? launch_absorbed<float>(ctx, p, st.T) : launch_heads(ctx, p, st.T));
    const dim3 grid(m.heads, st.T, (m.vdim + OUT_ROWS - 1) / OUT_ROWS), block(256);
    const size_t smem = (size_t)dc_pad8(m.kv_rank) * 8;
    const __nv_bfloat16* uv = m.ukv.w + (size_t)m.uv_row * m.ukv.ld;
    const float* gate = m.off_g < 0 ? nullptr : proj + m.off_g;
    if (c.f32)
        return dc_launch(ctx, "k_latent_out", k_latent_out, grid, block, smem, part, part_ml, m.heads, splits, m.kv_rank, uv, m.ukv.ld, m.vdim_p, m.vdim, gate, ldp,
                         mix, mixb, ldm);
    return dc_launch_drained(ctx, "k_latent_out", k_latent_out, grid, block, smem, part, part_ml, m.heads, splits, m.kv_rank, uv, m.ukv.ld, m.vdim_p, m.vdim, gate,
                             ldp, mix, mixb, ldm);
}

int dc_launch_latent_gather(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const dc_latent_cache& c, const int32_t* key_base,
                            int n_keys, __nv_bfloat16* keys_c, int ldc, __nv_bfloat16* keys_r, int ldr) {
    return dc_launch(ctx, "k_latent_gather", k_latent_gather, dim3((n_keys + 7) / 8), dim3(256), 0, cache_ref(c, m.row), st.seq_ids, st.positions,
                     st.starts, key_base, st.E, n_keys, m.window, m.kv_rank, m.rot_dim, keys_c, ldc, keys_r, ldr);
}

int dc_launch_latent_prefill(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const int32_t* key_base, const int32_t* tiles,
                             int n_tiles, const float* proj, int ldp, const __nv_bfloat16* keys_kv, int ldkv, const __nv_bfloat16* keys_r,
                             int ldr, __nv_bfloat16* mixb, int ldm) {
    PromptParams p = {proj, ldp, m.off_q, m.off_g, m.dim, m.rot_dim, m.dim_p, m.vdim, m.vdim_p, m.uv_row, m.window, m.scale, st.positions, st.starts,
                      key_base, tiles, keys_kv, ldkv, keys_r, ldr, (m.dim_p + ldr + 15) & ~15, mixb, ldm};
    const dim3 grid(n_tiles, m.heads);
    // 128 queries per CTA and three stages where they fit shared memory
#define DC_PROMPT(VD)                                                                                                       \
    do {                                                                                                                    \
        auto bytes = [&](int pq, int st) { return ((size_t)(pq + st * PK) * (p.dq + 8) + (size_t)st * PK * (VD + 8)) * 2; }; \
        if (bytes(128, 3) <= 227 * 1024) {                                                                                  \
            DC_TRY(dc_kernel_setup(ctx, (const void*)k_latent_prompt<VD, 128, 3>, (int)bytes(128, 3), "k_latent_prompt"));  \
            return dc_launch(ctx, "k_latent_prompt", k_latent_prompt<VD, 128, 3>, grid, dim3(256), bytes(128, 3), p);       \
        }                                                                                                                   \
        DC_TRY(dc_kernel_setup(ctx, (const void*)k_latent_prompt<VD, 64, 2>, (int)bytes(64, 2), "k_latent_prompt"));        \
        return dc_launch(ctx, "k_latent_prompt", k_latent_prompt<VD, 64, 2>, grid, dim3(128), bytes(64, 2), p);             \
    } while (0)
    if (m.vdim <= 32) DC_PROMPT(32);
    if (m.vdim <= 64) DC_PROMPT(64);
    if (m.vdim <= 128) DC_PROMPT(128);
    DC_PROMPT(256);
#undef DC_PROMPT
}
