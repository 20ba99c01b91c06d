// Grouped-query attention with its variants: a sliding window with or without the sequence's first tokens kept in sight, a
// soft cap on the scores, a sink in the softmax' denominator, unnormalized sigmoid weights instead of a softmax, short
// convolutions ahead of everything, norms of queries and keys over the whole projection or per head, norms of values, rotation of
// neighbouring or of half-distant pairs, values of their own or the key projection before norm and rotation, two maps per head
// whose outputs are subtracted, and a gate per head.
//
// A cached token is one row: the turned keys of all key heads (and maps), then the values.  Steps of up to DC_MAX_T tokens
// and f32 models take every token alone (k_gqa_tokens: keys split over CTAs, k_gqa_join); prompt-sized steps of bf16
// models run tiles of queries over the cached rows with bf16 products (k_gqa_prompt).  Scores, weights and their sums are
// f32.
#include <algorithm>

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

__device__ __forceinline__ void store_pair(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf2(a, b); }

__device__ __forceinline__ void store_four(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store_four(__nv_bfloat16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf2(v.x, v.y), pack_bf2(v.z, v.w)); }

// ---------------------------------------------------------------- norms, rotation, cache write
struct PrepParams {
    const float* proj;
    int ldp, off_q, off_k, heads, kv_heads, dim, dim_p, ldq, rot, max_pos, lanes;
    const float *q_norm, *k_norm, *cos_sin;
    float eps;
    const int32_t *seq_ids, *positions;
    CacheRef c;
    float* q;
    __nv_bfloat16* qb;       // instead of q
};

// One CTA per token and part: the last part is the keys and values, the others share the query heads (every one sums up
// the whole projection's squares).  A thread has one pair of dimensions (2^lanes threads a head) of several heads.
template <typename TC>
__global__ void __launch_bounds__(256) k_gqa_prep(const PrepParams p) {
    constexpr int U = 4, B = 8;
    __shared__ float red[33];
    pdl_launch_dependents();
    const bool keys = blockIdx.y == gridDim.y - 1;
    const int parts = gridDim.y - 1, share = (p.heads + parts - 1) / parts;
    const int h0 = keys ? 0 : blockIdx.y * share, h1 = keys ? p.kv_heads : min(p.heads, h0 + share), n = (keys ? p.kv_heads : p.heads) * p.dim;
    const int pitch = keys ? p.dim_p : p.ldq, step = 256 >> p.lanes;
    const int first = h0 + (threadIdx.x >> p.lanes), d = 2 * (threadIdx.x & ((1 << p.lanes) - 1));
    const float* w = (keys ? p.k_norm : p.q_norm) + d;
    const bool whole = d + 1 < p.dim && !(p.dim & 1), one = d < p.dim, two = d + 1 < p.dim;
    pdl_wait();
    const int t = blockIdx.x, at_pos = p.positions[t], seq = p.seq_ids[t];
    const float* x = p.proj + (size_t)t * p.ldp + (keys ? p.off_k : p.off_q);
    float2 raw[U], nw[U];
    auto fetch = [&](int head0) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int head = head0 + step * u;
            const float *xs = x + head * p.dim + d, *ws = w + head * p.dim;
            raw[u] = nw[u] = make_float2(0.0f, 0.0f);
            if (head >= h1) continue;
            if (whole) {
                raw[u] = *reinterpret_cast<const float2*>(xs), nw[u] = *reinterpret_cast<const float2*>(ws);
            } else {
                if (one) raw[u].x = xs[0], nw[u].x = ws[0];
                if (two) raw[u].y = xs[1], nw[u].y = ws[1];
            }
        }
    };
    fetch(first);                                        // on its way while the squares are summed up
    const int pos = min(max(at_pos, 0), p.max_pos - 1);
    const float2 turn = d < p.rot ? *reinterpret_cast<const float2*>(p.cos_sin + (size_t)pos * p.rot + d) : make_float2(1.0f, 0.0f);
    float ss = 0.0f;
    if ((keys || parts == 1) && h1 - h0 <= U * step) {   // ... from the same values
#pragma unroll
        for (int u = 0; u < U; ++u) ss = fmaf(raw[u].x, raw[u].x, fmaf(raw[u].y, raw[u].y, ss));
    } else {
        for (int i0 = threadIdx.x; i0 < n; i0 += 256 * B) {
            float v[B];
#pragma unroll
            for (int j = 0; j < B; ++j) v[j] = i0 + 256 * j < n ? x[i0 + 256 * j] : 0.0f;
#pragma unroll
            for (int j = 0; j < B; ++j) ss = fmaf(v[j], v[j], ss);
        }
    }
    TC* cache = keys ? reinterpret_cast<TC*>(p.c.arena) + p.c.at(seq, pos) + d : nullptr;
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)n + p.eps);
    if (d >= pitch) return;
    for (int head0 = first; head0 < h1; head0 += U * step) {
        if (head0 > first) fetch(head0);
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int head = head0 + step * u;
            if (head >= h1) break;
            const float a = raw[u].x * inv * nw[u].x, b = raw[u].y * inv * nw[u].y;
            const float c = a * turn.x - b * turn.y, e = b * turn.x + a * turn.y;
            if (keys) {
                TC* kd = cache + head * pitch;
                store_pair(kd, c, e);
                store_pair(kd + p.kv_heads * pitch, raw[u].x, raw[u].y);
            } else {
                const size_t at = ((size_t)t * p.heads + head) * pitch + d;
                if (p.qb) store_pair(p.qb + at, c, e);
                else store_pair(p.q + at, c, e);
            }
        }
    }
}

// The same with a norm per head or none: a warp per head of a token, a lane has the dimensions lane, lane + 32, ...
struct HeadsParams {
    const float* proj;
    int ldp, off_q, off_k, off_v, nq, nk, nv, dim, vdim, dim_p, vdim_p, v_at, ldq, rot, halves, max_pos;
    const float *q_norm, *k_norm, *cos_sin;
    float eps;
    const int32_t *seq_ids, *positions;
    CacheRef c;
    float* q;
    __nv_bfloat16* qb;       // instead of q
};

template <typename TC, int VP>      // VP: dimensions of a lane
__global__ void __launch_bounds__(256) k_gqa_prep_heads(const HeadsParams p) {
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, u = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (u >= p.nq + p.nk + p.nv) return;
    const bool query = u < p.nq, value = u >= p.nq + p.nk;
    const int head = query ? u : value ? u - p.nq - p.nk : u - p.nq, n = value ? p.vdim : p.dim;
    const float* w = value ? nullptr : query ? p.q_norm : p.k_norm;
    float nw[VP];
#pragma unroll
    for (int j = 0; j < VP; ++j) nw[j] = w && lane + 32 * j < n ? w[lane + 32 * j] : 1.0f;
    pdl_wait();
    const int t = blockIdx.x, pos = min(max(p.positions[t], 0), p.max_pos - 1);
    const float* x = p.proj + (size_t)t * p.ldp + (query ? p.off_q : value ? p.off_v : p.off_k) + head * n;
    const float* cs = p.cos_sin + (size_t)pos * p.rot;
    const int half = p.rot / 2;
    float v[VP], other[VP], ss = 0.0f;
    float2 turn[VP];
#pragma unroll
    for (int j = 0; j < VP; ++j) {
        const int d = lane + 32 * j;
        const bool first = p.halves ? d < half : !(d & 1), turned = !value && d < p.rot;
        const int mate = p.halves ? (first ? d + half : d - half) : d ^ 1;
        v[j] = d < n ? x[d] : 0.0f;
        other[j] = 0.0f, turn[j] = make_float2(1.0f, 0.0f);
        if (turned) {
            other[j] = x[mate] * (w ? w[mate] : 1.0f);
            turn[j] = *reinterpret_cast<const float2*>(cs + 2 * (p.halves ? min(d, mate) : d / 2));
            if (first) turn[j].y = -turn[j].y;
        }
        ss = fmaf(v[j], v[j], ss);
    }
    const float inv = w ? 1.0f / sqrtf(warp_sum(ss) / (float)n + p.eps) : 1.0f;
    TC* cache = query ? nullptr : reinterpret_cast<TC*>(p.c.arena) + p.c.at(p.seq_ids[t], pos) + (value ? p.v_at + head * p.vdim_p : head * p.dim_p);
    const int pitch = query ? p.ldq : value ? p.vdim_p : p.dim_p;
#pragma unroll
    for (int j = 0; j < VP; ++j) {
        const int d = lane + 32 * j;
        if (d >= pitch) break;
        const float r = (v[j] * nw[j] * turn[j].x + other[j] * turn[j].y) * inv;       // zero in the padding
        const size_t at = ((size_t)t * p.nq + head) * pitch + d;
        if (!query) store_as(cache + d, r);
        else if (p.qb) store_as(p.qb + at, r);
        else p.q[at] = r;
    }
}

// The same four dimensions at a time, for sizes that are multiples of four: a warp has U heads of a token in flight, a lane the
// dimensions 4 lane .. 4 lane + 3 (and, with NV 2, those 128 further on).
template <typename TC, int NV, int U>
__global__ void __launch_bounds__(256) k_gqa_prep_heads4(const HeadsParams p) {
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, u0 = blockIdx.y * 8 * U + (threadIdx.x >> 5), units = p.nq + p.nk + p.nv, half = p.rot / 2;
    pdl_wait();
    const int t = blockIdx.x, pos = min(max(p.positions[t], 0), p.max_pos - 1);
    const float* row = p.proj + (size_t)t * p.ldp;
    const float* cs = p.cos_sin + (size_t)pos * p.rot;
    float4 v[U][NV], mate[U][NV];
#pragma unroll
    for (int i = 0; i < U; ++i) {
        const int u = u0 + 8 * i;
        const bool query = u < p.nq, value = u >= p.nq + p.nk;
        const int head = query ? u : value ? u - p.nq - p.nk : u - p.nq, n = value ? p.vdim : p.dim;
        const float* x = row + (query ? p.off_q : value ? p.off_v : p.off_k) + head * n;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int d = 4 * lane + 128 * j;
            v[i][j] = u < units && d < n ? *reinterpret_cast<const float4*>(x + d) : make_float4(0.f, 0.f, 0.f, 0.f);
            mate[i][j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (u < units && !value && p.halves && d < p.rot) mate[i][j] = *reinterpret_cast<const float4*>(x + (d < half ? d + half : d - half));
        }
    }
    TC* cache = reinterpret_cast<TC*>(p.c.arena) + p.c.at(p.seq_ids[t], pos);
    float4 c[NV], s[NV];         // of the lane's dimensions; the sine has the sign of the mate's share
#pragma unroll
    for (int j = 0; j < NV; ++j) {
        const int d = 4 * lane + 128 * j;
        c[j] = make_float4(1.f, 1.f, 1.f, 1.f), s[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d >= p.rot) continue;
        if (p.halves) {
            const bool first = d < half;
            const float4* at = reinterpret_cast<const float4*>(cs + 2 * (first ? d : d - half));
            const float4 a = at[0], b = at[1];
            const float sign = first ? -1.0f : 1.0f;
            c[j] = make_float4(a.x, a.z, b.x, b.z), s[j] = make_float4(sign * a.y, sign * a.w, sign * b.y, sign * b.w);
        } else {
            const float4 a = *reinterpret_cast<const float4*>(cs + d);
            c[j] = make_float4(a.x, a.x, a.z, a.z), s[j] = make_float4(-a.y, a.y, -a.w, a.w);
        }
    }
#pragma unroll
    for (int i = 0; i < U; ++i) {
        const int u = u0 + 8 * i;
        if (u >= units) break;
        const bool query = u < p.nq, value = u >= p.nq + p.nk;
        const int head = query ? u : value ? u - p.nq - p.nk : u - p.nq, pitch = query ? p.ldq : value ? p.vdim_p : p.dim_p;
        const float* w = value ? nullptr : query ? p.q_norm : p.k_norm;
        float inv = 1.0f;
        if (w) {
            float ss = 0.0f;
#pragma unroll
            for (int j = 0; j < NV; ++j) ss += (v[i][j].x * v[i][j].x + v[i][j].y * v[i][j].y) + (v[i][j].z * v[i][j].z + v[i][j].w * v[i][j].w);
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
        }
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            const int d = 4 * lane + 128 * j;
            if (d >= pitch) break;
            float4 a = v[i][j], b = mate[i][j];
            if (w && d < p.dim) {
                const float4 f = *reinterpret_cast<const float4*>(w + d);
                a = make_float4(a.x * f.x, a.y * f.y, a.z * f.z, a.w * f.w);
                if (p.halves && d < p.rot) {
                    const float4 m = *reinterpret_cast<const float4*>(w + (d < half ? d + half : d - half));
                    b = make_float4(b.x * m.x, b.y * m.y, b.z * m.z, b.w * m.w);
                }
            }
            if (!p.halves) b = make_float4(a.y, a.x, a.w, a.z);
            const float4 r = value ? a : make_float4((a.x * c[j].x + b.x * s[j].x) * inv, (a.y * c[j].y + b.y * s[j].y) * inv,
                                                     (a.z * c[j].z + b.z * s[j].z) * inv, (a.w * c[j].w + b.w * s[j].w) * inv);
            const size_t at = ((size_t)t * p.nq + head) * pitch + d;
            if (!query) store_four(cache + (value ? p.v_at : 0) + head * pitch + d, r);
            else if (p.qb) store_four(p.qb + at, r);
            else store_four(p.q + at, r);
        }
    }
}

// Convolution and norms, no rotation: a warp takes a head of the queries, keys or values through a few tokens of an entry, a lane the
// dimensions lane, lane + 32, ...  The inputs ahead of the portion come from the sequence's ring.  TAPS: taps at most, 0: any number.
struct ConvParams {
    HeadsParams h;
    ConvRef cr;
    const float* conv;       // [taps][cr.ldw]
    bool q_unit, k_unit, v_unit, put_ring;      // put_ring: every entry is one token, whose input goes into the ring here
};
constexpr int conv_portion(int vp) { return vp <= 4 ? 8 : 4; }

template <typename TC, int VP, int TAPS>
__global__ void __launch_bounds__(256) k_gqa_prep_conv(const ConvParams p) {
    pdl_launch_dependents();
    const HeadsParams& a = p.h;
    const int lane = threadIdx.x & 31, u = blockIdx.y * 8 + (threadIdx.x >> 5), taps = p.cr.taps;
    if (u >= a.nq + a.nk + a.nv) return;
    const bool query = u < a.nq, value = u >= a.nq + a.nk;
    const int head = query ? u : value ? u - a.nq - a.nk : u - a.nq, n = value ? a.vdim : a.dim;
    const int col0 = (query ? a.off_q : value ? a.off_v : a.off_k) + head * n;
    const float* nw = value ? nullptr : query ? a.q_norm : a.k_norm;
    const bool unit = query ? p.q_unit : value ? p.v_unit : p.k_unit;
    constexpr int WN = TAPS > 0 ? TAPS : 1, PB = conv_portion(VP);
    float w[VP][WN];             // the last taps first: w[j][WN - 1] is the token's own
#pragma unroll
    for (int j = 0; j < VP; ++j)
#pragma unroll
        for (int k = 0; k < WN; ++k) {
            const int tap = taps - WN + k;
            w[j][k] = TAPS > 0 && tap >= 0 && lane + 32 * j < n ? p.conv[(size_t)tap * p.cr.ldw + col0 + lane + 32 * j] : 0.0f;
        }
    pdl_wait();
    const BlockRef br = block_at<PB>(p.cr.starts, p.cr.E, blockIdx.x);
    if (br.n <= 0) return;
    const int i0 = br.t0 - p.cr.starts[br.e], pos0 = p.cr.positions[br.t0], seq = p.cr.seq_ids[br.t0];
    float* ring = p.cr.ring(seq);
    float x[PB][VP], h[VP][WN > 1 ? WN - 1 : 1];
#pragma unroll
    for (int i = 0; i < PB; ++i)
#pragma unroll
        for (int j = 0; j < VP; ++j) {
            const int d = lane + 32 * j;
            x[i][j] = i < br.n && d < n ? a.proj[(size_t)(br.t0 + i) * a.ldp + col0 + d] : 0.0f;
        }
    if (TAPS > 1) {
#pragma unroll
        for (int j = 0; j < VP; ++j)
#pragma unroll
            for (int k = 0; k < WN - 1; ++k) {
                const int back = WN - 1 - k, d = lane + 32 * j;
                h[j][k] = 0.0f;
                if (back < taps && pos0 >= back && d < n)
                    h[j][k] = back <= i0 ? a.proj[(size_t)(br.t0 - back) * a.ldp + col0 + d] : ring[(size_t)((pos0 - back) % taps) * p.cr.C + col0 + d];
            }
    }
    if (p.put_ring)              // a row that no tap of this token reads
#pragma unroll
        for (int j = 0; j < VP; ++j)
            if (lane + 32 * j < n) ring[(size_t)(pos0 % taps) * p.cr.C + col0 + lane + 32 * j] = x[0][j];
    float y[PB][VP], ss[PB];
#pragma unroll
    for (int i = 0; i < PB; ++i) {
        ss[i] = 0.0f;
#pragma unroll
        for (int j = 0; j < VP; ++j) {
            const int d = lane + 32 * j;
            if (TAPS > 0) {
                float s = 0.0f;
#pragma unroll
                for (int k = 0; k < WN - 1; ++k) s = fmaf(w[j][k], h[j][k], s);
                y[i][j] = fmaf(w[j][WN - 1], x[i][j], s);
#pragma unroll
                for (int k = 0; k + 1 < WN - 1; ++k) h[j][k] = h[j][k + 1];
                if (TAPS > 1) h[j][WN > 1 ? WN - 2 : 0] = x[i][j];
            } else {
                y[i][j] = i < br.n && d < n ? conv_at(a.proj, a.ldp, ring, p.cr.C, col0 + d, taps, p.conv + col0 + d, p.cr.ldw, col0 + d, br.t0 + i, i0 + i, pos0 + i) : 0.0f;
            }
            ss[i] = fmaf(y[i][j], y[i][j], ss[i]);
        }
    }
    if (unit) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int i = 0; i < PB; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
    }
    const int pitch = query ? a.ldq : value ? a.vdim_p : a.dim_p;
#pragma unroll
    for (int i = 0; i < PB; ++i) {
        if (i >= br.n) break;
        const float inv = unit ? 1.0f / sqrtf(ss[i] / (float)n + a.eps) : 1.0f;
        const int t = br.t0 + i, pos = min(pos0 + i, a.max_pos - 1);
        TC* cache = query ? nullptr : reinterpret_cast<TC*>(a.c.arena) + a.c.at(seq, pos) + (value ? a.v_at + head * a.vdim_p : head * a.dim_p);
#pragma unroll
        for (int j = 0; j < VP; ++j) {
            const int d = lane + 32 * j;
            if (d >= pitch) break;
            const float r = y[i][j] * inv * (nw && d < n ? nw[d] : 1.0f);       // zero in the padding
            const size_t at = ((size_t)t * a.nq + head) * pitch + d;
            if (!query) store_as(cache + d, r);
            else if (a.qb) store_as(a.qb + at, r);
            else a.q[at] = r;
        }
    }
}

// The same for up to four taps and head sizes that are multiples of four up to 128: a lane has the dimensions 4 lane .. 4 lane + 3.
// PB: tokens of a warp; 1: every entry is one token.
template <typename TC, int PB>
__global__ void __launch_bounds__(256) k_gqa_prep_conv4(const ConvParams p) {
    pdl_launch_dependents();
    const HeadsParams& a = p.h;
    const int lane = threadIdx.x & 31, u = blockIdx.y * 8 + (threadIdx.x >> 5), taps = p.cr.taps, d = 4 * lane;
    if (u >= a.nq + a.nk + a.nv) return;
    const bool query = u < a.nq, value = u >= a.nq + a.nk;
    const int head = query ? u : value ? u - a.nq - a.nk : u - a.nq, n = value ? a.vdim : a.dim;
    const int col = (query ? a.off_q : value ? a.off_v : a.off_k) + head * n + min(d, n - 4);
    const bool unit = query ? p.q_unit : value ? p.v_unit : p.k_unit, in = d < n;
    const float* nw = value ? nullptr : query ? a.q_norm : a.k_norm;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    auto at4 = [](const float* q) { return *reinterpret_cast<const float4*>(q); };
    float4 w[4];                 // w[3] is the token's own
#pragma unroll
    for (int k = 0; k < 4; ++k) w[k] = in && taps - 4 + k >= 0 ? at4(p.conv + (size_t)(taps - 4 + k) * p.cr.ldw + col) : zero;
    const float4 nv = nw && in ? at4(nw + d) : make_float4(1.f, 1.f, 1.f, 1.f);
    pdl_wait();
    BlockRef br = {(int)blockIdx.x, (int)blockIdx.x, 1};
    if (PB > 1) br = block_at<PB>(p.cr.starts, p.cr.E, blockIdx.x);
    if (br.n <= 0) return;
    const int i0 = PB > 1 ? br.t0 - p.cr.starts[br.e] : 0, pos0 = p.cr.positions[br.t0], seq = p.cr.seq_ids[br.t0];
    float* ring = p.cr.ring(seq) + col;
    const float* x0 = a.proj + (size_t)br.t0 * a.ldp + col;
    float4 x[PB], h[3];
#pragma unroll
    for (int i = 0; i < PB; ++i) x[i] = i < br.n ? at4(x0 + (size_t)i * a.ldp) : zero;
#pragma unroll
    for (int k = 0; k < 3; ++k) {
        const int back = 3 - k;
        h[k] = back >= taps || pos0 < back ? zero : back <= i0 ? at4(x0 - (size_t)back * a.ldp) : at4(ring + (size_t)((pos0 - back) % taps) * p.cr.C);
    }
    if (p.put_ring && in) *reinterpret_cast<float4*>(ring + (size_t)(pos0 % taps) * p.cr.C) = x[0];       // a row that no tap of this token reads
    float ss[PB];
#pragma unroll
    for (int i = 0; i < PB; ++i) {
        float4 y;
#define DC_TAPS(e) y.e = fmaf(w[3].e, x[i].e, fmaf(w[2].e, h[2].e, fmaf(w[1].e, h[1].e, w[0].e * h[0].e)))
        DC_TAPS(x), DC_TAPS(y), DC_TAPS(z), DC_TAPS(w);
#undef DC_TAPS
        h[0] = h[1], h[1] = h[2], h[2] = x[i];
        x[i] = y;
        ss[i] = (y.x * y.x + y.y * y.y) + (y.z * y.z + y.w * y.w);       // zero beyond the head: its weights are
    }
    if (unit) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
            for (int i = 0; i < PB; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
    }
    const int pitch = query ? a.ldq : value ? a.vdim_p : a.dim_p;
    if (d >= pitch) return;
#pragma unroll
    for (int i = 0; i < PB; ++i) {
        if (i >= br.n) break;
        const float inv = unit ? 1.0f / sqrtf(ss[i] / (float)n + a.eps) : 1.0f;
        const float4 r = make_float4(x[i].x * inv * nv.x, x[i].y * inv * nv.y, x[i].z * inv * nv.z, x[i].w * inv * nv.w);
        const size_t q = ((size_t)(br.t0 + i) * a.nq + head) * pitch + d;
        if (!query) store_four(reinterpret_cast<TC*>(a.c.arena) + a.c.at(seq, min(pos0 + i, a.max_pos - 1)) + (value ? a.v_at + head * a.vdim_p : head * a.dim_p) + d, r);
        else if (a.qb) store_four(a.qb + q, r);
        else store_four(a.q + q, r);
    }
}

template <typename TC>
int launch_prep_conv4(dc_ctx* ctx, const ConvParams& p, const dc_step& st) {
    const int parts = (p.h.nq + p.h.nk + p.h.nv + 7) / 8;
    if (st.single) return dc_launch(ctx, "k_gqa_prep_conv4", k_gqa_prep_conv4<TC, 1>, dim3(st.T, parts), dim3(256), 0, p);
    return dc_launch(ctx, "k_gqa_prep_conv4", k_gqa_prep_conv4<TC, 8>, dim3(st.T / 8 + st.E, parts), dim3(256), 0, p);
}

template <typename TC, int VP>
int launch_prep_conv(dc_ctx* ctx, const ConvParams& p, const dc_step& st) {
    const dim3 grid(st.single ? st.T : st.T / conv_portion(VP) + st.E, (p.h.nq + p.h.nk + p.h.nv + 7) / 8);
    if (p.cr.taps <= 4) return dc_launch(ctx, "k_gqa_prep_conv", k_gqa_prep_conv<TC, VP, 4>, grid, dim3(256), 0, p);
    return dc_launch(ctx, "k_gqa_prep_conv", k_gqa_prep_conv<TC, VP, 0>, grid, dim3(256), 0, p);
}

// ---------------------------------------------------------------- every token alone
// The keys that a token sees, in order: the kept first ones that its window has left behind, then the window.
struct Keys {
    int first, kept, n;
    __device__ __forceinline__ int at(int i) const { return i < kept ? i : first + i - kept; }
};
__device__ __forceinline__ Keys keys_of(int pos, int last, int window, int keep) {
    Keys k;
    k.first = first_key(pos, window);
    k.kept = min(keep, k.first);
    k.n = k.kept + last - k.first + 1;
    return k;
}

struct TokenParams {
    const float* q;          // [T][heads * MAPS][ldq]
    int ldq, heads, per, groups, dim, vdim, dim_p, vdim_p, v_at, window, keep, splits;
    float scale, softcap;
    const int32_t *seq_ids, *positions;
    CacheRef c;
    const float* score_bias; // sigmoid weights; or null: softmax
    float *part, *part_ml;   // [T][heads * MAPS][splits][vdim], [T][heads * MAPS][splits][2]
};

constexpr int TK_KEYS = 32, TK_HEADS = 4;

// One CTA per (key split, four query heads of one key head, token); with two maps per head two heads and their maps.  A
// warp is a head and map.  Scores: a lane is a key; sums: a lane owns the value pairs lane, lane + 32, ... (VP of them).
template <typename TC, int VP, int MAPS>
__global__ void __launch_bounds__(TK_HEADS * 32) k_gqa_tokens(const TokenParams p) {
    constexpr int EPC = 16 / sizeof(TC);      // elements of a 16-byte chunk
    extern __shared__ __align__(16) uint8_t sm[];
    const int ldk = MAPS * p.dim_p + EPC, ldv = p.vdim_p + EPC, chunks = p.dim_p / EPC, vchunks = p.vdim_p / EPC;
    float* sq = reinterpret_cast<float*>(sm);                              // [TK_HEADS][dim_p]
    TC* sk = reinterpret_cast<TC*>(sm + (size_t)TK_HEADS * p.dim_p * 4);   // [TK_KEYS][ldk], then the values [TK_KEYS][ldv]
    TC* sv = sk + TK_KEYS * ldk;
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.x, g = blockIdx.y / p.groups, t = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int unit = (blockIdx.y % p.groups) * TK_HEADS + warp, map = unit % MAPS, h = g * p.per * MAPS + unit, pos = p.positions[t], seq = p.seq_ids[t];
    const bool live = unit < p.per * MAPS;
    const float bias = p.score_bias && live ? p.score_bias[h] : 0.0f;
    const Keys keys = keys_of(pos, pos, p.window, p.keep);
    const int per = ((keys.n + p.splits - 1) / p.splits + TK_KEYS - 1) / TK_KEYS * TK_KEYS;
    const int kb = s * per, ke = min(keys.n, kb + per);
    if (live)
        for (int c = lane; c < p.dim_p; c += 32) sq[warp * p.dim_p + c] = p.q[((size_t)t * p.heads * MAPS + h) * p.ldq + c] * p.scale;
    float m = -INFINITY, l = 0.0f, acc[VP][2];
#pragma unroll
    for (int j = 0; j < VP; ++j) acc[j][0] = acc[j][1] = 0.0f;
    for (int k0 = kb; k0 < ke; k0 += TK_KEYS) {
        __syncthreads();
        const TC* src[TK_KEYS / TK_HEADS];                  // a warp's keys: all rows asked for before any arrives
#pragma unroll
        for (int i = 0; i < TK_KEYS / TK_HEADS; ++i)
            src[i] = reinterpret_cast<const TC*>(p.c.arena) + p.c.at(seq, keys.at(min(k0 + warp * (TK_KEYS / TK_HEADS) + i, ke - 1)));
        for (int c = lane; c < MAPS * chunks + vchunks; c += 32) {
            const bool val = c >= MAPS * chunks;
            const int at = (val ? c - MAPS * chunks : c) * EPC, from = val ? p.v_at + g * p.vdim_p + at : g * MAPS * p.dim_p + at;
            TC* to = (val ? sv : sk) + at;
#pragma unroll
            for (int i = 0; i < TK_KEYS / TK_HEADS; ++i)
                cp_async16z(smem_u32(to + (warp * (TK_KEYS / TK_HEADS) + i) * (val ? ldv : ldk)), src[i] + from, true);
        }
        cp_async_commit();
        cp_async_wait<0>();
        __syncthreads();
        if (!live) continue;
        float part[EPC] = {};
        const float* q = sq + warp * p.dim_p;
#pragma unroll 8
        for (int c = 0; c < chunks; ++c) {
            float f[EPC];
            unpack16(*reinterpret_cast<const uint4*>(sk + lane * ldk + map * p.dim_p + c * EPC), f, TC());
#pragma unroll
            for (int i = 0; i < EPC; ++i) part[i] = fmaf(f[i], q[c * EPC + i], part[i]);
        }
        float sc = 0.0f;
#pragma unroll
        for (int i = 0; i < EPC; ++i) sc += part[i];
        if (p.softcap > 0.0f) sc = p.softcap * tanhf(sc / p.softcap);
        if (k0 + lane >= ke) sc = -INFINITY;
        float pr;
        if (p.score_bias) {
            pr = k0 + lane < ke ? sigmoid(sc + bias) : 0.0f;
        } else {
            float mx = sc;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m, mx), corr = expf(m - mn);
            pr = expf(sc - mn);
            m = mn;
            l = l * corr + warp_sum(pr);
#pragma unroll
            for (int j = 0; j < VP; ++j) acc[j][0] *= corr, acc[j][1] *= corr;
        }
#pragma unroll 8
        for (int kk = 0; kk < TK_KEYS; ++kk) {
            const float w = __shfl_sync(0xffffffffu, pr, kk);
#pragma unroll
            for (int j = 0; j < VP; ++j) {
                const TC* v = sv + kk * ldv + min(2 * (lane + 32 * j), p.vdim_p - 2);     // beyond the head: never stored
                acc[j][0] = fmaf(w, load_as(v), acc[j][0]);
                acc[j][1] = fmaf(w, load_as(v + 1), acc[j][1]);
            }
        }
    }
    if (!live) return;
    const size_t o = ((size_t)t * p.heads * MAPS + h) * p.splits + s;
    if (lane == 0 && !p.score_bias) {
        p.part_ml[2 * o] = m;
        p.part_ml[2 * o + 1] = l;
    }
#pragma unroll
    for (int j = 0; j < VP; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int d = 2 * (lane + 32 * j) + i;
            if (d < p.vdim) p.part[o * p.vdim + d] = acc[j][i];
        }
}

// Splits of one (head, token) and the sink joined; with two maps the second is taken off the first and the rest normed.  part_ml
// null: the splits' plain sum.  gate: the head's, or null.  Every fourth split is a warpgroup's.
constexpr int JOIN_PARTS = 4;
template <int MAPS>
__global__ void __launch_bounds__(128 * JOIN_PARTS) k_gqa_join(const float* __restrict__ part, const float* __restrict__ part_ml, int heads, int splits, int vdim,
                                                               float sink, float lambda, float mul, float eps, const float* __restrict__ gate, int ldg,
                                                               float* __restrict__ mix, __nv_bfloat16* __restrict__ mixb, int ldm) {
    __shared__ float sw[MAPS][DC_MAX_SPLITS], red[33], sum[JOIN_PARTS - 1][256];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, t = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, share = threadIdx.x >> 7, d0 = threadIdx.x & 127;
    const size_t o = ((size_t)t * heads + h) * MAPS * splits;
    float x[2][MAPS][DC_MAX_SPLITS / JOIN_PARTS];         // vdim <= 256
    if (!part_ml) {
        if (threadIdx.x < DC_MAX_SPLITS) sw[0][threadIdx.x] = 1.0f;
    } else if (warp < MAPS) join_weights(part_ml + 2 * (o + warp * splits), splits, lane, sink, warp ? -lambda : 1.0f, sw[warp]);
    float v[2] = {0.0f, 0.0f}, ss = 0.0f;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < MAPS; ++i)
#pragma unroll
            for (int k = 0; k < DC_MAX_SPLITS / JOIN_PARTS; ++k) {
                const int s = share + JOIN_PARTS * k, d = d0 + 128 * j;
                x[j][i][k] = s < splits && d < vdim ? part[(o + i * splits + s) * vdim + d] : 0.0f;
            }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < MAPS; ++i)
#pragma unroll
            for (int k = 0; k < DC_MAX_SPLITS / JOIN_PARTS; ++k) v[j] = fmaf(x[j][i][k], sw[i][share + JOIN_PARTS * k], v[j]);
    if (share > 0) sum[share - 1][d0] = v[0], sum[share - 1][d0 + 128] = v[1];
    __syncthreads();
    if (share > 0) v[0] = v[1] = 0.0f;
    else
#pragma unroll
        for (int k = 0; k < JOIN_PARTS - 1; ++k) v[0] += sum[k][d0], v[1] += sum[k][d0 + 128];
    ss = v[0] * v[0] + v[1] * v[1];
    float f = MAPS > 1 ? mul / sqrtf(block_sum(ss, red) / (float)vdim + eps) : 1.0f;
    if (gate) f *= sigmoid(gate[(size_t)t * ldg + h]);
    if (share > 0) return;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int d = d0 + 128 * j;
        if (d >= vdim) break;
        const size_t at = (size_t)t * ldm + (size_t)h * vdim + d;
        if (mixb) mixb[at] = __float2bfloat16_rn(v[j] * f);
        else mix[at] = v[j] * f;
    }
}

template <typename TC, int MAPS>
int launch_tokens(dc_ctx* ctx, const TokenParams& p, int kv_heads, int T) {
    const size_t smem = (size_t)TK_HEADS * p.dim_p * 4 + (size_t)TK_KEYS * ((MAPS * p.dim_p + p.vdim_p) * sizeof(TC) + 32);
    const dim3 grid(p.splits, kv_heads * p.groups, T), block(TK_HEADS * 32);
#define DC_TK(VP)                                                                                               \
    do {                                                                                                        \
        DC_TRY(dc_kernel_setup_small(ctx, (const void*)k_gqa_tokens<TC, VP, MAPS>, (int)smem, "k_gqa_tokens")); \
        return dc_launch(ctx, "k_gqa_tokens", k_gqa_tokens<TC, VP, MAPS>, grid, block, smem, p);                \
    } while (0)
    if (p.vdim <= 64) DC_TK(1);
    if (p.vdim <= 128) DC_TK(2);
    DC_TK(4);
#undef DC_TK
}

// ---------------------------------------------------------------- prompts
struct PromptParams {
    const __nv_bfloat16* q;  // [T][heads * MAPS][ldq]
    int ldq, heads, per, dim, vdim, dim_p, vdim_p, v_at, window, keep;
    float scale, softcap, sink;
    float lambda, mul, eps;  // two maps
    const float* score_bias; // sigmoid weights
    const float* gate;       // [T][ldg] per head, or null
    int ldg;
    const int32_t *seq_ids, *positions, *starts, *tiles;     // tiles: (entry, first query of the entry) pairs
    CacheRef c;
    __nv_bfloat16* out;
    int ldm;
};

constexpr int PK = 64;           // keys per tile

// cap tanh(s / cap), s in units of cap: to about 2e-7 of the cap
__device__ __forceinline__ float soft_cap(float z, float cap) {
    return cap - __fdividef(2.0f * cap, 1.0f + ex2(2.8853900817779268f * z));
}

// One CTA per (QT = PQ / MAPS queries of one entry, head), sixteen rows (queries of one map) a warp; key and value tiles in
// a ring of ST stages, two CTAs an SM.  DP, VP: key and value size, padded.  SIGMOID: sigmoid weights, no denominator.
template <int DP, int VP, int PQ, int ST, int MAPS, bool SIGMOID>
__global__ void __launch_bounds__(2 * PQ, PQ == 128 ? 2 : 1) k_gqa_prompt(const PromptParams p) {
    constexpr int LD = DP + 8, LDK = MAPS * DP + 8, LDV = VP + 8, NT = 2 * PQ, CH = DP / 8, VCH = VP / 8, QT = PQ / MAPS;
    extern __shared__ __align__(16) uint8_t smem[];
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem);     // [PQ][LD]
    __nv_bfloat16* sK = sQ + PQ * LD;                               // [ST][PK][LDK]
    __nv_bfloat16* sV = sK + ST * PK * LDK;                         // [ST][PK][LDV]
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, head = blockIdx.y;
    const int tile0 = (int)(gridDim.x - 1 - blockIdx.x);           // later queries see more keys: they start first
    const int e = p.tiles[2 * tile0], q0 = p.tiles[2 * tile0 + 1] + QT * blockIdx.z;
    const int t0 = p.starts[e], n = p.starts[e + 1] - t0, pos0 = p.positions[t0], seq = p.seq_ids[t0];
    if (q0 % QT || q0 >= n) return;                                 // tiles are listed per DC_LATENT_QTILE queries
    const int last = pos0 + min(q0 + QT, n) - 1;
    const Keys keys = keys_of(pos0 + q0, last, p.window, p.keep);
    const int n_tiles = (keys.n + PK - 1) / PK, kc = p.dim_p / 8, vc = p.vdim_p / 8;
    const __nv_bfloat16* cache = reinterpret_cast<const __nv_bfloat16*>(p.c.arena);
    const int k_at = (head / p.per) * MAPS * p.dim_p, v_at = p.v_at + (head / p.per) * p.vdim_p;

    const int lrow = tid >> 3, lc = tid & 7;                        // eight threads per key row
    auto load = [&](int tile, int buf) {
#pragma unroll
        for (int i = 0; i < PK * 8 / NT; ++i) {
            const int key = lrow + NT / 8 * i, at = tile * PK + key;
            const bool ok = at < keys.n;
            const __nv_bfloat16* src = cache + p.c.at(seq, ok ? keys.at(at) : last);
            const uint32_t dk = smem_u32(sK + (buf * PK + key) * LDK), dv = smem_u32(sV + (buf * PK + key) * LDV);
#pragma unroll
            for (int c0 = 0; c0 < MAPS * CH; c0 += 8) {
                const int c = c0 + lc, of = MAPS > 1 ? c % CH : c;
                if (MAPS * CH % 8 && c >= MAPS * CH) break;
                const bool in = ok && of < kc;
                cp_async16z(dk + 16 * c, in ? src + k_at + (MAPS > 1 ? c / CH * p.dim_p : 0) + 8 * of : src, in);
            }
#pragma unroll
            for (int c0 = 0; c0 < VCH; c0 += 8) {
                const int c = c0 + lc;
                if (VCH % 8 && c >= VCH) break;
                const bool in = ok && c < vc;
                cp_async16z(dv + 16 * c, in ? src + v_at + 8 * c : src, in);
            }
        }
        cp_async_commit();
    };
    for (int i = tid; i < PQ * CH; i += NT) {                       // the queries come with the first tile
        const int r = i / CH, c = i - r * CH, qr = r % QT;
        const bool in = q0 + qr < n && 8 * c < p.ldq;
        cp_async16z(smem_u32(sQ + r * LD + 8 * c),
                    p.q + ((size_t)(t0 + q0 + (in ? qr : 0)) * p.heads * MAPS + head * MAPS + r / QT) * p.ldq + (in ? 8 * c : 0), in);
    }
#pragma unroll
    for (int i = 0; i < ST - 1; ++i)
        if (i < n_tiles) load(i, i);
        else cp_async_commit();
    // capped scores are in units of log2 e already, others are multiplied on the way into the exponential
    const bool capped = p.softcap > 0.0f;
    const float cap = p.softcap * 1.4426950408889634f, to_cap = capped ? p.scale / p.softcap : 0.0f;
    const float sl2 = capped ? 1.0f : p.scale * 1.4426950408889634f, sink2 = p.sink * 1.4426950408889634f;
    const int g = lane >> 2, t4 = lane & 3, mi = lane >> 3, r8 = lane & 7;
    const int map = MAPS > 1 ? 16 * warp / QT : 0, qrow = 16 * warp - map * QT;       // first query of the warp
    const int qpos0 = pos0 + q0 + qrow + g;
    const int window = p.window > 0 ? p.window : 0x7fffffff;
    float o[VCH][4];
#pragma unroll
    for (int i = 0; i < VCH; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const float bias2 = SIGMOID ? p.score_bias[head] * 1.4426950408889634f : 0.0f;
    // the sink is the first term of the sum (one lane of a row's four counts it)
    const bool sink = p.sink > -INFINITY;
    float m_run[2], l_run[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) m_run[h] = sink ? sink2 : -1e30f, l_run[h] = sink && t4 == 0 ? 1.0f : 0.0f;

    for (int tile = 0; tile < n_tiles; ++tile) {
        const int buf = tile % ST, k0 = keys.at(tile * PK), k1 = keys.at(tile * PK + PK - 1);
        cp_async_wait<ST - 2>();
        __syncthreads();         // the tile has landed; every warp is done with the stage that the next load fills
        if (tile + ST - 1 < n_tiles) load(tile + ST - 1, (tile + ST - 1) % ST);
        else cp_async_commit();
        const int wq0 = pos0 + q0 + qrow;
        if (k0 > wq0 + 15 || (k1 <= wq0 - window && k0 >= p.keep)) continue;         // nothing of the tile is seen by these queries
        float s[8][4];
#pragma unroll
        for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        const uint32_t qa = smem_u32(sQ + (16 * warp + (mi & 1) * 8 + r8) * LD + (mi >> 1) * 8);
        const uint32_t ka = smem_u32(sK + (buf * PK + (mi >> 1) * 8 + r8) * LDK + map * DP + (mi & 1) * 8);
#pragma unroll
        for (int kk = 0; kk < DP; kk += 16) {
            uint32_t a[4];
            ldsm_x4(qa + 2 * kk, a);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                uint32_t b[4];
                ldsm_x4(ka + 2 * (16 * np * LDK + kk), b);
                mma_bf16(s[2 * np], a, b[0], b[1]);
                mma_bf16(s[2 * np + 1], a, b[2], b[3]);
            }
        }
        if (capped) {
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) s[nt][j] = soft_cap(s[nt][j] * to_cap, cap);
        }
        if constexpr (SIGMOID) {
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) s[nt][j] = __fdividef(1.0f, 1.0f + ex2(-fmaf(s[nt][j], sl2, bias2)));
        }
        // the warp's sixteen queries see the whole tile, or the mask decides key by key
        if (!(k1 <= wq0 && wq0 + 15 - k0 < window)) {
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int kp = keys.at(tile * PK + 8 * nt + 2 * t4 + (j & 1)), qp = qpos0 + (j >> 1) * 8;
                    if (!(kp <= qp && (qp - kp < window || kp < p.keep))) s[nt][j] = SIGMOID ? 0.0f : -INFINITY;
                }
        }
        if constexpr (!SIGMOID) {
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
                    for (int i = 0; i < VCH; ++i) {
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
            for (int dp = 0; dp < VP / 16; ++dp) {
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
    }
    float mul[2] = {1.0f, 1.0f};
    if (!SIGMOID) mul[0] = 1.0f / l_run[0], mul[1] = 1.0f / l_run[1];
    if (MAPS > 1) {
        constexpr int LDX = VP + 4;
        float* other = reinterpret_cast<float*>(smem);              // [QT][LDX]: the second map's answers
        __syncthreads();                                            // every warp is done with queries, keys and values
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int nt = 0; nt < VCH; ++nt)
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    if (map) other[(qrow + g + 8 * h) * LDX + 8 * nt + 2 * t4 + j] = o[nt][2 * h + j] * mul[h];
        __syncthreads();
        if (map) return;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            float ss = 0.0f;
#pragma unroll
            for (int nt = 0; nt < VCH; ++nt)
#pragma unroll
                for (int j = 0; j < 2; ++j) {                       // zero beyond the head
                    float& v = o[nt][2 * h + j];
                    v = v * mul[h] - p.lambda * other[(qrow + g + 8 * h) * LDX + 8 * nt + 2 * t4 + j];
                    ss = fmaf(v, v, ss);
                }
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            mul[h] = p.mul / sqrtf(ss / (float)p.vdim + p.eps);
        }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int row = q0 + qrow + g + 8 * h;
        if (row >= n) continue;
        if (p.gate) mul[h] *= sigmoid(p.gate[(size_t)(t0 + row) * p.ldg + head]);
        __nv_bfloat16* dst = p.out + (size_t)(t0 + row) * p.ldm + (size_t)head * p.vdim;
#pragma unroll
        for (int nt = 0; nt < VCH; ++nt)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int c = 8 * nt + 2 * t4 + j;
                if (c < p.vdim) dst[c] = __float2bfloat16_rn(o[nt][2 * h + j] * mul[h]);
            }
    }
}

template <int DP, int VP, int PQ, int ST, int MAPS, bool SIGMOID>
int launch_prompt(dc_ctx* ctx, const PromptParams& p, int n_tiles) {
    constexpr int QT = PQ / MAPS, bytes = (PQ * (DP + 8) + ST * PK * (MAPS * DP + VP + 16)) * 2;
    static_assert(bytes <= 227 * 1024 && (MAPS == 1 || QT * (VP + 4) * 4 <= bytes), "shared memory");
    DC_TRY(dc_kernel_setup(ctx, (const void*)k_gqa_prompt<DP, VP, PQ, ST, MAPS, SIGMOID>, bytes, "k_gqa_prompt"));
    const dim3 grid(n_tiles, p.heads, QT < DC_LATENT_QTILE ? DC_LATENT_QTILE / QT : 1);
    return dc_launch(ctx, "k_gqa_prompt", k_gqa_prompt<DP, VP, PQ, ST, MAPS, SIGMOID>, grid, dim3(2 * PQ), (size_t)bytes, p);
}

CacheRef cache_ref(const dc_gqa_cache& c, int row) { return CacheRef{c.arena, c.tables, c.max_blocks, row}; }
float sink_of(const dc_gqa_mixer& m) { return m.sink ? m.sink_score : -INFINITY; }

}  // namespace

int dc_launch_gqa_prep(dc_ctx* ctx, const dc_gqa_mixer& m, const dc_step& st, const dc_gqa_cache& c, const dc_state_ref* sr, const float* proj,
                       int ldp, float eps, int max_pos, float* q, __nv_bfloat16* qb) {
    if (m.taps > 0) {
        if (!sr || m.rot.dims || m.qk_norm == DC_QK_NORM_ALL || m.off_v == m.off_k) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "gqa_prep: form not available with convolutions");
        const int C = dc_gqa_conv_cols(m);
        ConvParams p = {{proj, ldp, m.off_q, m.off_k, m.off_v, m.heads * m.maps, m.kv_heads * m.maps, m.kv_heads, m.dim, m.vdim, m.dim_p, m.vdim_p, m.v_at,
                         dc_gqa_ldq(m), 0, 0, max_pos, m.q_norm, m.k_norm, nullptr, eps, st.seq_ids, st.positions, cache_ref(c, m.row), q, qb},
                        {sr->base, sr->slot_bytes, sr->ring_off, st.seq_ids, st.positions, st.starts, st.E, m.taps, C, C}, m.conv,
                        m.qk_norm == DC_QK_NORM_HEAD, m.qk_norm == DC_QK_NORM_HEAD, m.v_norm, st.single};
        const int most = std::max(std::max(p.h.ldq, p.h.dim_p), p.h.vdim_p);
#define DC_CONV(VP) DC_TRY((c.f32 ? launch_prep_conv<float, VP>(ctx, p, st) : launch_prep_conv<__nv_bfloat16, VP>(ctx, p, st)))
        if (m.taps <= 4 && m.dim % 4 == 0 && m.vdim % 4 == 0 && most <= 128 && ldp % 4 == 0)
            DC_TRY((c.f32 ? launch_prep_conv4<float>(ctx, p, st) : launch_prep_conv4<__nv_bfloat16>(ctx, p, st)));
        else if (most <= 64) DC_CONV(2);
        else if (most <= 128) DC_CONV(4);
        else DC_CONV(8);
#undef DC_CONV
        return st.single ? DC_B200_OK : dc_launch_ring_update(ctx, st, *sr, proj, ldp, 0, C, m.taps);
    }
    if (m.qk_norm != DC_QK_NORM_ALL) {
        if (m.off_v == m.off_k) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "gqa_prep: values from the keys need the norm over all heads");
        HeadsParams p = {proj, ldp, m.off_q, m.off_k, m.off_v, m.heads * m.maps, m.kv_heads * m.maps, m.kv_heads, m.dim, m.vdim, m.dim_p, m.vdim_p, m.v_at,
                         dc_gqa_ldq(m), m.rot.dims, m.halves, max_pos, m.q_norm, m.k_norm, m.cos_sin, eps, st.seq_ids, st.positions, cache_ref(c, m.row), q, qb};
        const int units = p.nq + p.nk + p.nv, most = std::max(std::max(p.ldq, p.dim_p), p.vdim_p);
        const dim3 grid(st.T, (units + 7) / 8), block(256);
        if (m.dim % 4 == 0 && m.vdim % 4 == 0 && m.rot.dims % (m.halves ? 8 : 4) == 0 && ldp % 4 == 0) {
#define DC_HEADS4(TC, NV)                                                                                                                                    \
    return st.T > DC_MAX_T ? dc_launch(ctx, "k_gqa_prep_heads4", k_gqa_prep_heads4<TC, NV, 3>, dim3(st.T, (units + 23) / 24), block, 0, p)                    \
                           : dc_launch(ctx, "k_gqa_prep_heads4", k_gqa_prep_heads4<TC, NV, 1>, grid, block, 0, p)
            if (c.f32 && most <= 128) DC_HEADS4(float, 1);
            if (c.f32) DC_HEADS4(float, 2);
            if (most <= 128) DC_HEADS4(__nv_bfloat16, 1);
            DC_HEADS4(__nv_bfloat16, 2);
#undef DC_HEADS4
        }
#define DC_HEADS(VP)                                                                                                          \
    return c.f32 ? dc_launch(ctx, "k_gqa_prep_heads", k_gqa_prep_heads<float, VP>, grid, block, 0, p)                          \
                 : dc_launch(ctx, "k_gqa_prep_heads", k_gqa_prep_heads<__nv_bfloat16, VP>, grid, block, 0, p)
        if (most <= 64) DC_HEADS(2);
        if (most <= 128) DC_HEADS(4);
        DC_HEADS(8);
#undef DC_HEADS
    }
    if (m.halves || m.maps > 1 || m.off_v != m.off_k) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "gqa_prep: form not available with the norm over all heads");
    int lanes = 3;               // a head's pairs, padding included, up to a power of two
    while (2 << lanes < dc_gqa_ldq(m)) ++lanes;
    PrepParams p = {proj, ldp, m.off_q, m.off_k, m.heads, m.kv_heads, m.dim, m.dim_p, dc_gqa_ldq(m), m.rot.dims, max_pos, lanes, m.q_norm, m.k_norm, m.cos_sin,
                    eps, st.seq_ids, st.positions, cache_ref(c, m.row), q, qb};
    const int parts = st.T > DC_MAX_T ? 1 : std::min(m.heads, (m.heads * m.dim + 511) / 512);      // few tokens: more CTAs each
    const dim3 grid(st.T, parts + 1), block(256);
    if (c.f32) return dc_launch(ctx, "k_gqa_prep", k_gqa_prep<float>, grid, block, 0, p);
    return dc_launch(ctx, "k_gqa_prep", k_gqa_prep<__nv_bfloat16>, grid, block, 0, p);
}

int dc_launch_gqa_tokens(dc_ctx* ctx, const dc_gqa_mixer& m, const dc_step& st, const dc_gqa_cache& c, const float* q, const float* proj, int ldp, int splits,
                         float* part, float* part_ml, float eps, float* mix, __nv_bfloat16* mixb, int ldm) {
    const float* gate = m.off_g < 0 ? nullptr : proj + m.off_g;
    const float* ml = m.score_bias ? nullptr : part_ml;
    if (m.score_bias && (m.maps > 1 || m.sink)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "gqa_tokens: form not available with sigmoid weights");
    const int per = m.heads / m.kv_heads;
    TokenParams p = {q, dc_gqa_ldq(m), m.heads, per, (per * m.maps + TK_HEADS - 1) / TK_HEADS, m.dim, m.vdim, m.dim_p, m.vdim_p, m.v_at, m.window, m.keep, splits,
                     m.scale, m.softcap, st.seq_ids, st.positions, cache_ref(c, m.row), m.score_bias, part, part_ml};
    if (m.maps > 1) {
        DC_TRY((c.f32 ? launch_tokens<float, 2>(ctx, p, m.kv_heads, st.T) : launch_tokens<__nv_bfloat16, 2>(ctx, p, m.kv_heads, st.T)));
        return dc_launch(ctx, "k_gqa_join", k_gqa_join<2>, dim3(m.heads, st.T), dim3(128 * JOIN_PARTS), 0, part, ml, m.heads, splits, m.vdim, sink_of(m), m.lambda,
                         1.0f - m.diff, eps, gate, ldp, mix, mixb, ldm);
    }
    DC_TRY((c.f32 ? launch_tokens<float, 1>(ctx, p, m.kv_heads, st.T) : launch_tokens<__nv_bfloat16, 1>(ctx, p, m.kv_heads, st.T)));
    return dc_launch(ctx, "k_gqa_join", k_gqa_join<1>, dim3(m.heads, st.T), dim3(128 * JOIN_PARTS), 0, part, ml, m.heads, splits, m.vdim, sink_of(m), 0.0f, 1.0f, eps,
                     gate, ldp, mix, mixb, ldm);
}

int dc_launch_gqa_prompt(dc_ctx* ctx, const dc_gqa_mixer& m, const dc_step& st, const dc_gqa_cache& c, const int32_t* tiles, int n_tiles,
                         const __nv_bfloat16* qb, const float* proj, int ldp, float eps, __nv_bfloat16* mixb, int ldm) {
    PromptParams p = {qb, dc_gqa_ldq(m), m.heads, m.heads / m.kv_heads, m.dim, m.vdim, m.dim_p, m.vdim_p, m.v_at, m.window, m.keep, m.scale, m.softcap, sink_of(m),
                      m.lambda, 1.0f - m.diff, eps, m.score_bias, m.off_g < 0 ? nullptr : proj + m.off_g, ldp, st.seq_ids, st.positions, st.starts, tiles, cache_ref(c, m.row), mixb, ldm};
    // the smallest pair of padded key and value sizes that holds the head
#define DC_PROMPT(DP, VP, PQ, ST, MAPS)                                                                  \
    if (m.maps == MAPS && !m.score_bias && m.dim <= DP && m.vdim <= VP) return launch_prompt<DP, VP, PQ, ST, MAPS, false>(ctx, p, n_tiles)
#define DC_PROMPT_SIGMOID(DP, VP, PQ, ST)                                                                \
    if (m.maps == 1 && m.score_bias && m.dim <= DP && m.vdim <= VP) return launch_prompt<DP, VP, PQ, ST, 1, true>(ctx, p, n_tiles)
    DC_PROMPT(32, 32, 128, 3, 1);
    DC_PROMPT(32, 64, 128, 3, 1);
    DC_PROMPT(64, 64, 128, 3, 1);
    DC_PROMPT(96, 96, 128, 2, 1);
    DC_PROMPT(64, 128, 128, 2, 1);
    DC_PROMPT(128, 128, 128, 2, 1);
    DC_PROMPT(256, 256, 64, 2, 1);
    DC_PROMPT(32, 32, 128, 3, 2);
    DC_PROMPT(32, 64, 128, 3, 2);
    DC_PROMPT(64, 64, 128, 3, 2);
    DC_PROMPT(64, 128, 128, 2, 2);
    DC_PROMPT(128, 128, 128, 2, 2);
    DC_PROMPT(128, 256, 64, 2, 2);
    DC_PROMPT_SIGMOID(32, 32, 128, 3);
    DC_PROMPT_SIGMOID(64, 32, 128, 3);
    DC_PROMPT_SIGMOID(64, 64, 128, 3);
    DC_PROMPT_SIGMOID(96, 96, 128, 2);
    DC_PROMPT_SIGMOID(128, 128, 128, 2);
    DC_PROMPT_SIGMOID(256, 256, 64, 2);
#undef DC_PROMPT_SIGMOID
#undef DC_PROMPT
    return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "gqa_prompt: head sizes %d and %d", m.dim, m.vdim);
}
