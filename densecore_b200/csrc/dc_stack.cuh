// Scalar device functions of the layer-list decoders' kernels (f32 throughout).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "dc_common.cuh"
#include "dc_stack.h"

namespace dc {

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float relu2(float z) {
    z = fmaxf(z, 0.0f);
    return z * z;
}
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ unsigned long long argmax_key(float f, int row) {
    uint32_t u = __float_as_uint(f);
    u = (f != f) ? 0u : ((u & 0x80000000u) ? ~u : (u | 0x80000000u));
    return ((unsigned long long)u << 32) | (0xFFFFFFFFu - (uint32_t)row);
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sum over a CTA of up to 1024 threads; red: 33 floats of shared memory.  Every thread gets the result.
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    if (threadIdx.x < 32) {
        float s = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.0f;
        s = warp_sum(s);
        if (threadIdx.x == 0) red[32] = s;
    }
    __syncthreads();
    return red[32];
}
// a pair of f32 values in one register pair, two multiply-adds per instruction
__device__ __forceinline__ uint64_t pair(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpair(uint64_t v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ void store_as(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_as(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float load_as(const float* p) { return *p; }
__device__ __forceinline__ float load_as(const __nv_bfloat16* p) { return __bfloat162float(*p); }
// ---- epilogues of the products (dc_lin_epi)
__device__ __forceinline__ float pair_value(const dc_lin_epi& e, float gate, float up) {
    if (e.pair_kind == DC_PAIR_GELU) return gelu_tanh(gate) * up;
    if (e.pair_kind == DC_PAIR_SILU) return silu(gate) * up;
    gate = fminf(gate, e.limit);
    up = fminf(fmaxf(up, -e.limit), e.limit);
    return gate * sigmoid(1.702f * gate) * (up + 1.0f);
}
__device__ __forceinline__ void put_pair(const dc_lin_epi& e, int t, int pair, float v) {
    const size_t at = (size_t)t * e.ldp + pair;
    if (e.poutb) e.poutb[at] = __float2bfloat16_rn(v);
    else e.pout[at] = v;
}
// returns the stored value
__device__ __forceinline__ float put_row(const dc_lin_epi& e, int t, int row, float v) {
    if (e.bias) v += e.bias[row];
    if (row < e.act_rows) v = e.act == DC_ACT_SILU ? silu(v) : relu2(v);
    if (e.tok_scale) v *= e.tok_scale[t];
    const size_t at = (size_t)t * e.ldo + row;
    if (e.outb) {
        e.outb[at] = __float2bfloat16_rn(v);
    } else {
        if (e.add) v += e.out[at];
        e.out[at] = v;
    }
    return v;
}

// ---- blocks of B tokens that entries are cut into from their own start
struct BlockRef {
    int e, t0, n;
};
template <int B>
__device__ __forceinline__ int block_base(const int32_t* starts, int e) {
    int b = 0;
    for (int i = 0; i < e; ++i) b += (starts[i + 1] - starts[i] + B - 1) / B;
    return b;
}
template <int B>
__device__ __forceinline__ BlockRef block_at(const int32_t* starts, int E, int blk) {
    for (int e = 0; e < E; ++e) {
        const int n = starts[e + 1] - starts[e], nb = (n + B - 1) / B;
        if (blk < nb) return BlockRef{e, starts[e] + blk * B, min(B, n - blk * B)};
        blk -= nb;
    }
    return BlockRef{0, 0, 0};
}
// ---- short causal convolutions
__device__ __forceinline__ int entry_of(const int32_t* starts, int E, int t) {
    int e = 0;
    while (e + 1 < E && starts[e + 1] <= t) ++e;
    return e;
}

// Convolution of one channel at token t (local index i in its entry, position pos): weights w[j * ldw], the last tap for
// the token itself; inputs before the entry come from the ring, before position 0 they are zero.
__device__ __forceinline__ float conv_at(const float* __restrict__ proj, int ldp, const float* __restrict__ ring, int C, int rc, int taps,
                                         const float* __restrict__ w, int ldw, int col, int t, int i, int pos) {
    float s = 0.0f;
    if (i >= taps - 1) {
        const float* in = proj + (size_t)(t - taps + 1) * ldp + col;
#pragma unroll 4
        for (int j = 0; j < taps; ++j) s = fmaf(w[(size_t)j * ldw], in[(size_t)j * ldp], s);
        return s;
    }
    for (int j0 = 0; j0 < taps; j0 += 4) {      // four taps' loads in flight, none behind a branch
        float in[4], wj[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int j = min(j0 + k, taps - 1), back = taps - 1 - j;
            const float* src = back <= i ? proj + (size_t)(t - back) * ldp + col : ring + (size_t)(max(pos - back, 0) % taps) * C + rc;
            in[k] = *src;
            wj[k] = w[(size_t)j * ldw];
            if (j0 + k >= taps || pos < back) in[k] = 0.0f;
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) s = fmaf(wj[k], in[k], s);
    }
    return s;
}

struct ConvRef {
    uint8_t* base;
    size_t slot_bytes, ring_off;
    const int32_t *seq_ids, *positions, *starts;
    int E, taps, C, ldw;     // C: channels of a ring row; ldw: pitch of the convolution weights [taps][ldw]
    __device__ float* ring(int seq) const { return reinterpret_cast<float*>(base + (size_t)seq * slot_bytes + ring_off); }
};

// ---- a residual of several streams (dc_hyper)
// Sixteen-byte groups of rows named by a sum, added up.
__device__ __forceinline__ void add4(float4& a, float4 b) { a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w; }
__device__ __forceinline__ float4 row_sum4(const dc_row_sum& sum, const int32_t* rows, int i) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int k = 0; k < sum.k; ++k) {
        const size_t at = (size_t)rows[k] * sum.ld + 4 * i;
        if (sum.yb) {
            const uint2 u = *reinterpret_cast<const uint2*>(sum.yb + at);
            add4(v, make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u)));
        } else {
            add4(v, *reinterpret_cast<const float4*>(sum.y + at));
        }
    }
    return v;
}
// Coefficient i of the table that hyper_mix reads, padded with zeros to S streams: in [S] | out [S], times mul | mix [S][S].  A
// thread below S (S + 2) has one and puts it there.
template <int S>
__device__ __forceinline__ float hyper_coefficient(const dc_hyper& h, int i) {
    const int n = h.streams;
    if (i < S) return i >= n ? 0.0f : h.next ? h.next[i] : 1.0f;
    if (i < 2 * S) return i - S < n && h.done ? h.mul * h.done[n + i - S] : 0.0f;
    const int s = (i - 2 * S) / S, t = (i - 2 * S) % S;
    return s >= n || t >= n ? 0.0f : h.done ? h.done[2 * n + s * n + t] : s == t ? 1.0f : 0.0f;
}
// Group i of four columns of token t: the streams,
template <int S>
__device__ __forceinline__ void hyper_load(const dc_hyper& h, int t, int i, int ld, float4 (&v)[S]) {
#pragma unroll
    for (int s = 0; s < S; ++s) {
        const size_t row = h.first ? t : (size_t)t * h.streams + s;
        v[s] = s < h.streams ? *reinterpret_cast<const float4*>(h.x + row * ld + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
}
// the streams anew with the sublayer's output y (to x_out if store), and u.
template <int S>
__device__ __forceinline__ float4 hyper_mix(const dc_hyper& h, const float* c, int t, int i, int ld, const float4 (&v)[S], float4 y, bool store) {
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int to = 0; to < S; ++to) {
        const float o = c[S + to], in = c[to];
        float4 r = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
        for (int s = 0; s < S; ++s) {
            const float m = c[2 * S + s * S + to];
            r.x = fmaf(m, v[s].x, r.x), r.y = fmaf(m, v[s].y, r.y), r.z = fmaf(m, v[s].z, r.z), r.w = fmaf(m, v[s].w, r.w);
        }
        if (store && to < h.streams) *reinterpret_cast<float4*>(h.x_out + ((size_t)t * h.streams + to) * ld + 4 * i) = r;
        u.x = fmaf(in, r.x, u.x), u.y = fmaf(in, r.y, u.y), u.z = fmaf(in, r.z, u.z), u.w = fmaf(in, r.w, u.w);
    }
    return u;
}

// ---- cached rows of a sequence's tokens
__device__ __forceinline__ int first_key(int pos, int window) { return window > 0 ? max(0, pos - window + 1) : 0; }

struct CacheRef {
    void* arena;
    const int32_t* tables;
    int max_blocks, row;     // row: elements per cached token
    __device__ size_t at(int seq, int pos) const {
        return ((size_t)tables[(size_t)seq * max_blocks + pos / DC_KV_BLOCK] * DC_KV_BLOCK + pos % DC_KV_BLOCK) * row;
    }
};

// One warp: what each of up to DC_MAX_SPLITS key splits, given as (largest score, sum of weights) pairs, counts in their join,
// times mul.  sink: score of one more term of the denominator (-inf: none).
__device__ __forceinline__ void join_weights(const float* ml, int splits, int lane, float sink, float mul, float* w) {
    constexpr int PER = DC_MAX_SPLITS / 32;
    float m[PER], l[PER], M = sink, L = 0.0f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int s = lane + 32 * j;
        const float2 v = s < splits ? *reinterpret_cast<const float2*>(ml + 2 * s) : make_float2(-INFINITY, 0.0f);
        m[j] = v.x, l[j] = v.y;
        M = fmaxf(M, m[j]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
#pragma unroll
    for (int j = 0; j < PER; ++j) m[j] = expf(m[j] - M), L += l[j] * m[j];
    L = warp_sum(L) + expf(sink - M);
#pragma unroll
    for (int j = 0; j < PER; ++j) w[lane + 32 * j] = m[j] / L * mul;
}

// ---- copies, fragments and products of the attention and chunk kernels
__device__ __forceinline__ void unpack16(const uint4& v, float (&f)[8], __nv_bfloat16) {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        f[2 * i] = __uint_as_float(u[i] << 16);
        f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void unpack16(const uint4& v, float (&f)[4], float) {
    f[0] = __uint_as_float(v.x), f[1] = __uint_as_float(v.y), f[2] = __uint_as_float(v.z), f[3] = __uint_as_float(v.w);
}

__device__ __forceinline__ void cp_async16z(uint32_t dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;   // 0: the 16 bytes are zero-filled, the address is not read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void cp_async4z(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(ok ? 4 : 0) : "memory");
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf2(float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&h);
}

// 2^x (the hardware's approximation, relative error about 2^-22)
__device__ __forceinline__ float ex2(float x) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
    return r;
}

// asks for a 128-byte line of global memory to be brought into L2
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

}  // namespace dc
