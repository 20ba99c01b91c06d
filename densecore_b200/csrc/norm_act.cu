// Norms around the sublayers of a layer-list decoder: RMS norm of a sublayer's output added to the f32 residual;
// RMS norm of residual rows (ahead of a layer's products, and the output norm on the rows whose logits are wanted), with
// what a step still owes the residual added on the way; the same over a residual of several streams.
#include "dc_common.cuh"
#include "dc_launch.cuh"
#include "dc_stack.h"
#include "dc_stack.cuh"

namespace {

// Rows are padded with zeros to ld (a multiple of eight); so are y's rows and the weight's allocation.  KEEP: groups of
// four values that a thread holds.
template <int KEEP>
__global__ void __launch_bounds__(256) k_post_norm(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, int H,
                                                   int ld, float eps, __nv_bfloat16* __restrict__ xb) {
    __shared__ float red[33];
    dc::pdl_launch_dependents();
    const int n4 = ld / 4;
    float4 wv[KEEP], xv[KEEP], yv[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        wv[j] = i < n4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    dc::pdl_wait();
    const size_t off = (size_t)blockIdx.x * ld;
    const float4 *y4 = reinterpret_cast<const float4*>(y + off), *x4 = reinterpret_cast<const float4*>(x + off);
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        yv[j] = i < n4 ? y4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        xv[j] = i < n4 ? x4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j) ss += (yv[j].x * yv[j].x + yv[j].y * yv[j].y) + (yv[j].z * yv[j].z + yv[j].w * yv[j].w);
    const float inv = 1.0f / sqrtf(dc::block_sum(ss, red) / (float)H + eps);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        if (i >= n4) continue;
        float4 r;
        r.x = fmaf(yv[j].x * inv, wv[j].x, xv[j].x);
        r.y = fmaf(yv[j].y * inv, wv[j].y, xv[j].y);
        r.z = fmaf(yv[j].z * inv, wv[j].z, xv[j].z);
        r.w = fmaf(yv[j].w * inv, wv[j].w, xv[j].w);
        reinterpret_cast<float4*>(x + off)[i] = r;
        if (xb) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(r.x, r.y), hi = __floats2bfloat162_rn(r.z, r.w);
            reinterpret_cast<uint2*>(xb + off)[i] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        }
    }
}

// Rows as above; KEEP as above.
template <int KEEP>
__global__ void __launch_bounds__(256) k_norm_rows(const float* __restrict__ x, const float* __restrict__ w, const int32_t* __restrict__ rows,
                                                   int first, int H, int ld, float eps, float* __restrict__ out,
                                                   __nv_bfloat16* __restrict__ outb, int ldo) {
    __shared__ float red[33];
    dc::pdl_launch_dependents();
    const int n4 = ld / 4;
    float4 wv[KEEP], xv[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        wv[j] = i < n4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    dc::pdl_wait();
    const int r = rows ? rows[blockIdx.x] : first + (int)blockIdx.x;
    const float4* x4 = reinterpret_cast<const float4*>(x + (size_t)r * ld);
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        xv[j] = i < n4 ? x4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j) ss += (xv[j].x * xv[j].x + xv[j].y * xv[j].y) + (xv[j].z * xv[j].z + xv[j].w * xv[j].w);
    const float inv = 1.0f / sqrtf(dc::block_sum(ss, red) / (float)H + eps);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        if (i >= n4) continue;
        const float4 v = make_float4(xv[j].x * inv * wv[j].x, xv[j].y * inv * wv[j].y, xv[j].z * inv * wv[j].z, xv[j].w * inv * wv[j].w);
        if (outb) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
            reinterpret_cast<uint2*>(outb + (size_t)blockIdx.x * ldo)[i] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
            reinterpret_cast<float4*>(out + (size_t)blockIdx.x * ldo)[i] = v;
        }
    }
}

// Rows as above.  The step's row and the gathered rows (bf16 or f32, pitch sum.ld, a multiple of eight) are added first.
template <int KEEP>
__global__ void __launch_bounds__(256) k_pre_norm(float* __restrict__ x, const float* __restrict__ step, const dc_row_sum sum,
                                                  const float* __restrict__ w, int H, int ld, float eps, float* __restrict__ out,
                                                  __nv_bfloat16* __restrict__ outb) {
    __shared__ float red[33];
    __shared__ int32_t s_rows[DC_MOE_MAX_TOP];
    dc::pdl_launch_dependents();
    const int n4 = ld / 4;
    float4 wv[KEEP], xv[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        wv[j] = w && i < n4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    dc::pdl_wait();
    const size_t off = (size_t)blockIdx.x * ld;
    float4* x4 = reinterpret_cast<float4*>(x + off);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        xv[j] = i < n4 ? x4[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (sum.k) {
        if (threadIdx.x < (unsigned)sum.k) s_rows[threadIdx.x] = sum.rows[blockIdx.x * sum.k + threadIdx.x];
        __syncthreads();
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
            const int i = threadIdx.x + 256 * j;
            if (i < n4) dc::add4(xv[j], dc::row_sum4(sum, s_rows, i));
        }
    }
    if (step)
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
            const int i = threadIdx.x + 256 * j;
            if (i < n4) dc::add4(xv[j], reinterpret_cast<const float4*>(step)[i]);
        }
    if (sum.k || step)
#pragma unroll
        for (int j = 0; j < KEEP; ++j) {
            const int i = threadIdx.x + 256 * j;
            if (i < n4) x4[i] = xv[j];
        }
    if (!w) return;
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) ss += (xv[j].x * xv[j].x + xv[j].y * xv[j].y) + (xv[j].z * xv[j].z + xv[j].w * xv[j].w);
    const float inv = 1.0f / sqrtf(dc::block_sum(ss, red) / (float)H + eps);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + 256 * j;
        if (i >= n4) continue;
        const float4 v = make_float4(xv[j].x * inv * wv[j].x, xv[j].y * inv * wv[j].y, xv[j].z * inv * wv[j].z, xv[j].w * inv * wv[j].w);
        if (outb) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
            reinterpret_cast<uint2*>(outb + off)[i] = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
        } else {
            reinterpret_cast<float4*>(out + off)[i] = v;
        }
    }
}

// S: streams at most.  Rows as above; NT threads, KEEP groups of four columns each.
template <int S, int KEEP, int NT>
__global__ void __launch_bounds__(NT) k_hyper_norm(const dc_hyper hy, const float* __restrict__ w, const int32_t* __restrict__ rows, int first, int H, int ld,
                                                   float eps, float* __restrict__ out, __nv_bfloat16* __restrict__ outb) {
    __shared__ float red[33], coef[S * (S + 2)];
    __shared__ int32_t s_rows[DC_MOE_MAX_TOP];
    constexpr int AHEAD = S * KEEP <= 8 ? KEEP : S >= 8 ? 1 : 8 / S;      // groups whose streams are in flight together
    dc::pdl_launch_dependents();
    const int n4 = ld / 4;
    float4 wv[KEEP], u[KEEP];
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + NT * j;
        wv[j] = w && i < n4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float own = threadIdx.x < S * (S + 2) ? dc::hyper_coefficient<S>(hy, threadIdx.x) : 0.0f;
    dc::pdl_wait();
    const int t = rows ? rows[blockIdx.x] : first + (int)blockIdx.x;
    float ss = 0.0f;
#pragma unroll
    for (int j0 = 0; j0 < KEEP; j0 += AHEAD) {
        float4 v[AHEAD][S], y[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int i = threadIdx.x + NT * (j0 + j);
            y[j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i >= n4) continue;
            dc::hyper_load<S>(hy, t, i, ld, v[j]);
            if (hy.y && !hy.sum.k) y[j] = *reinterpret_cast<const float4*>(hy.y + (size_t)t * ld + 4 * i);
        }
        if (j0 == 0) {
            if (threadIdx.x < (unsigned)hy.sum.k) s_rows[threadIdx.x] = hy.sum.rows[t * hy.sum.k + threadIdx.x];
            if (threadIdx.x < S * (S + 2)) coef[threadIdx.x] = own;
            __syncthreads();
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int i = threadIdx.x + NT * (j0 + j);
            u[j0 + j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i >= n4) continue;
            if (hy.sum.k) y[j] = dc::row_sum4(hy.sum, s_rows, i);
            const float4 r = u[j0 + j] = dc::hyper_mix<S>(hy, coef, t, i, ld, v[j], y[j], hy.x_out != nullptr);
            ss += (r.x * r.x + r.y * r.y) + (r.z * r.z + r.w * r.w);
        }
    }
    const float inv = w ? 1.0f / sqrtf(dc::block_sum(ss, red) / (float)H + eps) : 1.0f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
        const int i = threadIdx.x + NT * j;
        if (i >= n4) continue;
        float4 v = u[j];
        if (w) v = make_float4(v.x * inv * wv[j].x, v.y * inv * wv[j].y, v.z * inv * wv[j].z, v.w * inv * wv[j].w);
        if (outb) reinterpret_cast<uint2*>(outb + (size_t)blockIdx.x * ld)[i] = make_uint2(dc::pack_bf2(v.x, v.y), dc::pack_bf2(v.z, v.w));
        else reinterpret_cast<float4*>(out + (size_t)blockIdx.x * ld)[i] = v;
    }
}

template <int S>
int launch_hyper(dc_ctx* ctx, const dc_hyper& hy, const float* w, const int32_t* rows, int first, int R, int H, int ld, float eps, float* out, __nv_bfloat16* outb) {
#define DC_HYPER(KEEP, NT) return dc_launch(ctx, "k_hyper_norm", k_hyper_norm<S, KEEP, NT>, dim3(R), dim3(NT), 0, hy, w, rows, first, H, ld, eps, out, outb)
    if (R <= DC_MAX_T) {         // few tokens: a group a thread
        if (ld <= 1024) DC_HYPER(1, 256);
        if (ld <= 2048) DC_HYPER(1, 512);
        if (ld <= 4096) DC_HYPER(1, 1024);
        DC_HYPER(2, 1024);
    }
    if (ld <= 1024) DC_HYPER(1, 256);
    if (ld <= 2048) DC_HYPER(2, 256);
    if (ld <= 4096) DC_HYPER(4, 256);
    DC_HYPER(8, 256);
#undef DC_HYPER
}

}  // namespace

int dc_launch_hyper_norm(dc_ctx* ctx, const dc_hyper& hy, const float* w, const int32_t* rows, int first, int R, int H, int ld, float eps, float* out,
                         __nv_bfloat16* outb) {
    if (ld % 8 || ld > 8192 || hy.streams < 1 || hy.streams > DC_MAX_STREAMS || hy.sum.k > DC_MOE_MAX_TOP || (hy.sum.k && hy.sum.ld != ld) || hy.x == hy.x_out)
        return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "hyper_norm: bad operand");
    if (hy.streams <= 2) return launch_hyper<2>(ctx, hy, w, rows, first, R, H, ld, eps, out, outb);
    if (hy.streams <= 4) return launch_hyper<4>(ctx, hy, w, rows, first, R, H, ld, eps, out, outb);
    return launch_hyper<DC_MAX_STREAMS>(ctx, hy, w, rows, first, R, H, ld, eps, out, outb);
}

int dc_launch_pre_norm(dc_ctx* ctx, float* x, const float* step, const dc_row_sum& sum, const float* w, int T, int H, int ld, float eps, float* out,
                       __nv_bfloat16* outb) {
    const dim3 grid(T), block(256);
    if (ld % 8 || sum.k > DC_MOE_MAX_TOP || (sum.k && (sum.ld < ld || sum.ld % 8))) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "pre_norm: bad operand");
    if (ld <= 1024) return dc_launch(ctx, "k_pre_norm", k_pre_norm<1>, grid, block, 0, x, step, sum, w, H, ld, eps, out, outb);
    if (ld <= 2048) return dc_launch(ctx, "k_pre_norm", k_pre_norm<2>, grid, block, 0, x, step, sum, w, H, ld, eps, out, outb);
    if (ld <= 4096) return dc_launch(ctx, "k_pre_norm", k_pre_norm<4>, grid, block, 0, x, step, sum, w, H, ld, eps, out, outb);
    if (ld <= 8192) return dc_launch(ctx, "k_pre_norm", k_pre_norm<8>, grid, block, 0, x, step, sum, w, H, ld, eps, out, outb);
    return dc_fail(ctx, DC_B200_UNSUPPORTED, "pre_norm: width %d is too large", H);
}

int dc_launch_post_norm(dc_ctx* ctx, float* x, const float* y, const float* w, int T, int H, int ld, float eps, __nv_bfloat16* xb) {
    const dim3 grid(T), block(256);
    if (ld <= 1024) return dc_launch(ctx, "k_post_norm", k_post_norm<1>, grid, block, 0, x, y, w, H, ld, eps, xb);
    if (ld <= 2048) return dc_launch(ctx, "k_post_norm", k_post_norm<2>, grid, block, 0, x, y, w, H, ld, eps, xb);
    if (ld <= 4096) return dc_launch(ctx, "k_post_norm", k_post_norm<4>, grid, block, 0, x, y, w, H, ld, eps, xb);
    if (ld <= 8192) return dc_launch(ctx, "k_post_norm", k_post_norm<8>, grid, block, 0, x, y, w, H, ld, eps, xb);
    return dc_fail(ctx, DC_B200_UNSUPPORTED, "post_norm: width %d is too large", H);
}

int dc_launch_norm_rows(dc_ctx* ctx, const float* x, const float* w, const int32_t* rows, int first, int R, int H, int ld, float eps,
                        float* out, __nv_bfloat16* outb, int ldo) {
    const dim3 grid(R), block(256);
    if (ld % 8 || ldo < ld || ldo % 8) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "norm_rows: bad pitch");
    if (ld <= 1024) return dc_launch(ctx, "k_norm_rows", k_norm_rows<1>, grid, block, 0, x, w, rows, first, H, ld, eps, out, outb, ldo);
    if (ld <= 2048) return dc_launch(ctx, "k_norm_rows", k_norm_rows<2>, grid, block, 0, x, w, rows, first, H, ld, eps, out, outb, ldo);
    if (ld <= 4096) return dc_launch(ctx, "k_norm_rows", k_norm_rows<4>, grid, block, 0, x, w, rows, first, H, ld, eps, out, outb, ldo);
    if (ld <= 8192) return dc_launch(ctx, "k_norm_rows", k_norm_rows<8>, grid, block, 0, x, w, rows, first, H, ld, eps, out, outb, ldo);
    return dc_fail(ctx, DC_B200_UNSUPPORTED, "norm_rows: width %d is too large", H);
}
