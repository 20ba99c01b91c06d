// Norms around the sublayers of a layer-list decoder: RMS norm of a sublayer's output added to the f32 residual,
// and the output norm on the rows whose logits are wanted.
#include "dc_common.cuh"
#include "dc_launch.cuh"
#include "dc_stack.h"
#include "dc_stack.cuh"

namespace {

__global__ void __launch_bounds__(256) k_post_norm(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w, int H,
                                                   int ld, float eps, __nv_bfloat16* __restrict__ xb) {
    __shared__ float red[33];
    dc::pdl_launch_dependents();
    dc::pdl_wait();
    const size_t off = (size_t)blockIdx.x * ld;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < H; i += 256) {
        const float v = y[off + i];
        ss = fmaf(v, v, ss);
    }
    const float inv = 1.0f / sqrtf(dc::block_sum(ss, red) / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += 256) {
        const float v = x[off + i] + y[off + i] * inv * w[i];
        x[off + i] = v;
        if (xb) xb[off + i] = __float2bfloat16_rn(v);
    }
}

__global__ void __launch_bounds__(256) k_norm_rows(const float* __restrict__ x, const float* __restrict__ w, const int32_t* __restrict__ rows,
                                                   int first, int H, int ld, float eps, float* __restrict__ out,
                                                   __nv_bfloat16* __restrict__ outb, int ldo) {
    __shared__ float red[33];
    dc::pdl_launch_dependents();
    dc::pdl_wait();
    const int r = rows ? rows[blockIdx.x] : first + (int)blockIdx.x;
    const float* xr = x + (size_t)r * ld;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < H; i += 256) ss = fmaf(xr[i], xr[i], ss);
    const float inv = 1.0f / sqrtf(dc::block_sum(ss, red) / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += 256) {
        const float v = xr[i] * inv * w[i];
        if (outb) outb[(size_t)blockIdx.x * ldo + i] = __float2bfloat16_rn(v);
        else out[(size_t)blockIdx.x * ldo + i] = v;
    }
}

}  // namespace

int dc_launch_post_norm(dc_ctx* ctx, float* x, const float* y, const float* w, int T, int H, int ld, float eps, __nv_bfloat16* xb) {
    return dc_launch(ctx, "k_post_norm", k_post_norm, dim3(T), dim3(256), 0, x, y, w, H, ld, eps, xb);
}

int dc_launch_norm_rows(dc_ctx* ctx, const float* x, const float* w, const int32_t* rows, int first, int R, int H, int ld, float eps,
                        float* out, __nv_bfloat16* outb, int ldo) {
    return dc_launch(ctx, "k_norm_rows", k_norm_rows, dim3(R), dim3(256), 0, x, w, rows, first, H, ld, eps, out, outb, ldo);
}
