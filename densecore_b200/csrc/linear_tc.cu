// bf16 products y = W x for prompt-sized steps on the 5th-generation tensor cores.
//
// One CTA per 128 weight rows x 128 tokens: one thread keeps a ring of shared-memory stages full with tiled TMA
// loads (64 columns of both operands, 128-byte swizzle), one thread issues the UMMAs (128 x 128 x 16, f32
// accumulators in tensor memory), four warps read the accumulators out.  A weight row is a tensor-memory lane, so
// a warp's stores of one token are 32 consecutive outputs.  Two CTAs share an SM: one's read-out overlaps the
// other's products.  Large products use tiles of 128 x 256 instead (k_linear_tc_wide): one CTA per SM walks its share
// of them, with two sets of accumulators, so that the loads and products of a tile run while the tile before is read
// out by eight warps; the wider tile reads shared memory less often per product.  Its grouped form multiplies runs of sorted tokens with
// a matrix of their own each (experts); the runs' ends are device data, so every CTA lists the tiles itself, and a tile
// of few tokens takes narrower products.  All let the next kernel start only after every
// CTA has its tensor memory.  Columns beyond K and rows beyond the matrix are the zeros that TMA fills in.  Every wait is
// bounded; a CTA that gives up drains its copies, frees its tensor memory and leaves.
#include <algorithm>
#include <mutex>
#include <set>

#include "dc_common.cuh"
#include "dc_launch.cuh"
#include "dc_stack.h"
#include "dc_stack.cuh"
#include "dc_tcgen05.cuh"

using namespace dc;

namespace {

constexpr int LT_STAGES = 3, LT_TILE = 128 * 128;   // bytes of one operand of a stage: 128 rows of 64 bf16
constexpr int LT_THREADS = 192;
constexpr size_t LT_SMEM = (size_t)LT_STAGES * 2 * LT_TILE + 1024;

struct LtParams {
    int K, T;
    dc_lin_epi e;
    int* err;
};

// activations whose results are rounded to bf16: z / (1 + e^-z) with the hardware's exponential and division
__device__ __forceinline__ float quick_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float quick_clamped(float limit, float gate, float up) {
    gate = fminf(gate, limit);
    up = fminf(fmaxf(up, -limit), limit);
    return __fdividef(gate, 1.0f + __expf(-1.702f * gate)) * (up + 1.0f);
}

// f(v, c0) for every sixteen columns of the warp's tensor-memory lanes that belong to the step; the next ones are on their way
// meanwhile.
template <int COLS, typename F>
__device__ __forceinline__ void each16(uint32_t tmem, int n, F f) {
    int v[2][16];
    tmem_ld16(tmem, v[0]);
#pragma unroll 1
    for (int c0 = 0; c0 < COLS && c0 < n; c0 += 32) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int c = c0 + 16 * i;
            if (c >= n) break;
            tmem_ld_wait(v[i]);
            if (c + 16 < COLS && c + 16 < n) tmem_ld16(tmem + c + 16, v[i ^ 1]);
            f(v[i], c);
        }
    }
}

// Eight lanes (xor 1, 2, 4 times STEP) hold one row each, N pairs of tokens packed as bf16; afterwards a lane holds N / 4 tokens,
// eight rows each in a row of four registers.  Token of set k: 2 (N / 2 b1 + N / 4 b2 + k) + b0, b: the lane's bits.
template <int STEP, int N>
__device__ __forceinline__ void transpose8(const uint32_t (&r)[N], uint32_t (&out)[N / 4][4], int lane) {
    const bool b0 = lane & STEP, b1 = lane & 2 * STEP, b2 = lane & 4 * STEP;
    const uint32_t give = b0 ? 0x5410u : 0x7632u, mine0 = b0 ? 0x3254u : 0x5410u, mine1 = b0 ? 0x3276u : 0x7610u;
    uint32_t a[N];
#pragma unroll
    for (int j = 0; j < N; j += 2) {
        const uint32_t got = __shfl_xor_sync(0xffffffffu, __byte_perm(r[j], r[j + 1], give), STEP);
        a[j] = __byte_perm(r[j], got, mine0);
        a[j + 1] = __byte_perm(r[j + 1], got, mine1);
    }
    uint32_t b[N / 2][2];
#pragma unroll
    for (int j = 0; j < N / 2; ++j) {
        const uint32_t got = __shfl_xor_sync(0xffffffffu, b1 ? a[j] : a[j + N / 2], 2 * STEP), own = b1 ? a[j + N / 2] : a[j];
        b[j][0] = b1 ? got : own, b[j][1] = b1 ? own : got;
    }
#pragma unroll
    for (int j = 0; j < N / 4; ++j)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const uint32_t got = __shfl_xor_sync(0xffffffffu, b2 ? b[j][i] : b[j + N / 4][i], 4 * STEP), own = b2 ? b[j + N / 4][i] : b[j][i];
            out[j][i] = b2 ? got : own, out[j][2 + i] = b2 ? own : got;
        }
}

// Accumulators of a tile (rows: tensor-memory lanes, tokens: columns) to the output; a warp reads its quarter's lanes.  Grouped
// products end in clamped pairs or the rows' squares of relu, both with a factor per token, or in bf16 rows.
template <int COLS, bool GROUPED>
__device__ __forceinline__ void read_out(const LtParams& p, uint32_t tmem, int row0, int t0, int t1, int quarter, int lane) {
    const int row = row0 + 32 * quarter + lane, n = t1 - t0;
    const dc_lin_epi& e = p.e;
    tmem += (uint32_t)(32 * quarter) << 16;
    if (row0 + 32 * quarter >= e.pair0) {
        // lanes 2i (gate row) and 2i + 1 (up row) share one output row: each finishes eight tokens
        const bool up = lane & 1, gelu = !GROUPED && e.pair_kind == DC_PAIR_GELU, swish = !GROUPED && e.pair_kind == DC_PAIR_SILU;
        const int o = (row - e.pair0) >> 1, first = up ? 8 : 0;
        const bool in = o < e.n_pairs;
        const size_t at = (size_t)(t0 + first) * e.ldp + o;
        const bool wide = e.poutb && e.n_pairs % 8 == 0 && e.ldp % 8 == 0 && ((uintptr_t)e.poutb & 15) == 0;     // whole groups of eight outputs
        each16<COLS>(tmem, n, [&](int (&v)[16], int c0) {
            float h[8], f[8];        // factors: asked for ahead of the arithmetic
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] = GROUPED ? e.tok_scale[min(t0 + c0 + first + i, t1 - 1)] : 1.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float got = __int_as_float(__shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + 8], 1));
                const float mine = __int_as_float(up ? v[i + 8] : v[i]);
                const float gate = up ? got : mine, val = up ? mine : got;
                h[i] = (gelu ? gelu_tanh(gate) * val : swish ? quick_silu(gate) * val : quick_clamped(e.limit, gate, val)) * f[i];
            }
            const int m = in ? n - c0 - first : 0;
            if (wide) {
                uint32_t r[4], v8[1][4];
#pragma unroll
                for (int i = 0; i < 4; ++i) r[i] = pack_bf2(h[2 * i], h[2 * i + 1]);
                transpose8<2, 4>(r, v8, lane);
                const int tok = 2 * ((lane & 4 ? 2 : 0) + (lane & 8 ? 1 : 0)) + (lane & 2 ? 1 : 0);
                if (tok < m) *reinterpret_cast<uint4*>(e.poutb + at + (size_t)(c0 + tok) * e.ldp - ((lane >> 1) & 7)) = make_uint4(v8[0][0], v8[0][1], v8[0][2], v8[0][3]);
            } else if (GROUPED || e.poutb) {
                __nv_bfloat16* to = e.poutb + at + (size_t)c0 * e.ldp;
#pragma unroll
                for (int i = 0; i < 8; ++i, to += e.ldp)
                    if (i < m) *to = __float2bfloat16_rn(h[i]);
            } else {
                float* to = e.pout + at + (size_t)c0 * e.ldp;
#pragma unroll
                for (int i = 0; i < 8; ++i, to += e.ldp)
                    if (i < m) *to = h[i];
            }
        });
        return;
    }
    const bool in = row < e.n_store;
    const float bias = !GROUPED && in && e.bias ? e.bias[row] : 0.0f;
    const size_t at = (size_t)t0 * e.ldo + row;
    if (e.outb && e.n_store % 8 == 0 && e.ldo % 8 == 0 && ((uintptr_t)e.outb & 15) == 0) {       // whole groups of eight rows
        const bool act = !GROUPED && row < e.act_rows;
        const int tok = 2 * ((lane & 2 ? 4 : 0) + (lane & 4 ? 2 : 0)) + (lane & 1);
        each16<COLS>(tmem, n, [&](int (&v)[16], int c0) {
            uint32_t r[8], v8[2][4];
            if (GROUPED && e.act_rows) {
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    r[i] = pack_bf2(relu2(__int_as_float(v[2 * i])) * e.tok_scale[min(t0 + c0 + 2 * i, t1 - 1)],
                                    relu2(__int_as_float(v[2 * i + 1])) * e.tok_scale[min(t0 + c0 + 2 * i + 1, t1 - 1)]);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const float a = __int_as_float(v[2 * i]) + bias, b = __int_as_float(v[2 * i + 1]) + bias;
                    r[i] = act ? pack_bf2(quick_silu(a), quick_silu(b)) : pack_bf2(a, b);
                }
            }
            transpose8<1, 8>(r, v8, lane);
            const int m = in ? n - c0 : 0;
#pragma unroll
            for (int i = 0; i < 2; ++i)
                if (tok + 2 * i < m)
                    *reinterpret_cast<uint4*>(e.outb + at + (size_t)(c0 + tok + 2 * i) * e.ldo - (lane & 7)) = make_uint4(v8[i][0], v8[i][1], v8[i][2], v8[i][3]);
        });
    } else if (GROUPED || e.outb) {
        const bool act = row < e.act_rows;
        each16<COLS>(tmem, n, [&](int (&v)[16], int c0) {
            const int m = in ? n - c0 : 0;
            __nv_bfloat16* to = e.outb + at + (size_t)c0 * e.ldo;
#pragma unroll
            for (int i = 0; i < 16; ++i, to += e.ldo) {
                const float r = __int_as_float(v[i]) + bias;
                if (i < m) *to = __float2bfloat16_rn(!act ? r : GROUPED ? relu2(r) * e.tok_scale[t0 + c0 + i] : quick_silu(r));
            }
        });
    } else if (e.add) {
        each16<COLS>(tmem, n, [&](int (&v)[16], int c0) {
            const int m = in ? n - c0 : 0;
            float* to = e.out + at + (size_t)c0 * e.ldo;
#pragma unroll
            for (int i0 = 0; i0 < 16; i0 += 8, to += 8 * (size_t)e.ldo) {
                float old[8];
                float* at8 = to;
#pragma unroll
                for (int i = 0; i < 8; ++i, at8 += e.ldo) old[i] = i0 + i < m ? *at8 : 0.0f;          // loads ahead of the stores
                at8 = to;
#pragma unroll
                for (int i = 0; i < 8; ++i, at8 += e.ldo)
                    if (i0 + i < m) *at8 = old[i] + (__int_as_float(v[i0 + i]) + bias);
            }
        });
    } else {
        each16<COLS>(tmem, n, [&](int (&v)[16], int c0) {
            const int m = in ? n - c0 : 0;
            float* to = e.out + at + (size_t)c0 * e.ldo;
#pragma unroll
            for (int i = 0; i < 16; ++i, to += e.ldo)
                if (i < m) *to = __int_as_float(v[i]) + bias;
        });
    }
}

__global__ void __launch_bounds__(LT_THREADS, 2) k_linear_tc(const __grid_constant__ CUtensorMap wmap,
                                                             const __grid_constant__ CUtensorMap xmap, const LtParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bar[2 * LT_STAGES + 1];
    __shared__ uint32_t s_tmem;
    __shared__ int s_give_up;
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t full = smem_u32(s_bar), empty = full + 8 * LT_STAGES, acc = empty + 8 * LT_STAGES;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row0 = blockIdx.x * 128, t0 = blockIdx.y * 128;
    const int nk = (p.K + 63) / 64;
    volatile int* give_up = &s_give_up;
    if (warp == 1) {
        tmem_alloc(smem_u32(&s_tmem), 128);
        tmem_relinquish();
    }
    if (tid == 0) {
        s_give_up = 0;
        for (int i = 0; i < LT_STAGES; ++i) {
            mbar_init(full + 8 * i, 1);
            mbar_init(empty + 8 * i, 1);
        }
        mbar_init(acc, 1);
        mbar_fence_init();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    pdl_launch_dependents();
    pdl_wait();
    if (warp == 0) {
        if (lane == 0) {
            int issued = 0;
            for (; issued < nk; ++issued) {
                const int s = issued % LT_STAGES, use = issued / LT_STAGES;
                if (use > 0 && !tc_wait_raw(empty + 8 * s, (use - 1) & 1, give_up, p.err)) break;
                mbar_expect_tx(full + 8 * s, 2 * LT_TILE);
                tma_load_2d(base + s * 2 * LT_TILE, &wmap, issued * 64, row0, full + 8 * s);
                tma_load_2d(base + s * 2 * LT_TILE + LT_TILE, &xmap, issued * 64, t0, full + 8 * s);
            }
            // no copy may still be in flight when the CTA leaves (at once unless someone gave up)
            for (int s = 0; s < LT_STAGES; ++s) {
                const int uses = (issued - s + LT_STAGES - 1) / LT_STAGES;
                if (issued > s)
                    for (uint32_t i = 0; i < DC_WAIT_LIMIT && !mbar_try_wait(full + 8 * s, (uses - 1) & 1); ++i) {}
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = umma_idesc_bf16(128, 128);
            for (int k = 0; k < nk; ++k) {
                const int s = k % LT_STAGES;
                if (!tc_wait_raw(full + 8 * s, (k / LT_STAGES) & 1, give_up, p.err)) break;
                tc_fence_after();
                const uint32_t a = base + s * 2 * LT_TILE, b = a + LT_TILE;
#pragma unroll
                for (int j = 0; j < 4; ++j) umma_f16(tmem, umma_desc_sw128(a + 32 * j, 1024), umma_desc_sw128(b + 32 * j, 1024), idesc, k > 0 || j > 0);
                umma_commit(empty + 8 * s);
            }
            umma_commit(acc);
        }
    } else {
        const bool ok = tc_wait_raw(acc, 0, give_up, p.err) && !*give_up;
        tc_fence_after();
        if (__all_sync(0xffffffffu, ok)) read_out<128, false>(p, tmem, row0, t0, p.T, warp & 3, lane);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 1) tmem_dealloc(tmem, 128);
}

// ---- 128 x 256 tiles, one CTA per SM over its share of them
constexpr int LW_STAGES = 4, LW_STAGE = 3 * LT_TILE;       // 128 weight rows and 256 token rows of 64 columns
constexpr int LW_READERS = 2, LW_THREADS = 64 + 128 * LW_READERS;     // warps of a quarter's lanes share its columns
constexpr size_t LW_SMEM = (size_t)LW_STAGES * LW_STAGE + 1024;

struct LwTiles {
    int row_tiles, tok_tiles;        // one matrix
    int groups, group_rows;          // grouped: matrix g is rows g * group_rows .., its tokens are off[g] .. off[g + 1] - 1
    const int32_t* off;
};

template <bool GROUPED>
__global__ void __launch_bounds__(LW_THREADS, 1) k_linear_tc_wide(const __grid_constant__ CUtensorMap wmap,
                                                                  const __grid_constant__ CUtensorMap xmap, const LtParams p, const LwTiles tl) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t s_bar[2 * LW_STAGES + 4];
    __shared__ uint32_t s_tmem;
    __shared__ int s_give_up;
    __shared__ int s_off[GROUPED ? DC_MOE_MAX_EXPERTS + 1 : 1], s_first[GROUPED ? DC_MOE_MAX_EXPERTS + 1 : 1];
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t full = smem_u32(s_bar), empty = full + 8 * LW_STAGES, acc_full = empty + 8 * LW_STAGES, acc_free = acc_full + 16;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nk = (p.K + 63) / 64;
    volatile int* give_up = &s_give_up;
    if (warp == 1) {
        tmem_alloc(smem_u32(&s_tmem), 512);
        tmem_relinquish();
    }
    if (tid == 0) {
        s_give_up = 0;
        for (int i = 0; i < LW_STAGES; ++i) {
            mbar_init(full + 8 * i, 1);
            mbar_init(empty + 8 * i, 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(acc_full + 8 * i, 1);
            mbar_init(acc_free + 8 * i, 128 * LW_READERS);
        }
        mbar_fence_init();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    pdl_launch_dependents();
    pdl_wait();
    if (GROUPED) {               // the tiles of every group
        if (warp == 2) {
            int before = 0;
            for (int g0 = 0; g0 < tl.groups; g0 += 32) {
                const int g = g0 + lane, a = tl.off[min(g, tl.groups)], b = tl.off[min(g + 1, tl.groups)];
                int n = (b - a + 255) / 256 * tl.row_tiles;
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const int v = __shfl_up_sync(0xffffffffu, n, o);
                    if (lane >= o) n += v;
                }
                if (g < tl.groups) s_off[g + 1] = b, s_first[g + 1] = before + n;
                before += __shfl_sync(0xffffffffu, n, 31);
            }
            if (lane == 0) s_off[0] = s_first[0] = 0;
        }
        __syncthreads();
    }
    const int total = GROUPED ? s_first[tl.groups] : tl.row_tiles * tl.tok_tiles;
    struct Place {
        int wrow, row0, t0, t1;      // row of the map, row of the matrix, tokens
        __device__ int cols() const { return min(256, t1 - t0); }
    };
    auto place = [&](int tile, int& group) {
        Place at;
        if (GROUPED) {
            while (tile >= s_first[group + 1]) ++group;
            const int a = s_off[group], b = s_off[group + 1], tok_tiles = (b - a + 255) / 256, i = tile - s_first[group];
            at.row0 = i / tok_tiles * 128, at.t0 = a + i % tok_tiles * 256, at.t1 = b;
            at.wrow = group * tl.group_rows + at.row0;
        } else {
            at.row0 = at.wrow = tile / tl.tok_tiles * 128, at.t0 = tile % tl.tok_tiles * 256, at.t1 = p.T;
        }
        return at;
    };
    // Every role walks the same tiles; stages are counted on across tiles.
    if (warp == 0) {
        if (lane == 0) {
            int issued = 0, group = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
                const Place at = place(tile, group);
                const bool both = !GROUPED || at.cols() > 128;
                for (int k = 0; k < nk; ++k, ++issued) {
                    const int s = issued % LW_STAGES, use = issued / LW_STAGES;
                    if (use > 0 && !tc_wait_raw(empty + 8 * s, (use - 1) & 1, give_up, p.err)) {
                        ok = false;
                        break;
                    }
                    const uint32_t to = base + s * LW_STAGE;
                    mbar_expect_tx(full + 8 * s, both ? LW_STAGE : 2 * LT_TILE);
                    tma_load_2d(to, &wmap, k * 64, at.wrow, full + 8 * s);
                    tma_load_2d(to + LT_TILE, &xmap, k * 64, at.t0, full + 8 * s);
                    if (both) tma_load_2d(to + 2 * LT_TILE, &xmap, k * 64, at.t0 + 128, full + 8 * s);
                }
            }
            // no copy may still be in flight when the CTA leaves (at once unless someone gave up)
            for (int s = 0; s < LW_STAGES; ++s) {
                const int uses = (issued - s + LW_STAGES - 1) / LW_STAGES;
                if (issued > s)
                    for (uint32_t i = 0; i < DC_WAIT_LIMIT && !mbar_try_wait(full + 8 * s, (uses - 1) & 1); ++i) {}
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            int it = 0, j = 0, group = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x, ++j) {
                const int set = j & 1;
                const uint32_t idesc = umma_idesc_bf16(128, GROUPED ? (place(tile, group).cols() + 15) & ~15 : 256);
                if (j >= 2 && !tc_wait_raw(acc_free + 8 * set, ((j >> 1) - 1) & 1, give_up, p.err)) break;
                tc_fence_after();
                for (int k = 0; k < nk; ++k, ++it) {
                    const int s = it % LW_STAGES;
                    if (!tc_wait_raw(full + 8 * s, (it / LW_STAGES) & 1, give_up, p.err)) {
                        ok = false;
                        break;
                    }
                    tc_fence_after();
                    const uint32_t a = base + s * LW_STAGE, b = a + LT_TILE;
#pragma unroll
                    for (int q = 0; q < 4; ++q)
                        umma_f16(tmem + 256 * set, umma_desc_sw128(a + 32 * q, 1024), umma_desc_sw128(b + 32 * q, 1024), idesc, k > 0 || q > 0);
                    umma_commit(empty + 8 * s);
                }
                umma_commit(acc_full + 8 * set);
            }
        }
    } else {
        int j = 0, group = 0;
        for (int tile = blockIdx.x; tile < total; tile += gridDim.x, ++j) {
            const int set = j & 1;
            const bool ok = tc_wait_raw(acc_full + 8 * set, (j >> 1) & 1, give_up, p.err) && !*give_up;
            tc_fence_after();
            if (!__all_sync(0xffffffffu, ok)) break;
            const Place at = place(tile, group);
            const int per = (at.cols() + 16 * LW_READERS - 1) / (16 * LW_READERS) * 16, c0 = (warp - 2) / 4 * per;
            if (c0 < at.cols()) read_out<256 / LW_READERS, GROUPED>(p, tmem + 256 * set + c0, at.row0, at.t0 + c0, min(at.t1, at.t0 + c0 + per), warp & 3, lane);
            tc_fence_before();
            mbar_arrive(acc_free + 8 * set);
        }
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (warp == 1) tmem_dealloc(tmem, 512);
}

typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                             const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeFn encode_fn() {
    static EncodeFn fn = [] {
        void* f = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &f, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) f = nullptr;
        return (EncodeFn)f;
    }();
    return fn;
}

}  // namespace

// Loads from tensor memory land in their registers some time after the instruction; each16 uses others meanwhile.  A build that
// spills could store such a register too early and give it another use, which the load then overwrites: it may not run.
static int setup_unspilled(dc_ctx* ctx, const void* f, int smem, const char* name) {
    static std::mutex mu;
    static std::set<const void*> good;
    {
        std::lock_guard<std::mutex> lk(mu);
        if (!good.count(f)) {
            cudaFuncAttributes a;
            const int st = dc_check_cuda(ctx, cudaFuncGetAttributes(&a, f), name);
            if (st != DC_B200_OK) return st;
            if (a.localSizeBytes) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "%s was built with %d bytes of spilled registers", name, (int)a.localSizeBytes);
            good.insert(f);
        }
    }
    return dc_kernel_setup(ctx, f, smem, name);
}

// Tensor map of a bf16 matrix [rows][ld] whose first K columns count: boxes of 128 rows x 64 columns.
int dc_lin_encode(dc_ctx* ctx, CUtensorMap* map, const __nv_bfloat16* base, int rows, int K, int ld) {
    EncodeFn f = encode_fn();
    if (!f) return dc_fail(ctx, DC_B200_BACKEND_ERROR, "the driver has no cuTensorMapEncodeTiled");
    const cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {64, 128}, es[2] = {1, 1};
    const CUresult r = f(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (void*)base, dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? DC_B200_OK : dc_fail(ctx, DC_B200_BACKEND_ERROR, "cuTensorMapEncodeTiled failed (%d) for %d x %d, pitch %d", (int)r, rows, K, ld);
}

int dc_launch_linear_tc(dc_ctx* ctx, const dc_lin& w, const dc_tc_in& x, int T, const dc_lin_epi& epi) {
    if (w.K != x.K) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_tc: inner sizes %d and %d differ", w.K, x.K);
    if (epi.keys || epi.tok_scale || (epi.act_rows && epi.act != DC_ACT_SILU) || (epi.pair0 < (1 << 30) && epi.pair0 % DC_PAIR_ALIGN))
        return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_tc: epilogue not available");
    LtParams p = {w.K, T, epi, ctx->d_err};
    p.e.n_store = std::min(epi.n_store, std::min(w.N, epi.pair0));
    p.e.n_pairs = std::max(0, std::min(epi.n_pairs, (w.N - epi.pair0) / 2));
    const int row_tiles = (w.N + 127) / 128, tok_tiles = (T + 255) / 256, tiles = row_tiles * tok_tiles;
    if (T > 128 && tiles >= ctx->num_sms / 2) {
        int st = setup_unspilled(ctx, (const void*)k_linear_tc_wide<false>, (int)LW_SMEM, "k_linear_tc_wide");
        if (st != DC_B200_OK) return st;
        const LwTiles tl = {row_tiles, tok_tiles, 0, 0, nullptr};
        return dc_launch(ctx, "k_linear_tc_wide", k_linear_tc_wide<false>, dim3(tiles < ctx->num_sms ? tiles : ctx->num_sms), dim3(LW_THREADS), LW_SMEM,
                         w.map, x.map, p, tl);
    }
    int st = setup_unspilled(ctx, (const void*)k_linear_tc, (int)LT_SMEM, "k_linear_tc");
    if (st != DC_B200_OK) return st;
    return dc_launch(ctx, "k_linear_tc", k_linear_tc, dim3((w.N + 127) / 128, (T + 127) / 128), dim3(LT_THREADS), LT_SMEM, w.map, x.map, p);
}

int dc_launch_linear_grouped_tc(dc_ctx* ctx, const dc_lin& w, int groups, int group_rows, const int32_t* group_off, const dc_tc_in& x, int max_rows,
                                const dc_lin_epi& epi) {
    if (w.K != x.K) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_grouped_tc: inner sizes %d and %d differ", w.K, x.K);
    if (groups < 1 || groups > DC_MOE_MAX_EXPERTS || groups * group_rows != w.N || max_rows < 1) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_grouped_tc: bad groups");
    const bool pairs = epi.pair0 == 0 && epi.pair_kind == DC_PAIR_CLAMPED && epi.poutb && epi.tok_scale, rows = epi.pair0 >= (1 << 30) && epi.outb && !epi.bias && (epi.act_rows ? epi.act == DC_ACT_RELU2 && epi.act_rows >= group_rows && epi.tok_scale : !epi.tok_scale);
    if (epi.keys || epi.add || !(pairs || rows) || (epi.pair0 < (1 << 30) && epi.pair0 % DC_PAIR_ALIGN)) return dc_fail(ctx, DC_B200_INTERNAL_ERROR, "linear_grouped_tc: epilogue not available");
    LtParams p = {w.K, max_rows, epi, ctx->d_err};
    p.e.n_store = std::min(epi.n_store, std::min(group_rows, epi.pair0));
    p.e.n_pairs = std::max(0, std::min(epi.n_pairs, (group_rows - epi.pair0) / 2));
    const LwTiles tl = {(group_rows + 127) / 128, 0, groups, group_rows, group_off};
    const int st = setup_unspilled(ctx, (const void*)k_linear_tc_wide<true>, (int)LW_SMEM, "k_linear_tc_grouped");
    if (st != DC_B200_OK) return st;
    const long long most = (long long)tl.row_tiles * (max_rows / 256 + std::min(groups, max_rows));
    return dc_launch(ctx, "k_linear_tc_grouped", k_linear_tc_wide<true>, dim3((int)std::min<long long>(most, ctx->num_sms)), dim3(LW_THREADS), LW_SMEM, w.map, x.map,
                     p, tl);
}
