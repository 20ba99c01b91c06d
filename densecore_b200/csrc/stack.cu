// Layer-list decoders: weight upload, step buffers and the forward pass over dc_stack.h's mixers.  Host code plus
// the small kernels that lay random weights out; arithmetic is in linear*.cu, mix_*.cu, norm_act.cu and the greedy
// epilogue the other models use.
#include <math.h>
#include <string.h>

#include <algorithm>

#include "dc_common.cuh"
#include "dc_model.h"
#include "dc_stack.h"

#define DC_TRY(expr)                       \
    do {                                   \
        int st_ = (expr);                  \
        if (st_ != DC_B200_OK) return st_; \
    } while (0)

namespace {

uint64_t fnv1a64(const char* s) {
    uint64_t h = 1469598103934665603ull;
    for (; *s; ++s) {
        h ^= (uint8_t)*s;
        h *= 1099511628211ull;
    }
    return h;
}

float bf16_value(uint16_t b) {
    const uint32_t u = (uint32_t)b << 16;
    float f;
    memcpy(&f, &u, 4);
    return f;
}

int64_t elems(const dc_stack_tensor& t) {
    int64_t n = 1;
    for (int64_t d : t.shape) n *= d;
    return n;
}

// Random f32 values rounded to bf16 at the tensor's place in a fused matrix.
__global__ void k_place_rows(const float* __restrict__ src, int64_t n, int K, __nv_bfloat16* __restrict__ w, int ld, int row0, int step, int head_rows,
                             int head_pad, int col0) {
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
        const int r = (int)(i / K), c = (int)(i % K);
        const int64_t dst = row0 + (head_rows ? (int64_t)(r / head_rows) * head_pad + r % head_rows : (int64_t)r * step);
        w[dst * ld + col0 + c] = __float2bfloat16_rn(src[i]);
    }
}

// Values in the tensor's own order to their places in the device vector.
cudaError_t put_vector(const dc_stack_tensor& t, const std::vector<float>& v) {
    if (t.pitch) return cudaMemcpy2D(*t.vec + t.vec_off, (size_t)t.pitch * 4, v.data(), (size_t)t.shape[1] * 4, (size_t)t.shape[1] * 4, (size_t)t.shape[0], cudaMemcpyHostToDevice);
    if (!t.cols) return cudaMemcpy(*t.vec + t.vec_off, v.data(), v.size() * 4, cudaMemcpyHostToDevice);
    const size_t taps = (size_t)t.shape[1], n = v.size() / taps;
    std::vector<float> w(v.size());
    for (size_t c = 0; c < n; ++c)
        for (size_t j = 0; j < taps; ++j) w[j * n + c] = v[c * taps + j];
    return cudaMemcpy2D(*t.vec + t.vec_off, (size_t)t.cols * 4, w.data(), n * 4, n * 4, taps, cudaMemcpyHostToDevice);
}

template <typename T>
int alloc(dc_model* m, T** p, size_t n, const char* what = "step buffer") {
    DC_TRY(dc_check_cuda(m->ctx, cudaMalloc((void**)p, n * sizeof(T) + 256), what));
    m->stack->b.owned.push_back((void*)*p);
    return dc_check_cuda(m->ctx, cudaMemsetAsync(*p, 0, n * sizeof(T) + 256, m->ctx->stream), what);
}

}  // namespace

// ---------------------------------------------------------------- weights
int dc_stack_set_tensor(dc_model* m, const char* name, int type, const int64_t ne[4], const void* data) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    auto it = s->index.find(name);
    if (it == s->index.end()) return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "set_tensor: '%s' is not a tensor of this model", name);
    dc_stack_tensor& t = s->tensors[it->second];
    const bool matrix = t.shape.size() == 2;
    const int64_t K = matrix ? t.shape[1] : t.shape[0], N = matrix ? t.shape[0] : 1;
    if (ne[0] != K || (ne[1] > 0 ? ne[1] : 1) != N || (ne[2] > 1))
        return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "set_tensor: '%s' has shape [%lld, %lld], expected [%lld, %lld]", name, (long long)ne[1],
                       (long long)ne[0], (long long)N, (long long)K);
    if (t.loaded) return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "set_tensor: '%s' was already set", name);
    if (type != DC_TYPE_BF16 && !(type == DC_TYPE_F32 && t.vec))
        return dc_fail(ctx, DC_B200_UNSUPPORTED, "set_tensor: '%s' has type %d; matrices are bf16, vectors bf16 or f32", name, type);
    cudaError_t e = cudaSuccess;
    if (t.vec) {
        const int64_t n = elems(t);
        std::vector<float> v((size_t)n);
        for (int64_t i = 0; i < n; ++i) {
            v[i] = type == DC_TYPE_F32 ? ((const float*)data)[i] : bf16_value(((const uint16_t*)data)[i]);
            if (t.neg_exp) v[i] = (float)-exp((double)v[i]);
            v[i] += t.plus;
        }
        e = put_vector(t, v);
    } else if (!t.lin) {
        e = cudaMemcpy(s->embed->dev, data, s->embed->bytes, cudaMemcpyHostToDevice);
    } else {
        const size_t rb = (size_t)K * 2, pitch = (size_t)t.lin->ld * 2;
        const int per = t.head_rows ? t.head_rows : (int)N, blocks = (int)N / per;
        for (int b = 0; b < blocks && e == cudaSuccess; ++b)
            e = cudaMemcpy2D(t.lin->w + (size_t)(t.row0 + b * t.head_pad) * t.lin->ld + t.col0, pitch * t.row_step, (const uint8_t*)data + (size_t)b * per * rb, rb, rb,
                             per, cudaMemcpyHostToDevice);
    }
    DC_TRY(dc_check_cuda(ctx, e, "set_tensor"));
    t.loaded = true;
    return DC_B200_OK;
}

int dc_stack_init_synthetic(dc_model* m, uint64_t seed, float sigma) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    if (!dc_launch_synth_f32) return dc_fail(ctx, DC_B200_UNSUPPORTED, "init_synthetic: this library was built without the random-weight kernels");
    int64_t most = 0;
    for (auto& t : s->tensors) most = std::max(most, elems(t));
    float* tmp = nullptr;
    DC_TRY(dc_check_cuda(ctx, cudaMalloc((void**)&tmp, (size_t)most * 4), "init_synthetic"));
    int st = DC_B200_OK;
    for (auto& t : s->tensors) {
        if (t.loaded || st != DC_B200_OK) continue;
        const int64_t n = elems(t);
        // norm weights around 1, decay exponents and step biases in a useful range, convolution taps not tiny
        const float sg = t.synth == 4 ? 0.4f : t.synth == 2 ? 0.5f : sigma, off = t.synth == 1 ? 1.0f : t.synth == 3 ? -2.0f : t.synth == 5 ? 1.0f / s->cfg.streams : 0.0f;
        st = dc_launch_synth_f32(ctx, seed + fnv1a64(t.name.c_str()), n, sg, off, tmp);
        if (st != DC_B200_OK) break;
        if (t.vec) {
            std::vector<float> v((size_t)n);
            cudaStreamSynchronize(ctx->stream);
            cudaMemcpy(v.data(), tmp, (size_t)n * 4, cudaMemcpyDeviceToHost);
            if (t.neg_exp)
                for (float& x : v) x = (float)-exp((double)x);
            for (float& x : v) x += t.plus;
            st = dc_check_cuda(ctx, put_vector(t, v), "init_synthetic");
        } else {
            const int K = (int)t.shape[1];
            __nv_bfloat16* w = t.lin ? t.lin->w : (__nv_bfloat16*)s->embed->dev;
            k_place_rows<<<1184, 256, 0, ctx->stream>>>(tmp, n, K, w, t.lin ? t.lin->ld : K, t.row0, t.row_step, t.head_rows, t.head_pad, t.col0);
            st = dc_check_cuda(ctx, cudaGetLastError(), "k_place_rows");
        }
        t.loaded = true;
    }
    if (st == DC_B200_OK) st = dc_b200_synchronize(ctx);
    cudaFree(tmp);
    return st;
}

void dc_stack_release(dc_model* m) {
    dc_stack* s = m->stack;
    if (!s) return;
    for (void* p : s->owned) cudaFree(p);
    for (void* p : s->b.owned) cudaFree(p);
    for (auto& r : s->rot) cudaFree(r.second);
    if (s->b.h_meta) cudaFreeHost(s->b.h_meta);
    if (s->embed) {
        if (s->embed->dev && !s->cfg.tied) cudaFree(s->embed->dev);
        delete s->embed;
    }
    delete s;
    m->stack = nullptr;
}

// ---------------------------------------------------------------- cache, state slots, step buffers
namespace {

// The cos/sin table of a rotation, made at its first use.
int rotation_table(dc_model* m, const dc_rotation& r, const float** out) {
    float*& table = m->stack->rot[r];
    if (!table) {
        const int n = m->cfg.max_ctx, half = r.dims / 2;
        std::vector<double> f(half);
        double mul = 1.0, lo = 0.0, hi = 0.0;
        if (r.factor > 0.0) {
            // the pair that turns t times over the original context
            auto pair_of = [&](double t) { return r.dims * log(r.original / (2.0 * M_PI * t)) / (2.0 * log(r.base)); };
            lo = std::max(floor(pair_of(r.fast)), 0.0);
            hi = std::min(ceil(pair_of(r.slow)), r.dims - 1.0);
            mul = 0.1 * log(r.factor) + 1.0;
        }
        for (int i = 0; i < half; ++i) {
            f[i] = pow(r.base, -2.0 * i / r.dims);
            if (r.factor > 0.0) {
                const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
                f[i] = f[i] / r.factor * ramp + f[i] * (1.0 - ramp);
            }
        }
        std::vector<float> cs((size_t)n * r.dims);
        for (int p = 0; p < n; ++p)
            for (int i = 0; i < half; ++i) {
                cs[(size_t)p * r.dims + 2 * i] = (float)(mul * cos(p * f[i]));
                cs[(size_t)p * r.dims + 2 * i + 1] = (float)(mul * sin(p * f[i]));
            }
        DC_TRY(dc_check_cuda(m->ctx, cudaMalloc((void**)&table, cs.size() * 4), "rotation table"));
        DC_TRY(dc_check_cuda(m->ctx, cudaMemcpy(table, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice), "rotation table"));
    }
    *out = table;
    return DC_B200_OK;
}

}  // namespace

// Cache planes of the layers that write a latent, state slots of the recurrent layers, rotation tables.  The pool
// holds pool_tokens tokens (0: max_ctx for every sequence).
int dc_stack_create_cache(dc_model* m, int pool_tokens) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    const dc_model_config& c = m->cfg;
    const size_t elt = s->dtype == DC_DTYPE_F32 ? 4 : 2;
    std::vector<size_t> planes;
    size_t state = 0;
    auto carve = [&](size_t floats) {
        const size_t off = state;
        state += (floats * 4 + 255) & ~(size_t)255;
        return off;
    };
    int span = 1;
    auto key_range = [&](int window, int keep) {        // which of the distinct windows
        span = std::max(span, window > 0 ? std::min(window + keep, c.max_ctx) : c.max_ctx);
        auto w = std::find(s->windows.begin(), s->windows.end(), window);
        const int i = (int)(w - s->windows.begin());
        if (w == s->windows.end()) s->windows.push_back(window);
        return i;
    };
    auto plane = [&](int row) {
        planes.push_back((size_t)row * elt);
        return (int)planes.size() - 1;
    };
    std::vector<int> written(s->layers.size(), -1);     // plane of a layer's last run
    for (dc_stack_run& r : s->runs) {
        dc_stack_layer& L = s->layers[r.layer];
        if (L.kind == DC_MIX_LIGHTNING) {
            r.state_off = carve((size_t)L.li.heads * L.li.vdim * L.li.dim);
        } else if (L.kind == DC_MIX_GENERAL) {
            r.state_off = carve((size_t)L.ge.heads * L.ge.dim * L.ge.dim);
        } else if (L.kind == DC_MIX_GQA) {
            r.plane = plane(L.ga.row);
            L.ga.range = key_range(L.ga.window, L.ga.keep);
            if (L.ga.taps) r.ring_off = carve((size_t)L.ga.taps * dc_gqa_conv_cols(L.ga));
            if (L.ga.rot.dims) DC_TRY(rotation_table(m, L.ga.rot, &L.ga.cos_sin));
        } else if (L.kind == DC_MIX_DELTA) {
            r.state_off = carve((size_t)L.dl.heads * L.dl.vdim * L.dl.dim);
            r.ring_off = carve((size_t)L.dl.taps * (L.dl.off_v + L.dl.heads * L.dl.vdim));
        } else if (L.kind == DC_MIX_SSD) {
            r.state_off = carve((size_t)L.ssd.heads * L.ssd.vdim * L.ssd.state);
            r.ring_off = carve((size_t)L.ssd.taps * (L.ssd.heads * L.ssd.vdim + 2 * L.ssd.groups * L.ssd.state));
        } else {
            dc_latent_mixer& a = L.la;
            r.plane = written[r.layer] = a.kv_from < 0 ? plane(a.row) : written[a.kv_from];
            a.range = key_range(a.window, 0);
            dc_rotation rot;
            rot.dims = a.rot_dim, rot.base = a.rot_base;
            DC_TRY(rotation_table(m, rot, &a.cos_sin));
        }
    }
    // key splits of a decode step: about 32 keys each at the longest span
    s->splits = std::max(1, std::min(DC_MAX_SPLITS, (span + 31) / 32));
    const int per_seq = (c.max_ctx + DC_KV_BLOCK - 1) / DC_KV_BLOCK;
    const int blocks = pool_tokens > 0 ? (pool_tokens + DC_KV_BLOCK - 1) / DC_KV_BLOCK : per_seq * c.max_seqs;
    return dc_kv_init_planes(ctx, &m->kv, planes, state, blocks, c.max_seqs, per_seq);
}

// lambda of a differential attention layer, from its loaded vectors
static int map_weight(dc_model* m, dc_gqa_mixer* d) {
    std::vector<float> v[4];
    for (int i = 0; i < 4; ++i) {
        v[i].resize(d->dim);
        DC_TRY(dc_check_cuda(m->ctx, cudaMemcpy(v[i].data(), d->lam[i], (size_t)d->dim * 4, cudaMemcpyDeviceToHost), "finalize"));
    }
    double dot[2] = {0.0, 0.0};
    for (int i = 0; i < d->dim; ++i)
        for (int j = 0; j < 2; ++j) dot[j] += (double)v[2 * j][i] * v[2 * j + 1][i];
    d->lambda = (float)(exp(dot[0]) - exp(dot[1]) + (double)d->diff);
    return DC_B200_OK;
}

// rows of a layer's input product that are the mixer's
static int mixer_rows(const dc_stack_layer& L) { return L.pair0 ? L.pair0 : L.in.N; }

static constexpr int ENTRY_INTS = DC_MAX_T + 1;

int dc_stack_finalize(dc_model* m) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    dc_stack_buffers& b = s->b;
    if (b.cap) return DC_B200_OK;
    const size_t H = dc_pad8(s->cfg.width), V = s->cfg.vocab;
    const bool f32 = s->dtype == DC_DTYPE_F32;
    const long long all = (long long)m->cfg.max_seqs * m->cfg.max_ctx;
    const size_t C = std::max<long long>(DC_MAX_T, std::min<long long>(m->prefill_chunk, all));
    const size_t F = f32 ? C : DC_MAX_T;      // rows of buffers that only the f32 path uses
    size_t q = 0, actb = 0, head_state = 0;
    bool latent = false;
    size_t proj = 8, act = 8, low = 8, gate = 8, small = 8, mix = 8, ff = 8, lowb = 8, rank = 8, rot = 8, ukv = 8, blk = 8, qa = 0, part = 0, ml = 0;
    size_t top = 0, experts = 8, hid = 8;
    int span = 1;
    for (dc_stack_layer& L : s->layers) {
        auto up = [](size_t& a, long long v) { a = std::max(a, (size_t)dc_pad8((int)v)); };
        up(ff, L.ff);
        if (L.moe.experts) {
            top = std::max(top, (size_t)L.moe.top);
            up(experts, L.moe.experts), up(hid, L.moe.ff);
        }
        const size_t parts = std::max((size_t)DC_MAX_T * s->splits, f32 ? C : 0);
        auto attention = [&](int heads, int values, int window) {
            part = std::max(part, parts * heads * values);
            ml = std::max(ml, parts * heads * 2);
            span = std::max(span, window > 0 ? std::min(window, m->cfg.max_ctx) : m->cfg.max_ctx);
        };
        if (s->cfg.block == DC_BLOCK_PARALLEL) up(mix, L.out.K);
        if (L.kind == DC_MIX_GENERAL) {
            const dc_general_mixer& d = L.ge;
            up(proj, L.in.N), up(act, d.heads * d.dim), up(low, d.w2.N), up(lowb, d.rank), up(mix, L.out.K);
            blk = std::max(blk, dc_general_block_floats(d));
        } else if (L.kind == DC_MIX_GQA) {
            up(proj, mixer_rows(L));
            up(mix, L.out.K);
            q = std::max(q, (size_t)L.ga.heads * L.ga.maps * dc_gqa_ldq(L.ga));
            attention(L.ga.heads * L.ga.maps, L.ga.vdim, L.ga.window);
            if (L.ga.maps > 1) DC_TRY(map_weight(m, &L.ga));
        } else if (L.kind == DC_MIX_LIGHTNING) {
            up(f32 ? proj : actb, mixer_rows(L));
            up(act, L.li.heads * L.li.vdim);
            if (f32) blk = std::max(blk, dc_lightning_block_floats(L.li));
            else head_state = std::max(head_state, (size_t)L.li.heads * L.li.dim * L.li.vdim);
        } else if (L.kind == DC_MIX_DELTA) {
            const dc_delta_mixer& d = L.dl;
            up(proj, d.in.N), up(act, d.off_v + d.heads * d.vdim), up(low, d.a2.N), up(gate, d.g2.N), up(small, d.heads);
            blk = std::max(blk, dc_delta_block_floats(d));
            up(mix, d.heads * d.vdim), up(lowb, d.in.N - d.off_a);
        } else if (L.kind == DC_MIX_SSD) {
            const dc_ssd_mixer& d = L.ssd;
            up(proj, d.in.N), up(act, d.heads * d.vdim + 2 * d.groups * d.state), up(small, 2 * d.heads), up(mix, d.heads * d.vdim);
            blk = std::max(blk, dc_ssd_block_floats(d));
        } else {
            const dc_latent_mixer& d = L.la;
            up(proj, d.in.N), up(mix, d.heads * d.vdim), up(rank, d.kv_rank), up(rot, d.rot_dim), up(ukv, d.ukv.N);
            qa = std::max(qa, F * d.heads * dc_pad8(d.kv_rank));
            attention(d.heads, d.kv_rank, d.window);
            latent = true;
        }
    }
    b.key_cap = (int)std::min<long long>((long long)C + (long long)m->cfg.max_seqs * (span - 1), all);
    b.key_cap = std::max(b.key_cap, DC_MAX_T);
    const bool hyper = s->cfg.block == DC_BLOCK_HYPER;
    DC_TRY(alloc(m, &b.x, C * H * s->cfg.streams));
    if (hyper) {
        DC_TRY(alloc(m, &b.x2, C * H * s->cfg.streams));
        DC_TRY(alloc(m, &b.h, F * H));
    }
    DC_TRY(alloc(m, &b.y, C * H));
    DC_TRY(alloc(m, &b.proj, C * proj));
    DC_TRY(alloc(m, &b.act, C * act));
    DC_TRY(alloc(m, &b.scan, C * act));
    DC_TRY(alloc(m, &b.low, C * low));
    DC_TRY(alloc(m, &b.gate, C * gate));
    DC_TRY(alloc(m, &b.small, C * small));
    DC_TRY(alloc(m, &b.blk, (size_t)dc_scan_blocks((int)C, DC_MAX_T) * blk));
    DC_TRY(alloc(m, &b.mix, F * mix));
    DC_TRY(alloc(m, &b.ff, F * ff));
    DC_TRY(alloc(m, &b.lm_x, DC_MAX_T * H));
    if (!f32) {
        DC_TRY(alloc(m, &b.lm_xb, DC_MAX_T * H));
        DC_TRY(alloc(m, &b.xb, C * H));
        DC_TRY(alloc(m, &b.mixb, C * mix));
        DC_TRY(alloc(m, &b.ffb, C * ff));
        DC_TRY(alloc(m, &b.lowb, C * lowb));
    }
    if (actb) DC_TRY(alloc(m, &b.actb, C * actb));
    if (head_state) DC_TRY(alloc(m, &b.chunk_state, (size_t)dc_lightning_chunks((int)C, DC_MAX_T) * head_state));
    if (q) {
        DC_TRY(alloc(m, &b.q, F * q));
        if (!f32) DC_TRY(alloc(m, &b.qb, C * q));
    }
    if (top) {
        const size_t rows = C * top;
        b.moe_rows = (int)rows;
        DC_TRY(alloc(m, &b.moe_ids, rows));
        DC_TRY(alloc(m, &b.moe_row, rows));
        DC_TRY(alloc(m, &b.moe_src, rows));
        DC_TRY(alloc(m, &b.moe_w, rows));
        DC_TRY(alloc(m, &b.moe_row_w, rows));
        DC_TRY(alloc(m, &b.moe_off, experts + 1));
        DC_TRY(alloc(m, &b.moe_logits, C * experts));
        if (f32) {
            DC_TRY(alloc(m, &b.moe_hid, rows * hid));
            DC_TRY(alloc(m, &b.moe_y, rows * H));
        } else {
            DC_TRY(alloc(m, &b.moe_x, rows * H));
            DC_TRY(alloc(m, &b.moe_hidb, rows * hid));
            DC_TRY(alloc(m, &b.moe_yb, rows * H));
        }
    }
    if (!s->windows.empty()) {
        DC_TRY(alloc(m, &b.part, part));
        DC_TRY(alloc(m, &b.part_ml, ml));
    }
    if (latent) {
        DC_TRY(alloc(m, &b.qa, qa));
        if (!f32) {
            DC_TRY(alloc(m, &b.keys_c, b.key_cap * rank));
            DC_TRY(alloc(m, &b.keys_r, b.key_cap * rot));
            DC_TRY(alloc(m, &b.keys_kv, b.key_cap * ukv));
        }
    }
    // metadata of a step: tokens, sequences, positions, entry starts, wanted rows, key ranges per window, query tiles
    b.meta_ints = (int)(4 * C + ENTRY_INTS * (1 + s->windows.size()) + 2 * (C / DC_LATENT_QTILE + DC_MAX_T + 1));
    DC_TRY(alloc(m, &b.meta, (size_t)b.meta_ints));
    DC_TRY(dc_check_cuda(ctx, cudaMallocHost((void**)&b.h_meta, (size_t)b.meta_ints * DC_STACK_META_SLOTS * 4), "cudaMallocHost"));
    DC_TRY(alloc(m, &b.iota, ENTRY_INTS));
    DC_TRY(alloc(m, &b.chunk, 2 * ENTRY_INTS));
    int32_t iota[ENTRY_INTS], chunk[2 * ENTRY_INTS];
    for (int i = 0; i < ENTRY_INTS; ++i) iota[i] = i, chunk[2 * i] = 0, chunk[2 * i + 1] = i;
    DC_TRY(dc_check_cuda(ctx, cudaStreamSynchronize(ctx->stream), "finalize"));
    DC_TRY(dc_check_cuda(ctx, cudaMemcpy(b.iota, iota, sizeof(iota), cudaMemcpyHostToDevice), "finalize"));
    DC_TRY(dc_check_cuda(ctx, cudaMemcpy(b.chunk, chunk, sizeof(chunk), cudaMemcpyHostToDevice), "finalize"));
    // the step buffers every model has
    dc_step_buffers& g = m->buf;
    void** common[] = {(void**)&g.tokens, (void**)&g.seq_ids, (void**)&g.positions, (void**)&g.out_tokens, (void**)&g.argmax_keys,
                       (void**)&g.logits, (void**)&g.history, (void**)&g.history_len};
    const size_t bytes[] = {64, 64, 64, 64, 8 * DC_MAX_T, DC_MAX_T * V * 4, (size_t)DC_HISTORY_CAP * DC_MAX_T * 4, 4};
    for (int i = 0; i < 8; ++i) {
        DC_TRY(dc_check_cuda(ctx, cudaMalloc(common[i], bytes[i] + 256), "step buffer"));
        DC_TRY(dc_check_cuda(ctx, cudaMemsetAsync(*common[i], 0, bytes[i] + 256, ctx->stream), "step buffer"));
    }
    DC_TRY(dc_check_cuda(ctx, cudaMallocHost((void**)&m->h_stage, 4096), "cudaMallocHost"));
    b.cap = (int)C;
    DC_TRY(dc_check_cuda(ctx, cudaStreamSynchronize(cudaStreamLegacy), "finalize"));     // the tensors' copies
    return dc_check_cuda(ctx, cudaStreamSynchronize(ctx->stream), "finalize");
}

// ---------------------------------------------------------------- one step
namespace {

struct StepKeys {                       // prompt attention: gathered key ranges per window, query tiles
    std::vector<const int32_t*> base;   // device, [entries + 1]
    std::vector<int> count;
    const int32_t* tiles = nullptr;
    int n_tiles = 0;
};

// The tensor map of a step buffer's first K columns, made at its first use.
int tc_in(dc_model* m, dc_tc_in* out, const __nv_bfloat16* x, int K, int ld, int rows) {
    auto key = std::make_pair((const void*)x, K);
    auto it = m->stack->ins.find(key);
    if (it == m->stack->ins.end() || it->second.ld != ld) {
        dc_tc_in in;
        in.x = x, in.K = K, in.ld = ld;
        DC_TRY(dc_lin_encode(m->ctx, &in.map, x, rows, K, ld));
        m->stack->ins[key] = in;
        it = m->stack->ins.find(key);
    }
    *out = it->second;
    return DC_B200_OK;
}

// y = W x for the step's tokens: xf is the input of f32 models, xb that of bf16 models, same pitch.
int linear(dc_model* m, const dc_step& st, const dc_lin& w, const float* xf, const __nv_bfloat16* xb, int ldx, const dc_lin_epi& epi) {
    if (st.b16 && st.T <= DC_MAX_T) return dc_launch_linear_mma(m->ctx, w, xb, ldx, st.T, epi);
    if (st.b16) {
        dc_tc_in in;
        DC_TRY(tc_in(m, &in, xb, w.K, ldx, m->stack->b.cap));
        return dc_launch_linear_tc(m->ctx, w, in, st.T, epi);
    }
    if (st.T <= DC_MAX_T) return dc_launch_linear_rows(m->ctx, w, xf, ldx, st.T, epi);
    return dc_launch_linear_f32(m->ctx, w, xf, ldx, st.T, epi);
}
dc_lin_epi to(float* out, int ld) { return dc_lin_epi::store(out, nullptr, ld); }

// cls: kernel class of the per-class timing; bytes: what its launches have to read and write
#define L(cls, bytes, n, expr)                                           \
    do {                                                                 \
        dc_model::ProfRec r_ = {cls, nullptr, nullptr, (double)(bytes)}; \
        if (m->prof) {                                                   \
            cudaEventCreate(&r_.e0);                                     \
            cudaEventCreate(&r_.e1);                                     \
            cudaEventRecord(r_.e0, ctx->stream);                         \
        }                                                                \
        DC_TRY(expr);                                                    \
        if (m->prof) {                                                   \
            cudaEventRecord(r_.e1, ctx->stream);                         \
            m->prof_recs.push_back(r_);                                  \
        }                                                                \
        m->last_launches += (n);                                         \
    } while (0)

// a stream norm's: the streams in and out, y and the normed row
double hyper_bytes(const dc_model* m, int T) { return 8.0 * T * m->stack->cfg.width * (m->stack->cfg.streams + 1); }
double lin_bytes(const dc_lin& w, int T) { return (double)w.N * w.ld * 2 + (double)T * (w.N + w.K) * 4; }

int mix_delta(dc_model* m, const dc_step& st, const dc_stack_run& run, dc_stack_layer& Ly) {
    const dc_delta_mixer& d = Ly.dl;
    const dc_stack_buffers& b = m->stack->b;
    const dc_state_ref sr = {m->kv.state, m->kv.state_bytes, run.state_off, run.ring_off};
    const int ldp = d.in.N, lda = dc_pad8(d.off_v + d.heads * d.vdim), ldl = d.in.N - d.off_a, ldm = d.heads * d.vdim;
    if (st.single && st.T <= DC_MAX_T)
        return dc_launch_delta_decode(m->ctx, d, st, sr, b.proj, ldp, m->stack->cfg.eps, b.mix, st.b16 ? b.mixb : nullptr, dc_pad8(ldm));
    __nv_bfloat16* lowb = st.b16 ? b.lowb : nullptr;
    DC_TRY(dc_launch_delta_prep(m->ctx, d, st, sr, b.proj, ldp, b.act, lda, b.small, lowb, ldl));
    if (st.b16) {
        DC_TRY(linear(m, st, d.a2, nullptr, lowb, ldl, to(b.low, d.a2.N)));
        DC_TRY(linear(m, st, d.g2, nullptr, lowb + (d.off_g - d.off_a), ldl, to(b.gate, d.g2.N)));
    } else {
        DC_TRY(linear(m, st, d.a2, b.proj + d.off_a, nullptr, ldp, to(b.low, d.a2.N)));
        DC_TRY(linear(m, st, d.g2, b.proj + d.off_g, nullptr, ldp, to(b.gate, d.g2.N)));
    }
    return dc_launch_delta_scan(m->ctx, d, st, sr, b.act, lda, b.small, b.low, d.a2.N, b.blk, b.gate, d.g2.N, m->stack->cfg.eps, b.scan,
                                st.b16 ? nullptr : b.mix, st.b16 ? b.mixb : nullptr, dc_pad8(ldm));
}

int mix_ssd(dc_model* m, const dc_step& st, const dc_stack_run& run, dc_stack_layer& Ly) {
    const dc_ssd_mixer& d = Ly.ssd;
    const dc_stack_buffers& b = m->stack->b;
    const dc_state_ref sr = {m->kv.state, m->kv.state_bytes, run.state_off, run.ring_off};
    const int inner = d.heads * d.vdim, lda = dc_pad8(inner + 2 * d.groups * d.state);
    if (st.single && st.T <= DC_MAX_T)
        return dc_launch_ssd_decode(m->ctx, d, st, sr, b.proj, d.in.N, b.scan, lda, m->stack->cfg.eps, b.mix, st.b16 ? b.mixb : nullptr, dc_pad8(inner));
    return dc_launch_ssd(m->ctx, d, st, sr, b.proj, d.in.N, b.act, lda, b.small, b.blk, b.scan, m->stack->cfg.eps, st.b16 ? nullptr : b.mix,
                         st.b16 ? b.mixb : nullptr, dc_pad8(inner));
}

int mix_latent(dc_model* m, const dc_step& st, const StepKeys& sk, const dc_stack_run& run, dc_stack_layer& Ly) {
    const dc_latent_mixer& d = Ly.la;
    const dc_stack_buffers& b = m->stack->b;
    dc_latent_cache c;
    c.arena = m->kv.planes[run.plane].arena;
    c.f32 = m->stack->dtype == DC_DTYPE_F32;
    c.tables = m->kv.d_tables;
    c.max_blocks = m->kv.max_blocks_per_seq;
    const int ldp = d.in.N, ldm = dc_pad8(d.heads * d.vdim);
    DC_TRY(dc_launch_latent_prep(m->ctx, d, st, c, b.proj, ldp, m->stack->cfg.eps, m->cfg.max_ctx));
    if (!st.tc)
        return dc_launch_latent_absorbed(m->ctx, d, st, c, b.proj, ldp, st.T <= DC_MAX_T ? m->stack->splits : 1, b.qa, b.part, b.part_ml, b.mix,
                                         st.b16 ? b.mixb : nullptr, ldm);
    const int32_t* base = sk.base[d.range];
    const int nk = sk.count[d.range], ldc = dc_pad8(d.kv_rank), ldr = dc_pad8(d.rot_dim);
    DC_TRY(dc_launch_latent_gather(m->ctx, d, st, c, base, nk, b.keys_c, ldc, b.keys_r, ldr));
    dc_tc_in in;
    DC_TRY(tc_in(m, &in, b.keys_c, d.kv_rank, ldc, b.key_cap));
    DC_TRY(dc_launch_linear_tc(m->ctx, d.ukv, in, nk, dc_lin_epi::store(nullptr, b.keys_kv, d.ukv.N)));
    return dc_launch_latent_prefill(m->ctx, d, st, base, sk.tiles, sk.n_tiles, b.proj, ldp, b.keys_kv, d.ukv.N, b.keys_r, ldr, b.mixb, ldm);
}

int mix_gqa(dc_model* m, const dc_step& st, const StepKeys& sk, const dc_stack_run& run, dc_stack_layer& Ly) {
    const dc_gqa_mixer& d = Ly.ga;
    const dc_stack_buffers& b = m->stack->b;
    dc_gqa_cache c;
    c.arena = m->kv.planes[run.plane].arena;
    c.f32 = m->stack->dtype == DC_DTYPE_F32;
    c.tables = m->kv.d_tables;
    c.max_blocks = m->kv.max_blocks_per_seq;
    const int ldp = mixer_rows(Ly), ldm = dc_pad8(Ly.out.K);
    const dc_state_ref sr = {m->kv.state, m->kv.state_bytes, run.state_off, run.ring_off};
    DC_TRY(dc_launch_gqa_prep(m->ctx, d, st, c, d.taps ? &sr : nullptr, b.proj, ldp, m->stack->cfg.eps, m->cfg.max_ctx, b.q, st.tc ? b.qb : nullptr));
    if (st.tc) return dc_launch_gqa_prompt(m->ctx, d, st, c, sk.tiles, sk.n_tiles, b.qb, b.proj, ldp, m->stack->cfg.eps, b.mixb, ldm);
    return dc_launch_gqa_tokens(m->ctx, d, st, c, b.q, b.proj, ldp, st.T <= DC_MAX_T ? m->stack->splits : 1, b.part, b.part_ml, m->stack->cfg.eps, b.mix, st.b16 ? b.mixb : nullptr, ldm);
}

int mix_general(dc_model* m, const dc_step& st, const dc_stack_run& run, dc_stack_layer& Ly) {
    const dc_general_mixer& d = Ly.ge;
    const dc_stack_buffers& b = m->stack->b;
    const dc_state_ref sr = {m->kv.state, m->kv.state_bytes, run.state_off, 0};
    const int ldp = Ly.in.N, ldo = dc_pad8(d.heads * d.dim), ldl = dc_pad8(d.rank), ldm = dc_pad8(Ly.out.K);
    const float eps = m->stack->cfg.eps;
    __nv_bfloat16 *lowb = st.b16 ? b.lowb : nullptr, *mixb = st.b16 ? b.mixb : nullptr;
    if (st.single && st.T <= DC_MAX_T) return dc_launch_general_decode(m->ctx, d, st, sr, b.proj, ldp, eps, b.mix, mixb, ldm);
    DC_TRY(dc_launch_general_tanh(m->ctx, d, st.T, b.proj, ldp, lowb, ldl));
    DC_TRY(linear(m, st, d.w2, b.proj + d.off_w, lowb, st.b16 ? ldl : ldp, to(b.low, d.w2.N)));
    return dc_launch_general_scan(m->ctx, d, st, sr, b.proj, ldp, b.low, d.w2.N, b.blk, eps, b.scan, ldo, b.mix, mixb, ldm);
}

int mix_lightning(dc_model* m, const dc_step& st, const dc_stack_run& run, dc_stack_layer& Ly) {
    const dc_lightning_mixer& d = Ly.li;
    const dc_stack_buffers& b = m->stack->b;
    const dc_state_ref sr = {m->kv.state, m->kv.state_bytes, run.state_off, 0};
    const int lda = mixer_rows(Ly), ldy = dc_pad8(d.heads * d.vdim), ldm = dc_pad8(Ly.out.K);
    const __nv_bfloat16* actb = st.b16 ? b.actb : nullptr;
    if (st.single && st.T <= DC_MAX_T) DC_TRY(dc_launch_lightning_decode(m->ctx, d, st, sr, b.proj, actb, lda, b.scan, ldy));
    else if (st.b16) DC_TRY(dc_launch_lightning_chunks(m->ctx, d, st, sr, b.actb, lda, b.chunk_state, b.scan, ldy));
    else DC_TRY(dc_launch_lightning_scan(m->ctx, d, st, sr, b.proj, lda, b.blk, b.scan, ldy));
    return dc_launch_lightning_norm(m->ctx, d, st, b.scan, ldy, b.proj, actb, lda, m->stack->cfg.eps, b.mix, st.b16 ? b.mixb : nullptr, ldm);
}

// x += mixer(h) + ff(h) with h = norm1(x): one product from h, the mixer, one product back into the residual.  The
// feed-forward's hidden values lie beside the mixer's output.
int parallel_layer(dc_model* m, const dc_step& st, const StepKeys& sk, const dc_stack_run& run, dc_stack_layer& Ly) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    dc_stack_buffers& b = s->b;
    const int W = s->cfg.width, H = dc_pad8(W), T = st.T, rows = mixer_rows(Ly), ldm = dc_pad8(Ly.out.K);
    L(DC_K_PRE_NORM, 8.0 * T * W, 1, dc_launch_norm_rows(ctx, b.x, Ly.norm1, nullptr, 0, T, W, H, s->cfg.eps, b.y, st.b16 ? b.xb : nullptr, H));
    const bool light = Ly.kind == DC_MIX_LIGHTNING;
    dc_lin_epi in = dc_lin_epi::store(b.proj, light && st.b16 ? b.actb : nullptr, rows);
    if (light) in.act_rows = Ly.li.off_g;
    else in.bias = Ly.ga.bias;
    if (Ly.ff) in.pairs(Ly.pair0, DC_PAIR_CLAMPED, Ly.limit, b.mix + Ly.out_ff, st.b16 ? b.mixb + Ly.out_ff : nullptr, ldm, Ly.ff);
    L(DC_K_MIX_IN, lin_bytes(Ly.in, T), 1, linear(m, st, Ly.in, b.y, b.xb, H, in));
    if (light) L(DC_K_MIX_LIGHTNING, 8.0 * st.E * Ly.li.heads * Ly.li.dim * Ly.li.vdim, st.single && !st.tc ? 2 : 4, mix_lightning(m, st, run, Ly));
    else L(DC_K_MIX_GQA, 4.0 * T * Ly.in.N, st.tc ? 2 : 3, mix_gqa(m, st, sk, run, Ly));
    dc_lin_epi out = to(b.x, H);
    out.add = true;
    out.bias = Ly.out_bias;
    L(DC_K_MIX_OUT, lin_bytes(Ly.out, T), 1, linear(m, st, Ly.out, b.mix, b.mixb, ldm, out));
    return DC_B200_OK;
}

// The layer's experts on norm2 of the residual: of x, or (hy) of its streams, which are brought up to date on the way.  Steps of
// up to DC_MAX_T tokens of bf16 models add to x at once, with streams they leave y in b.y; the others leave a row of every chosen
// expert behind, which *owed names.
int moe_layer(dc_model* m, const dc_step& st, dc_stack_layer& Ly, const dc_hyper* hy, dc_row_sum* owed) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    dc_stack_buffers& b = s->b;
    const dc_moe_ffn& f = Ly.moe;
    const int W = s->cfg.width, H = dc_pad8(W), T = st.T, rows = T * f.top, F = dc_pad8(f.ff);
    __nv_bfloat16* xb = st.b16 ? b.xb : nullptr;
    float* h = hy ? b.h : b.y;
    const double up_bytes = (double)f.up_rows * f.up.ld * 2, down_bytes = (double)f.down_rows * f.down.ld * 2;
    const double touched = std::min<double>(f.experts, rows);
    if (dc_moe_norm_route_fits(f, st.b16, T, H)) {
        L(DC_K_ROUTER, lin_bytes(f.router, T), hy && T > DC_MAX_T ? 2 : 1, dc_launch_moe_norm_route(ctx, f, b.x, hy, Ly.norm2, T, W, H, s->cfg.eps, h, xb, b.moe_ids, b.moe_w));
    } else {
        if (hy) L(DC_K_PRE_NORM, hyper_bytes(m, T), 1, dc_launch_hyper_norm(ctx, *hy, Ly.norm2, nullptr, 0, T, W, H, s->cfg.eps, h, xb));
        else L(DC_K_PRE_NORM, 8.0 * T * W, 1, dc_launch_norm_rows(ctx, b.x, Ly.norm2, nullptr, 0, T, W, H, s->cfg.eps, h, xb, H));
        L(DC_K_ROUTER, lin_bytes(f.router, T), 1, linear(m, st, f.router, h, b.xb, H, to(b.moe_logits, f.router.N)));
        L(DC_K_ROUTER, 4.0 * T * f.experts, 1, dc_launch_moe_route(ctx, f, b.moe_logits, f.router.N, T, b.moe_ids, b.moe_w));
    }
    if (st.b16 && T <= DC_MAX_T) {
        L(DC_K_MOE_GATEUP, touched * up_bytes, 1, dc_launch_moe_up_mma(ctx, f, b.xb, H, T, b.moe_ids, b.moe_w, b.moe_hidb, F));
        L(DC_K_MOE_DOWN, touched * down_bytes, 1, dc_launch_moe_down_mma(ctx, f, b.moe_hidb, F, T, b.moe_ids, W, hy ? b.y : b.x, H, !hy));
        return DC_B200_OK;
    }
    L(DC_K_ROUTER, 16.0 * rows, 1, dc_launch_moe_order(ctx, f, b.moe_ids, b.moe_w, T, b.moe_off, b.moe_src, b.moe_row_w, b.moe_row));
    dc_lin_epi hid = f.plain ? dc_lin_epi::store(b.moe_hid, b.moe_hidb, F) : dc_lin_epi().pairs(0, DC_PAIR_CLAMPED, f.limit, b.moe_hid, b.moe_hidb, F, f.ff);
    if (f.plain) hid.act_rows = f.up_rows, hid.act = DC_ACT_RELU2;
    hid.tok_scale = b.moe_row_w;
    const dc_lin_epi y = dc_lin_epi::store(b.moe_y, b.moe_yb, H);
    if (st.b16) {
        dc_tc_in in;
        L(DC_K_MOE_GATEUP, 4.0 * rows * W, 1, dc_launch_moe_gather(ctx, b.xb, H, b.moe_src, rows, b.moe_x));
        DC_TRY(tc_in(m, &in, b.moe_x, W, H, b.moe_rows));
        L(DC_K_MOE_GATEUP, touched * up_bytes + 2.0 * rows * (W + f.ff), 1, dc_launch_linear_grouped_tc(ctx, f.up, f.experts, f.up_rows, b.moe_off, in, rows, hid));
        DC_TRY(tc_in(m, &in, b.moe_hidb, f.ff, F, b.moe_rows));
        L(DC_K_MOE_DOWN, touched * down_bytes + 2.0 * rows * (W + f.ff), 1, dc_launch_linear_grouped_tc(ctx, f.down, f.experts, f.down_rows, b.moe_off, in, rows, y));
    } else {
        L(DC_K_MOE_GATEUP, touched * up_bytes, 1, dc_launch_moe_f32(ctx, f.up, f.experts, f.up_rows, b.moe_off, rows, h, H, b.moe_src, hid));
        L(DC_K_MOE_DOWN, touched * down_bytes, 1, dc_launch_moe_f32(ctx, f.down, f.experts, f.down_rows, b.moe_off, rows, b.moe_hid, F, nullptr, y));
    }
    owed->y = b.moe_y, owed->yb = b.moe_yb, owed->rows = b.moe_row, owed->k = f.top, owed->ld = H;
    return DC_B200_OK;
}

// x += mixer(norm1(x)), then x += experts(norm2(x)).  *owed: rows that the feed-forward before has not added yet.
int pre_norm_layer(dc_model* m, const dc_step& st, const StepKeys& sk, const dc_stack_run& run, dc_stack_layer& Ly, dc_row_sum* owed) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    dc_stack_buffers& b = s->b;
    const int W = s->cfg.width, H = dc_pad8(W), T = st.T;
    const bool latent = Ly.kind == DC_MIX_LATENT;
    const dc_lin &in = latent ? Ly.la.in : Ly.in, &o = latent ? Ly.la.o : Ly.out;
    const float* step = run.step < 0 ? nullptr : s->loop_step + (size_t)run.step * H;
    L(DC_K_PRE_NORM, 8.0 * T * W, 1, dc_launch_pre_norm(ctx, b.x, step, *owed, Ly.norm1, T, W, H, s->cfg.eps, b.y, st.b16 ? b.xb : nullptr));
    *owed = dc_row_sum();
    dc_lin_epi proj = to(b.proj, in.N);
    if (!latent) proj.bias = Ly.ga.bias;
    L(DC_K_MIX_IN, lin_bytes(in, T), 1, linear(m, st, in, b.y, b.xb, H, proj));
    if (latent) L(DC_K_MIX_LATENT, (double)Ly.la.ukv.N * Ly.la.ukv.ld * 2, 4, mix_latent(m, st, sk, run, Ly));
    else L(DC_K_MIX_GQA, 4.0 * T * in.N, st.tc ? 2 : 3, mix_gqa(m, st, sk, run, Ly));
    dc_lin_epi out = to(b.x, H);
    out.add = true;
    L(DC_K_MIX_OUT, lin_bytes(o, T), 1, linear(m, st, o, b.mix, b.mixb, dc_pad8(o.K), out));
    return Ly.moe.experts ? moe_layer(m, st, Ly, nullptr, owed) : DC_B200_OK;
}

// The streams as the next sublayer (coefficients next) finds them; afterwards they lie in the other buffer and owe y.
dc_hyper hyper_next(dc_model* m, dc_hyper* hy, const float* next) {
    const dc_stack_buffers& b = m->stack->b;
    dc_hyper now = *hy;
    now.next = next;
    now.x_out = hy->x == b.x ? b.x2 : b.x;
    hy->x = now.x_out, hy->first = false, hy->done = next, hy->y = b.y, hy->sum = dc_row_sum();
    return now;
}

// Hyper-connected sublayers, mixer and feed-forward: u from the streams, y = f(norm(u)), which the streams then owe.
int hyper_layer(dc_model* m, const dc_step& st, const StepKeys& sk, const dc_stack_run& run, dc_stack_layer& Ly, dc_hyper* hy) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    dc_stack_buffers& b = s->b;
    const int W = s->cfg.width, H = dc_pad8(W), T = st.T;
    __nv_bfloat16* xb = st.b16 ? b.xb : nullptr;
    L(DC_K_PRE_NORM, hyper_bytes(m, T), 1, dc_launch_hyper_norm(ctx, hyper_next(m, hy, Ly.hyper[0]), Ly.norm1, nullptr, 0, T, W, H, s->cfg.eps, b.h, xb));
    L(DC_K_MIX_IN, lin_bytes(Ly.in, T), 1, linear(m, st, Ly.in, b.h, b.xb, H, to(b.proj, Ly.in.N)));
    if (Ly.kind == DC_MIX_GENERAL) L(DC_K_MIX_GENERAL, 8.0 * st.E * Ly.ge.heads * Ly.ge.dim * Ly.ge.dim, st.single && !st.tc ? 1 : 5, mix_general(m, st, run, Ly));
    else L(DC_K_MIX_GQA, 4.0 * T * Ly.in.N, st.tc ? 2 : 3, mix_gqa(m, st, sk, run, Ly));
    L(DC_K_MIX_OUT, lin_bytes(Ly.out, T), 1, linear(m, st, Ly.out, b.mix, b.mixb, dc_pad8(Ly.out.K), to(b.y, H)));
    if (Ly.moe.experts) {
        const dc_hyper now = hyper_next(m, hy, Ly.hyper[1]);
        return moe_layer(m, st, Ly, &now, &hy->sum);
    }
    if (!Ly.ff) return DC_B200_OK;
    const int F = dc_pad8(Ly.ff);
    L(DC_K_PRE_NORM, hyper_bytes(m, T), 1, dc_launch_hyper_norm(ctx, hyper_next(m, hy, Ly.hyper[1]), Ly.norm2, nullptr, 0, T, W, H, s->cfg.eps, b.h, xb));
    L(DC_K_FFN_GATEUP, lin_bytes(Ly.gate_up, T), 1, linear(m, st, Ly.gate_up, b.h, b.xb, H, dc_lin_epi().pairs(0, Ly.ff_pair, 0.0f, b.ff, st.b16 ? b.ffb : nullptr, F, F)));
    L(DC_K_FFN_DOWN, lin_bytes(Ly.down, T), 1, linear(m, st, Ly.down, b.ff, b.ffb, F, to(b.y, H)));
    return DC_B200_OK;
}

// Embedding and every layer; the residual ends in b.x, several streams in *hy.
int run_layers(dc_model* m, const dc_step& st, const StepKeys& sk, dc_hyper* hy) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    dc_stack_buffers& b = s->b;
    const int W = s->cfg.width, H = dc_pad8(W), T = st.T;
    const float eps = s->cfg.eps;
    __nv_bfloat16* xb = st.b16 ? b.xb : nullptr;
    const bool hyper = s->cfg.block == DC_BLOCK_HYPER;
    auto capture = [&](int il) -> int {     // parity aid: what enters layer il (the last slot: the output norm)
        if (!m->dbg_x || T > DC_MAX_T) return DC_B200_OK;
        const float* x = b.x;
        if (hyper) {                        // the streams' sum
            DC_TRY(dc_launch_hyper_norm(ctx, *hy, nullptr, nullptr, 0, T, W, H, eps, b.h, nullptr));
            x = b.h;
        }
        return dc_check_cuda(ctx, cudaMemcpy2DAsync(m->dbg_x + (size_t)il * DC_MAX_T * W, (size_t)W * 4, x, (size_t)H * 4, (size_t)W * 4, T,
                                                    cudaMemcpyDeviceToDevice, ctx->stream), "capture");
    };
    m->last_launches = 0;
    L(DC_K_EMBED, (double)T * W * 6, 1, dc_launch_embed(ctx, s->embed, st.tokens, T, hyper ? b.y : b.x, H, s->cfg.block == DC_BLOCK_POST_NORM ? xb : nullptr, s->cfg.embed_scale));
    if (hyper) hy->streams = s->cfg.streams, hy->mul = s->cfg.residual_mult, hy->x = b.y, hy->first = true;
    dc_row_sum owed;
    auto settle = [&]() -> int {
        if (!owed.k) return DC_B200_OK;
        L(DC_K_COMBINE, 4.0 * T * W * owed.k, 1, dc_launch_pre_norm(ctx, b.x, nullptr, owed, nullptr, T, W, H, eps, nullptr, nullptr));
        owed = dc_row_sum();
        return DC_B200_OK;
    };
    for (size_t il = 0; il < s->runs.size(); ++il) {
        const dc_stack_run& run = s->runs[il];
        dc_stack_layer& Ly = s->layers[run.layer];
        if (m->dbg_x) DC_TRY(settle());
        DC_TRY(capture((int)il));
        if (hyper) {
            DC_TRY(hyper_layer(m, st, sk, run, Ly, hy));
            continue;
        }
        if (s->cfg.block == DC_BLOCK_PARALLEL) {
            DC_TRY(parallel_layer(m, st, sk, run, Ly));
            continue;
        }
        if (s->cfg.block == DC_BLOCK_PRE_NORM) {
            DC_TRY(pre_norm_layer(m, st, sk, run, Ly, &owed));
            continue;
        }
        const dc_lin& in = Ly.kind == DC_MIX_DELTA ? Ly.dl.in : Ly.kind == DC_MIX_SSD ? Ly.ssd.in : Ly.la.in;
        const dc_lin& o = Ly.kind == DC_MIX_DELTA ? Ly.dl.o : Ly.kind == DC_MIX_SSD ? Ly.ssd.o : Ly.la.o;
        L(DC_K_MIX_IN, lin_bytes(in, T), 1, linear(m, st, in, b.x, xb, H, to(b.proj, in.N)));
        if (Ly.kind == DC_MIX_DELTA) L(DC_K_MIX_DELTA, 8.0 * st.E * Ly.dl.heads * Ly.dl.dim * Ly.dl.vdim, st.single && !st.tc ? 1 : 7, mix_delta(m, st, run, Ly));
        else if (Ly.kind == DC_MIX_SSD) L(DC_K_MIX_SSD, 8.0 * st.E * Ly.ssd.heads * Ly.ssd.state * Ly.ssd.vdim, st.single && !st.tc ? 2 : 5, mix_ssd(m, st, run, Ly));
        else L(DC_K_MIX_LATENT, (double)Ly.la.ukv.N * Ly.la.ukv.ld * 2, 4, mix_latent(m, st, sk, run, Ly));
        L(DC_K_MIX_OUT, lin_bytes(o, T), 1, linear(m, st, o, b.mix, b.mixb, dc_pad8(o.K), to(b.y, H)));
        L(DC_K_POST_NORM, 12.0 * T * W, 1, dc_launch_post_norm(ctx, b.x, b.y, Ly.norm1, T, W, H, eps, xb));
        if (!Ly.ff) continue;
        const int F = dc_pad8(Ly.ff);
        L(DC_K_FFN_GATEUP, lin_bytes(Ly.gate_up, T), 1, linear(m, st, Ly.gate_up, b.x, xb, H, dc_lin_epi().pairs(0, Ly.ff_pair, 0.0f, b.ff, st.b16 ? b.ffb : nullptr, F, F)));
        L(DC_K_FFN_DOWN, lin_bytes(Ly.down, T), 1, linear(m, st, Ly.down, b.ff, b.ffb, F, to(b.y, H)));
        L(DC_K_POST_NORM, 12.0 * T * W, 1, dc_launch_post_norm(ctx, b.x, b.y, Ly.norm2, T, W, H, eps, xb));
    }
    DC_TRY(settle());
    return capture((int)s->runs.size());
}

// Logits and greedy picks of R <= DC_MAX_T rows (rows: device list, or first, first + 1, ...).
int run_head(dc_model* m, const dc_hyper& hy, const int32_t* rows, int first, int R, bool feedback) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    const int W = s->cfg.width, H = dc_pad8(W);
    dc_step_buffers& g = m->buf;
    if (hy.x) L(DC_K_PRE_NORM, hyper_bytes(m, R), 1, dc_launch_hyper_norm(ctx, hy, s->final_norm, rows, first, R, W, H, s->cfg.eps, s->b.lm_x, s->b.lm_xb));
    else L(DC_K_POST_NORM, 8.0 * R * W, 1, dc_launch_norm_rows(ctx, s->b.x, s->final_norm, rows, first, R, W, H, s->cfg.eps, s->b.lm_x, s->b.lm_xb, H));
    L(DC_K_LM_HEAD, lin_bytes(s->head, R), 1,
      s->b.lm_xb ? dc_launch_linear_mma(ctx, s->head, s->b.lm_xb, H, R, dc_lin_epi::store(g.logits, nullptr, s->cfg.vocab, g.argmax_keys))
                 : dc_launch_linear_rows(ctx, s->head, s->b.lm_x, H, R, dc_lin_epi::store(g.logits, nullptr, s->cfg.vocab, g.argmax_keys)));
    L(DC_K_ARGMAX, 64.0, 1, dc_launch_argmax_finish(ctx, g.argmax_keys, R, g.out_tokens, feedback ? g.tokens : nullptr, feedback ? g.positions : nullptr,
                                                    feedback ? g.history : nullptr, feedback ? g.history_len : nullptr, DC_HISTORY_CAP));
    return DC_B200_OK;
}
#undef L

}  // namespace

int dc_stack_enqueue_small(dc_model* m, int T, bool chunk, int lm_mode, bool feedback) {
    dc_step st;
    st.T = T;
    st.E = chunk ? 1 : T;
    st.tokens = m->buf.tokens, st.seq_ids = m->buf.seq_ids, st.positions = m->buf.positions;
    st.starts = chunk ? m->stack->b.chunk + 2 * T : m->stack->b.iota;
    st.single = !chunk || T == 1;
    st.b16 = m->stack->dtype == DC_DTYPE_BF16;
    dc_hyper hy;
    DC_TRY(run_layers(m, st, StepKeys(), &hy));
    if (lm_mode == 1) return run_head(m, hy, nullptr, T - 1, 1, feedback);
    return lm_mode ? run_head(m, hy, nullptr, 0, T, feedback) : DC_B200_OK;
}

int dc_stack_batch(dc_model* m, int E, const int32_t* seqs, const int32_t* counts, const int32_t* tokens, int n_rows, const int32_t* rows,
                   float* logits_host, int32_t* picks_host) {
    dc_stack* s = m->stack;
    dc_ctx* ctx = m->ctx;
    dc_stack_buffers& b = s->b;
    const int C = b.cap, V = s->cfg.vocab;
    std::vector<int> done(E, 0), offset(E, 0);
    int total = 0;
    for (int e = 0; e < E; ++e) offset[e] = total, total += counts[e];
    int next_row = 0;                   // rows are ascending; sub-steps take entries front to back
    std::vector<int> order;             // flat token index of every token of the sub-step
    for (int left = total; left > 0;) {
        if (b.meta_slot == 0) DC_TRY(dc_check_cuda(ctx, cudaStreamSynchronize(ctx->stream), "sync"));
        int32_t* h = b.h_meta + (size_t)b.meta_slot * b.meta_ints;
        b.meta_slot = (b.meta_slot + 1) % DC_STACK_META_SLOTS;
        int32_t *h_tok = h, *h_seq = h + C, *h_pos = h + 2 * C, *h_rows = h + 3 * C, *h_start = h + 4 * C;
        int32_t* h_base = h_start + ENTRY_INTS;
        int32_t* h_tiles = h_base + ENTRY_INTS * s->windows.size();
        order.clear();
        StepKeys sk;
        sk.count.assign(s->windows.size(), 0);
        dc_step st;
        st.single = true;
        for (int e = 0; e < E && st.T < C; ++e) {
            const int n = std::min(counts[e] - done[e], C - st.T);
            if (n <= 0) continue;
            const int pos0 = m->kv.seqs[seqs[e]].len;
            h_start[st.E] = st.T;
            for (size_t w = 0; w < s->windows.size(); ++w) {
                h_base[w * ENTRY_INTS + st.E] = sk.count[w];
                sk.count[w] += pos0 + n - (s->windows[w] > 0 ? std::max(0, pos0 - s->windows[w] + 1) : 0);
            }
            for (int q = 0; q < n; q += DC_LATENT_QTILE) {
                h_tiles[2 * sk.n_tiles] = st.E;
                h_tiles[2 * sk.n_tiles + 1] = q;
                ++sk.n_tiles;
            }
            for (int i = 0; i < n; ++i) {
                h_tok[st.T + i] = tokens[offset[e] + done[e] + i];
                h_seq[st.T + i] = seqs[e];
                h_pos[st.T + i] = pos0 + i;
                order.push_back(offset[e] + done[e] + i);
            }
            st.single &= n == 1;
            st.T += n;
            ++st.E;
            done[e] += n;
            m->kv.seqs[seqs[e]].len += n;
        }
        h_start[st.E] = st.T;
        for (size_t w = 0; w < s->windows.size(); ++w) h_base[w * ENTRY_INTS + st.E] = sk.count[w];
        left -= st.T;
        int R = 0;
        for (int i = 0; i < st.T && next_row + R < n_rows; ++i)
            if (order[i] == rows[next_row + R]) h_rows[R++] = i;
        DC_TRY(dc_check_cuda(ctx, cudaMemcpyAsync(b.meta, h, (size_t)b.meta_ints * 4, cudaMemcpyHostToDevice, ctx->stream), "H2D step"));
        st.tokens = b.meta, st.seq_ids = b.meta + C, st.positions = b.meta + 2 * C, st.starts = b.meta + (h_start - h);
        for (size_t w = 0; w < s->windows.size(); ++w) sk.base.push_back(b.meta + (h_base - h) + w * ENTRY_INTS);
        sk.tiles = b.meta + (h_tiles - h);
        st.b16 = s->dtype == DC_DTYPE_BF16;
        st.tc = st.b16 && st.T > DC_MAX_T;
        dc_hyper hy;
        DC_TRY(run_layers(m, st, sk, &hy));
        for (int r = 0; r < R; r += DC_MAX_T) {
            const int n = std::min(DC_MAX_T, R - r);
            DC_TRY(run_head(m, hy, b.meta + 3 * C + r, 0, n, false));
            if (logits_host)
                DC_TRY(dc_check_cuda(ctx, cudaMemcpyAsync(logits_host + (size_t)(next_row + r) * V, m->buf.logits, (size_t)n * V * 4, cudaMemcpyDeviceToHost,
                                                          ctx->stream), "D2H logits"));
            if (picks_host)
                DC_TRY(dc_check_cuda(ctx, cudaMemcpyAsync(picks_host + next_row + r, m->buf.out_tokens, (size_t)n * 4, cudaMemcpyDeviceToHost, ctx->stream),
                                     "D2H picks"));
        }
        next_row += R;
    }
    return logits_host || picks_host ? dc_b200_synchronize(ctx) : DC_B200_OK;
}

void dc_stack_stats(dc_model* m, double* weight_bytes, double* kv_bytes_per_token) {
    dc_stack* s = m->stack;
    double w = (double)s->head.N * s->head.ld * 2 + (s->cfg.tied ? 0.0 : (double)s->embed->row_bytes), kv = 0.0;
    bool experts = false;
    for (const dc_stack_layer& L : s->layers) experts |= L.moe.experts > 0;
    if (!experts) {
        w = (double)s->weight_bytes - (double)s->embed->bytes + (s->cfg.tied ? 0.0 : (double)s->embed->row_bytes);
    } else {
        for (const dc_stack_run& r : s->runs) {         // every run reads its layer; of the experts, those that a token chooses
            const dc_stack_layer& L = s->layers[r.layer];
            const dc_moe_ffn& f = L.moe;
            for (const dc_lin* l : {&L.la.in, &L.la.ukv, &L.la.o, &L.in, &L.out, &L.ge.w2, &L.gate_up, &L.down, &f.router}) w += (double)l->N * l->ld * 2;
            if (f.experts) w += ((double)f.up.N * f.up.ld + (double)f.down.N * f.down.ld) * 2 * f.top / f.experts;
        }
    }
    for (const dc_stack_run& r : s->runs)
        if (r.plane >= 0) kv += (double)m->kv.planes[r.plane].row_bytes;
    if (weight_bytes) *weight_bytes = w;
    if (kv_bytes_per_token) *kv_bytes_per_token = kv;
}
