// Architecture table of the layer-list decoders: reads config.json's fields into the mixer structs of dc_stack.h,
// lays the weights out and lists the tensors the model needs.  A design is an entry of kArchs plus the mixers and
// feed-forwards it may use; constants that a design fixes are set here, everything else comes from its files.
#include <math.h>

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

using Shapes = std::map<std::string, std::vector<int64_t>>;

struct Reader {
    dc_model* m;
    dc_stack* s;
    const Shapes* shapes;
    std::string error;      // first problem found

    void bad(const std::string& what) {
        if (error.empty()) error = what;
    }
    double number(const dc_json& o, const char* key, const std::string& where) {
        const dc_json* v = o.get(key);
        if (!v || v->kind != dc_json::NUM) {
            bad(where + ": '" + key + "' is missing or not a number");
            return 0.0;
        }
        return v->num;
    }
    int size(const dc_json& o, const char* key, const std::string& where, int lo = 1, int hi = 1 << 24) {
        const double v = number(o, key, where);
        if (error.empty() && (v != floor(v) || v < lo || v > hi)) bad(where + ": '" + key + "' is out of range");
        return error.empty() ? (int)v : 1;
    }
    // length of dimension `dim` of a tensor, for sizes that only the tensor's shape gives
    int from_shape(const std::string& name, int dim) {
        auto it = shapes->find(name);
        if (it == shapes->end() || (int)it->second.size() <= dim || it->second[dim] < 1) {
            bad("the shape of tensor '" + name + "' is needed");
            return 1;
        }
        return (int)it->second[dim];
    }
    void tensor(dc_stack_tensor t) {
        s->index[t.name] = (int)s->tensors.size();
        s->tensors.push_back(std::move(t));
    }
    const dc_json* object(const dc_json& o, const char* key, const std::string& where) {
        const dc_json* v = o.get(key);
        if (v && v->kind == dc_json::OBJ) return v;
        bad(where + ": '" + key + "' is missing");
        return nullptr;
    }
    // {base, dims, scaling: {factor, original, fast, slow} or null}
    void rotation(const dc_json& o, const std::string& where, dc_rotation* r) {
        r->base = number(o, "base", where);
        r->dims = size(o, "dims", where, 2, 1024);
        if (r->dims % 2 || !(r->base > 1.0)) bad(where + ": dims must be even and base above 1");
        const dc_json* s = o.get("scaling");
        if (!s || s->is_null()) return;
        const std::string in = where + ".scaling";
        r->factor = number(*s, "factor", in), r->original = number(*s, "original", in);
        r->fast = number(*s, "fast", in), r->slow = number(*s, "slow", in);
        if (!(r->factor > 0.0 && r->original > 0.0 && r->fast > 0.0 && r->slow > 0.0)) bad(in + ": every value must be positive");
    }
    // rows of a matrix appended to lin (whose K must agree); returns the first row
    int matrix(dc_lin* lin, const std::string& name, int N, int K) {
        const int row0 = lin->N;
        lin->N += dc_pad8(N);
        lin->K = K;
        dc_stack_tensor t;
        t.name = name;
        t.shape = {N, K};
        t.lin = lin;
        t.row0 = row0;
        tensor(t);
        return row0;
    }
    void vec(float** p, const std::string& name, std::vector<int64_t> shape, int synth, int64_t off = 0, int64_t total = 0, bool neg_exp = false) {
        dc_stack_tensor t;
        t.name = name;
        int64_t n = 1;
        for (int64_t d : shape) n *= d;
        t.shape = std::move(shape);
        t.vec = p;
        t.vec_off = off;
        t.vec_len = total ? total : n;
        t.neg_exp = neg_exp;
        t.synth = synth;
        tensor(t);
    }
    // convolution weights [n, taps], kept as [taps][cols]
    void conv(float** p, const std::string& name, int n, int taps, int off, int cols) {
        vec(p, name, {n, taps}, 4, off, (int64_t)cols * taps);
        s->tensors.back().cols = cols;
    }
};

// ---------------------------------------------------------------- mixers
void read_delta(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L) {
    dc_delta_mixer& d = L->dl;
    const int H = r.s->cfg.width;
    d.heads = r.size(j, "heads", where);
    d.kv_heads = r.size(j, "kv_heads", where);
    d.dim = r.size(j, "dim", where, 1, 256);
    d.vdim = r.size(j, "vdim", where, 1, 512);
    d.taps = r.size(j, "conv", where, 1, 16);
    if (d.heads % d.kv_heads) r.bad(where + ": heads is not a multiple of kv_heads");
    d.unit_eps = 1e-6f;
    d.q_scale = (float)(1.0 / sqrt((double)d.dim));
    d.a_rank = r.from_shape(p + "a1", 0);
    d.g_rank = r.from_shape(p + "g1", 0);
    const int Q = d.kv_heads * d.dim, V = d.heads * d.vdim;
    d.off_q = r.matrix(&d.in, p + "q", Q, H);
    d.off_k = r.matrix(&d.in, p + "k", Q, H);
    d.off_v = r.matrix(&d.in, p + "v", V, H);
    d.off_b = r.matrix(&d.in, p + "b", d.heads, H);
    d.off_a = r.matrix(&d.in, p + "a1", d.a_rank, H);
    d.off_g = r.matrix(&d.in, p + "g1", d.g_rank, H);
    r.matrix(&d.a2, p + "a2", d.heads * d.dim, d.a_rank);
    r.matrix(&d.g2, p + "g2", V, d.g_rank);
    r.matrix(&d.o, p + "o", H, V);
    // convolution weights sit at the channels' projection columns, so that one index serves both
    const int C = d.off_v + dc_pad8(V);
    r.conv(&d.conv, p + "q.conv", Q, d.taps, d.off_q, C);
    r.conv(&d.conv, p + "k.conv", Q, d.taps, d.off_k, C);
    r.conv(&d.conv, p + "v.conv", V, d.taps, d.off_v, C);
    r.vec(&d.neg_a, p + "A_log", {d.heads}, 2, 0, 0, true);
    r.vec(&d.dt_bias, p + "dt_bias", {(int64_t)d.heads * d.dim}, 3);
    r.vec(&d.norm, p + "norm", {d.vdim}, 1);
}

void read_ssd(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L) {
    dc_ssd_mixer& d = L->ssd;
    const int H = r.s->cfg.width;
    d.heads = r.size(j, "heads", where);
    d.vdim = r.size(j, "vdim", where, 1, 512);
    d.state = r.size(j, "state", where, 1, 256);
    d.groups = r.size(j, "groups", where);
    d.norm_groups = r.size(j, "norm_groups", where);
    d.taps = r.size(j, "conv", where, 1, 16);
    const int inner = d.heads * d.vdim, C = inner + 2 * d.groups * d.state;
    if (d.heads % d.groups) r.bad(where + ": heads is not a multiple of groups");
    if (inner % d.norm_groups) r.bad(where + ": heads * vdim is not a multiple of norm_groups");
    // one tensor, one matrix: its rows z | x B C | dt keep their own offsets
    r.matrix(&d.in, p + "in", inner + C + d.heads, H);
    d.off_z = 0;
    d.off_x = inner;
    d.off_dt = inner + C;
    r.matrix(&d.o, p + "o", H, inner);
    r.conv(&d.conv, p + "conv", C, d.taps, 0, C);
    r.vec(&d.conv_b, p + "conv.b", {C}, 4);
    r.vec(&d.dt_bias, p + "dt_bias", {d.heads}, 3);
    r.vec(&d.neg_a, p + "A_log", {d.heads}, 2, 0, 0, true);
    r.vec(&d.D, p + "D", {d.heads}, 1);
    r.vec(&d.norm, p + "norm", {inner}, 1);
}

void read_latent(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L, int il) {
    dc_latent_mixer& d = L->la;
    const int H = r.s->cfg.width;
    d.heads = r.size(j, "heads", where);
    d.dim = r.size(j, "dim", where, 1, 512);
    d.rot_dim = r.size(j, "rot_dim", where, 2, 256);
    d.vdim = r.size(j, "vdim", where, 1, 256);
    d.kv_rank = r.size(j, "kv_rank", where, 1, 1024);
    d.scale = (float)r.number(j, "scale", where);
    if (const dc_json* rot = r.object(j, "rot", where)) {
        d.rot_base = r.number(*rot, "base", where + ".rot");
        if (r.size(*rot, "dims", where + ".rot") != d.rot_dim || d.rot_dim % 2) r.bad(where + ": rot.dims must be even and equal rot_dim");
    }
    const dc_json* mask = j.get("mask");
    d.window = mask && !mask->is_null() ? r.size(*mask, "size", where + ".mask") : 0;
    const dc_json* from = j.get("kv_from");
    d.kv_from = from && !from->is_null() ? r.size(j, "kv_from", where, 0) : -1;
    d.row = dc_pad8(d.kv_rank + d.rot_dim);
    d.dim_p = dc_pad8(d.dim);
    d.vdim_p = dc_pad8(d.vdim);
    d.off_q = r.matrix(&d.in, p + "q", d.heads * (d.dim + d.rot_dim), H);
    if (d.kv_from < 0) {
        d.off_kv = r.matrix(&d.in, p + "dkv", d.kv_rank + d.rot_dim, H);
        r.vec(&d.kv_norm, p + "dkv.norm", {d.kv_rank}, 1);
    } else {
        const dc_stack_layer* src = d.kv_from < il ? &r.s->layers[d.kv_from] : nullptr;
        if (!src || src->kind != DC_MIX_LATENT || src->la.kv_from >= 0 || src->la.kv_rank != d.kv_rank || src->la.rot_dim != d.rot_dim ||
            src->la.rot_base != d.rot_base) {
            r.bad(where + ": kv_from must name an earlier latent layer with a cache of its own and the same kv_rank, rot_dim and rotation");
            return;
        }
    }
    // every head's rows start at a multiple of eight in the expanded keys and values
    auto heads_of = [&](const char* n, int rows, int pad) {
        dc_stack_tensor t;
        t.name = p + n;
        t.shape = {(int64_t)d.heads * rows, d.kv_rank};
        t.lin = &d.ukv;
        t.row0 = d.ukv.N;
        t.head_rows = rows;
        t.head_pad = pad;
        d.ukv.N += d.heads * pad;
        d.ukv.K = d.kv_rank;
        r.tensor(t);
        return t.row0;
    };
    heads_of("uk", d.dim, d.dim_p);
    d.uv_row = heads_of("uv", d.vdim, d.vdim_p);
    r.matrix(&d.o, p + "o", H, d.heads * d.vdim);
}

// Mixers of parallel blocks: their input rows open L->in, their output matrix the columns of L->out.
void out_columns(Reader& r, const std::string& name, dc_stack_layer* L, int K) {
    const int H = r.s->cfg.width;
    dc_stack_tensor t;
    t.name = name;
    t.shape = {H, K};
    t.lin = &L->out;
    t.col0 = L->out.K;
    r.tensor(t);
    L->out.N = dc_pad8(H);
    L->out.K += K;
}

void read_gqa(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L) {
    dc_gqa_mixer& d = L->ga;
    const int H = r.s->cfg.width;
    d.heads = r.size(j, "heads", where);
    d.kv_heads = r.size(j, "kv_heads", where);
    d.dim = r.size(j, "dim", where, 1, 256);
    if (r.size(j, "vdim", where) != d.dim) r.bad(where + ": the values are the keys, so vdim must equal dim");
    if (d.heads % d.kv_heads) r.bad(where + ": heads is not a multiple of kv_heads");
    d.scale = (float)r.number(j, "scale", where);
    if (const dc_json* rot = r.object(j, "rot", where)) r.rotation(*rot, where + ".rot", &d.rot);
    if (d.rot.dims > d.dim) r.bad(where + ".rot: dims is larger than the head");
    const dc_json* mask = j.get("mask");
    d.window = mask && !mask->is_null() ? r.size(*mask, "size", where + ".mask") : 0;
    d.sink = true, d.sink_score = 0.0f;
    d.dim_p = dc_pad8(d.dim);
    d.row = 2 * d.kv_heads * d.dim_p;
    const int Q = d.heads * d.dim, K = d.kv_heads * d.dim;
    d.off_q = r.matrix(&L->in, p + "q", Q, H);
    d.off_k = r.matrix(&L->in, p + "k", K, H);
    const int rows = (L->in.N + DC_PAIR_ALIGN - 1) / DC_PAIR_ALIGN * DC_PAIR_ALIGN;     // as many as a product may store
    r.vec(&d.bias, p + "q.b", {Q}, 4, d.off_q, rows);
    r.vec(&d.bias, p + "k.b", {K}, 4, d.off_k, rows);
    r.vec(&d.q_norm, p + "q.norm", {Q}, 1);
    r.vec(&d.k_norm, p + "k.norm", {K}, 1);
    out_columns(r, p + "o", L, Q);
    r.vec(&L->out_bias, p + "o.b", {H}, 4);
}

void read_lightning(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L) {
    dc_lightning_mixer& d = L->li;
    const int H = r.s->cfg.width;
    d.heads = r.size(j, "heads", where);
    d.dim = r.size(j, "dim", where, 1, 256);
    d.vdim = r.size(j, "vdim", where, 1, 512);
    const dc_json* decay = j.get("decay");
    if (!decay || decay->kind != dc_json::ARR || (int)decay->arr.size() != d.heads) r.bad(where + ": 'decay' must list one number per head");
    else
        for (const dc_json& v : decay->arr) {
            if (v.kind != dc_json::NUM) r.bad(where + ": 'decay' must list one number per head");
            d.decays.push_back((float)v.num);
        }
    const int Q = d.heads * d.dim, V = d.heads * d.vdim;
    if (V > 16384) r.bad(where + ": heads * vdim is above 16384");
    d.off_q = r.matrix(&L->in, p + "q", Q, H);
    d.off_k = r.matrix(&L->in, p + "k", Q, H);
    d.off_v = r.matrix(&L->in, p + "v", V, H);
    d.off_g = r.matrix(&L->in, p + "g", V, H);
    r.vec(&d.norm, p + "norm", {V}, 1);
    out_columns(r, p + "o", L, V);
}

// Gate and up rows in turn from L->pair0 of the input matrix, the down matrix beside the mixer's output matrix.
void read_dense_clamped(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L) {
    const int H = r.s->cfg.width;
    L->ff = r.size(j, "ff", where);
    L->limit = (float)r.number(j, "limit", where);
    L->pair0 = L->in.N = (L->in.N + DC_PAIR_ALIGN - 1) / DC_PAIR_ALIGN * DC_PAIR_ALIGN;
    L->in.N += 2 * dc_pad8(L->ff);
    for (int i = 0; i < 2; ++i) {
        dc_stack_tensor t;
        t.name = p + (i ? "up" : "gate");
        t.shape = {L->ff, H};
        t.lin = &L->in;
        t.row0 = L->pair0 + i;
        t.row_step = 2;
        r.tensor(t);
    }
    L->out_ff = L->out.K = dc_pad8(L->out.K);
    out_columns(r, p + "down", L, L->ff);
}

void read_dense_gelu(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L) {
    const int H = r.s->cfg.width;
    L->ff = r.size(j, "ff", where);
    L->gate_up.N = 2 * dc_pad8(L->ff);
    L->gate_up.K = H;
    for (int i = 0; i < 2; ++i) {
        dc_stack_tensor t;
        t.name = p + (i ? "up" : "gate");
        t.shape = {L->ff, H};
        t.lin = &L->gate_up;
        t.row0 = i;
        t.row_step = 2;
        r.tensor(t);
    }
    r.matrix(&L->down, p + "down", H, L->ff);
}

// ---------------------------------------------------------------- designs
struct Arch {
    const char* name;
    unsigned mixers;        // bit per DC_MIX_*
    int block;              // DC_BLOCK_*; parallel blocks have the clamped feed-forward, the others the tanh-gelu one
    bool embed_scale;       // config.embedding.scale
    bool tied;
};
const Arch kArchs[] = {
    // Garilix: RMS norms on the sublayers' outputs only (x += norm(f(x))), tanh-gelu gated feed-forward
    {"Garilix", (1u << DC_MIX_DELTA) | (1u << DC_MIX_LATENT) | (1u << DC_MIX_SSD), DC_BLOCK_POST_NORM, false, false},
    // Datasun: mixer and clamped feed-forward side by side on one normed input, embedding table as output matrix
    {"Datasun", (1u << DC_MIX_GQA) | (1u << DC_MIX_LIGHTNING), DC_BLOCK_PARALLEL, true, true},
};
struct MixerType {
    const char* name;
    int kind;
};
const MixerType kMixers[] = {{"channel_delta", DC_MIX_DELTA}, {"latent_attention", DC_MIX_LATENT}, {"mamba2", DC_MIX_SSD},
                              {"attention", DC_MIX_GQA}, {"lightning", DC_MIX_LIGHTNING}};

int alloc_lin(dc_model* m, dc_lin* l) {
    if (!l->N) return DC_B200_OK;
    l->ld = (l->K + 63) & ~63;
    const size_t bytes = (size_t)l->N * l->ld * sizeof(__nv_bfloat16);
    DC_TRY(dc_check_cuda(m->ctx, cudaMalloc((void**)&l->w, bytes + 256), "weight memory"));
    m->stack->owned.push_back(l->w);
    m->stack->weight_bytes += bytes;
    DC_TRY(dc_check_cuda(m->ctx, cudaMemsetAsync(l->w, 0, bytes + 256, m->ctx->stream), "weight memory"));
    return dc_lin_encode(m->ctx, &l->map, l->w, l->N, l->K, l->ld);
}

}  // namespace

int dc_stack_parse(dc_model* m, const dc_json& cj, const Shapes& shapes) {
    dc_stack* s = m->stack = new dc_stack();
    Reader r{m, s, &shapes, ""};
    const dc_json* arch = cj.get("architecture");
    const Arch* a = nullptr;
    for (const Arch& e : kArchs)
        if (arch && arch->kind == dc_json::STR && arch->str == e.name) a = &e;
    if (!a)
        return dc_fail(m->ctx, DC_B200_UNSUPPORTED, "config: architecture '%s' is not registered", arch ? arch->str.c_str() : "(none)");
    s->cfg.arch = a->name;
    s->cfg.block = a->block;
    s->cfg.tied = a->tied;
    if (a->embed_scale)
        if (const dc_json* e = r.object(cj, "embedding", "config")) s->cfg.embed_scale = (float)r.number(*e, "scale", "config.embedding");
    s->cfg.vocab = r.size(cj, "vocab", "config", 2);
    s->cfg.width = r.size(cj, "width", "config", 1, 8192);
    const dc_json* norm = cj.get("norm");
    if (norm && norm->kind == dc_json::OBJ) s->cfg.eps = (float)r.number(*norm, "eps", "config.norm");
    else r.bad("config: 'norm' is missing");
    const dc_json* layers = cj.get("layers");
    if (!layers || layers->kind != dc_json::ARR || layers->arr.empty()) r.bad("config: 'layers' is missing");
    if (!r.error.empty()) return dc_fail(m->ctx, DC_B200_INVALID_ARGUMENT, "%s", r.error.c_str());

    const int H = s->cfg.width, n = (int)layers->arr.size();
    s->layers.resize(n);
    {
        dc_stack_tensor t;
        t.name = "embed";
        t.shape = {s->cfg.vocab, H};
        if (s->cfg.tied) {
            t.lin = &s->head;
            s->head.N = dc_pad8(s->cfg.vocab);
            s->head.K = H;
        }
        r.tensor(t);
    }
    for (int i = 0; i < n && r.error.empty(); ++i) {
        const dc_json& lj = layers->arr[i];
        const std::string p = "l" + std::to_string(i) + ".", where = "config.layers[" + std::to_string(i) + "]";
        dc_stack_layer& L = s->layers[i];
        const dc_json *type = lj.get("type"), *mixer = lj.get("mixer"), *mlp = lj.get("mlp");
        L.kind = -1;
        for (const MixerType& t : kMixers)
            if (type && type->kind == dc_json::STR && type->str == t.name && (a->mixers >> t.kind & 1)) L.kind = t.kind;
        if (L.kind < 0 || !mixer || mixer->kind != dc_json::OBJ) {
            r.bad(where + ": unknown mixer type '" + (type ? type->str : "") + "'");
            break;
        }
        if (L.kind == DC_MIX_DELTA) read_delta(r, *mixer, p + "mix.", where + ".mixer", &L);
        else if (L.kind == DC_MIX_SSD) read_ssd(r, *mixer, p + "mix.", where + ".mixer", &L);
        else if (L.kind == DC_MIX_GQA) read_gqa(r, *mixer, p + "mix.", where + ".mixer", &L);
        else if (L.kind == DC_MIX_LIGHTNING) read_lightning(r, *mixer, p + "mix.", where + ".mixer", &L);
        else read_latent(r, *mixer, p + "mix.", where + ".mixer", &L, i);
        r.vec(&L.norm1, p + "norm1", {H}, 1);
        if (mlp && !mlp->is_null()) {
            const dc_json* kind = mlp->get("kind");
            if (!kind || kind->str != "dense") {
                r.bad(where + ".mlp: unknown kind");
                break;
            }
            if (a->block == DC_BLOCK_PARALLEL) {
                read_dense_clamped(r, *mlp, p + "mlp.", where + ".mlp", &L);
            } else {
                read_dense_gelu(r, *mlp, p + "mlp.", where + ".mlp", &L);
                r.vec(&L.norm2, p + "norm2", {H}, 1);
            }
        }
    }
    r.vec(&s->final_norm, "final.norm", {H}, 1);
    if (!s->cfg.tied) r.matrix(&s->head, "head", s->cfg.vocab, H);
    if (!r.error.empty()) return dc_fail(m->ctx, DC_B200_INVALID_ARGUMENT, "%s", r.error.c_str());

    // weight memory
    s->embed = new dc_weight();
    s->embed->type = DC_TYPE_BF16;
    s->embed->K = H;
    s->embed->N = s->cfg.vocab;
    s->embed->E = 1;
    DC_TRY(alloc_lin(m, &s->head));
    if (s->cfg.tied) {              // rows of the output matrix; bytes 0: the memory is not the embedding's own
        s->embed->row_bytes = (size_t)s->head.ld * 2;
        s->embed->bytes = 0;
        s->embed->dev = (uint8_t*)s->head.w;
    } else {
        s->embed->row_bytes = (size_t)H * 2;
        s->embed->bytes = s->embed->row_bytes * s->cfg.vocab;
        DC_TRY(dc_check_cuda(m->ctx, cudaMalloc((void**)&s->embed->dev, s->embed->bytes + 64), "weight memory"));
    }
    for (dc_stack_layer& L : s->layers) {
        dc_lin* ls[] = {&L.dl.in, &L.dl.a2, &L.dl.g2, &L.dl.o, &L.ssd.in, &L.ssd.o, &L.la.in, &L.la.ukv, &L.la.o, &L.gate_up, &L.down, &L.in, &L.out};
        for (dc_lin* l : ls) DC_TRY(alloc_lin(m, l));
        if (!L.li.decays.empty()) {
            const size_t bytes = L.li.decays.size() * 4;
            DC_TRY(dc_check_cuda(m->ctx, cudaMalloc((void**)&L.li.decay, bytes), "weight memory"));
            s->owned.push_back(L.li.decay);
            DC_TRY(dc_check_cuda(m->ctx, cudaMemcpy(L.li.decay, L.li.decays.data(), bytes, cudaMemcpyHostToDevice), "weight memory"));
        }
    }
    for (dc_stack_tensor& t : s->tensors)
        if (t.vec && !*t.vec) {
            DC_TRY(dc_check_cuda(m->ctx, cudaMalloc((void**)t.vec, (size_t)t.vec_len * 4 + 64), "weight memory"));
            s->owned.push_back(*t.vec);
            s->weight_bytes += (size_t)t.vec_len * 4;
            DC_TRY(dc_check_cuda(m->ctx, cudaMemsetAsync(*t.vec, 0, (size_t)t.vec_len * 4 + 64, m->ctx->stream), "weight memory"));
        }
    s->weight_bytes += s->embed->bytes;
    // tensors are copied on another stream: the zeros have to be there first
    return dc_check_cuda(m->ctx, cudaStreamSynchronize(m->ctx->stream), "weight memory");
}
