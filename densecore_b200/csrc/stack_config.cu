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
    float norm_plus = 0.0f; // norm weights are stored as their distance from this

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
    // a sliding window, with the first tokens of the sequence kept in sight or not; no mask: every earlier token
    void mask(const dc_json& o, const std::string& where, int* window, int* keep) {
        const dc_json* v = o.get("mask");
        if (!v || v->is_null()) return;
        *window = size(*v, "size", where + ".mask");
        const dc_json* k = v->get("keep_first");
        if (k && !k->is_null()) {
            if (keep) *keep = size(*v, "keep_first", where + ".mask", 0);
            else bad(where + ".mask: 'keep_first' is not available here");
        }
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
    // a norm's weight over the residual
    void norm(float** p, const std::string& name) {
        vec(p, name, {s->cfg.width}, norm_plus > 0.0f ? 0 : 1);
        s->tensors.back().plus = norm_plus;
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

void read_latent(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L, int il, bool gate) {
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
    r.mask(j, where, &d.window, nullptr);
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
    if (gate) d.off_g = r.matrix(&d.in, p + "g", d.heads, H);
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

// The projections of these mixers open L->in, their output matrix the columns of L->out: a parallel block's feed-forward
// goes beside both.
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

// What a design fixes of its grouped-query attention
enum {
    GQA_KEY_VALUES = 1,     // the values are the key projection before norm and rotation
    GQA_BIAS = 2,           // of the projections
    GQA_OUT_BIAS = 4,
    GQA_NORM_ALL = 8,       // queries and keys normed over all heads
    GQA_NORM_HEAD = 16,     // ... per head and map
    GQA_HALVES = 32,        // rotated pairs (i, i + dims / 2)
    GQA_SINK = 64,          // a sink of score 0
    GQA_TWO_MAPS = 128,     // differential attention
    GQA_UNTURNED = 256,     // no rotation
    GQA_CONV = 512,         // short convolutions behind the projections
    GQA_UNIT = 1024,        // queries, keys and values over their root mean square per head, no weights
    GQA_SIGMOID = 2048,     // sigmoid weights with a bias per head
    GQA_GATE = 4096,        // a gate per head
};

void read_gqa(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L, unsigned form) {
    dc_gqa_mixer& d = L->ga;
    const int H = r.s->cfg.width;
    d.maps = form & GQA_TWO_MAPS ? 2 : 1;
    d.heads = r.size(j, "heads", where);
    d.kv_heads = r.size(j, "kv_heads", where);
    d.dim = r.size(j, "dim", where, 1, d.maps > 1 ? 128 : 256);
    d.vdim = r.size(j, "vdim", where, 1, 256);
    if (form & GQA_KEY_VALUES && d.vdim != d.dim) r.bad(where + ": the values are the keys, so vdim must equal dim");
    if (d.heads % d.kv_heads) r.bad(where + ": heads is not a multiple of kv_heads");
    d.scale = (float)r.number(j, "scale", where);
    if (!(form & GQA_UNTURNED))
        if (const dc_json* rot = r.object(j, "rot", where)) r.rotation(*rot, where + ".rot", &d.rot);
    if (d.rot.dims > d.dim) r.bad(where + ".rot: dims is larger than the head");
    d.halves = form & GQA_HALVES;
    r.mask(j, where, &d.window, &d.keep);
    const dc_json* cap = j.get("softcap");
    if (cap && !cap->is_null() && !((d.softcap = (float)r.number(j, "softcap", where)) > 0.0f)) r.bad(where + ": 'softcap' must be positive");
    d.sink = form & GQA_SINK, d.sink_score = 0.0f;
    d.qk_norm = form & GQA_NORM_ALL ? DC_QK_NORM_ALL : form & GQA_NORM_HEAD ? DC_QK_NORM_HEAD : DC_QK_PLAIN;
    d.dim_p = dc_pad8(d.dim);
    d.vdim_p = dc_pad8(d.vdim);
    d.v_at = d.kv_heads * d.maps * d.dim_p;
    d.row = d.v_at + d.kv_heads * d.vdim_p;
    const int Q = d.heads * d.maps * d.dim, K = d.kv_heads * d.maps * d.dim, V = d.kv_heads * d.vdim;
    const bool own_values = !(form & GQA_KEY_VALUES);
    d.off_q = r.matrix(&L->in, p + "q", Q, H);
    d.off_k = r.matrix(&L->in, p + "k", K, H);
    d.off_v = own_values ? r.matrix(&L->in, p + "v", V, H) : d.off_k;
    if (form & GQA_BIAS) {
        const int rows = (L->in.N + DC_PAIR_ALIGN - 1) / DC_PAIR_ALIGN * DC_PAIR_ALIGN;     // as many as a product may store
        r.vec(&d.bias, p + "q.b", {Q}, 4, d.off_q, rows);
        r.vec(&d.bias, p + "k.b", {K}, 4, d.off_k, rows);
        if (own_values) r.vec(&d.bias, p + "v.b", {V}, 4, d.off_v, rows);
    }
    if (form & GQA_UNIT) {
        d.qk_norm = DC_QK_NORM_HEAD, d.v_norm = true;
    } else if (d.qk_norm != DC_QK_PLAIN) {
        const bool all = d.qk_norm == DC_QK_NORM_ALL;
        r.vec(&d.q_norm, p + "q.norm", {all ? Q : d.dim}, 1);
        r.vec(&d.k_norm, p + "k.norm", {all ? K : d.dim}, 1);
    }
    if (form & GQA_CONV) {       // weights sit at the channels' projection columns, so that one index serves both
        d.taps = r.size(j, "conv", where, 1, 16);
        const int C = dc_gqa_conv_cols(d);
        r.conv(&d.conv, p + "q.conv", Q, d.taps, d.off_q, C);
        r.conv(&d.conv, p + "k.conv", K, d.taps, d.off_k, C);
        r.conv(&d.conv, p + "v.conv", V, d.taps, d.off_v, C);
    }
    if (form & GQA_SIGMOID) r.vec(&d.score_bias, p + "pb", {d.heads}, 3);
    if (form & GQA_GATE) d.off_g = r.matrix(&L->in, p + "g", d.heads, H);
    if (d.maps > 1) {
        const char* names[] = {"lq1", "lk1", "lq2", "lk2"};
        for (int i = 0; i < 4; ++i) r.vec(&d.lam[i], p + names[i], {d.dim}, 0);
        d.diff = (float)r.number(j, "diff", where);
    }
    out_columns(r, p + "o", L, d.heads * d.vdim);
    if (form & GQA_OUT_BIAS) r.vec(&L->out_bias, p + "o.b", {H}, 4);
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

void read_general(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L) {
    dc_general_mixer& d = L->ge;
    const int H = r.s->cfg.width;
    d.heads = r.size(j, "heads", where);
    d.dim = r.size(j, "dim", where, 1, 256);
    d.rank = r.from_shape(p + "w1", 0);
    const int Q = d.heads * d.dim;
    d.off_r = r.matrix(&L->in, p + "r", Q, H);
    d.off_k = r.matrix(&L->in, p + "k", Q, H);
    d.off_v = r.matrix(&L->in, p + "v", Q, H);
    d.off_g = r.matrix(&L->in, p + "g", Q, H);
    d.off_a = r.matrix(&L->in, p + "a", Q, H);
    d.off_w = r.matrix(&L->in, p + "w1", d.rank, H);
    r.matrix(&d.w2, p + "w2", Q, d.rank);
    r.vec(&d.w0, p + "w0", {Q}, 4);
    r.vec(&d.a_bias, p + "a.b", {Q}, 4);
    r.vec(&d.norm, p + "norm", {Q}, 1);
    out_columns(r, p + "o", L, Q);
}

// Coefficients of a sublayer's hyper-connections
void read_hyper(Reader& r, const std::string& p, float** to) {
    const int n = r.s->cfg.streams, all = n * (n + 2);
    r.vec(to, p + "in", {n}, 5, 0, all);
    r.vec(to, p + "out", {n}, 1, n, all);
    r.vec(to, p + "mix", {n, n}, 5, 2 * n, all);
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

void read_dense(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L, int pair) {
    const int H = r.s->cfg.width;
    L->ff_pair = pair;
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

// What a design fixes of its experts
enum {
    MOE_CLAMPED = 1,        // clamped gated experts behind a sigmoid router
    MOE_SOFTMAX = 2,        // softmax router, chosen scores divided by their sum
    MOE_PLAIN = 4,          // square of relu between two matrices
};

void read_moe(Reader& r, const dc_json& j, const std::string& p, const std::string& where, dc_stack_layer* L, unsigned form) {
    dc_moe_ffn& f = L->moe;
    const int H = r.s->cfg.width;
    const dc_json *router = r.object(j, "router", where), *expert = r.object(j, "expert", where);
    if (!router || !expert) return;
    f.experts = r.size(*router, "experts", where + ".router", 1, DC_MOE_MAX_EXPERTS);
    f.top = r.size(*router, "top", where + ".router", 1, DC_MOE_MAX_TOP);
    f.softmax = form & MOE_SOFTMAX, f.plain = form & MOE_PLAIN;
    if (!f.softmax) f.scale = (float)r.number(*router, "scale", where + ".router");
    const dc_json* groups = f.softmax ? nullptr : router->get("groups");
    if (groups && !groups->is_null()) {
        f.groups = r.size(*groups, "count", where + ".router.groups", 1, DC_MOE_MAX_GROUPS);
        f.keep = r.size(*groups, "keep", where + ".router.groups");
    }
    if (f.experts % f.groups) r.bad(where + ".router: experts is not a multiple of groups.count");
    else if (f.keep > f.groups || f.top > f.experts / f.groups * f.keep) r.bad(where + ".router: fewer experts than 'top' in the kept groups");
    f.ff = r.size(*expert, "ff", where + ".expert");
    if (!f.plain) f.limit = (float)r.number(*expert, "limit", where + ".expert");
    if (!r.error.empty()) return;
    f.up_rows = f.plain ? (f.ff + 15) & ~15 : 2 * dc_pad8(f.ff);
    f.down_rows = (H + 15) & ~15;
    r.matrix(&f.router, p + "router", f.experts, H);
    if (!f.softmax) r.vec(&f.correction, p + "correction", {f.experts}, 4);
    f.up.N = f.experts * f.up_rows, f.up.K = H;
    f.down.N = f.experts * f.down_rows, f.down.K = f.ff;
    for (int e = 0; e < f.experts; ++e) {
        const std::string in = p + "e" + std::to_string(e) + ".";
        for (int i = f.plain ? 1 : 0; i < 3; ++i) {
            const bool down = i == 2;
            dc_stack_tensor t;
            t.name = in + (down ? "down" : i ? "up" : "gate");
            t.shape = {down ? H : f.ff, down ? f.ff : H};
            t.lin = down ? &f.down : &f.up;
            t.row0 = down ? e * f.down_rows : e * f.up_rows + (f.plain ? 0 : i);
            t.row_step = down || f.plain ? 1 : 2;
            r.tensor(t);
        }
    }
}

// {start, stop, times}: layers start .. stop - 1 run `times` times in a row
void read_loop(Reader& r, const dc_json& j, int layers) {
    dc_stack_config& c = r.s->cfg;
    c.loop_start = r.size(j, "start", "config.loop", 0, layers - 1);
    c.loop_stop = r.size(j, "stop", "config.loop", c.loop_start + 1, layers);
    c.loop_times = r.size(j, "times", "config.loop", 1, 1024);
    if (!r.error.empty()) return;
    const int ld = dc_pad8(c.width);
    r.vec(&r.s->loop_step, "loop.step", {c.loop_times, c.width}, 0, 0, (int64_t)c.loop_times * ld);
    r.s->tensors.back().pitch = ld;
}

// ---------------------------------------------------------------- designs
struct MixerType {
    const char* name;
    int kind;
    unsigned form;          // GQA_* of grouped-query attention; latent attention: 1 if its heads are gated
};
struct Arch {
    const char* name;
    int block;              // DC_BLOCK_*
    bool embed_scale;       // config.embedding.scale
    bool tied;
    bool loops;             // config.loop
    float norm_plus;        // norm weights are stored as their distance from this
    int dense;              // pairs of the dense feed-forward (-1: none)
    unsigned moe;           // form of the experts (0: none)
    std::vector<MixerType> mixers;
};
const Arch kArchs[] = {
    // Garilix: RMS norms on the sublayers' outputs only (x += norm(f(x))), tanh-gelu gated feed-forward
    {"Garilix", DC_BLOCK_POST_NORM, false, false, false, 0.0f, DC_PAIR_GELU, 0,
     {{"channel_delta", DC_MIX_DELTA, 0}, {"latent_attention", DC_MIX_LATENT, 0}, {"mamba2", DC_MIX_SSD, 0}}},
    // Datasun: mixer and clamped feed-forward side by side on one normed input, embedding table as output matrix
    {"Datasun", DC_BLOCK_PARALLEL, true, true, false, 0.0f, DC_PAIR_CLAMPED, 0,
     {{"attention", DC_MIX_GQA, GQA_KEY_VALUES | GQA_BIAS | GQA_OUT_BIAS | GQA_NORM_ALL | GQA_SINK}, {"lightning", DC_MIX_LIGHTNING, 0}}},
    // Gomuzen: norms ahead of the sublayers, looped layers, gated latent attention, differential attention, biased attention over
    // a window and the first tokens, experts in groups
    {"Gomuzen", DC_BLOCK_PRE_NORM, false, false, true, 0.0f, -1, MOE_CLAMPED,
     {{"latent_attention", DC_MIX_LATENT, 1}, {"attention", DC_MIX_GQA, GQA_NORM_HEAD | GQA_HALVES | GQA_TWO_MAPS}, {"attention_2", DC_MIX_GQA, GQA_BIAS | GQA_HALVES}}},
    // Vepitar: hyper-connections over several streams, generalized delta rule, attention with sigmoid weights and short
    // convolutions, dense layers or experts behind a softmax router, embedding table as output matrix
    {"Vepitar", DC_BLOCK_HYPER, false, true, false, 1.0f, DC_PAIR_SILU, MOE_SOFTMAX | MOE_PLAIN,
     {{"general_delta", DC_MIX_GENERAL, 0}, {"attention", DC_MIX_GQA, GQA_UNTURNED | GQA_CONV | GQA_UNIT | GQA_SIGMOID | GQA_GATE}}},
};

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
    Reader r{m, s, &shapes, "", 0.0f};
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
    r.norm_plus = a->norm_plus;
    if (a->block == DC_BLOCK_HYPER) {
        s->cfg.streams = r.size(cj, "streams", "config", 1, DC_MAX_STREAMS);
        s->cfg.residual_mult = (float)r.number(cj, "residual_mult", "config");
    }
    const dc_json* layers = cj.get("layers");
    if (!layers || layers->kind != dc_json::ARR || layers->arr.empty()) r.bad("config: 'layers' is missing");
    if (!r.error.empty()) return dc_fail(m->ctx, DC_B200_INVALID_ARGUMENT, "%s", r.error.c_str());

    const int H = s->cfg.width, n = (int)layers->arr.size();
    s->layers.resize(n);
    if (const dc_json* loop = cj.get("loop"); loop && !loop->is_null()) {
        if (!a->loops) r.bad("config: 'loop' is not available in this architecture");
        else read_loop(r, *loop, n);
    }
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
        unsigned form = 0;
        for (const MixerType& t : a->mixers)
            if (type && type->kind == dc_json::STR && type->str == t.name) L.kind = t.kind, form = t.form;
        if (L.kind < 0 || !mixer || mixer->kind != dc_json::OBJ) {
            r.bad(where + ": unknown mixer type '" + (type ? type->str : "") + "'");
            break;
        }
        if (L.kind == DC_MIX_DELTA) read_delta(r, *mixer, p + "mix.", where + ".mixer", &L);
        else if (L.kind == DC_MIX_SSD) read_ssd(r, *mixer, p + "mix.", where + ".mixer", &L);
        else if (L.kind == DC_MIX_GQA) read_gqa(r, *mixer, p + "mix.", where + ".mixer", &L, form);
        else if (L.kind == DC_MIX_GENERAL) read_general(r, *mixer, p + "mix.", where + ".mixer", &L);
        else if (L.kind == DC_MIX_LIGHTNING) read_lightning(r, *mixer, p + "mix.", where + ".mixer", &L);
        else read_latent(r, *mixer, p + "mix.", where + ".mixer", &L, i, form);
        const bool hyper = a->block == DC_BLOCK_HYPER;
        r.norm(&L.norm1, p + "norm1");
        if (hyper) read_hyper(r, p + "hc1.", &L.hyper[0]);
        if (mlp && !mlp->is_null()) {
            const dc_json* kind = mlp->get("kind");
            const std::string name = kind && kind->kind == dc_json::STR ? kind->str : "";
            if (!(name == "dense" && a->dense >= 0) && !(name == "moe" && a->moe)) {
                r.bad(where + ".mlp: unknown kind");
                break;
            }
            if (name == "moe") read_moe(r, *mlp, p + "mlp.", where + ".mlp", &L, a->moe);
            else if (a->block == DC_BLOCK_PARALLEL) read_dense_clamped(r, *mlp, p + "mlp.", where + ".mlp", &L);
            else read_dense(r, *mlp, p + "mlp.", where + ".mlp", &L, a->dense);
            if (a->block != DC_BLOCK_PARALLEL) r.norm(&L.norm2, p + "norm2");
            if (hyper) read_hyper(r, p + "hc2.", &L.hyper[1]);
        } else if (hyper) {
            for (const char* t : {"norm2", "hc2.in", "hc2.out", "hc2.mix"}) s->unused.insert(p + t);
        }
    }
    // the order in which layers run
    const dc_stack_config& c = s->cfg;
    auto run = [&](int from, int to, int pass) {
        for (int i = from; i < to; ++i) {
            dc_stack_run e;
            e.layer = i;
            e.step = i == from ? pass : -1;
            s->runs.push_back(e);
        }
    };
    const int stop = c.loop_times ? c.loop_stop : n, start = c.loop_times ? c.loop_start : n;
    run(0, start, -1);
    for (int t = 0; t < c.loop_times; ++t) run(start, stop, t);
    run(stop, n, -1);
    r.norm(&s->final_norm, "final.norm");
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
        dc_lin* ls[] = {&L.dl.in, &L.dl.a2, &L.dl.g2, &L.dl.o, &L.ssd.in, &L.ssd.o, &L.la.in, &L.la.ukv, &L.la.o, &L.gate_up, &L.down, &L.in, &L.out, &L.moe.router, &L.moe.up, &L.moe.down, &L.ge.w2};
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
