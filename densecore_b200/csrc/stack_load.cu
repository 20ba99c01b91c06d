// Layer-list decoders from a folder with config.json and model.safetensors (an 8-byte little-endian header length,
// the header's JSON, the data), or from a config alone for models with random weights.  Host code.
#include <fcntl.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include "dc_common.cuh"
#include "dc_model.h"
#include "dc_stack.h"

#define DC_TRY(expr)                       \
    do {                                   \
        int st_ = (expr);                  \
        if (st_ != DC_B200_OK) return st_; \
    } while (0)

namespace {

struct Mapped {
    const uint8_t* p = nullptr;
    size_t n = 0;
    ~Mapped() {
        if (p) munmap((void*)p, n);
    }
    bool open(const std::string& path) {
        const int fd = ::open(path.c_str(), O_RDONLY);
        if (fd < 0) return false;
        struct stat sb;
        if (fstat(fd, &sb) == 0 && sb.st_size > 0) {
            void* v = mmap(nullptr, (size_t)sb.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
            if (v != MAP_FAILED) p = (const uint8_t*)v, n = (size_t)sb.st_size;
        }
        ::close(fd);
        return p != nullptr;
    }
};

using Shapes = std::map<std::string, std::vector<int64_t>>;

bool read_shape(const dc_json& a, std::vector<int64_t>* out) {
    if (a.kind != dc_json::ARR) return false;
    for (const dc_json& d : a.arr) {
        if (d.kind != dc_json::NUM || d.num < 0 || d.num > 1e12 || d.num != (double)(int64_t)d.num) return false;
        out->push_back((int64_t)d.num);
    }
    return true;
}

int create(dc_ctx* ctx, const dc_json& config, const Shapes& shapes, int dtype, int max_seqs, int max_ctx, int pool_tokens, dc_model** out) {
    if (dtype != DC_DTYPE_BF16 && dtype != DC_DTYPE_F32) return dc_fail(ctx, DC_B200_INVALID_ARGUMENT, "model: dtype must be 0 (bf16) or 1 (f32)");
    if (max_seqs < 1 || max_seqs > DC_MAX_T || max_ctx < 1) return dc_fail(ctx, DC_B200_INVALID_ARGUMENT, "model: bad max_seqs or max_ctx");
    cudaSetDevice(ctx->device);
    dc_model* m = new dc_model();
    m->ctx = ctx;
    int st = dc_stack_parse(m, config, shapes);
    if (st == DC_B200_OK) {
        m->stack->dtype = dtype;
        dc_model_config& c = m->cfg;
        c.n_layer = (int)m->stack->runs.size();
        c.hidden = m->stack->cfg.width;
        c.vocab = m->stack->cfg.vocab;
        c.rms_eps = m->stack->cfg.eps;
        c.max_seqs = max_seqs;
        c.max_ctx = max_ctx;
        c.ep_size = 1;
        st = dc_stack_create_cache(m, pool_tokens);
    }
    if (st != DC_B200_OK) {
        dc_b200_model_destroy(m);
        return st;
    }
    *out = m;
    return DC_B200_OK;
}

int parse_text(dc_ctx* ctx, const char* what, const char* text, size_t n, dc_json* out) {
    std::string err;
    if (!dc_json_parser(text, n).parse(out, &err) || out->kind != dc_json::OBJ)
        return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "%s is not a JSON object (%s)", what, err.c_str());
    return DC_B200_OK;
}

int load_dir(dc_ctx* ctx, const std::string& dir, int dtype, int max_seqs, int max_ctx, int pool_tokens, dc_model** out) {
    Mapped cfg, st;
    if (!cfg.open(dir + "/config.json")) return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "cannot read %s/config.json", dir.c_str());
    if (!st.open(dir + "/model.safetensors")) return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "cannot read %s/model.safetensors", dir.c_str());
    dc_json config, header;
    DC_TRY(parse_text(ctx, "config.json", (const char*)cfg.p, cfg.n, &config));
    uint64_t hn = 0;
    if (st.n >= 8) memcpy(&hn, st.p, 8);
    if (st.n < 8 || hn > st.n - 8) return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "model.safetensors: header length out of range");
    DC_TRY(parse_text(ctx, "model.safetensors header", (const char*)st.p + 8, (size_t)hn, &header));
    const uint8_t* data = st.p + 8 + hn;
    const size_t bytes = st.n - 8 - (size_t)hn;

    struct Entry {
        std::string name;
        int type;
        std::vector<int64_t> shape;
        size_t off;
    };
    std::vector<Entry> entries;
    Shapes shapes;
    for (auto& kv : header.obj) {
        if (kv.first == "__metadata__") continue;
        const dc_json *dt = kv.second.get("dtype"), *sh = kv.second.get("shape"), *of = kv.second.get("data_offsets");
        Entry e;
        std::vector<int64_t> span;
        e.name = kv.first;
        if (!dt || !sh || !of || !read_shape(*sh, &e.shape) || !read_shape(*of, &span) || span.size() != 2 || span[0] > span[1] || (size_t)span[1] > bytes)
            return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "model.safetensors: bad entry for '%s'", e.name.c_str());
        size_t n = 1, esz = 0;
        for (int64_t d : e.shape) n *= (size_t)d;
        if (dt->str == "BF16") e.type = DC_TYPE_BF16, esz = 2;
        else if (dt->str == "F32") e.type = DC_TYPE_F32, esz = 4;
        else return dc_fail(ctx, DC_B200_UNSUPPORTED, "model.safetensors: '%s' has type %s", e.name.c_str(), dt->str.c_str());
        if (n * esz != (size_t)(span[1] - span[0]))
            return dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "model.safetensors: '%s' has %lld bytes for its shape", e.name.c_str(), (long long)(span[1] - span[0]));
        e.off = (size_t)span[0];
        shapes[e.name] = e.shape;
        entries.push_back(e);
    }
    DC_TRY(create(ctx, config, shapes, dtype, max_seqs, max_ctx, pool_tokens, out));
    dc_model* m = *out;
    for (const Entry& e : entries) {
        if (m->stack->unused.count(e.name)) continue;
        auto it = m->stack->index.find(e.name);
        int rc = DC_B200_OK;
        if (it == m->stack->index.end()) {
            rc = dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "model.safetensors: '%s' is not a tensor of this model", e.name.c_str());
        } else {
            // vectors may come with any shape of the same length
            const dc_stack_tensor& t = m->stack->tensors[it->second];
            int64_t n = 1, want = 1;
            for (int64_t d : e.shape) n *= d;
            for (int64_t d : t.shape) want *= d;
            const bool ok = t.vec ? n == want : e.shape == t.shape;
            const int64_t ne[4] = {t.shape.back(), t.shape.size() > 1 ? t.shape[0] : 1, 1, 1};
            std::vector<uint8_t> copy;     // the file aligns nothing: element reads want an aligned copy of vectors
            const uint8_t* src = data + e.off;
            if (t.vec) copy.assign(src, src + (size_t)n * (e.type == DC_TYPE_F32 ? 4 : 2)), src = copy.data();
            rc = ok ? dc_b200_model_set_tensor(m, e.name.c_str(), e.type, ne, src)
                    : dc_fail(ctx, DC_B200_MODEL_LOAD_FAILED, "model.safetensors: '%s' has the wrong shape", e.name.c_str());
        }
        if (rc != DC_B200_OK) {
            dc_b200_model_destroy(m);
            *out = nullptr;
            return rc;
        }
    }
    return DC_B200_OK;
}

}  // namespace

extern "C" {

int dc_b200_model_from_dir(dc_ctx* ctx, const char* dir, int dtype, int max_seqs, int max_ctx, int pool_tokens, dc_model** out) {
    if (!ctx || !dir || !out) return DC_B200_INVALID_ARGUMENT;
    *out = nullptr;
    return load_dir(ctx, dir, dtype, max_seqs, max_ctx, pool_tokens, out);
}

int dc_b200_model_from_config(dc_ctx* ctx, const char* config_json, const char* shapes_json, int dtype, int max_seqs, int max_ctx, int pool_tokens,
                              dc_model** out) {
    if (!ctx || !config_json || !out) return DC_B200_INVALID_ARGUMENT;
    *out = nullptr;
    dc_json config, sj;
    DC_TRY(parse_text(ctx, "config", config_json, strlen(config_json), &config));
    Shapes shapes;
    if (shapes_json) {
        DC_TRY(parse_text(ctx, "shapes", shapes_json, strlen(shapes_json), &sj));
        for (auto& kv : sj.obj)
            if (!read_shape(kv.second, &shapes[kv.first])) return dc_fail(ctx, DC_B200_INVALID_ARGUMENT, "shapes: bad shape for '%s'", kv.first.c_str());
    }
    return create(ctx, config, shapes, dtype, max_seqs, max_ctx, pool_tokens, out);
}

}  // extern "C"
