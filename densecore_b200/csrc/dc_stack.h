// Layer-list decoders: models whose config.json names the mixer and the feed-forward of every layer.  A model
// is a list of layers built from the mechanisms below; every size and constant is a field, so that a design is
// a line in the architecture table (stack_config.cu) and not a forward pass of its own.
//
// Numbers: weights are bf16 in HBM; the residual, norms, decays, gates, recurrent state and attention scores are
// f32.  A bf16 model rounds the inputs of matrix products to bf16 (accumulation is f32), an f32 model keeps every
// activation in f32.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>

#include <map>
#include <set>
#include <string>
#include <tuple>
#include <vector>

#include "dc_internal.h"
#include "dc_json.h"
#include "dc_kv.h"

struct dc_model;

enum { DC_MIX_DELTA = 0, DC_MIX_LATENT = 1, DC_MIX_SSD = 2, DC_MIX_GQA = 3, DC_MIX_LIGHTNING = 4, DC_MIX_GENERAL = 5 };
enum { DC_DTYPE_BF16 = 0, DC_DTYPE_F32 = 1 };
// How a layer's sublayers meet the residual.  POST_NORM: x += norm1(mixer(x)), then x += norm2(ff(x)).  PARALLEL: with
// h = norm1(x), x += mixer(h) + ff(h); the input matrices of both are one product, and so are the output matrices.
// PRE_NORM: x += mixer(norm1(x)), then x += ff(norm2(x)).  HYPER: pre-norm over a residual of several streams, see dc_hyper.
enum { DC_BLOCK_POST_NORM = 0, DC_BLOCK_PARALLEL = 1, DC_BLOCK_PRE_NORM = 2, DC_BLOCK_HYPER = 3 };
enum { DC_PAIR_GELU = 0, DC_PAIR_CLAMPED = 1, DC_PAIR_SILU = 2 };
enum { DC_ACT_SILU = 0, DC_ACT_RELU2 = 1 };     // of single rows

#define DC_MAX_SPLITS 64        // key splits of a decode step's attention

static inline int dc_pad8(int n) { return (n + 7) & ~7; }

// Rows of one or more weight matrices that share their input, bf16, every row padded with zeros to `ld`
// elements.  Segments start at row offsets that are multiples of eight (unused rows are zero).
struct dc_lin {
    __nv_bfloat16* w = nullptr;
    int N = 0, K = 0, ld = 0;
    CUtensorMap map;            // [N rows][K], box 128 x 64, 128-byte swizzle
};

// What becomes of a product's rows.  Rows below pair0 are stored (to outb if given, else to out) after the bias and, for
// the first act_rows of them, silu or the square of relu; `add` adds to what out holds.  Rows from pair0 on are gate and
// up rows in turn and each pair is one value of poutb / pout: gelu_tanh(gate) up, silu(gate) up, or with both clamped
// (gate from above only) gate sigmoid(1.702 gate) (up + 1).
#define DC_PAIR_ALIGN 32        // pair0 is a multiple of this
struct dc_lin_epi {
    float* out = nullptr;
    __nv_bfloat16* outb = nullptr;
    int ldo = 0, n_store = 0;   // rows stored: at most n_store (launchers: also at most the matrix' rows)
    const float* bias = nullptr;
    int act_rows = 0, act = DC_ACT_SILU;
    bool add = false;
    int pair0 = 1 << 30, pair_kind = DC_PAIR_GELU;
    float limit = 0.0f;
    float* pout = nullptr;
    __nv_bfloat16* poutb = nullptr;
    int ldp = 0, n_pairs = 0;
    const float* tok_scale = nullptr;        // factor of every pair value, or of every row after its activation, of a token (grouped products)
    unsigned long long* keys = nullptr;      // packed greedy picks per token (products of up to DC_MAX_T tokens)

    static dc_lin_epi store(float* out, __nv_bfloat16* outb, int ldo, unsigned long long* keys = nullptr) {
        dc_lin_epi e;
        e.out = out, e.outb = outb, e.ldo = e.n_store = ldo, e.keys = keys;
        return e;
    }
    dc_lin_epi& pairs(int row0, int kind, float clamp, float* o, __nv_bfloat16* ob, int ld, int n) {
        pair0 = row0, pair_kind = kind, limit = clamp, pout = o, poutb = ob, ldp = ld, n_pairs = n;
        if (n_store > row0) n_store = row0;
        return *this;
    }
};

// Input of a tensor-core product: a bf16 buffer [rows][ld] with the tensor map that reads its first K columns.
struct dc_tc_in {
    const __nv_bfloat16* x = nullptr;
    int K = 0, ld = 0;
    CUtensorMap map;            // box 128 x 64
};

struct dc_delta_mixer {         // gated delta rule with one decay per key channel
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 0, a_rank = 0, g_rank = 0;
    float unit_eps = 1e-6f, q_scale = 1.0f;
    dc_lin in, a2, g2, o;       // in: q | k | v | b | a1 | g1
    int off_q = 0, off_k = 0, off_v = 0, off_b = 0, off_a = 0, off_g = 0;
    float *conv = nullptr;      // [taps][C], C = q, k and v projection columns
    float *neg_a = nullptr;     // [heads]: -exp(A_log)
    float *dt_bias = nullptr;   // [heads * dim]
    float *norm = nullptr;      // [vdim]
};

struct dc_ssd_mixer {           // Mamba-2
    int heads = 0, vdim = 0, state = 0, groups = 0, norm_groups = 0, taps = 0;
    dc_lin in, o;               // in: z | x B C | dt
    int off_z = 0, off_x = 0, off_dt = 0;
    float *conv = nullptr, *conv_b = nullptr, *neg_a = nullptr, *dt_bias = nullptr, *D = nullptr, *norm = nullptr;
};

struct dc_latent_mixer {        // attention over a compressed key/value latent with a shared rotated key part
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, window = 0;   // window 0: every earlier token
    int kv_from = -1;           // layer whose cached latent this layer reads (-1: its own)
    float scale = 1.0f;
    double rot_base = 10000.0;
    dc_lin in, ukv, o;          // in: q | c and rotated key part;  ukv: per head uk, then per head uv (rows padded to 8)
    int off_q = 0, off_kv = 0, dim_p = 0, vdim_p = 0, uv_row = 0;
    int off_g = -1;             // one gate per head: the head's output is multiplied by sigmoid of this row (-1: none)
    float* kv_norm = nullptr;   // [kv_rank]
    const float* cos_sin = nullptr;   // [max_ctx][rot_dim / 2][2]
    int row = 0;                // elements per cached token
    int range = 0;              // which of the step's key ranges (distinct windows)
};

// Rotary angles: pair i of `dims` turns by pos * f_i with f_i = base^(-2i / dims).  YaRN (factor > 0): pairs that turn
// less than `slow` times over `original` positions turn slower by the factor, those above `fast` turns are left alone,
// linear in between; cos and sin are multiplied by 0.1 ln(factor) + 1.
struct dc_rotation {
    int dims = 0;
    double base = 10000.0, factor = 0.0, original = 0.0, fast = 0.0, slow = 0.0;
    bool operator<(const dc_rotation& o) const {
        return std::tie(dims, base, factor, original, fast, slow) < std::tie(o.dims, o.base, o.factor, o.original, o.fast, o.slow);
    }
};

enum { DC_QK_PLAIN = 0, DC_QK_NORM_ALL = 1, DC_QK_NORM_HEAD = 2 };

// Grouped-query attention.  maps 2: every head has two queries and keys over the same values; the second map's output is
// taken off the first's, weighted by lambda, and the difference is normed per head and multiplied by 1 - diff.  score_bias:
// no softmax, a visible key counts sigmoid(score + the head's bias), unnormalized.
struct dc_gqa_mixer {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, maps = 1;
    int window = 0, keep = 0;   // window 0: every earlier token; else the last `window` and the sequence's first `keep`
    float scale = 1.0f, softcap = 0.0f;     // softcap c > 0: scores become c tanh(score / c)
    bool sink = false;          // a term of the softmax' denominator with score sink_score and no value
    float sink_score = 0.0f;
    dc_rotation rot;
    bool halves = false;        // pairs (i, i + dims / 2) instead of (2i, 2i + 1)
    int qk_norm = DC_QK_PLAIN;  // RMS norm of queries and keys ahead of the rotation: none, over all heads, per head and map
    int off_q = 0, off_k = 0, off_v = 0;    // projection rows; off_v = off_k: the values are the keys before norm and rotation
    int dim_p = 0, vdim_p = 0;  // padded sizes in the cached rows
    float *bias = nullptr;      // of the projection rows
    float *q_norm = nullptr, *k_norm = nullptr;             // [heads * dim] and [kv_heads * dim], or [dim] (null: no weight)
    bool v_norm = false;        // every head's value over its root mean square
    int taps = 0;               // short causal convolution of the projections ahead of everything else (0: none)
    float *conv = nullptr;      // [taps][projection columns up to the values' end]
    float *score_bias = nullptr;            // [heads]
    int off_g = -1;             // one gate per head: the head's output is multiplied by sigmoid of this row (-1: none)
    float diff = 0.0f, lambda = 0.0f;       // lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
    float* lam[4] = {};         // lq1, lk1, lq2, lk2 [dim]
    const float* cos_sin = nullptr;
    int row = 0, v_at = 0;      // row: kv_heads * maps keys of dim_p, from v_at kv_heads values of vdim_p
    int range = 0;
};

struct dc_lightning_mixer {     // linear attention with one constant decay per head: S <- decay S + k v^T, o = S^T q
    int heads = 0, dim = 0, vdim = 0;
    int off_q = 0, off_k = 0, off_v = 0, off_g = 0;         // q, k, v pass through silu
    std::vector<float> decays;  // one per head, from the configuration
    float *decay = nullptr;     // their device copy
    float *norm = nullptr;      // [heads * vdim]: all heads are normed together, then gated by sigmoid(g)
};

// Generalized delta rule: S <- diag(w) S - (a u)(u^T S) + k v^T, o = S^T r, with the unit key u, a removal rate a and a decay
// w = exp(-e^(-1/2) sigmoid(W2 tanh(W1 h) + w0)) per key channel.  Heads are normed, weighted and gated by sigmoid(g).
struct dc_general_mixer {
    int heads = 0, dim = 0, rank = 0;       // values have the keys' size
    float unit_eps = 1e-6f;
    int off_r = 0, off_k = 0, off_v = 0, off_g = 0, off_a = 0, off_w = 0;   // projection rows; off_w: W1
    dc_lin w2;
    float *w0 = nullptr, *a_bias = nullptr, *norm = nullptr;                // [heads * dim]
};

// Mixture of experts.  Scores are sigmoid(router); choices are made on score + correction, among the experts of the `keep`
// groups whose two best choice scores sum up highest; an expert's weight is its score times scale.  softmax: scores are the
// softmax over all experts, and the chosen ones' are divided by their sum.  Experts are clamped and gated, or (plain) the
// square of relu between two matrices.
#define DC_MOE_MAX_EXPERTS 512
#define DC_MOE_MAX_TOP 32
#define DC_MOE_MAX_GROUPS 32
struct dc_moe_ffn {
    int experts = 0, top = 0, groups = 1, keep = 1, ff = 0;
    float scale = 1.0f, limit = 0.0f;
    bool softmax = false, plain = false;
    dc_lin router, up, down;    // up: per expert up_rows rows (gate and up in turn, or up alone), down: per expert down_rows
    int up_rows = 0, down_rows = 0;
    float* correction = nullptr;
};

struct dc_stack_layer {
    int kind = DC_MIX_DELTA;
    dc_delta_mixer dl;
    dc_ssd_mixer ssd;
    dc_latent_mixer la;
    dc_gqa_mixer ga;
    dc_lightning_mixer li;
    dc_general_mixer ge;
    // parallel blocks: mixer rows, then (from pair0) gate and up rows in turn; mixer columns, then (from out_ff) the
    // feed-forward's
    dc_lin in, out;
    int pair0 = 0, out_ff = 0;
    float* out_bias = nullptr;
    float limit = 0.0f;         // of the clamped pairs
    int ff = 0;                 // 0: no dense feed-forward
    dc_moe_ffn moe;             // experts 0: none
    dc_lin gate_up, down;       // gate_up: rows 2i = gate row i, 2i + 1 = up row i
    int ff_pair = DC_PAIR_GELU; // dense feed-forward of its own
    float *norm1 = nullptr, *norm2 = nullptr;
    float* hyper[2] = {};       // coefficients of the sublayers: in [streams] | out [streams] | mix [from][to]
};

// One run of a layer: a looped layer has several, each with a cache or state of its own.
struct dc_stack_run {
    int layer = 0;
    int step = -1;              // row of the loop's vectors that is added to the residual ahead of this run
    int plane = -1;             // cache plane of an attention layer
    size_t state_off = 0, ring_off = 0;     // byte offsets in a sequence's state slot
};

// Where a named tensor goes: rows of a dc_lin, or a vector of floats.
struct dc_stack_tensor {
    std::string name;
    std::vector<int64_t> shape;
    dc_lin* lin = nullptr;
    int row0 = 0, row_step = 1; // destination row of tensor row i: row0 + i * row_step (head_rows 0) ...
    int head_rows = 0, head_pad = 0;      // ... or row0 + (i / head_rows) * head_pad + i % head_rows
    int col0 = 0;               // destination column
    float** vec = nullptr;
    int64_t vec_off = 0, vec_len = 0;     // destination range and the vector's whole length
    bool neg_exp = false;       // stored as -exp(value)
    float plus = 0.0f;          // added to what the file holds
    int64_t pitch = 0;          // a vector of shape [n, k] stored with rows of this many floats
    int64_t cols = 0;           // a vector of shape [n, taps] stored transposed: element (c, j) at j * cols + vec_off + c
    bool loaded = false;
    int synth = 0;              // random-weight kind: 0 matrix, 1 norm weight, 2 decay exponent, 3 step bias, 4 small vector, 5 one over the streams
};

struct dc_stack_config {
    std::string arch;
    int vocab = 0, width = 0, block = DC_BLOCK_POST_NORM;
    int loop_start = 0, loop_stop = 0, loop_times = 0;      // layers start .. stop - 1 run `times` times in a row (0: no loop)
    float eps = 1e-5f, embed_scale = 1.0f;
    bool tied = false;          // the output matrix is the embedding table
    int streams = 1;            // of the residual
    float residual_mult = 1.0f;
};

// One step's tokens on the device.  Entry e is tokens starts[e] .. starts[e + 1] - 1, consecutive positions of one
// sequence.
struct dc_step {
    int T = 0, E = 0;
    const int32_t *tokens = nullptr, *seq_ids = nullptr, *positions = nullptr, *starts = nullptr;
    bool b16 = false;           // inputs of matrix products in bf16
    bool tc = false;            // ... and more than DC_MAX_T tokens: tiled products, prompt attention
    bool single = false;        // every entry is one token
};

struct dc_stack_buffers {
    int cap = 0;                // tokens of a step
    int key_cap = 0;            // gathered keys of a step
    int32_t* meta = nullptr;    // device copy of one step's metadata
    int32_t* h_meta = nullptr;  // pinned, DC_STACK_META_SLOTS slots
    int meta_ints = 0, meta_slot = 0;
    int32_t *iota = nullptr, *chunk = nullptr;   // constant entry starts: one token each; one entry of n tokens at chunk + 2 n
    float *x = nullptr, *x2 = nullptr, *h = nullptr, *y = nullptr, *proj = nullptr, *act = nullptr, *scan = nullptr, *low = nullptr, *gate = nullptr, *small = nullptr, *blk = nullptr;
    float *mix = nullptr, *ff = nullptr, *lm_x = nullptr;   // mix, ff, lm_x: f32 models
    __nv_bfloat16 *lm_xb = nullptr, *xb = nullptr, *mixb = nullptr, *ffb = nullptr, *lowb = nullptr;
    __nv_bfloat16 *keys_c = nullptr, *keys_r = nullptr, *keys_kv = nullptr;
    float *qa = nullptr, *part = nullptr, *part_ml = nullptr;
    float* q = nullptr;         // grouped-query attention: turned queries (qb: bf16, prompts)
    __nv_bfloat16 *qb = nullptr, *actb = nullptr;
    float* chunk_state = nullptr;        // linear attention: the state ahead of every chunk
    // mixture of experts: an assignment is a (token, choice); rows are assignments sorted by expert
    int32_t *moe_ids = nullptr, *moe_row = nullptr, *moe_src = nullptr, *moe_off = nullptr;
    float *moe_w = nullptr, *moe_row_w = nullptr, *moe_logits = nullptr, *moe_hid = nullptr, *moe_y = nullptr;
    __nv_bfloat16 *moe_x = nullptr, *moe_hidb = nullptr, *moe_yb = nullptr;
    int moe_rows = 0;
    std::vector<void*> owned;
};
#define DC_STACK_META_SLOTS 4

struct dc_stack {
    dc_stack_config cfg;
    int dtype = DC_DTYPE_BF16;
    std::vector<dc_stack_layer> layers;
    std::vector<dc_stack_run> runs;
    float* hyper_sum = nullptr; // [streams]: ones
    float* loop_step = nullptr; // [loop_times][width padded to 8]
    dc_weight* embed = nullptr;
    dc_lin head;
    float* final_norm = nullptr;
    std::vector<dc_stack_tensor> tensors;
    std::map<std::string, int> index;
    std::set<std::string> unused;        // files may hold these too: norms and coefficients of sublayers that a layer does not have
    std::vector<void*> owned;   // weight memory
    size_t weight_bytes = 0;
    std::map<dc_rotation, float*> rot;   // cos/sin tables [max_ctx][dims / 2][2]
    std::vector<int> windows;   // distinct windows of the attention layers
    int splits = 1;             // key splits of a decode step's attention
    dc_stack_buffers b;
    std::map<std::pair<const void*, int>, dc_tc_in> ins;
};

// ---- stack_config.cu: architecture table, config.json -> layers and tensor slots
int dc_stack_parse(dc_model* m, const dc_json& config, const std::map<std::string, std::vector<int64_t>>& shapes);
// ---- stack.cu
int dc_stack_finalize(dc_model* m);
void dc_stack_release(dc_model* m);
int dc_stack_set_tensor(dc_model* m, const char* name, int type, const int64_t ne[4], const void* data);
int dc_stack_init_synthetic(dc_model* m, uint64_t seed, float sigma);
int dc_stack_create_cache(dc_model* m, int pool_tokens);
// a step of up to DC_MAX_T tokens whose inputs are in the model's step buffers: one token per sequence, or (chunk)
// consecutive tokens of one sequence
int dc_stack_enqueue_small(dc_model* m, int T, bool chunk, int lm_mode, bool feedback);
// entries of any length as one batch: counts[e] next tokens of seqs[e].  rows: places (flat token index, ascending)
// whose logits are wanted; logits_host / picks_host may be null.
int dc_stack_batch(dc_model* m, int E, const int32_t* seqs, const int32_t* counts, const int32_t* tokens, int n_rows,
                   const int32_t* rows, float* logits_host, int32_t* picks_host);
void dc_stack_stats(dc_model* m, double* weight_bytes, double* kv_bytes_per_token);

// ---- linear.cu / linear_tc.cu: y = W x
// T <= DC_MAX_T tokens, bf16 or f32 inputs: one pass over the weights
int dc_launch_linear_mma(dc_ctx* ctx, const dc_lin& w, const __nv_bfloat16* x, int ldx, int T, const dc_lin_epi& epi);
int dc_launch_linear_rows(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, const dc_lin_epi& epi);
// any T, f32 inputs (f32 models)
int dc_launch_linear_f32(dc_ctx* ctx, const dc_lin& w, const float* x, int ldx, int T, const dc_lin_epi& epi);
// any T, bf16 inputs on the tensor cores
int dc_launch_linear_tc(dc_ctx* ctx, const dc_lin& w, const dc_tc_in& x, int T, const dc_lin_epi& epi);
// the same per expert: rows group_off[e] .. group_off[e + 1] - 1 of x (of max_rows) with rows e * group_rows .. of w
int dc_launch_linear_grouped_tc(dc_ctx* ctx, const dc_lin& w, int groups, int group_rows, const int32_t* group_off, const dc_tc_in& x, int max_rows,
                                const dc_lin_epi& epi);
int dc_lin_encode(dc_ctx* ctx, CUtensorMap* map, const __nv_bfloat16* base, int rows, int K, int ld);

// ---- norm_act.cu
// x += rms(y) * w per token; xb (optional): bf16 copy of the new x
int dc_launch_post_norm(dc_ctx* ctx, float* x, const float* y, const float* w, int T, int H, int ld, float eps, __nv_bfloat16* xb);
// out[r] = rms(x[rows ? rows[r] : first + r]) * w
int dc_launch_norm_rows(dc_ctx* ctx, const float* x, const float* w, const int32_t* rows, int first, int R, int H, int ld, float eps,
                        float* out, __nv_bfloat16* outb, int ldo);

// x += step (one row, optional) + for every token the sum of its k rows y[rows[t * k + i]] (optional, yb: bf16); then, with
// w, out = rms(x) * w as above.  x is rewritten where something was added.
struct dc_row_sum {
    const float* y = nullptr;
    const __nv_bfloat16* yb = nullptr;
    const int32_t* rows = nullptr;
    int k = 0, ld = 0;
};
int dc_launch_pre_norm(dc_ctx* ctx, float* x, const float* step, const dc_row_sum& sum, const float* w, int T, int H, int ld, float eps, float* out,
                       __nv_bfloat16* outb);

// A residual of `streams` streams, [token][stream][ld], and what it still owes: the sublayer before left y (one row a token, or
// the sum of rows) and its coefficients `done`; stream t becomes sum_s mix[s][t] x_s + mul out[t] y.  u = sum_t next[t] x_t is
// what the next sublayer's norm takes.  Without `done` nothing is owed.  x_out (optional) is another buffer than x: several
// CTAs of a token read x.
#define DC_MAX_STREAMS 8
struct dc_hyper {
    int streams = 1;
    bool first = false;         // x has one row per token that all streams share
    const float* x = nullptr;
    float* x_out = nullptr;
    const float* y = nullptr;
    dc_row_sum sum;
    const float *done = nullptr, *next = nullptr;
    float mul = 1.0f;
};
// out row r: u of token rows[r] (rows null: first + r), normed with w (w null: as it is)
int dc_launch_hyper_norm(dc_ctx* ctx, const dc_hyper& hy, const float* w, const int32_t* rows, int first, int R, int H, int ld, float eps, float* out,
                         __nv_bfloat16* outb);

// ---- ffn_moe.cu
// norm of the residual (out / outb), router logits, choices (ids and weights [T][top]); where it fits: few tokens, or a bf16
// model whose width and experts leave room in shared memory
bool dc_moe_norm_route_fits(const dc_moe_ffn& f, bool b16, int T, int ld);
// hy: the row that is normed comes from the streams instead of x
int dc_launch_moe_norm_route(dc_ctx* ctx, const dc_moe_ffn& f, const float* x, const dc_hyper* hy, const float* w, int T, int H, int ld, float eps, float* out,
                             __nv_bfloat16* outb, int32_t* ids, float* weights);
// choices from logits [T][ldl]
int dc_launch_moe_route(dc_ctx* ctx, const dc_moe_ffn& f, const float* logits, int ldl, int T, int32_t* ids, float* weights);
// assignments sorted by expert: off [experts + 1]; src, row_w [rows]: token and weight of a row; row [T][top]: an assignment's row
int dc_launch_moe_order(dc_ctx* ctx, const dc_moe_ffn& f, const int32_t* ids, const float* weights, int T, int32_t* off, int32_t* src, float* row_w,
                        int32_t* row);
int dc_launch_moe_gather(dc_ctx* ctx, const __nv_bfloat16* x, int ldx, const int32_t* src, int rows, __nv_bfloat16* out);
// up to DC_MAX_T tokens of bf16 models: hidden values of every assignment times its weight, then x = or += their products
int dc_launch_moe_up_mma(dc_ctx* ctx, const dc_moe_ffn& f, const __nv_bfloat16* xb, int ldx, int T, const int32_t* ids, const float* weights,
                         __nv_bfloat16* hid, int ldh);
int dc_launch_moe_down_mma(dc_ctx* ctx, const dc_moe_ffn& f, const __nv_bfloat16* hid, int ldh, int T, const int32_t* ids, int H, float* x, int ldx,
                             bool add);
// f32 models: sorted rows; src: input row of a row (null: itself)
int dc_launch_moe_f32(dc_ctx* ctx, const dc_lin& w, int experts, int group_rows, const int32_t* off, int rows, const float* x, int ldx,
                      const int32_t* src, const dc_lin_epi& epi);

// ---- mix_recur.cu
struct dc_state_ref {           // per-sequence state in the cache manager's slots
    uint8_t* base = nullptr;
    size_t slot_bytes = 0, state_off = 0, ring_off = 0;
};
// most blocks that T tokens of E entries make; floats of one block's shared factors, all heads
int dc_scan_blocks(int T, int E);
size_t dc_delta_block_floats(const dc_delta_mixer& m);
size_t dc_ssd_block_floats(const dc_ssd_mixer& m);
int dc_launch_delta_prep(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp,
                         float* act, int lda, float* small, __nv_bfloat16* lowb, int ldl);
int dc_launch_delta_scan(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* act, int lda,
                         const float* small, const float* low, int ldd, float* blk, const float* raw_g, int ldg, float eps, float* o,
                         float* mix, __nv_bfloat16* mixb, int ldm);
int dc_launch_delta_decode(dc_ctx* ctx, const dc_delta_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp,
                           float eps, float* mix, __nv_bfloat16* mixb, int ldm);
int dc_launch_ssd(dc_ctx* ctx, const dc_ssd_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float* act,
                  int lda, float* small, float* blk, float* y, float eps, float* mix, __nv_bfloat16* mixb, int ldm);
int dc_launch_ssd_decode(dc_ctx* ctx, const dc_ssd_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float* y, int ldy,
                         float eps, float* mix, __nv_bfloat16* mixb, int ldm);
// generalized delta rule.  tanh: columns off_w .. of proj, to lowb or in place.  scan: entries of any length; low: decay
// projections [T][ldd].  decode: one token per sequence, everything from the projections.
size_t dc_general_block_floats(const dc_general_mixer& m);
int dc_launch_general_tanh(dc_ctx* ctx, const dc_general_mixer& m, int T, float* proj, int ldp, __nv_bfloat16* lowb, int ldl);
int dc_launch_general_scan(dc_ctx* ctx, const dc_general_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, const float* low,
                           int ldd, float* blk, float eps, float* o, int ldo, float* mix, __nv_bfloat16* mixb, int ldm);
int dc_launch_general_decode(dc_ctx* ctx, const dc_general_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, float eps,
                             float* mix, __nv_bfloat16* mixb, int ldm);
int dc_launch_ring_update(dc_ctx* ctx, const dc_step& st, const dc_state_ref& sr, const float* proj, int ldp, int off, int C, int taps);

// lightning attention.  decode: one token per sequence.  scan: entries of any length in f32 (blocks of sixteen tokens).
// act: q, k and v after silu and the gate's input, columns off_q ..; y: the states' answers [T][ldy], all heads.
size_t dc_lightning_block_floats(const dc_lightning_mixer& m);
int dc_launch_lightning_decode(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* act,
                               const __nv_bfloat16* actb, int lda, float* y, int ldy);
int dc_launch_lightning_scan(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const dc_state_ref& sr, const float* act, int lda,
                             float* blk, float* y, int ldy);
// y / rms(y) * norm * sigmoid(gate) over all heads
int dc_launch_lightning_norm(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const float* y, int ldy, const float* act,
                             const __nv_bfloat16* actb, int lda, float eps, float* mix, __nv_bfloat16* mixb, int ldm);
// ---- mix_lightning.cu: the same for entries of bf16 models on the tensor cores, in chunks of 64 tokens
int dc_lightning_chunks(int T, int E);       // most chunks that T tokens of E entries make
int dc_launch_lightning_chunks(dc_ctx* ctx, const dc_lightning_mixer& m, const dc_step& st, const dc_state_ref& sr, const __nv_bfloat16* act,
                               int lda, float* chunk_state, float* y, int ldy);

// ---- mix_gqa.cu
struct dc_gqa_cache {
    void* arena = nullptr;      // [block][DC_KV_BLOCK][row], bf16 or f32
    bool f32 = false;
    const int32_t* tables = nullptr;
    int max_blocks = 0;
};
static inline int dc_gqa_ldq(const dc_gqa_mixer& m) { return (m.dim + 15) & ~15; }      // pitch of a turned query
// convolution, norms, rotation, cache rows of the step's tokens; queries to q or qb [T][heads * maps][dc_gqa_ldq].  sr: the
// convolution's ring (null without one)
int dc_launch_gqa_prep(dc_ctx* ctx, const dc_gqa_mixer& m, const dc_step& st, const dc_gqa_cache& c, const dc_state_ref* sr, const float* proj, int ldp, float eps,
                       int max_pos, float* q, __nv_bfloat16* qb);
static inline int dc_gqa_conv_cols(const dc_gqa_mixer& m) { return m.off_v + m.kv_heads * m.vdim; }     // projection columns under the convolution
// every token alone: keys split over CTAs, then joined.  proj: for the heads' gates
int dc_launch_gqa_tokens(dc_ctx* ctx, const dc_gqa_mixer& m, const dc_step& st, const dc_gqa_cache& c, const float* q, const float* proj, int ldp, int splits,
                         float* part, float* part_ml, float eps, float* mix, __nv_bfloat16* mixb, int ldm);
// prompts of bf16 models: tiles of queries over the cached rows
int dc_launch_gqa_prompt(dc_ctx* ctx, const dc_gqa_mixer& m, const dc_step& st, const dc_gqa_cache& c, const int32_t* tiles, int n_tiles,
                         const __nv_bfloat16* qb, const float* proj, int ldp, float eps, __nv_bfloat16* mixb, int ldm);

// ---- mix_latent.cu
struct dc_latent_cache {
    void* arena = nullptr;      // [block][DC_KV_BLOCK][row], bf16 or f32
    bool f32 = false;
    const int32_t* tables = nullptr;
    int max_blocks = 0;
};
int dc_launch_latent_prep(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const dc_latent_cache& c, float* proj, int ldp, float eps,
                          int max_pos);
int dc_launch_latent_absorbed(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const dc_latent_cache& c, const float* proj, int ldp,
                              int splits, float* qa, float* part, float* part_ml, float* mix, __nv_bfloat16* mixb, int ldm);
int dc_launch_latent_gather(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const dc_latent_cache& c, const int32_t* key_base,
                            int n_keys, __nv_bfloat16* keys_c, int ldc, __nv_bfloat16* keys_r, int ldr);
int dc_launch_latent_prefill(dc_ctx* ctx, const dc_latent_mixer& m, const dc_step& st, const int32_t* key_base, const int32_t* tiles,
                             int n_tiles, const float* proj, int ldp, const __nv_bfloat16* keys_kv, int ldkv, const __nv_bfloat16* keys_r,
                             int ldr, __nv_bfloat16* mixb, int ldm);
#define DC_LATENT_QTILE 64      // queries per tile of the prompt attention
