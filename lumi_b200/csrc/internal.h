// Internal structures shared by the translation units of liblumi_b200.so.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <cstdint>
#include <map>
#include <string>
#include <vector>

#include "../../include/lumi_b200.h"

namespace lumi {

// ---- errors -----------------------------------------------------------------------------------
void set_error(const char* fmt, ...);
int32_t fail(int32_t code, const char* fmt, ...);

#define LUMI_CUDA(expr)                                                                            \
    do {                                                                                           \
        cudaError_t _e = (expr);                                                                   \
        if (_e != cudaSuccess)                                                                     \
            return ::lumi::fail(_e == cudaErrorMemoryAllocation ? LUMI_E_NOMEM : LUMI_E_CUDA,      \
                                "%s failed: %s (%s:%d)", #expr, cudaGetErrorString(_e), __FILE__, __LINE__); \
    } while (0)

#define LUMI_TRY(expr)                    \
    do {                                  \
        int32_t _s = (expr);              \
        if (_s != LUMI_OK) return _s;     \
    } while (0)

// ---- configuration (ModelConfig of the reference, inference/src/model.rs:20-86) -----------------
// One layer of a model whose config lists its layers one by one: a mixer and, behind it, an optional feed-forward, each
// either behind a norm of the residual stream (pre_norm) or followed by a norm of its OUTPUT before it joins the stream.
// Every mixer constant is a field here, so that another design can combine them differently.
enum MixerKind { MIXER_NONE = 0, MIXER_DELTA, MIXER_ATTENTION, MIXER_RETENTION, MIXER_RGLRU, MIXER_LATENT };
// Rotary positions: `dims` of a head's dimensions turn by p * base^(-2i/dims), dimension i with i + dims/2, or (pairs) 2i with 2i + 1.
struct RotSpec {
    int dims = 0;
    bool pairs = false;
    double base = 10000.0;
};
struct MixerSpec {
    MixerKind kind = MIXER_NONE;
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int taps = 1;              // delta rule, gated linear recurrence: length of the short convolutions
    float unit_eps = 1e-6f;    // delta rule: epsilon inside the root of the unit vectors
    float scale = 1.f;         // attention: factor of the scores
    int window = 0;            // attention: tokens a position sees, itself included (0 = all)
    int kv_from = -1;          // attention: layer whose keys and values are read (-1 = this layer's own)
    bool qk_norm = false;      // attention: q and k over their root mean square
    bool sink = false;         // attention: one score of `sink_score` without a value joins the softmax
    float sink_score = 0.f;
    RotSpec rot;               // retention (first dimensions of q and k), latent attention (the rot_dim part of q and k)
    int kv_rank = 0;           // latent attention: size of the cached latent
    int rot_dim = 0;           // latent attention: rotated dimensions per query head and of the shared key part
    int channels = 0;          // gated linear recurrence: width of its two branches
    int blocks = 0;            // gated linear recurrence: blocks of the gates' matrices
    float decay_rate = 8.f;    // gated linear recurrence: log a = -decay_rate * r * softplus(lam)
    bool recurrent() const { return kind == MIXER_DELTA || kind == MIXER_RETENTION || kind == MIXER_RGLRU; }
    bool cached() const { return kind == MIXER_ATTENTION || kind == MIXER_LATENT; }
};
// Activations of a product.  Gated ones take the rows of W in groups of 16 gate rows and the 16 up rows that belong to them:
// result n = act(gate n) * up n.  ACT_SIGMOID_GATE is the hybrid's form (gate rows first, then the up rows).
enum Act { ACT_NONE = 0, ACT_SIGMOID_GATE = 1, ACT_RELU2 = 2, ACT_RELU_GATE = 3, ACT_SILU_GATE = 4 };
struct FfSpec {
    int ff = 0;                // width (0 = no feed-forward)
    int act = ACT_RELU2;       // gated kinds have a gate matrix beside the up matrix
    bool bias = false;
    int experts = 0, top = 0;  // mixture of experts (0 = dense): sigmoid scores, the weight multiplies the expert's input
    bool gated() const { return act == ACT_RELU_GATE || act == ACT_SILU_GATE; }
};
struct LayerSpec {
    MixerSpec mixer;
    FfSpec ff;
    bool pre_norm = false;
    int weights_of = -1;       // layer whose weights are used (-1 = its own); cache and state are always its own
    std::vector<float> decay;  // retention: decay per head
};

struct Config;
struct JsonValue;
// A model design: how its config.json is read and what its tensors are called.  `name` is the config's "architecture";
// a config without that key is the Mamba-3 / attention hybrid.
struct Architecture {
    const char* name;
    const char* tensor_prefix;                            // names without it are not looked at ("" = every name counts)
    int32_t (*parse)(const JsonValue& root, Config& out);
    // shape of a tensor by its name (prefix removed); rank 0 = not a tensor of this model.  `wide` is set for tensors
    // that are kept in fp32 whatever their rank
    int (*expected_shape)(const Config& c, const std::string& name, int64_t shp[3], bool& wide);
};
const Architecture* find_architecture(const char* name);  // null if there is none of that name

struct Config {
    int d_model = 0, n_layers = 0, d_state = 0, expand = 0, n_heads = 0, n_groups = 0, vocab = 0, max_seq_len = 0;
    int attention_interval = 0, attn_n_heads = 16, attn_kv_heads = 4, attn_mlp_expand = 4;
    std::vector<int> attn_window_sizes, attention_layers;
    bool byte_level = false;
    int attn_mlp_dim = 0;        // extension: 0 = attn_mlp_expand * d_model
    float attn_rope_base = 0.f;  // extension: 0 = no rotary embedding in attention
    float eps = 1e-5f;           // the reference hard-codes 1e-5 (model.rs:97) and has no norm_eps key
    const Architecture* arch = nullptr;
    std::vector<LayerSpec> specs;          // one entry per layer for designs that list them; empty for the hybrid
    float embed_scale = 1.f;
    bool embed_positions = false;          // sinusoidal position vectors are added to the embedding
    bool own_head = false;                 // the output matrix is a tensor of its own, not the embedding
    bool norm_offset = true;               // norm weights of listed designs are stored as offsets from one

    bool stacked() const { return !specs.empty(); }
    // elements per row of the residual stream on the device: rows of listed designs are padded with zeros to whole
    // 64-element blocks, so that any width goes through the tensor-core products
    int x_ld() const { return stacked() ? (d_model + 63) / 64 * 64 : d_model; }
    int max_window() const {               // most tokens an attention layer looks back over; 0 = one of them sees all
        int w = 1;
        for (const LayerSpec& l : specs) if (l.mixer.cached()) { if (l.mixer.window <= 0) return 0; if (l.mixer.window > w) w = l.mixer.window; }
        return w;
    }

    int d_inner() const { return expand * d_model; }
    int head_dim() const { return n_heads > 0 ? d_inner() / n_heads : 0; }
    int bc() const { return n_groups * d_state; }
    int in_proj_out() const { return 2 * d_inner() + 2 * bc() + 3 * n_heads + n_heads * d_state / 2; }
    int attn_head_dim() const { return d_model / attn_n_heads; }
    int kv_dim() const { return attn_kv_heads * attn_head_dim(); }
    int mlp_dim() const { return attn_mlp_dim > 0 ? attn_mlp_dim : attn_mlp_expand * d_model; }
    bool is_attention_layer(int i) const;
    int n_attn_layers() const;
    int attn_window_size(int attn_idx) const {
        return attn_idx < (int)attn_window_sizes.size() ? attn_window_sizes[attn_idx] : 0;
    }
};
int32_t parse_config(const char* json, Config& out);

// ---- device tensors -----------------------------------------------------------------------------
struct DevTensor {
    void* p = nullptr;
    int dtype = LUMI_DTYPE_F32;
    int64_t rows = 0, cols = 0;   // rank-1 tensors: rows = 1
    size_t bytes = 0;
};

struct MambaW {
    const float* norm_g = nullptr;
    DevTensor in_proj, out_proj;
    const float *b_gamma = nullptr, *c_gamma = nullptr, *b_bias = nullptr, *c_bias = nullptr;
    const float *d_skip = nullptr, *dt_bias = nullptr, *h_init = nullptr;   // h_init may stay null (zeros)
};
struct AttnW {
    const float *attn_norm_g = nullptr, *mlp_norm_g = nullptr;
    DevTensor qkv, o, gate_up, down;     // q|k|v and gate|up rows concatenated at finalize
};
// Weights of a listed layer.  `in` holds the input projections stacked by rows, each part padded to a multiple of 8 rows;
// columns (and the stacked total) are padded to multiples of 64 with zeros.  Norm weights are stored as the factor itself.
struct SubW {
    DevTensor in, out, up, down;
    int off_q = 0, off_k = 0, off_v = 0, off_b = 0, off_a = 0, off_g = 0;
    const float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr;      // [channels][taps]
    const float *a_log = nullptr, *dt_bias = nullptr, *o_norm = nullptr;
    const float *norm1 = nullptr, *norm2 = nullptr;                           // [x_ld]
    const float *in_b = nullptr, *up_b = nullptr, *down_b = nullptr;          // biases by weight row (may be null)
    const double* rot_freq = nullptr;                                         // [rot.dims / 2] frequencies in half turns per position
    const float* decay_pow = nullptr;                                         // retention: [heads][kDecayPowers] powers 0, 1, ... of the decay
    // gated linear recurrence: [block][2 bp][bp], rows in groups of 16 of the decay gate and 16 of the input gate (bp: block size
    // padded to 64), biases in the same order; conv_q holds the filter
    DevTensor rg; const float *rg_b = nullptr, *conv_b = nullptr, *lam = nullptr;
    int off_x = 0, off_y = 0, off_c = 0;
    // latent attention: key up-projection per head transposed [head][lp][dp], value up-projection [head][vdim][lp], and both as one
    // matrix over a cache row for prompts [head][dk_pad + dv_pad][row]; norm weight of the latent
    DevTensor uk, uv, ukv; const float* c_norm = nullptr;
    // experts: up [expert][2 ffp][x_ld] (gate and up rows in groups of 16), down [expert][x_ld][ffp]
    DevTensor router;
};
constexpr int kDecayPowers = 65;
// Padded sizes of a latent attention layer: latent, unrotated query part, cache row.
struct LatentShape {
    int lp, dp, row, dk, dk_pad, dv_pad;
    __host__ __device__ explicit LatentShape(const MixerSpec& m)
        : lp((m.kv_rank + 63) / 64 * 64), dp((m.dim + 63) / 64 * 64), row((lp + m.rot_dim + 63) / 64 * 64), dk(m.dim + m.rot_dim),
          dk_pad((dk + 15) / 16 * 16), dv_pad((m.vdim + 15) / 16 * 16) {}
};
struct Layer {
    bool is_attn = false;
    int kind_idx = 0;     // index among the Mamba layers, or among the attention layers
    int window = 0;
    MambaW m;
    AttnW a;
    const LayerSpec* spec = nullptr;      // set for layers of a design that lists them; `s` then holds the weights
    SubW s;
    bool is_mamba() const { return !is_attn && spec == nullptr; }
};

}  // namespace lumi

struct lumi_model {
    lumi::Config cfg;
    int device = 0;
    bool finalized = false;
    int wdtype = -1;                                  // dtype of rank-2 tensors (all must agree)
    bool widen = false;                               // bf16 tensors are widened to fp32 when they are loaded
    std::map<std::string, lumi::DevTensor> tensors;   // by name without the "item." prefix
    std::vector<void*> owned;                         // extra device allocations made at finalize
    std::vector<lumi::Layer> layers;
    lumi::DevTensor embedding;
    lumi::DevTensor head;                             // listed designs: the embedding, or a matrix of its own
    const float* final_norm_g = nullptr;
    int n_mamba = 0, n_attn = 0;
    int n_recur = 0, n_wattn = 0;                     // listed layers with a recurrent state, and with a cache
    int64_t weight_bytes = 0;                         // bytes of weights one decode step reads
};

namespace lumi {

// Device-resident control block read by the kernels of a step, so that a captured CUDA graph stays
// valid from call to call: the host rewrites these fields, not kernel arguments.
struct StepCtl {
    int32_t step;            // index of the token being generated (Philox counter, output row)
    int32_t status;          // 0 ok; kernels OR in LUMI_STATUS_* bits
    int32_t record;          // 1: write sampled tokens to out_tokens[step][b] and track eos
    int32_t want_dump;       // 1: copy logits to dump[step][b][:]
    float temperature;
    int32_t top_k;
    uint32_t seed_lo, seed_hi;
    uint32_t eos_id;
    int32_t ignore_eos;
    uint32_t* out_tokens;    // [n_new][batch]
    float* dump;             // [n_new][batch][vocab]
    int32_t batch;
    int32_t prompt_len;      // prefill: tokens per sequence still to come from `prompt`
    int32_t prompt_pos;      // next prompt position; >= prompt_len means "consume tok_cur"
    int32_t pad;
    const uint32_t* prompt;  // [prompt_len][batch]
};
enum { STATUS_BAD_TOKEN = 1, STATUS_KV_FULL = 2, STATUS_TIMEOUT = 4 };

struct GraphEntry {
    cudaGraphExec_t exec = nullptr;
    int64_t launches = 0;
};

}  // namespace lumi

namespace lumi {
struct B1Layer;
// Per-sequence state of one listed layer for all slots of a session.
struct LayerState {
    void* kv = nullptr;         // attention: page pool [slot pages][kv_head][K rows | V rows of 64 tokens], rows padded to dk_pad / dv_pad
    size_t kv_bytes = 0;
    int dk_pad = 0, dv_pad = 0;
    float* S = nullptr;         // delta rule, retention: [slot][head][dim][dv_pad]; gated linear recurrence: [slot][channels]
    float* conv = nullptr;      // [slot][taps][channels] raw inputs of the short convolutions, ring over positions
    int dvp = 0, channels = 0;
    size_t s_seq = 0, conv_seq = 0;      // floats per sequence
};
// Buffers of a mixture of experts over `rows` token rows at a time: the (row, expert) pairs sorted by expert, operand halves, hidden
// halves and results; fp32 hidden rows where no tensor cores are used.
struct MoeBufs {
    int rows = 0;
    float *logits = nullptr, *y = nullptr, *h32 = nullptr;
    __nv_bfloat16 *gh = nullptr, *gl = nullptr, *hh = nullptr, *hl = nullptr;
    int32_t* plan = nullptr;                         // see MoeArgs
};
// Row buffers of a pass over listed layers (one set for decode steps, one for prompt slices).
struct RowBufs {
    size_t rows = 0;
    float *x = nullptr;                              // residual stream [rows][x_ld] (the decode set uses the session's x)
    float *x2 = nullptr;                             // where x goes when a product's prologue adds to it (few rows)
    float *proj = nullptr, *mix = nullptr, *qkv = nullptr, *gates = nullptr, *y32 = nullptr;
    __nv_bfloat16 *xh = nullptr, *xl = nullptr, *ah = nullptr, *al = nullptr;
    float* ssq = nullptr; int ssq_stride = 0;        // pre-norm layers: sums of squares beside xh / xl
    __nv_bfloat16 *bh = nullptr, *bl = nullptr;      // operand rows of products by blocks (gated linear recurrence)
    // latent attention with queries in the latent space: queries, contexts, and either as halves
    size_t lat_rows = 0;
    float *qlat = nullptr, *ctx = nullptr;
    __nv_bfloat16 *lh = nullptr, *ll = nullptr;
    lumi::MoeBufs moe;
};
}

struct lumi_session {
    lumi_model* m = nullptr;
    int max_batch = 0, max_tokens_kv = 0;
    cudaStream_t stream = nullptr;
    cudaEvent_t ev0 = nullptr, ev1 = nullptr, ev2 = nullptr;
    // two-lane execution of large tensor-core batches: GEMM kernels of each lane on a high-priority
    // stream, state steps on a low-priority one
    cudaStream_t lane_hi[2] = {nullptr, nullptr}, lane_lo[2] = {nullptr, nullptr};
    cudaEvent_t lane_ev[2][2] = {{nullptr, nullptr}, {nullptr, nullptr}}, ev_fork = nullptr, ev_stagger = nullptr, ev_join[2] = {nullptr, nullptr};
    int opt_overlap = 0;              // minimum batch for two-lane execution (0 = never)
    size_t act_ld = 0;                // elements per row of the activation-half buffers
    int opt_chunked_prefill = 128;    // minimum prompt length for the chunked SSD prefill (0 = never)
    int opt_prefill_rows = 131072;    // token rows processed per chunked-prefill pass (workspace size)
    // chunked-prefill workspace (grow-only): residual rows, in_proj output, bf16 halves, BCNorm scales
    float *pf_x = nullptr, *pf_proj = nullptr, *pf_rb = nullptr, *pf_rc = nullptr;
    __nv_bfloat16 *pf_hi = nullptr, *pf_lo = nullptr;
    size_t pf_rows = 0;
    // options
    int opt_gemm = 0, opt_split = 1, opt_graph = 1, opt_pdl = 1, opt_mega = 0;
    // greedy head with the argmax fused behind the lm_head GEMV (batch <= 8): set by the caller of a step that wants
    // neither sampling nor the logits; per (row, CTA) partials
    bool fused_head = false;
    float* amax_val = nullptr;
    int* amax_idx = nullptr;
    int amax_stride = 0;
    // batch-1 persistent kernel
    bool b1_ok = false;
    lumi::B1Layer* b1_layers = nullptr;
    void* b1_grid_ctl = nullptr;
    float* b1_amax_val = nullptr;
    int* b1_amax_idx = nullptr;
    unsigned long long* b1_timing = nullptr;
    unsigned long long* b1_tagged = nullptr;   // xt | pt | yt
    uint32_t b1_epoch = 1;
    // state, per Mamba layer l: base + l * max_batch * per-sequence size
    float *h = nullptr, *xprev = nullptr, *bprev = nullptr, *cum = nullptr;
    // attention cache: pool of pages of kPageTokens tokens, [n_attn][pages][2][kv_heads][kPageTokens][head_dim]
    void* kv_pool = nullptr;           // element type follows the weights (fp32 or bf16)
    size_t kv_layer_bytes = 0;
    int32_t* page_table = nullptr;     // [max_batch][pages_per_seq]
    int32_t* kv_pos = nullptr;         // [max_batch] tokens consumed so far (absolute position)
    float* attn_part = nullptr;        // partial (max, sum, context) of attention contexts split over CTAs
    int32_t* attn_part_count = nullptr;
    int32_t* slot_buf = nullptr;       // [max_batch] slot list of a partial reset
    int32_t* row_len = nullptr;        // [max_batch] prompt lengths of a ragged prefill
    float* xlast = nullptr;            // [max_batch][d_model] residual rows at each sequence's last prompt token
    int pages_per_seq = 0;
    // designs that list their layers
    std::vector<lumi::LayerState> lstate;
    __nv_bfloat16* lat_kv = nullptr;   // latent attention, prompt slices: keys and values per head of a few sequences' rings
    size_t lat_kv_cap = 0;
    float* ret_seg = nullptr;          // retention, prompt slices: states of segments
    size_t ret_seg_cap = 0;
    lumi::RowBufs dec, pre;
    int kv_limit = 0;                  // positions at or past it are refused (0 = the ring takes any)
    int slice_max = 0;                 // most tokens of a sequence per pass (what the ring leaves beside the widest window)
    double* pos_freq = nullptr;        // [d_model / 2] frequencies of the position vectors
    int32_t* want_idx = nullptr; size_t want_cap = 0;
    // activations
    float *x = nullptr, *proj = nullptr, *y32 = nullptr, *logits = nullptr;
    __nv_bfloat16 *act_hi = nullptr, *act_lo = nullptr;
    __nv_bfloat16 *xn_hi = nullptr, *xn_lo = nullptr;   // residual rows x the next norm's weights, bf16 halves [rows][d_model]
    float* ssq = nullptr;              // [rows][ssq_stride] partial sums of squares of the residual rows
    int ssq_stride = 0;
    uint32_t *tok_cur = nullptr;       // [max_batch] tokens the next step consumes
    int32_t *finished = nullptr, *out_len = nullptr;   // [max_batch]
    int32_t* gemm_counters = nullptr;  // [2][kGemmCounters] zeroed ints for the split-K GEMM (second half: second lane)
    float* gemm_scratch = nullptr;     // [2][kGemmScratchFloats] partial tiles of the split-K GEMM
    lumi::StepCtl* ctl = nullptr;      // device
    lumi::StepCtl* ctl_host = nullptr; // pinned mirror
    uint32_t* pin_tokens = nullptr;    // pinned staging [max_batch]
    // grow-only buffers for lumi_generate outputs
    uint32_t* gen_out = nullptr; size_t gen_out_cap = 0;
    uint32_t* prompt_dev = nullptr; size_t prompt_cap = 0;
    float* gen_dump = nullptr; size_t gen_dump_cap = 0;
    float* score_logits = nullptr; size_t score_logits_cap = 0;    // logits of a block of prefill rows (scoring)
    std::map<int64_t, lumi::GraphEntry> graphs;
    int64_t launches = 0;              // kernels enqueued outside graphs since last reset of the counter
    int64_t launches_per_step = 0;
};

namespace lumi {

constexpr int kPageTokens = 64;
constexpr int kGemmCounters = 4096;
constexpr size_t kGemmScratchFloats = (size_t)4 << 20;      // 16 MiB per lane

// ---- kernel launchers (kernels.cu) --------------------------------------------------------------
// All take the stream to enqueue on and return a cudaError_t from the launch.
// A row operand that is still to take the norm of a sublayer's output: A + o / rms(o) * w over `width` elements (rows of K
// elements); the product is taken of the sum, which also goes to x_out (not the memory of A or o).  o null: nothing.
struct PostAdd {
    const float* o = nullptr;
    const float* w = nullptr;
    float* x_out = nullptr;
    int width = 0;
};
struct GemvArgs {
    const float* A; int lda;         // [M][K] fp32
    const void* W; int w_dtype;      // [N][K]
    float* D; int ldd;               // [M][N]
    const float* R;                  // residual, same layout as D, or null
    const float* gamma;              // RMSNorm weight applied to rows of A first, or null
    int M, N, K;
    float eps;
    int act;                         // Act; gated kinds: N = results (pairs of rows)
    int32_t* status = nullptr;       // device word that receives STATUS_TIMEOUT if a bounded wait gives up; may be null
    bool allow_preload = true;       // false: never the single-wave preloading kernel (the only GEMV with a device-side wait)
    // greedy head: per (batch row, CTA) the best (value, row) of the CTA's rows goes to amax_val / amax_idx
    // [M][amax_stride]; *amax_parts (host) receives the number of partials per row; D may then be null (no logits written)
    float* amax_val = nullptr;
    int* amax_idx = nullptr;
    int amax_stride = 0;
    int* amax_parts = nullptr;
    PostAdd post;                    // applied before gamma
    int norm_width = 0;              // elements the norm under gamma runs over (0 = K; the others are zero padding)
    const float* bias = nullptr;     // by weight row
};
cudaError_t launch_gemv(const GemvArgs& a, cudaStream_t st);
cudaError_t launch_logprob(const float* logits, int B, int V, const uint32_t* targets, float* out, int out_stride, int out_col,
                           cudaStream_t st);
cudaError_t launch_logprob_rows(const float* logits, int rows, int V, const uint32_t* prompt, int batch_total, int T, int ts, int t0,
                                int b0, int row0, float* out, cudaStream_t st);
// Kernels of kernels.cu launched by the calling thread from now on carry (or not) the
// programmatic-dependent-launch attribute.
void set_launch_pdl(bool on);
bool launch_pdl_on();
// The same for the tensor-core GEMM launches alone (their set-up may overlap the predecessor's tail at batch sizes where
// an early start of the CUDA-core kernels does not pay).
void set_launch_pdl_gemm(bool on);
bool launch_pdl_gemm_on();

// What some designs do to an embedding row before it becomes the residual stream: a factor, a sinusoidal position vector
// (freq: [width / 2], pos: position of each sequence's first row in this pass), and the bf16 halves of the result for the
// first product.  The defaults leave the row as the table holds it.
struct EmbedPost {
    float scale = 1.f;
    const double* freq = nullptr;
    const int32_t* pos = nullptr;
    int width = 0;
    __nv_bfloat16 *hi = nullptr, *lo = nullptr;
};
cudaError_t launch_embed(const void* emb, int dtype, const uint32_t* tok_cur, float* x, int B, int D, int vocab,
                         StepCtl* ctl, cudaStream_t st, const int32_t* row_len = nullptr, const EmbedPost& post = EmbedPost());
// x[B][D] fp32 -> RMSNorm(gamma) -> bf16 hi (+ lo if lo != null); gamma null = plain split.
// ssq != null: hi / lo = x * gamma without the per-row scale, ssq[b * ssq_stride] = sum of x^2 (for a GEMM with a folded norm)
cudaError_t launch_norm_split(const float* x, const float* gamma, __nv_bfloat16* hi, __nv_bfloat16* lo, int B, int D,
                              float eps, cudaStream_t st, float* ssq = nullptr, int ssq_stride = 0);

struct SsmArgs {
    const float* proj; int ldp;      // [B][in_proj_out]
    const float *bg, *cg, *bb, *cb, *dskip, *dtb;
    float *h, *xprev, *bprev, *cum;  // this layer's slices
    float* y32;                      // [B][d_inner] fp32, or null
    __nv_bfloat16 *yhi, *ylo;        // [B][d_inner] bf16 halves, or null
    int B, H, P, N, G;
    float eps;
    // prompts of different lengths (null otherwise): sequences whose prompt has ended (ctl->prompt_pos >= row_len[b]
    // while the prefill runs) are left untouched
    const int32_t* row_len = nullptr;
    const StepCtl* ctl = nullptr;
};
cudaError_t launch_ssm_step(const SsmArgs& a, cudaStream_t st);
bool ssm_shape_supported(int P, int N);

cudaError_t launch_state_reset(float* h, float* xprev, float* bprev, float* cum, const float* h_init, const int32_t* slots,
                               int n_slots, int H, int P, int N, cudaStream_t st);

cudaError_t launch_sample(const float* logits, int B, int V, StepCtl* ctl, uint32_t* tok_cur, int32_t* finished,
                          int32_t* out_len, cudaStream_t st);
cudaError_t launch_advance_step(StepCtl* ctl, int32_t* kv_pos, int B, int sampled, cudaStream_t st, const int32_t* row_len = nullptr);
cudaError_t launch_capture_last(const float* x, float* xlast, const int32_t* row_len, const StepCtl* ctl, int B, int D, cudaStream_t st);
// greedy head, second stage for batch <= 8: argmax over the GEMV's partials, token bookkeeping, end-of-step bookkeeping
cudaError_t launch_head_finish(const float* amax_val, const int* amax_idx, int nparts, int stride, int B, StepCtl* ctl, uint32_t* tok_cur,
                               int32_t* finished, int32_t* out_len, int32_t* kv_pos, cudaStream_t st);

// ---- attention (attention.cu) ---------------------------------------------------------------------
struct AttnArgs {
    const float* qkv; int ldq;       // [B][d_model + 2 kv_dim] fp32 (q | k | v) of the current token
    void* pool;                      // this layer's page pool (fp32 or bf16 elements)
    int kv_is_f32;
    const int32_t* page_table; int pages_per_seq;
    const int32_t* pos;              // [B] absolute position of the current token
    float* ctx32;                    // [B][d_model] fp32 or null
    __nv_bfloat16 *chi, *clo;        // bf16 halves or null
    int B, n_heads, kv_heads, head_dim, window, max_tokens;
    float rope_base;
    StepCtl* ctl;
    // Batched prefill: B counts token rows, row r = sequence (b0 + r / rows_per_seq), position pos[sequence] + r % rows_per_seq;
    // the rows of a slice are appended to the cache by one launch (phase 1) and attend to it in a second one (phase 2).
    // Decode: rows_per_seq = 1, phase 0 (append, then attend, in one launch).
    int rows_per_seq = 1, b0 = 0, phase = 0;
    // decode only: room for the partial results of a context split over several CTAs — part: [B * kv_heads][16 slices]
    // [hpk * (head_dim + 2)] floats, part_count: [B * kv_heads] zeroed ints (left zero) — and the longest context of the
    // batch as far as the host knows it (bounds the number of slices); null / 0: one CTA per (row, KV head)
    float* part = nullptr;
    int32_t* part_count = nullptr;
    int max_ctx_hint = 0;
    const int32_t* row_len = nullptr;    // prompts of different lengths: rows at or past their sequence's prompt length are skipped (decode form: by the
                                         // step's prompt position; prompt slices: by the row's own position, and their output rows are zero)
    size_t pool_bytes = 0;               // size of this layer's page pool (bounds the tensor map of the tensor-core kernel); 0: not given
};
constexpr int kAttnPartSlices = 16;
constexpr int kAttnPartUnits = 296;        // (row, KV head) pairs below which a context is split over CTAs: two CTAs per SM (sizes the partial-result buffer)
cudaError_t launch_attention_decode(const AttnArgs& a, cudaStream_t st);
cudaError_t launch_kv_advance(int32_t* kv_pos, int b0, int nb, int by, cudaStream_t st, const int32_t* lens = nullptr, int t_abs0 = 0);


// ---- tcgen05 GEMM (gemm_tcgen05.cu) ---------------------------------------------------------------
// D[M][N] (+)= A[M][K] W[N][K]^T ; A as bf16 hi (+ lo) halves, W bf16, fp32 accumulate and output.
// epi: 0 store, 1 add to existing D (residual), 2 sigmoid-gate: D[m][n] = sigmoid(acc[n]) * acc[n + N] is NOT
// done here (see gate kernel).  status_word: device int that receives STATUS_TIMEOUT if a bounded wait gives up.
// RMSNorm folded around a tensor-core product.  Consumer side (ssq_in): the A rows hold x * gamma without the
// per-row scale; the kernel sums `ssq_parts` partial sums of x^2 per row (stride ssq_stride) and multiplies its
// accumulator rows by 1 / sqrt(sum * inv_k + eps).  Producer side (out_hi): beside D the kernel writes
// D * gamma_next as bf16 hi (+ lo) rows of width N and, per row, the sum of D^2 over each strip of 32 columns into
// ssq_out[row * ssq_stride + column / 32] (independent of the tile width, so results do not depend on the row
// count) — the next product's consumer side.  All null: plain product.
struct NormFuse {
    const float* ssq_in = nullptr;
    int ssq_parts = 0;
    int ssq_stride = 0;
    float inv_k = 0.f, eps = 0.f;
    const float* gamma_next = nullptr;
    __nv_bfloat16 *out_hi = nullptr, *out_lo = nullptr;
    float* ssq_out = nullptr;
    // activation before the result is stored: ACT_NONE, ACT_RELU2 (the gated ones belong to GemmExt).  With gamma_next null,
    // out_hi / out_lo receive the result itself (width N) and no sums of squares are written; D may then be null
    int act = 0;
    const float* bias = nullptr;         // [N], added before the activation
};

// Products in groups, and gated results (persistent kernel, rows of W in `groups` blocks of group_rows each).
//   by columns:  group g multiplies columns [g K, (g + 1) K) of A (rows of lda elements); its results go to columns g * out_step + n,
//                n < out_n.  groups == 1 is an ordinary product.
//   by rows (tiles given): rows of A are sorted by group; row tile i holds tiles[i] = (first row, rows, group, 0), *n_tiles of them.
// gate: ACT_RELU_GATE / ACT_SILU_GATE (rows of W as Act says; out_n and out_step count results).  mul: the result is multiplied
// by sigmoid(mul[row * ldmul + column]).  Results go to D (ldd) and / or out_hi / out_lo (ldo).
struct GemmExt {
    int groups = 1, group_rows = 0, lda = 0, out_step = 0, out_n = 0;
    const int4* tiles = nullptr;
    const int32_t* n_tiles = nullptr;
    int max_tiles = 0;                   // row tiles there can be (bounds the launch)
    int gate = 0;
    const float* mul = nullptr; int ldmul = 0;
    int ldo = 0;
};

struct GemmArgs {
    const __nv_bfloat16 *a_hi, *a_lo;   // [M][K]
    const __nv_bfloat16* w;             // [N][K]
    float* d; int ldd;
    int M, N, K;
    int accumulate;
    int32_t* status_word;               // may be null
    int32_t* tile_counters = nullptr;   // zeroed device ints for split-K (the kernel leaves them zero); null: no split-K
    int n_counters = 0;
    float* scratch = nullptr;           // partial tiles of the splits
    size_t scratch_floats = 0;
    uint64_t wait_limit_ns = 0;         // limit of every device-side wait (0 = the default, 0.5 s)
    int debug_skip_unit = -1;           // test hook: the producer stops before this work unit, so the consumers' waits run out
    NormFuse nf;                        // RMSNorm folded around the product (persistent kernel only)
    const GemmExt* ext = nullptr;       // products in groups, gated results
};
int32_t launch_gemm_tcgen05(const GemmArgs& a, cudaStream_t st);   // returns LUMI_* status
void gemm_tcgen05_plan(const GemmArgs& a, int* width, int* splits);     // the tile width and K split that launch would take
int32_t gemm_tcgen05_init();                                        // resolves the driver entry point

// ---- batch-1 persistent decode kernel (decode_b1.cu) ---------------------------------------------
struct B1Layer {
    const void *in_proj, *out_proj;
    const float *norm_g, *bg, *cg, *bb, *cb, *dskip, *dtb;
    float *h, *xprev, *bprev, *cum;          // slot 0 of this layer's state
};
struct B1Args {
    const B1Layer* layers; int n_layers;
    const void* emb; const float* final_g;
    int vocab, D, DI, R, H, G, BC;
    float eps;
    unsigned long long *xt, *pt, *yt;        // epoch-tagged activations: [D], [R], [DI]
    uint32_t epoch_base;                     // epochs used by this launch start at epoch_base (+1 per layer, token, ...)
    float* logits;
    uint32_t* tok_cur;
    int32_t *finished, *out_len;
    StepCtl* ctl;
    void* grid_ctl;                          // 32 bytes of barrier counters, zeroed per launch
    float* amax_val; int* amax_idx;          // [grid] argmax partials
    int n_tokens;
    int head_mode;                           // 0: never run the lm_head; 1: at the last prompt position and every decode position
    int do_argmax;                           // 1: pick the greedy token on the device and advance the step counter
    unsigned long long* timing;              // optional: [2][n_layers][10] globaltimer stamps of the last token (CTA 0 and CTA 100)
};
bool decode_b1_supported(const Config& c, int n_attn, int device);
cudaError_t launch_decode_b1(const B1Args& a, int w_dtype, int device, cudaStream_t st);

// ---- chunked SSD prefill (prefill_ssd.cu) ----------------------------------------------------------
struct PrefillArgs {
    const float* proj; int ldp;              // [nb * ts][in_proj_out], row = sequence * ts + token
    const float *bg, *cg, *bb, *cb, *dskip, *dtb;
    float *h, *xprev, *bprev, *cum;          // this layer's state, slot 0
    float *rb, *rc;                          // [nb * ts] BCNorm scales (scratch)
    __nv_bfloat16 *yhi, *ylo;                // [nb * ts][d_inner] gated output halves
    int H, G, ts, nb, b0;                    // heads, groups, tokens per sequence in this launch, sequences, first slot
    float eps;
    int32_t* status = nullptr;               // device word that receives STATUS_TIMEOUT if the bounded wait gives up
    // prompts of different lengths: lens[slot] = prompt length of the sequence, t_abs0 = prompt position of this launch's first
    // token; a sequence takes min(ts, lens - t_abs0) tokens of the launch (none: its state is left alone).  null: all take ts
    const int32_t* lens = nullptr;
    int t_abs0 = 0;
};
bool prefill_ssd_supported(const Config& c);
cudaError_t launch_prefill_embed(const void* emb, int dtype, const uint32_t* prompt, float* x, int D, int vocab, int rows, int ts,
                                 int t_abs0, int b_abs0, int batch_total, StepCtl* ctl, cudaStream_t st, const int32_t* lens = nullptr,
                                 const EmbedPost& post = EmbedPost());
cudaError_t launch_prefill_scan(const PrefillArgs& a, cudaStream_t st);
cudaError_t launch_gather_last(const float* xr, float* x, int D, int ts, int nb, int b0, cudaStream_t st, const int32_t* lens = nullptr, int t_abs0 = 0);

// ---- listed layers: norm of a sublayer's output into the residual stream (sublayer.cu) --------------------
// x[r] += o[r] / sqrt(mean(o[r]^2) + eps) * w over `width` elements (rows of ld elements, padding stays zero); with hi set,
// the new residual also goes out as bf16 halves for the next product.  o == null: rows of x are normalised into y32 and / or
// hi / lo instead and x is left alone; row_idx (device, may be null) then picks the rows of x.
struct RowNormArgs {
    float* x; const float* o; const float* w;
    float* y32; __nv_bfloat16 *hi, *lo;
    const int32_t* row_idx;
    int rows, width, ld;
    float eps;
    float* x_out;                        // where the new residual rows go (null = back into x)
};
cudaError_t launch_row_norm(const RowNormArgs& a, cudaStream_t st);

// Read-outs of a recurrence head by head: o / rms(o) * w * silu(gate), rows of the pass as in DeltaArgs (dead rows are zero).
struct HeadGateArgs {
    const float* o; int H, dv, dvp;                  // [rows][H][dvp]
    const float* gate; int ldg;                      // [rows][ldg], H dv elements used
    const float* w;                                  // [dv], or null
    float eps;
    const int32_t* row_len; int t_abs0; const StepCtl* ctl;
    int nseq, ts, b0;
    float* y32; __nv_bfloat16 *yhi, *ylo; int ldy;
};
cudaError_t launch_head_gate(const HeadGateArgs& a, cudaStream_t st);

// ---- gated delta rule (delta_rule.cu) ----------------------------------------------------------------------
// Rows of the stacked input projections; row r = sequence b0 + r / ts, token r % ts of this pass.
struct DeltaArgs {
    const float* proj; int ldp;
    int off_q, off_k, off_v, off_b, off_a, off_g;
    const float *conv_q, *conv_k, *conv_v;           // [channels][taps]; channels of the ring: q | k | v
    const float *a_log, *dt_bias, *o_norm;
    float* S; float* conv;                           // this layer's state, slot 0
    int H, G, dk, dv, dvp, taps;
    float eps, unit_eps;
    const int32_t* pos;                              // [slot] position of the pass's first token
    const int32_t* row_len; int t_abs0;              // prompts of different lengths (null otherwise), as in PrefillArgs
    const StepCtl* ctl;                              // decode form (ts == 1) with row_len: the step's prompt position decides
    int nseq, ts, b0;
    float* y32; __nv_bfloat16 *yhi, *ylo; int ldy;   // gated, normalised output rows
    // chunked form: prepared q | k | v rows (unit vectors, activations applied), [rows][2 G dk + H dv] padded, and per (row, head)
    // beta and the logarithm of the decay; the read-out before its norm
    float* qkv; int ldqkv; float* gates; float* o32;
    int32_t* status;                                 // receives STATUS_TIMEOUT if a bounded wait gives up; may be null
};
cudaError_t launch_delta_step(const DeltaArgs& a, cudaStream_t st, int* launches);
bool delta_chunk_supported(int dk, int dv);
cudaError_t launch_delta_chunk(const DeltaArgs& a, cudaStream_t st, int* launches);

// ---- windowed attention with a softmax sink (window_attention.cu) -----------------------------------------
struct WinAttnArgs {
    const float* proj; int ldp; int off_q, off_k, off_v;
    void* kv; int kv_is_f32; int dk_pad, dv_pad;
    const int32_t* page_table; int pages_per_seq;    // ring of pages_per_seq pages per slot
    const int32_t* pos;                              // [slot] position of the pass's first token
    int H, G, dk, dv;
    MixerSpec m;
    int append;                                      // 0: the keys and values are another layer's and already in the cache
    float eps;
    const int32_t* row_len; int t_abs0; StepCtl* ctl;
    int nseq, ts, b0;
    int limit;                                       // positions at or past it are refused (0 = the ring takes any)
    float* y32; __nv_bfloat16 *yhi, *ylo; int ldy;
    float* part; int32_t* part_count;                // as in AttnArgs, decode only
    // where the rows lie, if not as LayerState says (page_elems 0): elements per page, from one head's rows to the next one's,
    // from a K row to the next, from a V row to the next, and from a head's first K row to its first V row
    long page_elems = 0; int head_step = 0, k_ld = 0, v_ld = 0, v_off = 0;
    bool plain = false;                              // always the plain form
    const float* gate = nullptr; int ldg = 0;        // the contexts are multiplied by sigmoid(gate[row * ldg + h * dv + d])
};
cudaError_t launch_window_attention(const WinAttnArgs& a, cudaStream_t st, int* launches);
size_t window_attention_part_floats(const MixerSpec& m);      // room for the partial results of one (row, head group)

// ---- retention (retention.cu) ------------------------------------------------------------------------------
// Linear attention with a fixed decay per head: S_t = decay S_{t-1} + k_t v_t^T, o_t = S_t^T q_t; q and k rotated, k times k_scale;
// o over its root mean square, times silu of the gate rows.
struct RetentionArgs {
    const float* proj; int ldp; int off_q, off_k, off_v, off_g;
    float* S;                                        // this layer's state, slot 0
    int H, dk, dv, dvp;
    RotSpec rot; const double* freq;
    const float* decay_pow;                          // [H][kDecayPowers]
    float k_scale, eps;
    const int32_t* pos;
    const int32_t* row_len; int t_abs0; const StepCtl* ctl;      // as in DeltaArgs
    int nseq, ts, b0;
    float* y32; __nv_bfloat16 *yhi, *ylo; int ldy;
    float* o32;                                      // chunked form: read-out before its norm, [rows][H][dvp]
    int32_t* status;                                 // receives STATUS_TIMEOUT if a bounded wait gives up; may be null
    float* seg;                                      // chunked form: retention_segment_floats elements, or null (in one piece)
};
// chunked form: room for the states of segments that run side by side (0: the slice goes in one piece)
size_t retention_segment_floats(const MixerSpec& m, int nseq, int ts);
cudaError_t launch_retention_step(const RetentionArgs& a, cudaStream_t st, int* launches);
bool retention_chunk_supported(int dk, int dv);
cudaError_t launch_retention_chunk(const RetentionArgs& a, cudaStream_t st, int* launches);

// ---- gated linear recurrence (rglru.cu) --------------------------------------------------------------------
// u = conv(x) per channel; r, i = sigmoid of block-diagonal products of u; log a = -rate r softplus(lam);
// S_t = a S_{t-1} + sqrt(1 - a^2) i u; output S * gelu(y).
struct RglruArgs {
    const float* proj; int ldp; int off_x, off_y;
    const float *conv_w, *conv_b, *lam;
    const void* rg; int rg_dtype; const float* rg_b; // as in SubW
    int channels, blocks, bp, taps;                  // bp: block size padded to 64
    float rate;
    float *S, *conv;                                 // this layer's state, slot 0
    const int32_t* pos;
    const int32_t* row_len; int t_abs0; const StepCtl* ctl;
    int nseq, ts, b0;
    float* u32; __nv_bfloat16 *uh, *ul;              // convolution output: [rows][channels], halves [rows][blocks bp] (may be null)
    const float* gates;                              // [rows][blocks][2 bp] gate rows before the sigmoid (SubW order, bias included)
    float* y32; __nv_bfloat16 *yhi, *ylo; int ldy;
};
cudaError_t launch_rglru_conv(const RglruArgs& a, cudaStream_t st);
cudaError_t launch_rglru_scan(const RglruArgs& a, cudaStream_t st, int* launches);      // and the ring's new contents
constexpr int kRglruStepRows = 32;                    // rows up to which a decode token takes the one-launch form
bool rglru_step_supported(const RglruArgs& a);
cudaError_t launch_rglru_step(const RglruArgs& a, cudaStream_t st);      // a decode token, everything in one launch

// ---- latent attention (latent_attention.cu) ----------------------------------------------------------------
struct LatentArgs {
    float* proj; int ldp; int off_q, off_c;          // q rows are rotated in place
    void* kv; int kv_is_f32;                         // cache rows [latent lp | rotated key | 0] of `row` elements, pages of 64
    const int32_t* page_table; int pages_per_seq;
    const int32_t* pos;
    MixerSpec m; const double* freq; const float* c_norm;
    float eps;
    const int32_t* row_len; int t_abs0; StepCtl* ctl;
    int nseq, ts, b0, limit;
    __nv_bfloat16 *qh, *ql;                          // unrotated query parts [rows][H][dp] as halves (may be null)
    float* qlat;                                     // queries over a cache row [rows][H][row]; the prep kernel writes the rotated part and padding
    float* ctx; __nv_bfloat16 *ch, *cl;              // contexts over the latent [rows][H][lp]
    float* part; int32_t* part_count;
};
cudaError_t launch_latent_prep(const LatentArgs& a, cudaStream_t st);
cudaError_t launch_latent_attention(const LatentArgs& a, cudaStream_t st);       // queries absorbed into the latent space
size_t latent_part_floats(const MixerSpec& m);

// ---- products of a few rows by groups (block_product.cu) ---------------------------------------------------
// D[r][g * out_step + n] = (sum_k A[r][g * a_step + k] W[g][n][k] + bias[g][n]) * sigmoid(mul[r][g * out_step + n]), n < n_out <= group_rows, k < K
// (K <= the padded row length ldw of W).  fp32 or bf16 weights, fp32 products.
struct BlockProductArgs {
    const float* A; int lda, a_step;
    const void* W; int w_dtype; int ldw, group_rows;
    const float* bias; const float* mul; int ldmul;
    float* D; int ldd, out_step;
    int rows, groups, n_out, K;
};
cudaError_t launch_block_product(const BlockProductArgs& a, cudaStream_t st);
// dst[(r / rg * rs + r % rg + ro) * ld + co + c] = src[r][c]; transpose: dst[(r / rg * rs + c + ro) * ld + co + r % rg]
cudaError_t launch_pack_rows(void* dst, long ld, const void* src, long rows, long cols, int esz, long rg, long rs, long ro, long co, bool transpose,
                             cudaStream_t st);

// ---- mixture of experts (moe.cu) -----------------------------------------------------------------------------
// plan (int32): [0] row tiles, [1] ticket, [4 ...] counts [E_max] (zeros between launches), offsets [E_max], then per pair expert and
// place [2 pairs], weights [pairs] (as float bits) and the row tiles (int4 each, 16-byte aligned).
struct MoeArgs {
    const float* logits; int ldl;                    // router logits [rows][ldl]
    int rows, E, E_max, top, D, ldx, ff, ffp;        // E_max: most experts of any layer that uses the plan
    float* x; const float* gamma; float eps;         // residual rows and the norm in front of the router and the experts
    int32_t* plan;
    __nv_bfloat16 *gh, *gl;                          // experts' inputs sorted by expert [pairs][ldx]
    float* y;                                        // experts' results [pairs][ldx]
    // few rows: hidden rows [pairs][ffp] fp32 and the experts' weights
    float* h32; const void *w_up, *w_down; int w_dtype, act;
    // what the next product takes (tensor-core path): x * gamma_next as halves and its sum of squares
    const float* gamma_next; __nv_bfloat16 *xh, *xl; float* ssq; int ssq_stride;
};
size_t moe_plan_ints(int rows, int top, int E_max);
int moe_max_tiles(int rows, int top, int E);
const int4* moe_tiles(const MoeArgs& a);
cudaError_t launch_moe_route(const MoeArgs& a, cudaStream_t st);
cudaError_t launch_moe_gather(const MoeArgs& a, cudaStream_t st);
cudaError_t launch_moe_combine(const MoeArgs& a, cudaStream_t st);
cudaError_t launch_moe_few(const MoeArgs& a, cudaStream_t st);       // two launches: route + gate and up rows, then down rows into x

cudaError_t launch_gate_mul(const float* gu, int ld, float* out32, __nv_bfloat16* hi, __nv_bfloat16* lo, int B, int mlp,
                            cudaStream_t st);

}  // namespace lumi
