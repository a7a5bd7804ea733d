// Layered models: decoders whose configuration lists every layer with its own sizes and mechanisms (LayerSpec), on a
// 32-bit residual stream.  This header holds the layer description and the launch prototypes of the kernels such a
// layer is made of (layered_ops.cu, tanh_rows.cu, recurrence.cu, moe.cu; the bf16 matrix products and attention are gemm_umma.cu and tree_attn.cu).
//
// Every kernel that handles activations exists for bf16 and for fp32 (T): bf16 is what a model is served in, fp32 runs
// everything in true 32-bit through plain SIMT matrix products.  Weights are bf16 in both.
//
// Row buffers have their width padded to a multiple of 64 with zeros (`ld`), so every matrix product has a K that the
// tensor-core kernels take and every row starts on a 16-byte boundary, whatever the model's width is.
#pragma once
#include "common.cuh"

enum RecurrenceKind : int {
    REC_NONE = 0,
    REC_TIME_MIX = 1,    // decay per token and key channel, bonus for the current token, inputs mixed with the token before
    REC_LIGHTNING = 2,   // constant decay per head, silu on queries, keys and values
};

struct LayerSpec {
    // ---- mixer: softmax attention (heads == 0: none) and / or a recurrence; with both, they read the same input side by
    // side and their outputs are added
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 0.f;
    int window = 0;          // > 0: a token sees itself and the window - 1 tokens before it
    float bias_exp = 0.f;    // > 0: distance bias, slope of head h = 2^(-bias_exp * (h + 1) / heads)
    int qk_norm = 0;         // RMS norm over all query rows and over all key rows at once, before the split into heads
    int kv_from = -1;        // >= 0: the keys and values of that layer's cache
    int sink = 0;            // one more score of 0, without a value, in every softmax
    int rot_dims = 0;        // > 0: rotary positions on the first rot_dims of each query and key head (i paired with i + rot_dims / 2)
    float attn_scale = 1.f;  // factor of the attention's output
    int rec = REC_NONE;
    int rec_heads = 0, rec_dim = 0, rec_vdim = 0;   // key / query and value width of a head
    int rec_rank = 0;        // REC_TIME_MIX: inner width of the decay's two matrices
    float rec_scale = 1.f;   // factor of the recurrence's output
    // ---- feed-forward: mixture of experts (experts + identity == 0: none)
    int experts = 0, identity = 0, top = 0, groups = 1, keep_groups = 1;
    float router_scale = 1.f;
    int expert_ff = 0;
    int shared_ff = 0;       // > 0: an expert of this width that runs for every token
    // ---- feed-forward: one dense one (ff == 0: none), y = g sigmoid(ff_alpha g) (u + 1) with g <= ff_limit, |u| <= ff_limit
    int ff = 0;
    float ff_limit = 0.f, ff_alpha = 0.f;
};

// Norms of a layered model
enum NormKind : int {
    NORM_OUTPUT_RMS = 0,     // x += m * rms(sublayer(x)) * (1 + w)
    NORM_DYNAMIC_TANH = 1,   // x += N'(sublayer(N(x))), N(x) = tanh(alpha x) * w + b
};
struct DynTanh {
    const bf16 *w = nullptr, *b = nullptr;
    float alpha = 0.f;
};

inline int pad64(int n) { return (n + 63) / 64 * 64; }

// ---------------------------------------------------------------- rows (layered_ops.cu)
// x32 = embed[id] * scale (fp32), xh the same in T; `ld` columns per row.  Ids outside [0, vocab) raise ERR_BAD_TOKEN.
// state_len (models with recurrent layers): tokens the recurrent state holds; the pass must begin there (*kv_len + kv_off)
// or at 0, otherwise ERR_STATE_POS; advanced by `rows`.
struct StateCheck {
    int32_t* state_len = nullptr;
    const int32_t* kv_len = nullptr;
    int kv_off = 0;
};
template <typename T>
void launch_embed_rows(const int32_t* ids, const bf16* table, int vocab, float scale, float* x32, T* xh, int ld, int rows,
                       const StateCheck& check, cudaStream_t s);

// Query / key norm over the whole projections, rotation, then queries to q_out[rows][heads][dim_p] and keys / values to rows
// *kv_len + kv_off + r of the caches ([.][kv_heads][dim_p], [.][kv_heads][vdim_p]).  qkv: [rows][ld] q | k | v.
struct QkvNormArgs {
    const void* qkv;
    int ld;
    int heads, kv_heads, dim, dim_p, vdim, vdim_p;
    const bf16 *wq, *wk;     // null: no norm
    float eps;
    int rot_dims = 0;        // rotated dimensions per query / key head; the position is the cache row
    const float* inv_freq = nullptr;   // [rot_dims / 2]
    void* q_out;
    void *k_cache, *v_cache; // null: queries only
    const int32_t* kv_len;
    int kv_off, cache_rows;
    int* error;
};
template <typename T>
void launch_qkv_norm_append(const QkvNormArgs& a, int rows, cudaStream_t s);

// x32 += mult * rms(delta) * (1 + w), xh = x32 rounded to T.  delta is a T matrix, or with `mix` the weighted sum of a
// token's expert outputs (MoeMix).
struct MoeMix {
    const void* y = nullptr;         // expert outputs in T, [.][ld]; the null pointer selects the plain form
    const int32_t* expert = nullptr; // [rows][top]
    const float* weight = nullptr;   // [rows][top]
    const int32_t* rank = nullptr;   // [rows][top]: row of expert e's slot = offset[e] + rank
    const int32_t* offset = nullptr; // [experts]
    const float* id_weight = nullptr;// [rows]: weight of the input itself (identity experts)
    int top = 0, experts = 0;
    int shared_row0 = -1;            // >= 0: y rows from here are the shared expert's
};
template <typename T>
void launch_out_norm(float* x32, T* xh, const T* delta, const MoeMix& mix, float mult, const bf16* w, int rows, int width, int ld,
                     float eps, cudaStream_t s);
// y[i] = rms(x32[rows_idx ? rows_idx[i] : i]) * (1 + w)
template <typename T>
void launch_norm_rows(const float* x32, const int32_t* rows_idx, const bf16* w, T* y, int rows, int width, int ld, float eps,
                      cudaStream_t s);

// ---- dynamic tanh models
// What a time-mix layer reads instead of h itself: out[s][r] = h + (h_before - h) * mu[s], s = r, k, v, g, w; h_before is the
// row before, or `prev` ([ld] fp32, written with the last row's h) for the first row, zero at position 0.
constexpr int kMixes = 5;
struct TokenShift {
    const bf16* mu = nullptr;    // [kMixes][ld]; null: no mixes
    void* out = nullptr;         // [kMixes][stride] T
    size_t stride = 0;           // elements between two mixes
    float* prev = nullptr;
    const int32_t* kv_len = nullptr;   // position of the first row = *kv_len + kv_off
    int kv_off = 0;
};
// h[i] = N(x32[rows_idx ? rows_idx[i] : i]) in T, and the mixes
template <typename T>
void launch_tanh_norm(const float* x32, const int32_t* rows_idx, const DynTanh& n, T* h, const TokenShift& shift, int rows, int ld,
                      cudaStream_t s);
// x32 += post(delta); out = next(x32) in T, or x32 itself where next has no weights
template <typename T>
void launch_tanh_residual(float* x32, const T* delta, const DynTanh& post, const DynTanh& next, T* out, int rows, int ld, cudaStream_t s);
// act = clamped gate of gu (two blocks of ff columns, or interleaved in groups of 64: see launch_silu_gate)
template <typename T>
void launch_clamped_gate(const T* gu, int ld_gu, T* act, int ld_act, int rows, int ff, float limit, float alpha, bool interleaved, cudaStream_t s);
// Token side input: g[r] = gelu_tanh(z[r]) * table[ids[r]][col0 ..], dim columns, zero up to ld
template <typename T>
void launch_side_gate(const T* z, int ld, const int32_t* ids, const bf16* table, int table_ld, int col0, int dim, int vocab, T* g, int rows,
                      cudaStream_t s);
// x32 += rms(y) * w; with `next`, h = next(x32) in T and, for a single row, its mixes
template <typename T>
void launch_side_add(float* x32, const T* y, const bf16* w, const DynTanh& next, T* h, const TokenShift& shift, int rows, int width, int ld,
                     float eps, cudaStream_t s);
// A single row from a sublayer's output to the next layer's input in one launch: x32 += post(delta), then the token side input
// (gate product, launch_side_gate, projection, launch_side_add).  The two matrices are tile-major for bf16, row-major for fp32.
struct SideStepArgs {
    float* x32 = nullptr;
    const void* delta = nullptr;
    DynTanh post;
    const bf16 *gate = nullptr, *proj = nullptr, *norm = nullptr;
    const int32_t* ids = nullptr;
    const bf16* table = nullptr;
    int table_ld = 0, col0 = 0, dim = 0, vocab = 0;
    DynTanh next;
    void* h = nullptr;
    TokenShift shift;
    int width = 0, ld = 0;
    float eps = 0.f;
};
template <typename T>
void launch_side_step(const SideStepArgs& a, cudaStream_t s);
// dst [cols][rows] = src [rows][cols], host or device memory
void upload_transposed(const void* src, int rows, int cols, bf16* dst, cudaStream_t s);
// Decays of a time-mix layer: out[r][c] = exp(-exp(sum_k w2[k][c] tanh(x[r][k]) + w0[c])), c < channels; x: `rank` columns of
// T, w2 [rank][channels] (upload_transposed)
template <typename T>
void launch_decay(const T* x, int ld_x, const bf16* w2, const bf16* w0, int rank, int channels, float* out, int ld_out, int rows, cudaStream_t s);
// out[r][c] = rms over each group of `group` columns of o[r] * w[c] * gate(g[r][c]) * scale; gate: silu, or sigmoid
template <typename T>
void launch_norm_gate(const float* o, int ld_o, int groups, int group, const bf16* w, const T* gate, int ld_gate, bool silu, float eps,
                      float scale, T* out, int ld_out, int rows, cudaStream_t s);

// ---------------------------------------------------------------- recurrences (recurrence.cu)
// Per head, with a state S [dim][vdim] in fp32:
//   bonus != null:  o_t = (S + diag(u) k_t v_t^T)^T r_t,  then S = diag(w_t) S + k_t v_t^T
//   bonus == null:  S = diag(w_t) S + k_t v_t^T,  then o_t = S^T r_t
// w_t is given per token and channel, or constant per head.  Everything is fp32 from r, k, v on.
struct ScanArgs {
    const void *r = nullptr, *k = nullptr, *v = nullptr;   // T, head after head in a row
    int ld_r = 0, ld_k = 0, ld_v = 0;
    bool silu = false;             // r, k, v pass through silu first
    const float* w = nullptr;      // [rows][ld_w] decays, channel h * dim + c; null: constant decay
    int ld_w = 0;
    const float* decay = nullptr;  // [heads]
    const bf16* bonus = nullptr;   // [heads * dim]
    int heads = 0, dim = 0, vdim = 0, rows = 0;
    float* state = nullptr;        // scan_state_floats(heads, dim, vdim)
    const int32_t* kv_len = nullptr;   // position of the first row = *kv_len + kv_off; at 0 the state starts at zero
    int kv_off = 0;
    float* out = nullptr;          // [rows][ld_out], column h * vdim + c
    int ld_out = 0;
    float* ws = nullptr;           // scan_workspace_floats(heads, dim, vdim, rows)
};
bool scan_fits(int dim, int vdim);
size_t scan_state_floats(int heads, int dim, int vdim);
size_t scan_workspace_floats(int heads, int dim, int vdim, int rows);
template <typename T>
void launch_scan(const ScanArgs& a, cudaStream_t s);

// A single token's recurrence in one launch together with the decays before it (time mix: launch_decay of `inner`; a.w unused) and
// the norm and gate behind it (launch_norm_gate per head for a time mix, over all heads otherwise).
struct ScanStepArgs {
    ScanArgs scan;
    const void* inner = nullptr;   // T [rank]
    const bf16 *w2 = nullptr, *w0 = nullptr;
    int rank = 0;
    const bf16* norm = nullptr;    // [heads * vdim]
    const void* gate = nullptr;    // T [heads * vdim]
    float eps = 0.f, scale = 1.f;
    void* out = nullptr;           // T [heads * vdim]
    int32_t* ticket = nullptr;     // zero between launches
};
bool scan_step_fits(int dim, int vdim, bool time_mix);
template <typename T>
void launch_scan_step(const ScanStepArgs& a, cudaStream_t s);

// Attention of any head width up to 512, one warp per (token, head); q [tq][hq][dk], caches [.][hkv][dk | dv], out rows
// of hq * out_cols.  The bias, window and kv_len arguments are those of make_biased_attn_plan.
struct PlainAttnArgs {
    const void *q, *k_cache, *v_cache;
    void* out;
    int tq, hq, hkv, dk, dv, out_cols, out_ld;
    const int32_t* kv_len;
    int kv_len_add;
    float scale;
    int window;
    float bias_exp;
    int sink = 0;
    float out_scale = 1.f;
};
template <typename T>
void launch_plain_attention(const PlainAttnArgs& a, cudaStream_t s);

// fp32 Y[M][ldy] = X[M][ldx] W[N][K]^T with bf16 W, row-major.  With `entries` the rows come in groups, one per blockIdx.z:
// {expert, first x row, first y row, rows <= kF32Rows}; expert e's matrix is w + e * w_stride.  x_at_y: the
// rows of x are those of y (a product of what an earlier grouped product wrote).
constexpr int kF32Rows = 64;
void launch_linear_f32(const float* x, int ldx, const bf16* w, size_t w_stride, float* y, int ldy, int M, int N, int K,
                       const int4* entries, const int32_t* n_entries, int max_entries, bool x_at_y, cudaStream_t s);
// act[r][c] = silu(gu[r][c]) * gu[r][ff + c], IEEE exponential and division
void launch_silu_f32(const float* gu, int ld_gu, float* act, int ld_act, int rows, int ff, cudaStream_t s);

// ---------------------------------------------------------------- mixture of experts (moe.cu)
constexpr int kMoeMaxOutputs = 1024;   // router outputs (experts + identity experts)
constexpr int kMoeMaxTop = 32;
constexpr int kMoeMaxEntries = 1024;   // row groups of one launch of the expert products

struct MoeBuffers {
    float* z = nullptr;           // [rows][outputs] router logits
    int32_t* expert = nullptr;    // [rows][top]
    float* weight = nullptr;      // [rows][top]
    int32_t* rank = nullptr;      // [rows][top]
    float* id_weight = nullptr;   // [rows]
    int32_t* counts = nullptr;    // [outputs], zero between launches
    int32_t* offset = nullptr;    // [outputs]
    int4* entries = nullptr;      // [kMoeMaxEntries] {expert, first x row, first y row, rows}
    int32_t* n_entries = nullptr;
    int32_t* tickets = nullptr;   // [1 + row blocks], zero between launches
};

// Router: logits in fp32 from the fp32 stream, softmax over all outputs, choice by score + correction inside the best
// keep_groups groups, weights = the chosen scores over their sum, times router_scale.  The last CTA lays the rows of every
// expert out one after the other and cuts them into groups of at most `tile` rows.
// `direct`: a single row feeds every expert, its input is not copied (x row 0 in every entry).
void launch_moe_route(const LayerSpec& sp, const float* x32, const bf16* w, const float* correction, const MoeBuffers& b, int rows,
                      int ld, int tile, bool direct, cudaStream_t s);
size_t moe_ticket_ints(int max_rows);
// Rows per group for `rows` tokens (16 .. 256) and the most groups that can come out.
int moe_pick_tile(const LayerSpec& sp, int rows);
int moe_max_entries(const LayerSpec& sp, int rows, int tile);
// dst[offset[e] + rank] = src[r] for every chosen expert e of row r
template <typename T>
void launch_moe_gather(const LayerSpec& sp, const T* src, T* dst, const MoeBuffers& b, int rows, int ld, cudaStream_t s);

// One grouped product on the tensor cores: every expert's rows times its matrix, and the shared expert's rows (all tokens)
// times its own.  Weights tile-major, expert after expert, the shared expert last.
struct MoeGemmPlan {
    CUtensorMap tm_w, tm_x, tm_xs;   // weights, expert rows, shared expert's rows
    int tile = 0, rows = 0;          // rows per group; tokens
    int max_entries = 0;
    int swiglu = 0;
    int n_tiles = 0, kblocks = 0, N = 0;          // per expert
    int n_tiles_s = 0, kblocks_s = 0, N_s = 0;    // shared expert; n_tiles_s == 0: none
    long long w_row_s = 0;                        // first row of the shared expert's tiles in the weight map
    int xs_row0 = 0, ys_row0 = 0;                 // first row of the shared expert's input / output
    bf16* y = nullptr;
    int ldy = 0;
    const int4* entries = nullptr;
    const int32_t* n_entries = nullptr;
    int uniform = 0;                 // > 0: no router, this many matrices whose rows lie one block of `rows` after the other
};
// `n` products of the same shape in one launch: rows [i * rows, (i + 1) * rows) of x times matrix i [N][K], into the same rows
// of y; with N_s > 0 one more, of N_s outputs, on rows n * rows ... .  w: linear_weight_elems(N, K) per matrix, the extra one
// last.
MoeGemmPlan make_grouped_plan(const bf16* w, int n, int N, int N_s, int K, const bf16* x, bf16* y, int ldy, int rows);
// gate/up with the SwiGLU epilogue: y[row][ff_p columns]; x rows of K = ld columns
MoeGemmPlan make_moe_gate_up_plan(const LayerSpec& sp, const bf16* w, const bf16* x, int x_rows, const bf16* xs, int K, bf16* act,
                                  int ld_act, int rows, int tile, const MoeBuffers& b);
// down: y[row][width]; act rows of ld_act columns
MoeGemmPlan make_moe_down_plan(const LayerSpec& sp, const bf16* w, const bf16* act, int act_rows, int ld_act, int width, bf16* y,
                               int ld_y, int rows, int tile, const MoeBuffers& b);
void launch_moe_gemm(const MoeGemmPlan& p, cudaStream_t s);
// elements of the two weight buffers (tile-major), and where an expert's (index `experts`: the shared expert's) part begins
size_t moe_gate_up_elems(const LayerSpec& sp, int K);
size_t moe_down_elems(const LayerSpec& sp, int width);
size_t moe_gate_up_offset(const LayerSpec& sp, int K, int expert);
size_t moe_down_offset(const LayerSpec& sp, int width, int expert);
