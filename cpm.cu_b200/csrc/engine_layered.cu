// Engine: layered models (ModelConfig::specs) - storage, weight loading and the forward pass over LayerSpec layers.
// They share the engine's pool, K/V budget, prefill / decode entry points and error handling with Llama-format targets.
//
//   x   = embed[token]                                    fp32 stream, with a copy in T for the matrix products
//   x  += m * rms(o(attention(x))) * (1 + w1)             the sublayers read x itself; the norm is on their output
//   x  += m * rms(mixture(x)) * (1 + w2)
//   out = head(rms(x) * (1 + wf))
//
// or, with dynamic tanh norms N (NORM_DYNAMIC_TANH) before and after the sublayers and an input of each layer's own per token:
//
//   x   = c * embed[token]
//   x  += N1b(o([attention(N1(x)) | recurrence(N1(x))]));  x += N2b(ff(N2(x)));  x += rms(P (gelu(G x) * e[token, layer])) * w
//   out = head(Nf(x))
//
// Positions are cache rows: token r of a pass that starts at row L has position L + r.
#include <algorithm>
#include <cstdlib>
#include <cstring>

#include "engine.cuh"

namespace {
// Tensor names of a layer's mixer: two mixers side by side are told apart
std::string attn_prefix(const LayerSpec& s) { return s.rec != REC_NONE ? "mix.left." : "mix."; }
std::string rec_prefix(const LayerSpec& s) { return s.heads > 0 ? "mix.right." : "mix."; }
constexpr char kMixNames[kMixes + 1] = "rkvgw";   // the order of the mixes, and of the matrices of a time mix
}  // namespace

void Engine::check_specs() const {
    CPM_REQUIRE(mc_.hidden >= 1 && mc_.vocab >= 1, "layered model: empty width or vocabulary");
    CPM_REQUIRE(ld() <= 16384, "layered model: width above 16384 is not supported");
    CPM_REQUIRE(mc_.norm == NORM_OUTPUT_RMS || mc_.norm == NORM_DYNAMIC_TANH, "layered model: unknown norm");
    CPM_REQUIRE(mc_.side_dim >= 0 && (mc_.side_dim == 0 || mc_.norm == NORM_DYNAMIC_TANH), "layered model: token inputs per layer need dynamic tanh norms");
    CPM_REQUIRE(!mc_.sparse.enabled && !mc_.w4a16, "layered model: block selection and int4 weights belong to Llama-format targets");
    for (size_t i = 0; i < mc_.specs.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        const bool tanh_norms = mc_.norm == NORM_DYNAMIC_TANH;
        CPM_REQUIRE(s.heads > 0 || s.rec != REC_NONE, at + "no mixer");
        if (s.heads != 0) {
            CPM_REQUIRE(s.heads >= 1 && s.kv_heads >= 1 && s.heads % s.kv_heads == 0, at + "query heads must be a multiple of key/value heads");
            CPM_REQUIRE(s.dim >= 1 && s.vdim >= 1 && pad64(s.dim) <= 512 && s.vdim <= 512, at + "head widths must be in [1, 512]");
            CPM_REQUIRE(s.rot_dims >= 0 && s.rot_dims % 2 == 0 && s.rot_dims <= s.dim, at + "rotated dimensions must be even and within the head");
        }
        if (s.rec != REC_NONE) {
            CPM_REQUIRE(s.rec == REC_TIME_MIX || s.rec == REC_LIGHTNING, at + "unknown recurrence");
            CPM_REQUIRE(tanh_norms, at + "recurrences need norms in front of the sublayers");
            CPM_REQUIRE(s.rec_heads >= 1 && scan_fits(s.rec_dim, s.rec_vdim), at + "recurrence: head widths must be at most 256 (keys) and 512 (values)");
            CPM_REQUIRE(s.rec != REC_TIME_MIX || (s.rec_dim == s.rec_vdim && s.rec_rank >= 1 && s.rec_rank <= 1024), at + "time mix: bad widths");
        }
        CPM_REQUIRE(s.ff >= 0 && (s.ff == 0 || (tanh_norms && s.ff_limit > 0.f)), at + "dense feed-forwards need dynamic tanh norms and a limit");
        CPM_REQUIRE(!tanh_norms || s.experts + s.identity == 0, at + "mixtures of experts need norms on the sublayers' outputs");
        CPM_REQUIRE(s.window >= 0, at + "negative window");
        if (s.kv_from >= 0) {
            CPM_REQUIRE(s.kv_from < static_cast<int>(i), at + "keys and values must come from an earlier layer");
            const LayerSpec& f = mc_.specs[s.kv_from];
            CPM_REQUIRE(f.heads > 0 && f.kv_from < 0 && f.kv_heads == s.kv_heads && f.dim == s.dim && f.vdim == s.vdim,
                        at + "the layer whose keys and values are shared must have its own, of the same shape");
        }
        if (s.experts + s.identity == 0) continue;
        const int n = s.experts + s.identity;
        CPM_REQUIRE(s.experts >= 1 && s.identity >= 0 && n <= kMoeMaxOutputs, at + "number of experts out of range");
        CPM_REQUIRE(s.groups >= 1 && n % s.groups == 0 && s.keep_groups >= 1 && s.keep_groups <= s.groups, at + "bad expert groups");
        CPM_REQUIRE(s.top >= 1 && s.top <= kMoeMaxTop && s.top <= n / s.groups * s.keep_groups, at + "more experts per token than can be chosen");
        CPM_REQUIRE(s.expert_ff >= 1 && s.shared_ff >= 0, at + "bad expert widths");
    }
}

size_t Engine::layered_bytes_per_token() const {
    size_t b = 0;
    for (const LayerSpec& s : mc_.specs) {
        if (s.heads > 0 && s.kv_from < 0) b += static_cast<size_t>(s.kv_heads) * (pad64(s.dim) + pad64(s.vdim)) * elem_bytes();
    }
    return std::max<size_t>(b, 1);   // purely recurrent models hold any number of tokens
}

bool Engine::has_recurrence() const {
    for (const LayerSpec& s : mc_.specs) {
        if (s.rec != REC_NONE) return true;
    }
    return false;
}

int Engine::layered_attn_splits(const LayerSpec& sp, int rows) const {
    if (rows > 64) return 1;
    const int tok = 128 / std::min(128, sp.heads / sp.kv_heads);
    int n = runtime().num_sms / (ceil_div(rows, tok) * sp.kv_heads);
    if (sp.window > 0) n = std::min(n, ceil_div(sp.window + tok, 128) + 1);   // key tiles one token tile can touch
    return std::max(1, std::min(n, 24));
}

void Engine::lay_out_layered(Pool& p) {
    const size_t R = max_rows_, es = elem_bytes();
    const int L = ld(), V = mc_.vocab;
    // ---- weights
    embed_ = take<bf16>(p, static_cast<size_t>(V) * L);
    lm_head_ = take<bf16>(p, linear_weight_elems(V, L));
    final_norm_ = take<bf16>(p, L);
    const bool tanh_norms = mc_.norm == NORM_DYNAMIC_TANH;
    auto take_tanh = [&](DynTanh& n) {
        n.w = take<bf16>(p, L);
        n.b = take<bf16>(p, L);
    };
    if (tanh_norms) take_tanh(tanh_final_);
    const int side = mc_.side_dim, side_ld = pad64(side);
    if (side > 0) side_embed_ = take<bf16>(p, static_cast<size_t>(V) * mc_.specs.size() * side);
    size_t qkv = 1, q = 1, attn = 0, ws = 256, slots = 1, x_slots = 1, act_ld = 64, outputs = 1, top = 1;
    size_t mix = 0, rec = 0, channels = 0, rec_out = 0, rec_ws = 0, ff = 0;
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        LayeredWeights& w = lw_[i];
        w.o = take<bf16>(p, linear_weight_elems(mc_.hidden, o_cols(s)));
        attn = std::max<size_t>(attn, o_cols(s));
        if (tanh_norms) {
            take_tanh(w.tanh1);
            take_tanh(w.tanh1b);
        } else {
            w.norm1 = take<bf16>(p, L);
        }
        if (s.heads > 0) {
            const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim;
            const int n = s.kv_from >= 0 ? nq : nq + nk + nv;
            w.qkv = take<bf16>(p, linear_weight_elems(n, L));
            if (s.qk_norm) {
                w.q_norm = take<bf16>(p, nq);
                if (s.kv_from < 0) w.k_norm = take<bf16>(p, nk);
            }
            if (s.rot_dims > 0) w.inv_freq = take<float>(p, s.rot_dims / 2);
            qkv = std::max<size_t>(qkv, n);
            q = std::max<size_t>(q, static_cast<size_t>(s.heads) * pad64(s.dim));
            for (int rows = 1; rows <= 64; ++rows) {
                ws = std::max(ws, attn_workspace_bytes(rows, s.heads, std::max(128, pad64(s.vdim)), layered_attn_splits(s, rows)));
            }
        }
        if (s.rec != REC_NONE) {
            const int nk = s.rec_heads * s.rec_dim, nv = s.rec_heads * s.rec_vdim;
            if (s.rec == REC_TIME_MIX) {
                w.rec_part = linear_weight_elems(nk, L);
                w.rec_proj = take<bf16>(p, 4 * w.rec_part + linear_weight_elems(s.rec_rank, L));
                w.w2 = take<bf16>(p, static_cast<size_t>(nk) * s.rec_rank);
                w.w0 = take<bf16>(p, nk);
                w.bonus = take<bf16>(p, nk);
                w.mu = take<bf16>(p, static_cast<size_t>(kMixes) * L);
                w.prev = take<float>(p, L);
                mix = kMixes * R * L;
                rec = std::max(rec, kMixes * R * rec_ld(s));
                channels = std::max<size_t>(channels, nk);
            } else {
                w.rec_proj = take<bf16>(p, linear_weight_elems(2 * (nk + nv), L));
                w.decay = take<float>(p, s.rec_heads);
                rec = std::max(rec, R * rec_ld(s));
            }
            w.rec_norm = take<bf16>(p, nv);
            w.state = take<float>(p, scan_state_floats(s.rec_heads, s.rec_dim, s.rec_vdim));
            rec_out = std::max<size_t>(rec_out, nv);
            rec_ws = std::max(rec_ws, scan_workspace_floats(s.rec_heads, s.rec_dim, s.rec_vdim, max_rows_));
        }
        if (s.ff > 0) {
            take_tanh(w.tanh2);
            take_tanh(w.tanh2b);
            w.gate_up = take<bf16>(p, linear_weight_elems(2 * pad64(s.ff), L));
            w.down = take<bf16>(p, linear_weight_elems(mc_.hidden, pad64(s.ff)));
            ff = std::max<size_t>(ff, pad64(s.ff));
        }
        if (side > 0) {
            w.side_gate = take<bf16>(p, linear_weight_elems(side, L));
            w.side_proj = take<bf16>(p, linear_weight_elems(mc_.hidden, side_ld));
            w.side_norm = take<bf16>(p, L);
        }
        if (s.experts + s.identity > 0) {
            const int outs = s.experts + s.identity;
            w.norm2 = take<bf16>(p, L);
            w.router = take<bf16>(p, static_cast<size_t>(outs) * L);
            w.correction = take<float>(p, outs);
            w.gate_up = take<bf16>(p, moe_gate_up_elems(s, L));
            w.down = take<bf16>(p, moe_down_elems(s, mc_.hidden));
            x_slots = std::max(x_slots, R * s.top);
            slots = std::max(slots, R * (s.top + (s.shared_ff > 0 ? 1 : 0)));
            act_ld = std::max<size_t>(act_ld, std::max(pad64(s.expert_ff), pad64(s.shared_ff)));
            outputs = std::max<size_t>(outputs, outs);
            top = std::max<size_t>(top, s.top);
        }
    }
    // ---- activations
    x32_ = take<float>(p, R * L);
    lx_ = p.take(R * L * es);
    lqkv_ = p.take(R * qkv * es);
    lq_ = p.take(R * q * es);
    lattn_ = p.take(R * attn * es);
    ldelta_ = p.take(R * L * es);
    lnorm_ = p.take(R * L * es);
    want_ = take<int32_t>(p, R);
    lmix_ = p.take(mix * es);
    lrec_ = p.take(rec * es);
    ldecay_ = take<float>(p, R * channels);
    lo_ = take<float>(p, R * rec_out);
    rec_ws_ = take<float>(p, rec_ws);
    lgu_ = p.take(R * 2 * ff * es);
    lact_ = p.take(R * ff * es);
    lside_ = p.take(R * side_ld * es);
    lsg_ = p.take(R * side_ld * es);
    state_len_ = take<int32_t>(p, 2);   // and the counter of a one-token recurrence
    moe_rows_ = slots;
    moe_x_ = p.take(x_slots * L * es);
    moe_act_ = p.take(slots * act_ld * es);
    moe_gu_ = mc_.fp32 ? p.take(slots * 2 * act_ld * es) : nullptr;
    moe_y_ = p.take(slots * L * es);
    moe_.z = take<float>(p, R * outputs);
    moe_.expert = take<int32_t>(p, R * top);
    moe_.weight = take<float>(p, R * top);
    moe_.rank = take<int32_t>(p, R * top);
    moe_.id_weight = take<float>(p, R);
    moe_.counts = take<int32_t>(p, outputs);
    moe_.offset = take<int32_t>(p, outputs);
    moe_.entries = take<int4>(p, kMoeMaxEntries);
    moe_.n_entries = take<int32_t>(p, 1);
    moe_.tickets = take<int32_t>(p, moe_ticket_ints(max_rows_));
    gemm_ws_ = reinterpret_cast<float*>(p.take(linear_workspace_bytes(256, runtime().num_sms)));
    tickets_ = take<int>(p, kTicketInts);
    attn_ws_o_ = reinterpret_cast<float*>(p.take(ws));
    attn_ws_ml_ = reinterpret_cast<float*>(p.take(ws / 32 + 1024));
    st_ = take<int32_t>(p, S_COUNT);
    // ---- K/V caches last
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        LayeredWeights& w = lw_[i];
        if (s.heads == 0) continue;
        if (s.kv_from >= 0) {
            w.k = lw_[s.kv_from].k;
            w.v = lw_[s.kv_from].v;
        } else {
            w.k = p.take(static_cast<size_t>(budget_) * s.kv_heads * pad64(s.dim) * es);
            w.v = p.take(static_cast<size_t>(budget_) * s.kv_heads * pad64(s.vdim) * es);
        }
    }
    if (p.counting) return;
    // ---- the tensors load() has to see
    not_loaded_ = {"embed"};
    auto need_norm = [&](const std::string& n) {
        not_loaded_.insert(n);
        if (!tanh_norms) return;
        not_loaded_.insert(n + ".b");
        not_loaded_.insert(n + ".alpha");
    };
    need_norm("final.norm");
    if (!mc_.tied_head) not_loaded_.insert("head");
    if (side > 0) not_loaded_.insert("side.embed");
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        const std::string l = "l" + std::to_string(i) + ".";
        auto need = [&](const std::string& n) { not_loaded_.insert(l + n); };
        need_norm(l + "norm1");
        if (tanh_norms) need_norm(l + "norm1b");
        if (s.heads > 0) {
            const std::string m = attn_prefix(s);
            need(m + "q"); need(m + "o");
            if (s.kv_from < 0) { need(m + "k"); need(m + "v"); }
            if (s.rot_dims > 0) need(m + "inv_freq");
            if (s.qk_norm) {
                need(m + "q.norm");
                if (s.kv_from < 0) need(m + "k.norm");
            }
        }
        if (s.rec != REC_NONE) {
            const std::string m = rec_prefix(s);
            need(m + "k"); need(m + "v"); need(m + "g"); need(m + "norm"); need(m + "o");
            if (s.rec == REC_LIGHTNING) {
                need(m + "q"); need(m + "decay");
            } else {
                need(m + "r"); need(m + "w0"); need(m + "w1"); need(m + "w2"); need(m + "u");
                for (int k = 0; k < kMixes; ++k) need(m + "mu." + kMixNames[k]);
            }
        }
        if (s.ff > 0) {
            need_norm(l + "norm2");
            need_norm(l + "norm2b");
            need("mlp.gate"); need("mlp.up"); need("mlp.down");
        }
        if (side > 0) { need("side.gate"); need("side.proj"); need("side.norm"); }
        if (s.experts + s.identity == 0) continue;
        need("norm2"); need("mlp.router"); need("mlp.correction");
        for (int e = 0; e < s.experts + (s.shared_ff > 0 ? 1 : 0); ++e) {
            const std::string x = e < s.experts ? "mlp.e" + std::to_string(e) : std::string("mlp.shared");
            need(x + ".gate"); need(x + ".up"); need(x + ".down");
        }
    }
}

void Engine::load_layered(const std::string& name, const void* src) {
    cudaStream_t st = runtime().stream;
    const int W = mc_.hidden, L = ld();
    // row-major rows x cols -> dst; K: padded columns of dst
    auto plain = [&](bf16* dst, int rows, int cols, int K) {
        CUDA_CHECK(cudaMemcpy2DAsync(dst, static_cast<size_t>(K) * 2, src, static_cast<size_t>(cols) * 2, static_cast<size_t>(cols) * 2, rows,
                                     cudaMemcpyDefault, st));
    };
    auto plain_f32 = [&](float* dst, size_t n) { CUDA_CHECK(cudaMemcpyAsync(dst, src, n * 4, cudaMemcpyDefault, st)); };
    // a matrix of a product; mode 1 / 2: gate / up rows of a SwiGLU pair of `half` padded rows each
    auto matrix = [&](bf16* dst, int rows, int cols, int K, int row_offset, int mode, int half, int k_offset = 0) {
        if (mc_.fp32) plain(dst + static_cast<size_t>(mode == 2 ? half : row_offset) * K + k_offset, rows, cols, K);
        else retile_weight_rows(src, rows, cols, dst, K, mode, row_offset, k_offset, st);
    };
    // "<base>", "<base>.b" or "<base>.alpha" of a dynamic tanh norm
    auto tanh_part = [&](const std::string& n, const std::string& base, DynTanh& t) -> bool {
        if (mc_.norm != NORM_DYNAMIC_TANH || n.rfind(base, 0) != 0) return false;
        const std::string rest = n.substr(base.size());
        if (rest == "") plain(const_cast<bf16*>(t.w), 1, W, L);
        else if (rest == ".b") plain(const_cast<bf16*>(t.b), 1, W, L);
        else if (rest == ".alpha") {
            bf16 h;
            CUDA_CHECK(cudaMemcpyAsync(&h, src, 2, cudaMemcpyDefault, st));
            CUDA_CHECK(cudaStreamSynchronize(st));
            t.alpha = __bfloat162float(h);
        } else {
            return false;
        }
        return true;
    };
    if (decode_graph_ != nullptr) {   // alpha is an argument of captured kernels
        cudaGraphExecDestroy(decode_graph_);
        decode_graph_ = nullptr;
        memset(decode_key_, 0, sizeof(decode_key_));
    }
    const std::set<std::string>::iterator known = not_loaded_.find(name);
    int li = -1;
    std::string sub;
    if (name.size() > 1 && name[0] == 'l' && isdigit(static_cast<unsigned char>(name[1]))) {
        const size_t dot = name.find('.');
        CPM_REQUIRE(dot != std::string::npos, "Unsupported name " + name);
        li = atoi(name.c_str() + 1);
        sub = name.substr(dot + 1);
        CPM_REQUIRE(li >= 0 && li < static_cast<int>(lw_.size()), "layer index out of range: " + name);
    }
    if (name == "embed") {
        plain(embed_, mc_.vocab, W, L);
        if (mc_.tied_head) matrix(lm_head_, mc_.vocab, W, L, 0, 0, 0);
    } else if (name == "side.embed" && mc_.side_dim > 0) {
        const int cols = static_cast<int>(lw_.size()) * mc_.side_dim;
        plain(side_embed_, mc_.vocab, cols, cols);
    } else if (tanh_part(name, "final.norm", tanh_final_)) {
    } else if (name == "head" && !mc_.tied_head) matrix(lm_head_, mc_.vocab, W, L, 0, 0, 0);
    else if (name == "final.norm") plain(final_norm_, 1, W, L);
    else {
        CPM_REQUIRE(li >= 0, "Unsupported name " + name);
        const LayerSpec& s = mc_.specs[li];
        LayeredWeights& w = lw_[li];
        const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim;
        const bool own = s.kv_from < 0, moe = s.experts + s.identity > 0;
        if (s.heads > 0 && sub.rfind(attn_prefix(s), 0) == 0) {
            const std::string m = sub.substr(attn_prefix(s).size());
            if (m == "q") matrix(w.qkv, nq, W, L, 0, 0, 0);
            else if (m == "k" && own) matrix(w.qkv, nk, W, L, nq, 0, 0);
            else if (m == "v" && own) matrix(w.qkv, nv, W, L, nq + nk, 0, 0);
            else if (m == "o") matrix(w.o, W, s.heads * s.vdim, o_cols(s), 0, 0, 0);
            else if (m == "inv_freq" && s.rot_dims > 0) plain_f32(w.inv_freq, s.rot_dims / 2);
            else if (m == "q.norm" && s.qk_norm) plain(w.q_norm, 1, nq, nq);
            else if (m == "k.norm" && s.qk_norm && own) plain(w.k_norm, 1, nk, nk);
            else throw std::invalid_argument("Unsupported name " + name);
        } else if (s.rec != REC_NONE && sub.rfind(rec_prefix(s), 0) == 0) {
            const std::string m = sub.substr(rec_prefix(s).size());
            const int ck = s.rec_heads * s.rec_dim, cv = s.rec_heads * s.rec_vdim;
            if (m == "o") matrix(w.o, W, cv, o_cols(s), 0, 0, 0, o_left(s));
            else if (m == "norm") plain(w.rec_norm, 1, cv, cv);
            else if (s.rec == REC_LIGHTNING) {
                if (m == "q") matrix(w.rec_proj, ck, W, L, 0, 0, 0);
                else if (m == "k") matrix(w.rec_proj, ck, W, L, ck, 0, 0);
                else if (m == "v") matrix(w.rec_proj, cv, W, L, 2 * ck, 0, 0);
                else if (m == "g") matrix(w.rec_proj, cv, W, L, 2 * ck + cv, 0, 0);
                else if (m == "decay") plain_f32(w.decay, s.rec_heads);
                else throw std::invalid_argument("Unsupported name " + name);
            } else if (m == "w0") plain(w.w0, 1, ck, ck);
            else if (m == "w1") matrix(w.rec_proj + 4 * w.rec_part, s.rec_rank, W, L, 0, 0, 0);
            else if (m == "w2") upload_transposed(src, ck, s.rec_rank, w.w2, st);
            else if (m == "u") plain(w.bonus, 1, ck, ck);
            else {
                const bool mu = m.rfind("mu.", 0) == 0;
                const std::string which = mu ? m.substr(3) : m;
                const char* at = which.size() == 1 ? strchr(kMixNames, which[0]) : nullptr;
                const int k = at != nullptr ? static_cast<int>(at - kMixNames) : kMixes;
                if (mu && k < kMixes) plain(w.mu + static_cast<size_t>(k) * L, 1, W, L);
                else if (!mu && k < 4) matrix(w.rec_proj + k * w.rec_part, ck, W, L, 0, 0, 0);
                else throw std::invalid_argument("Unsupported name " + name);
            }
        } else if (tanh_part(sub, "norm1b", w.tanh1b) || tanh_part(sub, "norm1", w.tanh1)) {
        } else if (s.ff > 0 && (tanh_part(sub, "norm2b", w.tanh2b) || tanh_part(sub, "norm2", w.tanh2))) {
        } else if (s.ff > 0 && sub == "mlp.gate") matrix(w.gate_up, s.ff, W, L, 0, 1, pad64(s.ff));
        else if (s.ff > 0 && sub == "mlp.up") matrix(w.gate_up, s.ff, W, L, 0, 2, pad64(s.ff));
        else if (s.ff > 0 && sub == "mlp.down") matrix(w.down, W, s.ff, pad64(s.ff), 0, 0, 0);
        else if (mc_.side_dim > 0 && sub == "side.gate") matrix(w.side_gate, mc_.side_dim, W, L, 0, 0, 0);
        else if (mc_.side_dim > 0 && sub == "side.proj") matrix(w.side_proj, W, mc_.side_dim, pad64(mc_.side_dim), 0, 0, 0);
        else if (mc_.side_dim > 0 && sub == "side.norm") plain(w.side_norm, 1, W, L);
        else if (sub == "norm1" && w.norm1 != nullptr) plain(w.norm1, 1, W, L);
        else if (sub == "norm2" && moe) plain(w.norm2, 1, W, L);
        else if (sub == "mlp.router" && moe) plain(w.router, s.experts + s.identity, W, L);
        else if (sub == "mlp.correction" && moe) {
            std::vector<bf16> h(s.experts + s.identity);
            CUDA_CHECK(cudaMemcpyAsync(h.data(), src, h.size() * 2, cudaMemcpyDefault, st));
            CUDA_CHECK(cudaStreamSynchronize(st));
            std::vector<float> f(h.size());
            for (size_t i = 0; i < h.size(); ++i) f[i] = __bfloat162float(h[i]);
            CUDA_CHECK(cudaMemcpyAsync(w.correction, f.data(), f.size() * 4, cudaMemcpyHostToDevice, st));
            CUDA_CHECK(cudaStreamSynchronize(st));
        } else {
            const size_t dot = sub.rfind('.');
            CPM_REQUIRE(moe && sub.rfind("mlp.", 0) == 0 && dot != std::string::npos && dot > 4, "Unsupported name " + name);
            const std::string who = sub.substr(4, dot - 4), what = sub.substr(dot + 1);
            int e = -1;
            if (who == "shared" && s.shared_ff > 0) e = s.experts;
            else if (who.size() > 1 && who[0] == 'e' && isdigit(static_cast<unsigned char>(who[1]))) e = atoi(who.c_str() + 1);
            CPM_REQUIRE(e >= 0 && (e < s.experts || who == "shared"), "Unsupported name " + name);
            const int ff = e < s.experts ? s.expert_ff : s.shared_ff;
            bf16* gu = w.gate_up + moe_gate_up_offset(s, L, e);
            if (what == "gate") matrix(gu, ff, W, L, 0, 1, pad64(ff));
            else if (what == "up") matrix(gu, ff, W, L, 0, 2, pad64(ff));
            else if (what == "down") matrix(w.down + moe_down_offset(s, W, e), W, ff, pad64(ff), 0, 0, 0);
            else throw std::invalid_argument("Unsupported name " + name);
        }
    }
    CUDA_CHECK(cudaStreamSynchronize(st));
    if (known != not_loaded_.end()) not_loaded_.erase(known);
}

// ------------------------------------------------------------------ plans (bf16)
LayeredPlans& Engine::layered_plans(int rows) {
    auto it = lplans_.find(rows);
    if (it != lplans_.end()) return *it->second;
    if (lplans_.size() >= 256) lplans_.clear();   // a stream of odd chunk sizes
    auto plans = std::make_unique<LayeredPlans>();
    LayeredPlans& lp = *plans;
    lp.rows = rows;
    lp.layers.resize(lw_.size());
    const int L = ld(), W = mc_.hidden;
    auto product = [&](const void* x, int K, const bf16* w, int N, void* y, int ldy) {
        LayeredProduct p;
        p.x = x; p.w = w; p.N = N; p.K = K; p.y = y; p.ldy = ldy;
        if (!mc_.fp32) {
            p.plan = make_linear_plan(static_cast<const bf16*>(x), rows, w, rows, N, K, static_cast<bf16*>(y), ldy, nullptr, gemm_ws_, tickets_,
                                      runtime().num_sms);
            CPM_REQUIRE(2LL * ceil_div(p.plan.N, 128) * ceil_div(p.plan.M, p.plan.mt) <= kTicketInts,
                        "linear: more output tiles than the split-K counters cover");
        }
        return p;
    };
    auto at = [&](void* p, size_t elems) { return static_cast<void*>(static_cast<uint8_t*>(p) + elems * elem_bytes()); };
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        const LayeredWeights& w = lw_[i];
        LayeredPlans::Layer& l = lp.layers[i];
        const int nq = s.heads * s.dim, n = s.kv_from >= 0 ? nq : nq + s.kv_heads * (s.dim + s.vdim);
        if (s.heads > 0) l.qkv = product(lx_, L, w.qkv, n, lqkv_, n);
        l.o = product(lattn_, o_cols(s), w.o, W, ldelta_, L);
        if (s.rec != REC_NONE) {
            const int nk = s.rec_heads * s.rec_dim, nv = s.rec_heads * s.rec_vdim, ldr = rec_ld(s);
            if (s.rec == REC_LIGHTNING) {
                l.rec.push_back(product(lx_, L, w.rec_proj, 2 * (nk + nv), lrec_, ldr));
            } else if (!mc_.fp32) {
                l.mixes = make_grouped_plan(w.rec_proj, 4, nk, s.rec_rank, L, static_cast<const bf16*>(lmix_), static_cast<bf16*>(lrec_), ldr, rows);
            } else {
                for (int k = 0; k < kMixes; ++k) {
                    l.rec.push_back(product(at(lmix_, static_cast<size_t>(k) * rows * L), L, w.rec_proj + k * w.rec_part, k < 4 ? nk : s.rec_rank,
                                            at(lrec_, static_cast<size_t>(k) * rows * ldr), ldr));
                }
            }
        }
        if (s.ff > 0) {
            const int ff = pad64(s.ff);
            l.ff_fused = !mc_.fp32 && linear_swiglu_fits(rows, ff, runtime().num_sms);
            if (l.ff_fused) {
                l.ff_gate_up.plan = make_linear_swiglu_plan(static_cast<const bf16*>(lx_), rows, w.gate_up, rows, ff, L, static_cast<bf16*>(lact_), ff,
                                                            runtime().num_sms);
                l.ff_gate_up.plan.gate_limit = s.ff_limit;
                l.ff_gate_up.plan.gate_alpha = s.ff_alpha;
            } else {
                l.ff_gate_up = product(lx_, L, w.gate_up, 2 * ff, lgu_, 2 * ff);
            }
            l.ff_down = product(lact_, ff, w.down, W, ldelta_, L);
        }
        if (mc_.side_dim > 0) {
            l.side_gate = product(lx_, L, w.side_gate, mc_.side_dim, lside_, pad64(mc_.side_dim));
            l.side_proj = product(lsg_, pad64(mc_.side_dim), w.side_proj, W, ldelta_, L);
        }
    }
    if (!mc_.fp32) {
        bf16 *x = static_cast<bf16*>(lx_), *q = static_cast<bf16*>(lq_), *at = static_cast<bf16*>(lattn_), *mx = static_cast<bf16*>(moe_x_),
             *act = static_cast<bf16*>(moe_act_), *y = static_cast<bf16*>(moe_y_);
        for (size_t i = 0; i < lw_.size(); ++i) {
            const LayerSpec& s = mc_.specs[i];
            const LayeredWeights& w = lw_[i];
            LayeredPlans::Layer& l = lp.layers[i];
            const int dk = pad64(s.dim), dv = pad64(s.vdim);
            l.tensor_attn = s.heads > 0 && biased_attn_fits(s.heads, s.kv_heads, dk, dv);
            if (l.tensor_attn) {
                l.attn = make_biased_attn_plan(q, s.heads * dk, static_cast<const bf16*>(w.k), static_cast<const bf16*>(w.v), budget_, rows,
                                               s.heads, s.kv_heads, dk, dv, s.vdim, layered_attn_splits(s, rows), s.scale, s.window,
                                               s.bias_exp, at, o_cols(s), attn_ws_o_, attn_ws_ml_);
                l.attn.sink = s.sink;
                l.attn.out_scale = s.attn_scale;
            }
            if (s.experts + s.identity > 0) {
                const int tile = moe_pick_tile(s, rows);
                const int ld_act = std::max(pad64(s.expert_ff), pad64(s.shared_ff));
                const int slots = rows * (s.top + (s.shared_ff > 0 ? 1 : 0));
                // a single token's input is every expert's input: nothing is copied
                l.gate_up = make_moe_gate_up_plan(s, w.gate_up, rows == 1 ? x : mx, rows == 1 ? 1 : rows * s.top, x, L, act, ld_act, rows, tile, moe_);
                l.down = make_moe_down_plan(s, w.down, act, slots, ld_act, W, y, L, rows, tile, moe_);
            }
        }
    }
    lplans_[rows] = std::move(plans);
    return lp;
}

// ------------------------------------------------------------------ forward
// Mixture of experts of the stream rows, then the output norm and the residual add.
template <typename T>
void Engine::layered_mixture(int i, LayeredPlans& lp, cudaStream_t s) {
    const LayerSpec& sp = mc_.specs[i];
    const LayeredWeights& w = lw_[i];
    const int rows = lp.rows, L = ld(), W = mc_.hidden;
    const bool single = rows == 1;
    const int tile = mc_.fp32 ? kF32Rows : lp.layers[i].gate_up.tile;
    launch_moe_route(sp, x32_, w.router, w.correction, moe_, rows, L, tile, single, s);
    if (!single) launch_moe_gather<T>(sp, static_cast<const T*>(lx_), static_cast<T*>(moe_x_), moe_, rows, L, s);
    if constexpr (sizeof(T) == 2) {
        launch_moe_gemm(lp.layers[i].gate_up, s);
        launch_moe_gemm(lp.layers[i].down, s);
    } else {
        const float* x = static_cast<const float*>(lx_);
        float *gu = static_cast<float*>(moe_gu_), *act = static_cast<float*>(moe_act_), *y = static_cast<float*>(moe_y_);
        const int ff = pad64(sp.expert_ff), ffs = pad64(sp.shared_ff), slots = rows * sp.top;
        const int most = moe_max_entries(sp, rows, tile);
        launch_linear_f32(single ? x : static_cast<const float*>(moe_x_), L, w.gate_up, moe_gate_up_offset(sp, L, 1), gu, 2 * ff, 0, 2 * ff, L,
                          moe_.entries, moe_.n_entries, most, false, s);
        launch_silu_f32(gu, 2 * ff, act, ff, slots, ff, s);
        launch_linear_f32(act, ff, w.down, moe_down_offset(sp, W, 1), y, L, 0, W, ff, moe_.entries, moe_.n_entries, most, true, s);
        if (ffs > 0) {
            launch_linear_f32(x, L, w.gate_up + moe_gate_up_offset(sp, L, sp.experts), 0, gu, 2 * ffs, rows, 2 * ffs, L, nullptr, nullptr, 0, false, s);
            launch_silu_f32(gu, 2 * ffs, act, ffs, rows, ffs, s);
            launch_linear_f32(act, ffs, w.down + moe_down_offset(sp, W, sp.experts), 0, y + static_cast<size_t>(slots) * L, L, rows, W, ffs, nullptr,
                              nullptr, 0, false, s);
        }
    }
    MoeMix mix;
    mix.y = moe_y_;
    mix.expert = moe_.expert; mix.weight = moe_.weight; mix.rank = moe_.rank; mix.offset = moe_.offset; mix.id_weight = moe_.id_weight;
    mix.top = sp.top; mix.experts = sp.experts;
    mix.shared_row0 = sp.shared_ff > 0 ? rows * sp.top : -1;
    launch_out_norm<T>(x32_, static_cast<T*>(lx_), nullptr, mix, mc_.scale_residual, w.norm2, rows, W, L, mc_.eps, s);
}

template <typename T>
void Engine::run_product(const LayeredProduct& p, int rows, cudaStream_t s) {
    if constexpr (sizeof(T) == 2) launch_linear(p.plan, s);
    else launch_linear_f32(static_cast<const float*>(p.x), p.K, p.w, 0, static_cast<float*>(p.y), p.ldy, rows, p.N, p.K, nullptr, nullptr, 0, false, s);
}

template <typename T>
void Engine::layered_attention(int i, LayeredPlans& lp, const int32_t* kv_len, int kv_off, cudaStream_t s) {
    const LayerSpec& sp = mc_.specs[i];
    const LayeredWeights& w = lw_[i];
    LayeredPlans::Layer& l = lp.layers[i];
    const int rows = lp.rows;
    run_product<T>(l.qkv, rows, s);
    QkvNormArgs a;
    a.qkv = lqkv_; a.ld = l.qkv.N;
    a.heads = sp.heads; a.kv_heads = sp.kv_heads;
    a.dim = sp.dim; a.dim_p = pad64(sp.dim); a.vdim = sp.vdim; a.vdim_p = pad64(sp.vdim);
    a.wq = w.q_norm; a.wk = w.k_norm; a.eps = mc_.eps;
    a.rot_dims = sp.rot_dims; a.inv_freq = w.inv_freq;
    a.q_out = lq_;
    a.k_cache = sp.kv_from >= 0 ? nullptr : w.k;
    a.v_cache = sp.kv_from >= 0 ? nullptr : w.v;
    a.kv_len = kv_len; a.kv_off = kv_off; a.cache_rows = budget_; a.error = runtime().d_error;
    launch_qkv_norm_append<T>(a, rows, s);
    if (l.tensor_attn) {
        l.attn.kv_len = kv_len;
        l.attn.kv_len_add = kv_off + rows;
        launch_tree_attention(l.attn, s);
    } else {
        PlainAttnArgs pa;
        pa.q = lq_; pa.k_cache = w.k; pa.v_cache = w.v; pa.out = lattn_;
        pa.tq = rows; pa.hq = sp.heads; pa.hkv = sp.kv_heads;
        pa.dk = pad64(sp.dim); pa.dv = pad64(sp.vdim); pa.out_cols = sp.vdim; pa.out_ld = o_cols(sp);
        pa.kv_len = kv_len; pa.kv_len_add = kv_off + rows;
        pa.scale = sp.scale; pa.window = sp.window; pa.bias_exp = sp.bias_exp;
        pa.sink = sp.sink; pa.out_scale = sp.attn_scale;
        launch_plain_attention<T>(pa, s);
    }
}

template <typename T>
void Engine::layered_recurrence(int i, LayeredPlans& lp, const int32_t* kv_len, int kv_off, cudaStream_t s) {
    const LayerSpec& sp = mc_.specs[i];
    const LayeredWeights& w = lw_[i];
    LayeredPlans::Layer& l = lp.layers[i];
    const int rows = lp.rows, nk = sp.rec_heads * sp.rec_dim, nv = sp.rec_heads * sp.rec_vdim, ldr = rec_ld(sp);
    const T* proj = static_cast<const T*>(lrec_);
    if (sizeof(T) == 2 && sp.rec == REC_TIME_MIX) {
        launch_moe_gemm(l.mixes, s);
    } else {
        for (const LayeredProduct& p : l.rec) run_product<T>(p, rows, s);
    }
    ScanArgs a;
    a.heads = sp.rec_heads; a.dim = sp.rec_dim; a.vdim = sp.rec_vdim; a.rows = rows;
    a.ld_r = a.ld_k = a.ld_v = ldr;
    a.state = w.state; a.ws = rec_ws_;
    a.kv_len = kv_len; a.kv_off = kv_off;
    a.out = lo_; a.ld_out = nv;
    const T* gate;
    const bool per_head = sp.rec == REC_TIME_MIX;
    T* out = static_cast<T*>(lattn_) + o_left(sp);
    const bool step = rows == 1 && scan_step_fits(sp.rec_dim, sp.rec_vdim, per_head);
    if (per_head) {
        const size_t part = static_cast<size_t>(rows) * ldr;
        if (!step) launch_decay<T>(proj + 4 * part, ldr, w.w2, w.w0, sp.rec_rank, nk, ldecay_, nk, rows, s);
        a.r = proj; a.k = proj + part; a.v = proj + 2 * part;
        gate = proj + 3 * part;
        a.w = ldecay_; a.ld_w = nk;
        a.bonus = w.bonus;
    } else {
        a.r = proj; a.k = proj + nk; a.v = proj + 2 * nk;
        gate = proj + 2 * nk + nv;
        a.silu = true;
        a.decay = w.decay;
    }
    if (step) {
        ScanStepArgs st;
        st.scan = a;
        st.inner = proj + 4 * static_cast<size_t>(ldr);
        st.w2 = w.w2; st.w0 = w.w0; st.rank = sp.rec_rank;
        st.norm = w.rec_norm; st.gate = gate;
        st.eps = mc_.eps; st.scale = sp.rec_scale;
        st.out = out;
        st.ticket = state_len_ + 1;
        launch_scan_step<T>(st, s);
        return;
    }
    launch_scan<T>(a, s);
    launch_norm_gate<T>(lo_, nv, per_head ? sp.rec_heads : 1, per_head ? sp.rec_vdim : nv, w.rec_norm, gate, ldr, per_head, mc_.eps, sp.rec_scale, out,
                        o_cols(sp), rows, s);
}

template <typename T>
void Engine::layered_dense(int i, LayeredPlans& lp, cudaStream_t s) {
    const LayerSpec& sp = mc_.specs[i];
    LayeredPlans::Layer& l = lp.layers[i];
    const int ff = pad64(sp.ff);
    if (l.ff_fused) {
        launch_linear(l.ff_gate_up.plan, s);
    } else {
        run_product<T>(l.ff_gate_up, lp.rows, s);
        launch_clamped_gate<T>(static_cast<const T*>(lgu_), 2 * ff, static_cast<T*>(lact_), ff, lp.rows, ff, sp.ff_limit, sp.ff_alpha, sizeof(T) == 2, s);
    }
    run_product<T>(l.ff_down, lp.rows, s);
}

TokenShift Engine::token_shift(int i, int rows, const int32_t* kv_len, int kv_off) const {
    TokenShift t;
    if (mc_.specs[i].rec != REC_TIME_MIX) return t;
    t.mu = lw_[i].mu;
    t.out = lmix_;
    t.stride = static_cast<size_t>(rows) * ld();
    t.prev = lw_[i].prev;
    t.kv_len = kv_len; t.kv_off = kv_off;
    return t;
}

template <typename T>
bool Engine::layered_tanh_layer(int i, LayeredPlans& lp, const int32_t* ids, const int32_t* kv_len, int kv_off, cudaStream_t s) {
    const LayerSpec& sp = mc_.specs[i];
    const LayeredWeights& w = lw_[i];
    LayeredPlans::Layer& l = lp.layers[i];
    const int rows = lp.rows, L = ld(), W = mc_.hidden, layers = static_cast<int>(lw_.size());
    T *x = static_cast<T*>(lx_), *delta = static_cast<T*>(ldelta_);
    if (sp.heads > 0) layered_attention<T>(i, lp, kv_len, kv_off, s);
    if (sp.rec != REC_NONE) layered_recurrence<T>(i, lp, kv_len, kv_off, s);
    run_product<T>(l.o, rows, s);
    // a row's mixes need the row before it, which only a single row has at hand at a layer's end
    const bool next = i + 1 < layers && mc_.side_dim > 0 && (rows == 1 || mc_.specs[i + 1].rec != REC_TIME_MIX);
    const DynTanh next_norm = next ? lw_[i + 1].tanh1 : DynTanh();
    const TokenShift next_shift = next ? token_shift(i + 1, rows, kv_len, kv_off) : TokenShift();
    const bool side_step = rows == 1 && mc_.side_dim > 0 && mc_.side_dim <= 4096;
    if (sp.ff > 0) {
        launch_tanh_residual<T>(x32_, delta, w.tanh1b, w.tanh2, x, rows, L, s);
        layered_dense<T>(i, lp, s);
    }
    const DynTanh& last = sp.ff > 0 ? w.tanh2b : w.tanh1b;
    if (side_step) {
        SideStepArgs a;
        a.x32 = x32_; a.delta = ldelta_;
        a.post = last;
        a.gate = w.side_gate; a.proj = w.side_proj; a.norm = w.side_norm;
        a.ids = ids; a.table = side_embed_; a.table_ld = layers * mc_.side_dim; a.col0 = i * mc_.side_dim;
        a.dim = mc_.side_dim; a.vocab = mc_.vocab;
        a.next = next_norm; a.h = lx_; a.shift = next_shift;
        a.width = W; a.ld = L; a.eps = mc_.eps;
        launch_side_step<T>(a, s);
        return next;
    }
    launch_tanh_residual<T>(x32_, delta, last, DynTanh(), x, rows, L, s);
    if (mc_.side_dim == 0) return false;
    run_product<T>(l.side_gate, rows, s);
    launch_side_gate<T>(static_cast<const T*>(lside_), pad64(mc_.side_dim), ids, side_embed_, layers * mc_.side_dim, i * mc_.side_dim, mc_.side_dim,
                        mc_.vocab, static_cast<T*>(lsg_), rows, s);
    run_product<T>(l.side_proj, rows, s);
    launch_side_add<T>(x32_, delta, w.side_norm, next_norm, x, next_shift, rows, W, L, mc_.eps, s);
    return next;
}

template <typename T>
void Engine::layered_forward(int rows, const int32_t* ids, const int32_t* kv_len, int kv_off, cudaStream_t s) {
    const int L = ld(), W = mc_.hidden;
    LayeredPlans& lp = layered_plans(rows);
    StateCheck check;
    if (has_recurrence()) {
        check.state_len = state_len_;
        check.kv_len = kv_len; check.kv_off = kv_off;
    }
    launch_embed_rows<T>(ids, embed_, mc_.vocab, mc_.scale_embed, x32_, static_cast<T*>(lx_), L, rows, check, s);
    bool ready = false;   // the layer's first norm has been taken
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& sp = mc_.specs[i];
        const LayeredWeights& w = lw_[i];
        if (mc_.norm == NORM_DYNAMIC_TANH) {
            const int li = static_cast<int>(i);
            if (!ready) launch_tanh_norm<T>(x32_, nullptr, w.tanh1, static_cast<T*>(lx_), token_shift(li, rows, kv_len, kv_off), rows, L, s);
            ready = layered_tanh_layer<T>(li, lp, ids, kv_len, kv_off, s);
        } else {
            layered_attention<T>(static_cast<int>(i), lp, kv_len, kv_off, s);
            run_product<T>(lp.layers[i].o, rows, s);
            launch_out_norm<T>(x32_, static_cast<T*>(lx_), static_cast<const T*>(ldelta_), MoeMix(), mc_.scale_residual, w.norm1, rows, W, L, mc_.eps, s);
            if (sp.experts + sp.identity > 0) layered_mixture<T>(static_cast<int>(i), lp, s);
        }
        if (layer_capture_ != nullptr) {
            CUDA_CHECK(cudaMemcpy2DAsync(layer_capture_ + i * static_cast<size_t>(rows) * W, static_cast<size_t>(W) * 4, x32_,
                                         static_cast<size_t>(L) * 4, static_cast<size_t>(W) * 4, rows, cudaMemcpyDeviceToDevice, s));
        }
    }
}

template <typename T>
void Engine::layered_logits(const int32_t* rows_idx, int n, void* out, cudaStream_t s) {
    const int L = ld(), V = mc_.vocab;
    if (mc_.norm == NORM_DYNAMIC_TANH) launch_tanh_norm<T>(x32_, rows_idx, tanh_final_, static_cast<T*>(lnorm_), TokenShift(), n, L, s);
    else launch_norm_rows<T>(x32_, rows_idx, final_norm_, static_cast<T*>(lnorm_), n, mc_.hidden, L, mc_.eps, s);
    if constexpr (sizeof(T) == 2) {
        LinearPlan p = make_linear_plan(static_cast<const bf16*>(lnorm_), n, lm_head_, n, V, L, static_cast<bf16*>(out), V, nullptr, gemm_ws_,
                                        tickets_, runtime().num_sms);
        CPM_REQUIRE(2LL * ceil_div(p.N, 128) * ceil_div(p.M, p.mt) <= kTicketInts, "linear: more output tiles than the split-K counters cover");
        launch_linear(p, s);
    } else {
        launch_linear_f32(static_cast<const float*>(lnorm_), L, lm_head_, 0, static_cast<float*>(out), V, n, V, L, nullptr, nullptr, 0, false, s);
    }
}

// A pass that reported an error may have left anything in the recurrent states: only position 0 is open afterwards.
void Engine::layered_check_errors(const char* where) {
    try {
        check_errors(where);
    } catch (...) {
        cudaMemsetAsync(state_len_, 0xff, sizeof(int32_t), runtime().stream);
        throw;
    }
}

void Engine::layered_prefill(int n, int history, const int32_t* ids, const int32_t* want, int n_want, void* logits_out) {
    CPM_REQUIRE(not_loaded_.empty(), "weights missing, for instance " + *not_loaded_.begin());
    cudaStream_t s = runtime().stream;
    CUDA_CHECK(cudaMemcpyAsync(st_ + 6, &history, sizeof(int), cudaMemcpyHostToDevice, s));
    if (n_want > 0) CUDA_CHECK(cudaMemcpyAsync(want_, want, static_cast<size_t>(n_want) * 4, cudaMemcpyHostToDevice, s));
    if (mc_.fp32) layered_forward<float>(n, ids, st_ + 6, 0, s);
    else layered_forward<bf16>(n, ids, st_ + 6, 0, s);
    if (n_want > 0) {
        if (mc_.fp32) layered_logits<float>(want_, n_want, logits_out, s);
        else layered_logits<bf16>(want_, n_want, logits_out, s);
    }
    host_len_ = static_cast<long>(history) + n;
    CUDA_CHECK(cudaStreamSynchronize(s));
    layered_check_errors("prefill");
}

// cache_length (device) already counts the n new tokens.  With cuda_graph a one-token step is captured on its second
// call with the same buffers and replayed from then on.
void Engine::layered_decode(int n, const int32_t* ids, const int32_t* cache_length, void* logits_out, bool cuda_graph) {
    CPM_REQUIRE(not_loaded_.empty(), "weights missing, for instance " + *not_loaded_.begin());
    Runtime& rt = runtime();
    cudaStream_t s = rt.stream;
    auto enqueue = [&]() {
        if (mc_.fp32) {
            layered_forward<float>(n, ids, cache_length, -n, s);
            layered_logits<float>(nullptr, n, logits_out, s);
        } else {
            layered_forward<bf16>(n, ids, cache_length, -n, s);
            layered_logits<bf16>(nullptr, n, logits_out, s);
        }
    };
    const void* key[3] = {ids, cache_length, logits_out};
    const bool graph = cuda_graph && n == 1 && layer_capture_ == nullptr && !rt.profile;
    if (graph && memcmp(key, decode_key_, sizeof(key)) == 0) {
        if (decode_graph_ == nullptr) {
            const long before = rt.launches;
            cudaGraph_t g = nullptr;
            CUDA_CHECK(cudaStreamBeginCapture(s, cudaStreamCaptureModeRelaxed));
            try {
                enqueue();
            } catch (...) {
                cudaStreamEndCapture(s, &g);
                if (g) cudaGraphDestroy(g);
                throw;
            }
            CUDA_CHECK(cudaStreamEndCapture(s, &g));
            CUDA_CHECK(cudaGraphInstantiate(&decode_graph_, g, 0));
            CUDA_CHECK(cudaGraphDestroy(g));
            decode_launches_ = rt.launches - before;
            rt.launches = before;
        }
        CUDA_CHECK(cudaEventRecord(ev0_, s));
        CUDA_CHECK(cudaGraphLaunch(decode_graph_, s));
        CUDA_CHECK(cudaEventRecord(ev1_, s));
        rt.launches += decode_launches_;
    } else {
        if (graph) {
            if (decode_graph_) {
                cudaGraphExecDestroy(decode_graph_);
                decode_graph_ = nullptr;
            }
            memcpy(decode_key_, key, sizeof(key));
        }
        CUDA_CHECK(cudaEventRecord(ev0_, s));
        enqueue();
        CUDA_CHECK(cudaEventRecord(ev1_, s));
    }
    CUDA_CHECK(cudaStreamSynchronize(s));
    float ms = 0.f;
    CUDA_CHECK(cudaEventElapsedTime(&ms, ev0_, ev1_));
    last_step_ms_ = ms;
    layered_check_errors("decode");
}
