// Engine: layered models (ModelConfig::specs) - storage, weight loading and the forward pass over LayerSpec layers.
// They share the engine's pool, K/V budget, prefill / decode entry points and error handling with Llama-format targets.
//
//   x   = embed[token]                                    fp32 stream, with a copy in T for the matrix products
//   x  += m * rms(o(attention(x))) * (1 + w1)             the sublayers read x itself; the norm is on their output
//   x  += m * rms(mixture(x)) * (1 + w2)
//   out = head(rms(x) * (1 + wf))
//
// Positions are cache rows: token r of a pass that starts at row L has position L + r.
#include <algorithm>
#include <cstdlib>
#include <cstring>

#include "engine.cuh"

void Engine::check_specs() const {
    CPM_REQUIRE(mc_.hidden >= 1 && mc_.vocab >= 1, "layered model: empty width or vocabulary");
    CPM_REQUIRE(ld() <= 16384, "layered model: width above 16384 is not supported");
    CPM_REQUIRE(!mc_.sparse.enabled && !mc_.w4a16, "layered model: block selection and int4 weights belong to Llama-format targets");
    for (size_t i = 0; i < mc_.specs.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        const std::string at = "layer " + std::to_string(i) + ": ";
        CPM_REQUIRE(s.heads >= 1 && s.kv_heads >= 1 && s.heads % s.kv_heads == 0, at + "query heads must be a multiple of key/value heads");
        CPM_REQUIRE(s.dim >= 1 && s.vdim >= 1 && pad64(s.dim) <= 512 && s.vdim <= 512, at + "head widths must be in [1, 512]");
        CPM_REQUIRE(s.window >= 0, at + "negative window");
        if (s.kv_from >= 0) {
            CPM_REQUIRE(s.kv_from < static_cast<int>(i), at + "keys and values must come from an earlier layer");
            const LayerSpec& f = mc_.specs[s.kv_from];
            CPM_REQUIRE(f.kv_from < 0 && f.kv_heads == s.kv_heads && f.dim == s.dim && f.vdim == s.vdim,
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
        if (s.kv_from < 0) b += static_cast<size_t>(s.kv_heads) * (pad64(s.dim) + pad64(s.vdim)) * elem_bytes();
    }
    return b;
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
    size_t qkv = 0, q = 0, attn = 0, ws = 256, slots = 1, x_slots = 1, act_ld = 64, outputs = 1, top = 1;
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        LayeredWeights& w = lw_[i];
        const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim, ko = pad64(s.heads * s.vdim);
        const int n = s.kv_from >= 0 ? nq : nq + nk + nv;
        w.qkv = take<bf16>(p, linear_weight_elems(n, L));
        w.o = take<bf16>(p, linear_weight_elems(mc_.hidden, ko));
        w.norm1 = take<bf16>(p, L);
        if (s.qk_norm) {
            w.q_norm = take<bf16>(p, nq);
            if (s.kv_from < 0) w.k_norm = take<bf16>(p, nk);
        }
        qkv = std::max<size_t>(qkv, n);
        q = std::max<size_t>(q, static_cast<size_t>(s.heads) * pad64(s.dim));
        attn = std::max<size_t>(attn, ko);
        for (int rows = 1; rows <= 64; ++rows) {
            ws = std::max(ws, attn_workspace_bytes(rows, s.heads, std::max(128, pad64(s.vdim)), layered_attn_splits(s, rows)));
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
    not_loaded_ = {"embed", "head", "final.norm"};
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& s = mc_.specs[i];
        const std::string l = "l" + std::to_string(i) + ".";
        auto need = [&](const std::string& n) { not_loaded_.insert(l + n); };
        need("norm1"); need("mix.q"); need("mix.o");
        if (s.kv_from < 0) { need("mix.k"); need("mix.v"); }
        if (s.qk_norm) {
            need("mix.q.norm");
            if (s.kv_from < 0) need("mix.k.norm");
        }
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
    // a matrix of a product; mode 1 / 2: gate / up rows of a SwiGLU pair of `half` padded rows each
    auto matrix = [&](bf16* dst, int rows, int cols, int K, int row_offset, int mode, int half) {
        if (mc_.fp32) plain(dst + static_cast<size_t>(mode == 2 ? half : row_offset) * K, rows, cols, K);
        else retile_weight_rows(src, rows, cols, dst, K, mode, row_offset, 0, st);
    };
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
    if (name == "embed") plain(embed_, mc_.vocab, W, L);
    else if (name == "head") matrix(lm_head_, mc_.vocab, W, L, 0, 0, 0);
    else if (name == "final.norm") plain(final_norm_, 1, W, L);
    else {
        CPM_REQUIRE(li >= 0, "Unsupported name " + name);
        const LayerSpec& s = mc_.specs[li];
        LayeredWeights& w = lw_[li];
        const int nq = s.heads * s.dim, nk = s.kv_heads * s.dim, nv = s.kv_heads * s.vdim;
        const bool own = s.kv_from < 0, moe = s.experts + s.identity > 0;
        if (sub == "norm1") plain(w.norm1, 1, W, L);
        else if (sub == "norm2" && moe) plain(w.norm2, 1, W, L);
        else if (sub == "mix.q") matrix(w.qkv, nq, W, L, 0, 0, 0);
        else if (sub == "mix.k" && own) matrix(w.qkv, nk, W, L, nq, 0, 0);
        else if (sub == "mix.v" && own) matrix(w.qkv, nv, W, L, nq + nk, 0, 0);
        else if (sub == "mix.o") matrix(w.o, W, s.heads * s.vdim, pad64(s.heads * s.vdim), 0, 0, 0);
        else if (sub == "mix.q.norm" && s.qk_norm) plain(w.q_norm, 1, nq, nq);
        else if (sub == "mix.k.norm" && s.qk_norm && own) plain(w.k_norm, 1, nk, nk);
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
    if (!mc_.fp32) {
        const int L = ld(), W = mc_.hidden, sms = runtime().num_sms;
        bf16 *x = static_cast<bf16*>(lx_), *qkv = static_cast<bf16*>(lqkv_), *q = static_cast<bf16*>(lq_), *at = static_cast<bf16*>(lattn_),
             *delta = static_cast<bf16*>(ldelta_), *mx = static_cast<bf16*>(moe_x_), *act = static_cast<bf16*>(moe_act_),
             *y = static_cast<bf16*>(moe_y_);
        for (size_t i = 0; i < lw_.size(); ++i) {
            const LayerSpec& s = mc_.specs[i];
            const LayeredWeights& w = lw_[i];
            LayeredPlans::Layer& l = lp.layers[i];
            const int nq = s.heads * s.dim, n = s.kv_from >= 0 ? nq : nq + s.kv_heads * (s.dim + s.vdim), ko = pad64(s.heads * s.vdim);
            const int dk = pad64(s.dim), dv = pad64(s.vdim);
            l.qkv = make_linear_plan(x, rows, w.qkv, rows, n, L, qkv, n, nullptr, gemm_ws_, tickets_, sms);
            l.o = make_linear_plan(at, rows, w.o, rows, W, ko, delta, L, nullptr, gemm_ws_, tickets_, sms);
            for (const LinearPlan* p : {&l.qkv, &l.o}) {
                CPM_REQUIRE(2LL * ceil_div(p->N, 128) * ceil_div(p->M, p->mt) <= kTicketInts, "linear: more output tiles than the split-K counters cover");
            }
            l.tensor_attn = biased_attn_fits(s.heads, s.kv_heads, dk, dv);
            if (l.tensor_attn) {
                l.attn = make_biased_attn_plan(q, s.heads * dk, static_cast<const bf16*>(w.k), static_cast<const bf16*>(w.v), budget_, rows,
                                               s.heads, s.kv_heads, dk, dv, s.vdim, layered_attn_splits(s, rows), s.scale, s.window,
                                               s.bias_exp, at, ko, attn_ws_o_, attn_ws_ml_);
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
void Engine::layered_forward(int rows, const int32_t* ids, const int32_t* kv_len, int kv_off, cudaStream_t s) {
    const int L = ld(), W = mc_.hidden;
    LayeredPlans& lp = layered_plans(rows);
    launch_embed_rows<T>(ids, embed_, mc_.vocab, x32_, static_cast<T*>(lx_), L, rows, s);
    for (size_t i = 0; i < lw_.size(); ++i) {
        const LayerSpec& sp = mc_.specs[i];
        const LayeredWeights& w = lw_[i];
        LayeredPlans::Layer& l = lp.layers[i];
        const int nq = sp.heads * sp.dim, n = sp.kv_from >= 0 ? nq : nq + sp.kv_heads * (sp.dim + sp.vdim), ko = pad64(sp.heads * sp.vdim);
        if constexpr (sizeof(T) == 2) launch_linear(l.qkv, s);
        else launch_linear_f32(static_cast<const float*>(lx_), L, w.qkv, 0, static_cast<float*>(lqkv_), n, rows, n, L, nullptr, nullptr, 0, false, s);
        QkvNormArgs a;
        a.qkv = lqkv_; a.ld = n;
        a.heads = sp.heads; a.kv_heads = sp.kv_heads;
        a.dim = sp.dim; a.dim_p = pad64(sp.dim); a.vdim = sp.vdim; a.vdim_p = pad64(sp.vdim);
        a.wq = w.q_norm; a.wk = w.k_norm; a.eps = mc_.eps;
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
            pa.dk = pad64(sp.dim); pa.dv = pad64(sp.vdim); pa.out_cols = sp.vdim; pa.out_ld = ko;
            pa.kv_len = kv_len; pa.kv_len_add = kv_off + rows;
            pa.scale = sp.scale; pa.window = sp.window; pa.bias_exp = sp.bias_exp;
            launch_plain_attention<T>(pa, s);
        }
        if constexpr (sizeof(T) == 2) launch_linear(l.o, s);
        else launch_linear_f32(static_cast<const float*>(lattn_), ko, w.o, 0, static_cast<float*>(ldelta_), L, rows, W, ko, nullptr, nullptr, 0, false, s);
        launch_out_norm<T>(x32_, static_cast<T*>(lx_), static_cast<const T*>(ldelta_), MoeMix(), mc_.scale_residual, w.norm1, rows, W, L, mc_.eps, s);
        if (sp.experts + sp.identity > 0) layered_mixture<T>(static_cast<int>(i), lp, s);
        if (layer_capture_ != nullptr) {
            CUDA_CHECK(cudaMemcpy2DAsync(layer_capture_ + i * static_cast<size_t>(rows) * W, static_cast<size_t>(W) * 4, x32_,
                                         static_cast<size_t>(L) * 4, static_cast<size_t>(W) * 4, rows, cudaMemcpyDeviceToDevice, s));
        }
    }
}

template <typename T>
void Engine::layered_logits(const int32_t* rows_idx, int n, void* out, cudaStream_t s) {
    const int L = ld(), V = mc_.vocab;
    launch_norm_rows<T>(x32_, rows_idx, final_norm_, static_cast<T*>(lnorm_), n, mc_.hidden, L, mc_.eps, s);
    if constexpr (sizeof(T) == 2) {
        LinearPlan p = make_linear_plan(static_cast<const bf16*>(lnorm_), n, lm_head_, n, V, L, static_cast<bf16*>(out), V, nullptr, gemm_ws_,
                                        tickets_, runtime().num_sms);
        CPM_REQUIRE(2LL * ceil_div(p.N, 128) * ceil_div(p.M, p.mt) <= kTicketInts, "linear: more output tiles than the split-K counters cover");
        launch_linear(p, s);
    } else {
        launch_linear_f32(static_cast<const float*>(lnorm_), L, lm_head_, 0, static_cast<float*>(out), V, n, V, L, nullptr, nullptr, 0, false, s);
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
    check_errors("prefill");
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
    check_errors("decode");
}
