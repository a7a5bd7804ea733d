"""Prefill and decode throughput of a layered design beside the Llama-format model of equal size (`bench.py --model tipetar`,
`--model fabulix`).

Three sizes with the layer shapes of real models, few layers, random weights.  The Llama-format model has the same width,
layers, vocabulary and attention width, and as much feed-forward width as gives both the same matrix work per token (Tipetar:
chosen experts + shared expert).  For each size and model:

  prefill   4096 tokens in one chunk: host clock around LLM.prefill after a warm-up pass, best of three
  decode    one token at a time behind those 4096: host clock around LLM.decode (median step), and the engine's device time
  kernels   CUDA events around every launch of one more pass, summed per class, as a fraction of the roofline: weight
            (or K/V, or state) bytes at the measured HBM bandwidth for decode; for prefill FLOPs at the measured bf16 peak,
            for recurrences fp32 FLOPs at the nominal peak of the fp32 pipes, for row kernels bytes

One JSON line.
"""
import json
import os
import statistics
import time
import types

CONTEXT = 4096
VOCAB = 32768


def _moe(experts, top, ff, identity, groups, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "top": top, "identity": identity, "groups": {"count": groups[0], "keep": groups[1]},
                       "scale": 2.0}}


def _model(width, heads, kv_heads, dim, window, layers, mlp):
    out = []
    for i in range(layers):
        mix = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": window}}
        if i >= layers // 2:                     # the second half of the layers shares one cache
            mix["kv_from"] = layers // 2 - 1
        out.append({"type": "attention", "mixer": mix, "mlp": mlp})
    return {"architecture": "Tipetar", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-5}, "residual_mult": 0.5, "layers": out}


TIPETAR_SIZES = {
    "2k": _model(2048, 16, 4, 128, 1024, 8, _moe(60, 6, 1024, 4, (8, 4), 2048)),
    "4k": _model(4096, 32, 8, 128, 2048, 6, _moe(30, 4, 2048, 2, (4, 3), 4096)),
    "3k-narrow": _model(3072, 48, 6, 64, 4096, 8, _moe(14, 2, 4096, 2, (4, 3), 2048)),
}


def _fabulix(width, left, right, light, ff, side, layers):
    """left: (heads, kv heads, head width), right and light: (heads, head width); every third layer is a lightning layer without
    feed-forward."""
    out = []
    for i in range(layers):
        if i % 3 == 0:
            mix = {"heads": light[0], "dim": light[1], "vdim": light[1], "decay": [0.9 + 0.099 * h / light[0] for h in range(light[0])]}
            out.append({"type": "lightning", "mixer": mix, "mlp": None})
            continue
        h, g, d = left
        mix = {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": d, "scale": d ** -0.5, "rot": {"base": 500000.0, "dims": d}},
               "right": {"heads": right[0], "dim": right[1]}, "left_scale": 0.7, "right_scale": 0.6}
        out.append({"type": "parallel", "mixer": mix, "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}})
    return {"architecture": "Fabulix", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
            "token_side": {"dim": side}, "layers": out}


FABULIX_SIZES = {
    "2k": _fabulix(2048, (16, 4, 128), (32, 64), (16, 128), 5632, 128, 9),
    "4k": _fabulix(4096, (32, 8, 128), (64, 64), (32, 128), 11008, 256, 6),
    "3k-narrow": _fabulix(3072, (48, 12, 64), (48, 64), (24, 128), 8192, 192, 9),
}
DECAY_RANK = 64
FP32_FLOPS = 148 * 128 * 2 * 1.965e9   # nominal: SMs x lanes x fused multiply-add x clock


def fabulix_layer(cfg, layer):
    """(multiply-adds of the matrix products, recurrence (heads, key, value width), elements row kernels move) of a token."""
    W, s, m = cfg["width"], cfg["token_side"]["dim"], layer["mixer"]
    n, f = 2 * W * s, layer["mlp"]
    if f:
        n += 3 * W * f["ff"]
    if layer["type"] == "lightning":
        nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        return n + W * (2 * nk + 3 * nv), (m["heads"], m["dim"], m["vdim"])
    a, r = m["left"], m["right"]
    nr = r["heads"] * r["dim"]
    n += W * (a["heads"] * (a["dim"] + a["vdim"]) + a["kv_heads"] * (a["dim"] + a["vdim"])) + 5 * W * nr + DECAY_RANK * (W + nr)
    return n, (r["heads"], r["dim"], r["dim"])


def llama_shape(design, cfg):
    """(attention heads of 128, key heads, feed-forward width) of the Llama-format model of equal size."""
    if design == "tipetar":
        m, r = cfg["layers"][0]["mixer"], cfg["layers"][0]["mlp"]
        ff = r["router"]["top"] * r["expert"]["ff"] + r["shared"]["ff"]
    else:
        m = cfg["layers"][1]["mixer"]["left"]
    hq, hkv = m["heads"] * m["dim"] // 128, max(1, m["kv_heads"] * m["dim"] // 128)    # 128-wide heads only
    if design == "fabulix":
        W, L = cfg["width"], len(cfg["layers"])
        total = sum(fabulix_layer(cfg, x)[0] for x in cfg["layers"])
        ff = round((total / L - W * 128 * (2 * hq + 2 * hkv)) / (3 * W) / 128) * 128
    return hq, hkv, ff


def _attention_work(rows, context, heads, kv_heads, dim, window):
    pairs = sum(min(window, context - rows + r + 1) for r in range(rows))
    return 2 * min(window, context) * kv_heads * dim * 2, 4 * pairs * heads * dim


def bytes_and_flops(design, cfg, kind, rows, context):
    """(decode bytes, prefill FLOPs) per kernel class of one pass of `rows` tokens behind context - rows others."""
    W, V = cfg["width"], cfg["vocab"]
    lin = experts = kv = att = scan = state = 0
    for layer in cfg["layers"]:
        m, f = layer["mixer"], layer["mlp"]
        if kind == "llama":
            hq, hkv, ff = llama_shape(design, cfg)
            lin += W * 128 * (2 * hq + 2 * hkv) + 3 * W * ff
            work = _attention_work(rows, context, hq, hkv, 128, context)
        elif kind == "tipetar":
            h, g, d = m["heads"], m["kv_heads"], m["dim"]
            lin += W * h * d * 2 + (2 * g * d * W if m.get("kv_from") is None else 0)
            experts += 3 * W * llama_shape(design, cfg)[2]
            work = _attention_work(rows, context, h, g, d, m["mask"]["size"])
        else:
            n, (h, dk, dv) = fabulix_layer(cfg, layer)
            lin += n
            scan += 5 * h * dk * dv          # S = w S + k v: three, o += r S: two
            state += 2 * 4 * h * dk * dv
            a = m.get("left")
            work = _attention_work(rows, context, a["heads"], a["kv_heads"], a["dim"], context) if a else (0, 0)
        kv, att = kv + work[0], att + work[1]
    return ({"linear": 2 * (lin + V * W), "experts": 2 * experts, "attention": kv, "scan": state},
            {"linear": 2 * rows * lin + 2 * V * W, "experts": 2 * rows * experts, "attention": att, "scan": rows * scan})


def weights_tipetar(cfg, seed=1):
    import torch
    g = torch.Generator(device="cuda").manual_seed(seed)
    W = cfg["width"]

    def mat(*shape, std=None):
        return (torch.randn(*shape, device="cuda", generator=g) * (std or shape[-1] ** -0.5)).to(torch.bfloat16)

    yield "embed", mat(VOCAB, W, std=1.0)
    yield "head", mat(VOCAB, W)
    yield "final.norm", mat(W, std=0.1)
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        yield p + "mix.q", mat(m["heads"] * m["dim"], W)
        yield p + "mix.q.norm", 1 + mat(m["heads"] * m["dim"], std=0.1)
        if m.get("kv_from") is None:
            yield p + "mix.k", mat(m["kv_heads"] * m["dim"], W)
            yield p + "mix.k.norm", 1 + mat(m["kv_heads"] * m["dim"], std=0.1)
            yield p + "mix.v", mat(m["kv_heads"] * m["vdim"], W)
        yield p + "mix.o", mat(W, m["heads"] * m["vdim"])
        yield p + "norm1", mat(W, std=0.1)
        yield p + "norm2", mat(W, std=0.1)
        n = f["router"]["experts"] + f["router"]["identity"]
        yield p + "mlp.router", mat(n, W)
        yield p + "mlp.correction", mat(n, std=0.01)
        for e in range(f["router"]["experts"]):
            for part, shape in (("gate", (f["expert"]["ff"], W)), ("up", (f["expert"]["ff"], W)), ("down", (W, f["expert"]["ff"]))):
                yield f"{p}mlp.e{e}.{part}", mat(*shape)
        for part, shape in (("gate", (f["shared"]["ff"], W)), ("up", (f["shared"]["ff"], W)), ("down", (W, f["shared"]["ff"]))):
            yield f"{p}mlp.shared.{part}", mat(*shape)


def weights_fabulix(cfg, seed=1):
    import torch
    g = torch.Generator(device="cuda").manual_seed(seed)
    W, side = cfg["width"], cfg["token_side"]["dim"]

    def mat(*shape, std=None, mean=0.0):
        return (torch.randn(*shape, device="cuda", generator=g) * (std or shape[-1] ** -0.5) + mean).to(torch.bfloat16)

    def norm(name):
        yield name, mat(W, std=0.1, mean=1.0)
        yield name + ".b", mat(W, std=0.1)
        yield name + ".alpha", torch.tensor(0.5, dtype=torch.bfloat16, device="cuda")

    yield "embed", mat(VOCAB, W, std=1.0)
    yield "side.embed", mat(VOCAB, len(cfg["layers"]) * side, std=1.0)
    yield from norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        yield from norm(p + "norm1")
        yield from norm(p + "norm1b")
        if layer["type"] == "lightning":
            nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", nk), ("k", nk), ("v", nv), ("g", nv)):
                yield f"{p}mix.{n}", mat(rows, W)
            yield p + "mix.o", mat(W, nv)
            yield p + "mix.norm", mat(nv, std=0.1, mean=1.0)
        else:
            a, r = m["left"], m["right"]
            nr = r["heads"] * r["dim"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                yield f"{p}mix.left.{n}", mat(rows, W)
            yield p + "mix.left.o", mat(W, a["heads"] * a["vdim"])
            for n in "rkvg":
                yield f"{p}mix.right.{n}", mat(nr, W)
            for n in "rkvgw":
                yield f"{p}mix.right.mu.{n}", mat(W, std=0.2, mean=0.5)
            yield p + "mix.right.w1", mat(DECAY_RANK, W)
            yield p + "mix.right.w2", mat(nr, DECAY_RANK)
            yield p + "mix.right.w0", mat(nr, std=1.0, mean=-3.0)
            yield p + "mix.right.u", mat(r["heads"], r["dim"], std=0.3)
            yield p + "mix.right.norm", mat(nr, std=0.1, mean=1.0)
            yield p + "mix.right.o", mat(W, nr)
        f = layer["mlp"]
        if f:
            yield from norm(p + "norm2")
            yield from norm(p + "norm2b")
            yield p + "mlp.gate", mat(f["ff"], W)
            yield p + "mlp.up", mat(f["ff"], W)
            yield p + "mlp.down", mat(W, f["ff"])
        yield p + "side.gate", mat(side, W)
        yield p + "side.proj", mat(W, side)
        yield p + "side.norm", mat(W, std=0.1, mean=0.2)


def open_design(design, cfg):
    import torch
    from cpmcu.fabulix import FabulixLLM
    from cpmcu.tipetar import TipetarLLM
    kw = dict(config=cfg, dtype=torch.bfloat16, chunk_length=CONTEXT, memory_limit=0.7)
    if design == "tipetar":
        llm, weights = TipetarLLM(**kw), weights_tipetar
    else:
        ranks = {f"l{i}.mix.right.w1": (DECAY_RANK, cfg["width"]) for i in range(len(cfg["layers"]))}
        llm, weights = FabulixLLM(shapes=ranks, **kw), weights_fabulix
    llm.init_storage()
    for name, t in weights(cfg):
        llm._load(name, t)
    return llm


def open_llama(design, cfg):
    import torch
    from cpmcu.llm import LLM
    W = cfg["width"]
    hq, hkv, I = llama_shape(design, cfg)
    hf = types.SimpleNamespace(vocab_size=VOCAB, num_hidden_layers=len(cfg["layers"]), hidden_size=W, intermediate_size=I,
                               num_attention_heads=hq, num_key_value_heads=hkv, head_dim=128, rms_norm_eps=1e-5,
                               rope_theta=10000.0, torch_dtype=torch.bfloat16)
    llm = LLM(None, config=hf, dtype=torch.bfloat16, chunk_length=CONTEXT, memory_limit=0.7)
    llm.init_storage()
    g = torch.Generator(device="cuda").manual_seed(1)

    def mat(*shape):
        return (torch.randn(*shape, device="cuda", generator=g) * 0.02).to(torch.bfloat16)

    ones = torch.ones(W, device="cuda", dtype=torch.bfloat16)
    llm._load("model.embed_tokens.weight", mat(VOCAB, W))
    llm._load("lm_head.weight", mat(VOCAB, W))
    llm._load("model.norm.weight", ones)
    for i in range(len(cfg["layers"])):
        p = f"model.layers.{i}."
        for n, shape in (("self_attn.q_proj", (hq * 128, W)), ("self_attn.k_proj", (hkv * 128, W)), ("self_attn.v_proj", (hkv * 128, W)),
                         ("self_attn.o_proj", (W, hq * 128)), ("mlp.gate_proj", (I, W)), ("mlp.up_proj", (I, W)), ("mlp.down_proj", (W, I))):
            llm._load(p + n + ".weight", mat(*shape))
        llm._load(p + "input_layernorm.weight", ones)
        llm._load(p + "post_attention_layernorm.weight", ones)
    llm._load("model.rotary_emb.inv_freq", llm._rope_inv_freq(), dtype=torch.float32)
    return llm


def measure(llm, design, cfg, kind, steps, peaks):
    import torch
    import cpmcu.C as C
    ids = torch.randint(0, VOCAB, (CONTEXT,), dtype=torch.int32, device="cuda", generator=torch.Generator(device="cuda").manual_seed(3))
    pos = torch.arange(CONTEXT, dtype=torch.int32, device="cuda")
    runs = []
    for _ in range(4):
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        llm.prefill(ids, pos)
        torch.cuda.synchronize()
        runs.append(time.perf_counter() - t0)
    prefill_s = min(runs[1:])
    C.profile(True)
    llm.prefill(ids, pos)
    pre = C.profile(False)
    tok, wall, dev = 1, [], []
    for i in range(steps + 4):
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        llm._decode_one(tok + i, CONTEXT + i)
        torch.cuda.synchronize()
        wall.append(time.perf_counter() - t0)
        dev.append(C.last_step_ms())
    C.profile(True)
    for i in range(4):
        llm._decode_one(tok + i, CONTEXT + steps + 4 + i)
    dec = {k: (v[0] / 4, v[1] // 4) for k, v in C.profile(False).items()}
    nbytes, _ = bytes_and_flops(design, cfg, kind, 1, CONTEXT + steps)
    _, flops = bytes_and_flops(design, cfg, kind, CONTEXT, CONTEXT)
    hbm, tf = peaks

    def frac(times, amount, peak, scan_peak):
        return {k: {"ms": round(times[k][0], 4), "launches": times[k][1],
                    "of_peak": round(amount[k] / (times[k][0] * 1e-3) / (scan_peak if k == "scan" else peak), 3) if amount.get(k) else None}
                for k in times if times[k][1]}

    out = {"prefill_tokens_per_s": round(CONTEXT / prefill_s), "prefill_ms": round(prefill_s * 1e3, 3),
           "decode_tokens_per_s": round(1 / statistics.median(wall[4:]), 1), "decode_ms": round(1e3 * statistics.median(wall[4:]), 4),
           "prefill_kernels": frac(pre, flops, tf * 1e12, FP32_FLOPS),
           "decode_kernels": frac(dec, nbytes, hbm * 1e9, hbm * 1e9)}
    if kind != "llama":
        out["decode_device_ms"] = round(statistics.median(dev[4:]), 4)
    return out


def run(args, sampler_cls, peaks):
    import torch
    import cpmcu.C as C
    os.environ["CPMCU_MAX_TOKENS"] = str(CONTEXT + 1024)
    sampler = sampler_cls(0)
    sampler.start()
    sizes, design = {}, args.model
    configs = {"tipetar": TIPETAR_SIZES, "fabulix": FABULIX_SIZES}[design]
    for name in args.sizes.split(",") if args.sizes else configs:
        cfg = configs[name]
        sizes[name] = {"width": cfg["width"], "layers": len(cfg["layers"]), "llama_ff": llama_shape(design, cfg)[2]}
        for kind, opener in ((design, open_design), ("llama", open_llama)):
            llm = opener(design, cfg)
            torch.cuda.empty_cache()
            sizes[name][kind] = measure(llm, design, cfg, kind, args.steps, peaks)
            C.release()
    sampler.stop_flag.set()
    sampler.join(timeout=2)
    first = next(iter(sizes.values()))[design]
    print(json.dumps({"metric": "decode_tokens_per_s", "value": first["decode_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1,
                      "steps": args.steps, "higher_is_better": True, "dtype": "bf16", "data": "synthetic",
                      "config": {"model": design.capitalize(), "context": CONTEXT, "batch": 1}, "clocks": sampler.summary(), "sizes": sizes,
                      "gpu_launches": int(C.total_launches())}), flush=True)
