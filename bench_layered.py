"""Prefill and decode throughput of a Tipetar model beside the Llama-format model of equal size (`bench.py --model tipetar`).

Three sizes with the layer shapes of real models, few layers, random weights.  The Llama-format model has the same width,
layers, vocabulary and attention width, and the feed-forward width a token of the mixture uses (chosen experts + shared
expert), so both do about the same work per token.  For each size and model:

  prefill   4096 tokens in one chunk: host clock around LLM.prefill after a warm-up pass, best of three
  decode    one token at a time behind those 4096: host clock around LLM.decode (median step), and the engine's device time
  kernels   CUDA events around every launch of one more pass, summed per class, as a fraction of the roofline: weight
            (or K/V) bytes at the measured HBM bandwidth for decode, FLOPs at the measured bf16 peak for prefill

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


SIZES = {
    "2k": _model(2048, 16, 4, 128, 1024, 8, _moe(60, 6, 1024, 4, (8, 4), 2048)),
    "4k": _model(4096, 32, 8, 128, 2048, 6, _moe(30, 4, 2048, 2, (4, 3), 4096)),
    "3k-narrow": _model(3072, 48, 6, 64, 4096, 8, _moe(14, 2, 4096, 2, (4, 3), 2048)),
}


def active_ff(cfg):
    """Feed-forward width of the Llama-format model: what a token's experts add up to."""
    r = cfg["layers"][0]["mlp"]
    return r["router"]["top"] * r["expert"]["ff"] + r["shared"]["ff"]


def bytes_and_flops(cfg, kind, rows, context):
    """(decode bytes, prefill FLOPs) per kernel class of one pass of `rows` tokens behind context - rows others."""
    W, V, L = cfg["width"], cfg["vocab"], len(cfg["layers"])
    lin = experts = kv = att = 0
    for layer in cfg["layers"]:
        m, f = layer["mixer"], layer["mlp"]
        h, g, d = m["heads"], m["kv_heads"], m["dim"]
        own = m.get("kv_from") is None or kind == "llama"
        lin += W * h * d * 2 + (2 * g * d * W if own else 0)
        win = m["mask"]["size"] if kind == "tipetar" else context
        kv += 2 * min(win, context) * g * d * 2
        pairs = sum(min(win, context - rows + r + 1) for r in range(rows))
        att += 4 * pairs * h * d
        n = 3 * W * active_ff(cfg)
        if kind == "tipetar":
            experts += n
        else:
            lin += n
    return ({"linear": 2 * (lin + V * W), "experts": 2 * experts, "attention": kv},
            {"linear": 2 * rows * lin + 2 * V * W, "experts": 2 * rows * experts, "attention": att})


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


def open_tipetar(cfg):
    import torch
    from cpmcu.tipetar import TipetarLLM
    llm = TipetarLLM(config=cfg, dtype=torch.bfloat16, chunk_length=CONTEXT, memory_limit=0.7)
    llm.init_storage()
    for name, t in weights_tipetar(cfg):
        llm._load(name, t)
    return llm


def open_llama(cfg):
    import torch
    from cpmcu.llm import LLM
    W, I = cfg["width"], active_ff(cfg)
    m = cfg["layers"][0]["mixer"]
    hq, hkv = m["heads"] * m["dim"] // 128, max(1, m["kv_heads"] * m["dim"] // 128)    # 128-wide heads only
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


def measure(llm, cfg, kind, steps, peaks):
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
    nbytes, _ = bytes_and_flops(cfg, kind, 1, CONTEXT + steps)
    _, flops = bytes_and_flops(cfg, kind, CONTEXT, CONTEXT)
    hbm, tf = peaks

    def frac(times, amount, peak):
        return {k: {"ms": round(times[k][0], 4), "launches": times[k][1],
                    "of_measured": round(amount[k] / (times[k][0] * 1e-3) / peak, 3) if amount.get(k) else None}
                for k in times if times[k][1]}

    out = {"prefill_tokens_per_s": round(CONTEXT / prefill_s), "prefill_ms": round(prefill_s * 1e3, 3),
           "decode_tokens_per_s": round(1 / statistics.median(wall[4:]), 1), "decode_ms": round(1e3 * statistics.median(wall[4:]), 4),
           "prefill_kernels": frac(pre, flops, tf * 1e12), "decode_kernels": frac(dec, nbytes, hbm * 1e9)}
    if kind == "tipetar":
        out["decode_device_ms"] = round(statistics.median(dev[4:]), 4)
    return out


def run(args, sampler_cls, peaks):
    import torch
    import cpmcu.C as C
    os.environ["CPMCU_MAX_TOKENS"] = str(CONTEXT + 1024)
    sampler = sampler_cls(0)
    sampler.start()
    sizes = {}
    for name in args.sizes.split(",") if args.sizes else SIZES:
        cfg = SIZES[name]
        sizes[name] = {"width": cfg["width"], "layers": len(cfg["layers"]), "active_ff": active_ff(cfg)}
        for kind, opener in (("tipetar", open_tipetar), ("llama", open_llama)):
            llm = opener(cfg)
            torch.cuda.empty_cache()
            sizes[name][kind] = measure(llm, cfg, kind, args.steps, peaks)
            C.release()
    sampler.stop_flag.set()
    sampler.join(timeout=2)
    first = next(iter(sizes.values()))["tipetar"]
    print(json.dumps({"metric": "decode_tokens_per_s", "value": first["decode_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1,
                      "steps": args.steps, "higher_is_better": True, "dtype": "bf16", "data": "synthetic",
                      "config": {"model": "Tipetar", "context": CONTEXT, "batch": 1}, "clocks": sampler.summary(), "sizes": sizes,
                      "gpu_launches": int(C.total_launches())}), flush=True)
