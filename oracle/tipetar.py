"""Plain implementation of the Tipetar design: the slow, obvious form of every mechanism, one function each, for the
parity tests.  Everything runs in the dtype of the tensors it is given (float64 for a sharp reference).  Nothing here
is used by the product.

The model (x: residual stream, all positions of one sequence at once):

    x   = embed[token]
    x  += m * rms(mixer(x)) * (1 + w1)          per layer; the sublayers read x itself, the norm is on their output
    x  += m * rms(ff(x)) * (1 + w2)
    out = head @ (rms(x) * (1 + wf))

`config` is the parsed config.json of a model, `weights` a mapping name -> tensor.
"""
import torch
import torch.nn.functional as F


# ---------------------------------------------------------------- norms
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_one(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


# ---------------------------------------------------------------- attention
def distance_slopes(heads, dtype=torch.float64):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=dtype)


def window_mask(rows, keys, first_row, size):
    """[rows, keys] booleans: query first_row + r may see key c.  size None: every key up to the query."""
    i = torch.arange(first_row, first_row + rows)[:, None]
    j = torch.arange(keys)[None, :]
    seen = j <= i
    if size is not None:
        seen &= (i - j) < size
    return seen


def attention(q, k, v, scale, size, first_row=0):
    """q [rows, H, d] at positions first_row ..; k [keys, G, d], v [keys, G, dv] from position 0.  Returns [rows, H * dv]."""
    rows, H, _ = q.shape
    keys, G, dv = v.shape
    slopes = distance_slopes(H, q.dtype)
    seen = window_mask(rows, keys, first_row, size)
    i = torch.arange(first_row, first_row + rows)[:, None]
    dist = (i - torch.arange(keys)[None, :]).to(q.dtype)
    out = []
    for h in range(H):
        g = h // (H // G)
        score = (q[:, h] @ k[:, g].T) * scale - slopes[h] * dist
        score = score.masked_fill(~seen, float("-inf"))
        out.append(torch.softmax(score, dim=-1) @ v[:, g])
    return torch.cat(out, dim=-1)


def project_queries(x, mix, w, p, eps):
    q = norm_plain(x @ w[p + ".q"].T, w[p + ".q.norm"], eps)
    return q.view(x.shape[0], mix["heads"], mix["dim"])


def project_keys_values(x, mix, w, p, eps):
    k = norm_plain(x @ w[p + ".k"].T, w[p + ".k.norm"], eps)
    v = x @ w[p + ".v"].T
    return k.view(x.shape[0], mix["kv_heads"], mix["dim"]), v.view(x.shape[0], mix["kv_heads"], mix["vdim"])


def mask_size(mix):
    return (mix.get("mask") or {}).get("size")


# ---------------------------------------------------------------- mixture of experts
def gated(x, w, p):
    """One feed-forward: W_down(silu(W_gate x) * W_up x)."""
    g = x @ w[p + ".gate"].T
    return (F.silu(g) * (x @ w[p + ".up"].T)) @ w[p + ".down"].T


def route(logits, correction, router):
    """(indices [rows, top], weights [rows, top]) of the chosen experts."""
    s = torch.softmax(logits, dim=-1)
    choice = s if correction is None else s + correction
    n = s.shape[-1]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    per = n // groups["count"]
    best = choice.view(-1, groups["count"], per).max(dim=-1).values
    keep = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(groups["keep"], dim=-1).indices, True)
    choice = choice.masked_fill(~keep.repeat_interleave(per, dim=1), float("-inf"))
    idx = choice.topk(router["top"], dim=-1).indices
    wt = s.gather(1, idx)
    wt = wt / (wt.sum(dim=-1, keepdim=True) + 1e-20) * router["scale"]
    return idx, wt


def choice_margin(logits, correction, router):
    """[rows]: how far the closest call among a row's choices (of groups, then of experts) is from going the other way, as
    the gap of the two choice scores over the sum of their scores s (and a thousandth of the choice score, whose own last
    bits count when s is tiny).  Rounding moves s by a small fraction of itself, so rows with a small margin may choose
    differently in low precision."""
    s = torch.softmax(logits, dim=-1)
    choice = s if correction is None else s + correction
    n = s.shape[-1]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    per = n // groups["count"]

    def gap(values, scores, k):
        if k >= values.shape[-1]:
            return torch.full(values.shape[:1], float("inf"), dtype=values.dtype)
        top = values.topk(k + 1, dim=-1)
        at = top.indices[:, k - 1:k + 1]
        return (top.values[:, k - 1] - top.values[:, k]) / (scores.gather(1, at).sum(-1) + 1e-3 * top.values[:, k].abs())

    best = choice.view(-1, groups["count"], per).max(dim=-1)
    best_s = s.view(-1, groups["count"], per).gather(2, best.indices[..., None]).squeeze(-1)
    margin = gap(best.values, best_s, groups["keep"])
    keep = torch.zeros_like(best_s, dtype=torch.bool).scatter_(1, best.values.topk(groups["keep"], dim=-1).indices, True)
    masked = choice.masked_fill(~keep.repeat_interleave(per, dim=1), -1e30)
    return torch.minimum(margin, gap(masked, s, router["top"]))


def mixture(x, mlp, w, p, margins_out=None):
    router = mlp["router"]
    logits = x @ w[p + ".router"].T
    idx, wt = route(logits, w.get(p + ".correction"), router)
    if margins_out is not None:
        margins_out.append(choice_margin(logits, w.get(p + ".correction"), router))
    out = torch.zeros_like(x)
    for e in range(router["experts"]):
        rows, slot = (idx == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += wt[rows, slot, None] * gated(x[rows], w, f"{p}.e{e}")
    # identity experts hand the input on
    out += x * (wt * (idx >= router["experts"])).sum(dim=-1, keepdim=True)
    if mlp.get("shared"):
        out += gated(x, w, p + ".shared")
    return out


# ---------------------------------------------------------------- the model
class Sequence:
    """Keys and values of one sequence, per layer that has its own."""

    def __init__(self):
        self.length = 0
        self.kv = {}


def forward(config, weights, tokens, seq=None, layers_out=None, margins_out=None):
    """Logits [len(tokens), vocab] of the next tokens of `seq` (a fresh sequence when None).  layers_out receives the stream
    after every layer, margins_out the choice margins of every mixture."""
    seq = seq if seq is not None else Sequence()
    w, eps, m = weights, config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        mix, p = layer["mixer"], f"l{i}"
        q = project_queries(x, mix, w, p + ".mix", eps)
        src = mix.get("kv_from")
        if src is None:
            k, v = project_keys_values(x, mix, w, p + ".mix", eps)
            if seq.length:
                k, v = torch.cat([seq.kv[i][0], k]), torch.cat([seq.kv[i][1], v])
            seq.kv[i] = (k, v)
        k, v = seq.kv[i if src is None else src]
        a = attention(q, k, v, mix["scale"], mask_size(mix), seq.length)
        x = x + m * norm_around_one(a @ w[p + ".mix.o"].T, w[p + ".norm1"], eps)
        if layer.get("mlp"):
            x = x + m * norm_around_one(mixture(x, layer["mlp"], w, p + ".mlp", margins_out), w[p + ".norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    seq.length += len(tokens)
    return norm_around_one(x, w["final.norm"], eps) @ w["head"].T


def greedy(config, weights, prompt, count):
    """`count` greedy tokens after `prompt`, recomputing everything each time (no cache)."""
    seq = list(prompt)
    for _ in range(count):
        seq.append(int(forward(config, weights, seq)[-1].argmax()))
    return seq[len(prompt):]


# ---------------------------------------------------------------- models for tests
def random_weights(config, seed=0, gain=1.0, dtype=torch.float64):
    """Seeded weights of every tensor the configuration needs, rounded to bfloat16 values."""
    g = torch.Generator().manual_seed(seed)
    H = config["width"]

    def mat(*shape, std=None):
        t = torch.randn(*shape, generator=g) * (std if std is not None else gain / shape[-1] ** 0.5)
        return t.to(torch.bfloat16)

    w = {"embed": mat(config["vocab"], H, std=1.0), "head": mat(config["vocab"], H), "final.norm": mat(H, std=0.2)}
    for i, layer in enumerate(config["layers"]):
        mix, p = layer["mixer"], f"l{i}"
        nq, nk, nv = mix["heads"] * mix["dim"], mix["kv_heads"] * mix["dim"], mix["kv_heads"] * mix["vdim"]
        w[p + ".mix.q"], w[p + ".mix.q.norm"] = mat(nq, H), (1 + mat(nq, std=0.2).float()).to(torch.bfloat16)
        if mix.get("kv_from") is None:
            w[p + ".mix.k"], w[p + ".mix.k.norm"] = mat(nk, H), (1 + mat(nk, std=0.2).float()).to(torch.bfloat16)
            w[p + ".mix.v"] = mat(nv, H)
        w[p + ".mix.o"] = mat(H, mix["heads"] * mix["vdim"])
        w[p + ".norm1"] = mat(H, std=0.2)
        if layer.get("mlp"):
            w[p + ".norm2"] = mat(H, std=0.2)
            mlp, r = layer["mlp"], layer["mlp"]["router"]
            n = r["experts"] + (r.get("identity") or 0)
            w[p + ".mlp.router"] = mat(n, H, std=2.0 / H ** 0.5)
            w[p + ".mlp.correction"] = mat(n, std=0.1)
            widths = {f"e{e}": mlp["expert"]["ff"] for e in range(r["experts"])}
            if mlp.get("shared"):
                widths["shared"] = mlp["shared"]["ff"]
            for name, ff in widths.items():
                w[f"{p}.mlp.{name}.gate"], w[f"{p}.mlp.{name}.up"] = mat(ff, H), mat(ff, H)
                w[f"{p}.mlp.{name}.down"] = mat(H, ff)
    return {k: v.to(dtype) for k, v in w.items()}
