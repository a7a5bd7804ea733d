"""Plain implementation of the Fabulix design: the slow, obvious form of every mechanism, one function each, for the
parity tests.  Everything runs in the dtype of the tensors it is given (float64 for a sharp reference), recurrences token
by token.  Nothing here is used by the product.

The model (x: residual stream, all positions of one portion of a sequence at once; N: dynamic tanh with its own weights):

    x   = embed[token] * c
    x  += N1b(mixer(N1(x)));  x += N2b(ff(N2(x)));  x += rms(P (gelu(G x) * e[token, layer])) * w      per layer
    out = embed @ Nf(x)

`config` is the parsed config.json of a model, `weights` a mapping name -> tensor.
"""
import math

import torch


# ---------------------------------------------------------------- elementwise
def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def norm(x, weights, name):
    return dynamic_tanh(x, weights[name + ".alpha"], weights[name], weights[name + ".b"])


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


# ---------------------------------------------------------------- softmax attention with rotation and a sink
def rotate(x, first, dims, base):
    """x [rows, heads, d] at positions first ..: dimensions i and i + dims / 2 turn by position * base^(-2 i / dims)."""
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = torch.arange(first, first + x.shape[0], dtype=x.dtype)[:, None, None] * freq
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([u * angle.cos() - v * angle.sin(), v * angle.cos() + u * angle.sin(), rest], dim=-1)


def sink_softmax(score):
    """exp(s_j) / (1 + sum_j exp(s_j)): one more score of 0 that has no value."""
    top = score.max(dim=-1, keepdim=True).values.clamp_min(0)
    e = torch.exp(score - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def attention(q, k, v, scale, first=0):
    """q [rows, H, d] at positions first ..; k [keys, G, d], v [keys, G, dv] from position 0.  Returns [rows, H * dv]."""
    rows, H, _ = q.shape
    keys, G, _ = v.shape
    seen = torch.arange(keys)[None, :] <= torch.arange(first, first + rows)[:, None]
    out = []
    for h in range(H):
        g = h // (H // G)
        score = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, float("-inf"))
        out.append(sink_softmax(score) @ v[:, g])
    return torch.cat(out, dim=-1)


def softmax_mixer(h, mix, w, p, state):
    rows, first = h.shape[0], state.tokens
    H, G, d, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    turn = (lambda x: rotate(x, first, mix["rot"]["dims"], mix["rot"]["base"])) if mix.get("rot") else (lambda x: x)
    q = turn((h @ w[p + ".q"].T).view(rows, H, d))
    k = turn((h @ w[p + ".k"].T).view(rows, G, d))
    v = (h @ w[p + ".v"].T).view(rows, G, dv)
    k, v = state.append(p, k, v)
    return attention(q, k, v, mix["scale"], first) @ w[p + ".o"].T


# ---------------------------------------------------------------- recurrences
def time_mix_scan(r, k, v, decay, bonus, S):
    """r, k, decay [rows, H, d], v [rows, H, dv], bonus [H, d], S [H, d, dv].  Returns outputs [rows, H, dv] and the state."""
    out = []
    for t in range(r.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append((r[t][:, :, None] * (S + bonus[:, :, None] * kv)).sum(dim=1))
        S = decay[t][:, :, None] * S + kv
    return torch.stack(out), S


def log_log_decay(mixed, w, p):
    return torch.tanh(mixed @ w[p + ".w1"].T) @ w[p + ".w2"].T + w[p + ".w0"]


def time_mixer(h, mix, w, p, state, eps):
    rows, H, d = h.shape[0], mix["heads"], mix["dim"]
    before = torch.cat([state.get(p + ".h", torch.zeros_like(h[:1])), h[:-1]])
    m = {s: h + (before - h) * w[p + ".mu." + s] for s in "rkvgw"}
    r, k, v = ((m[s] @ w[p + "." + s].T).view(rows, H, d) for s in "rkv")
    gate = silu(m["g"] @ w[p + ".g"].T)
    decay = torch.exp(-torch.exp(log_log_decay(m["w"], w, p))).view(rows, H, d)
    o, S = time_mix_scan(r, k, v, decay, w[p + ".u"], state.get(p + ".S", torch.zeros(H, d, d, dtype=h.dtype)))
    state.put(p + ".h", h[-1:])
    state.put(p + ".S", S)
    return (unit_rms(o, eps).reshape(rows, H * d) * w[p + ".norm"] * gate) @ w[p + ".o"].T


def constant_decay_scan(q, k, v, decay, S):
    """q, k [rows, H, d], v [rows, H, dv], decay [H], S [H, d, dv]: the current token is in the state it reads."""
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((q[t][:, :, None] * S).sum(dim=1))
    return torch.stack(out), S


def lightning_mixer(h, mix, w, p, state, eps):
    rows, H, d, dv = h.shape[0], mix["heads"], mix["dim"], mix["vdim"]
    q, k, v = (silu(h @ w[p + "." + s].T).view(rows, H, n) for s, n in (("q", d), ("k", d), ("v", dv)))
    decay = torch.tensor(mix["decay"], dtype=h.dtype)
    o, S = constant_decay_scan(q, k, v, decay, state.get(p + ".S", torch.zeros(H, d, dv, dtype=h.dtype)))
    state.put(p + ".S", S)
    return (unit_rms(o.reshape(rows, H * dv), eps) * w[p + ".norm"] / (1 + torch.exp(-(h @ w[p + ".g"].T)))) @ w[p + ".o"].T


def parallel_mixer(h, mix, w, p, state, eps):
    left = softmax_mixer(h, mix["left"], w, p + ".left", state)
    right = time_mixer(h, mix["right"], w, p + ".right", state, eps)
    return mix["left_scale"] * left + mix["right_scale"] * right


MIXERS = {"parallel": parallel_mixer, "lightning": lightning_mixer}


# ---------------------------------------------------------------- feed-forward, token side input
def clamped_gate(gate, up, limit):
    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def feed_forward(h, mlp, w, p):
    return clamped_gate(h @ w[p + ".gate"].T, h @ w[p + ".up"].T, mlp["limit"]) @ w[p + ".down"].T


def token_side(x, e, w, p, eps):
    """What layer p adds for the tokens' own rows e [rows, dim]."""
    return unit_rms((gelu_tanh(x @ w[p + ".side.gate"].T) * e) @ w[p + ".side.proj"].T, eps) * w[p + ".side.norm"]


# ---------------------------------------------------------------- model
class Sequence:
    """What a sequence carries from one portion to the next."""

    def __init__(self):
        self.tokens, self.kept = 0, {}

    def append(self, name, k, v):
        if name in self.kept:
            k, v = (torch.cat([old, new]) for old, new in zip(self.kept[name], (k, v)))
        self.kept[name] = (k, v)
        return k, v

    def get(self, name, start):
        return self.kept.get(name, start)

    def put(self, name, value):
        self.kept[name] = value


def forward(config, weights, tokens, seq=None, layers_out=None):
    """Logits [len(tokens), vocab] of the next tokens of a sequence."""
    seq = Sequence() if seq is None else seq
    ids = torch.as_tensor(tokens, dtype=torch.long)
    eps, dim = config["norm"]["eps"], config["token_side"]["dim"]
    x = weights["embed"][ids] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        y = MIXERS[layer["type"]](norm(x, weights, p + ".norm1"), layer["mixer"], weights, p + ".mix", seq, eps)
        x = x + norm(y, weights, p + ".norm1b")
        if layer.get("mlp"):
            y = feed_forward(norm(x, weights, p + ".norm2"), layer["mlp"], weights, p + ".mlp")
            x = x + norm(y, weights, p + ".norm2b")
        x = x + token_side(x, weights["side.embed"][ids][:, i * dim:(i + 1) * dim], weights, p, eps)
        if layers_out is not None:
            layers_out.append(x)
    seq.tokens += len(ids)
    return norm(x, weights, "final.norm") @ weights["embed"].T


def greedy(config, weights, prompt, n):
    seq, out, tokens = Sequence(), [], list(prompt)
    for _ in range(n):
        out.append(int(forward(config, weights, tokens, seq)[-1].argmax()))
        tokens = out[-1:]
    return out


# ---------------------------------------------------------------- models for tests
def random_weights(config, seed=0, dtype=torch.float64):
    """Seeded weights of every tensor the configuration needs, rounded to bfloat16 values.  The inner width of a decay differs
    from layer to layer; decays reach from almost nothing kept to almost everything."""
    g = torch.Generator().manual_seed(seed)
    W, V, side, scale = config["width"], config["vocab"], config["token_side"]["dim"], config["embedding"]["scale"]

    def mat(*shape, std=None, mean=0.0):
        return (torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5) + mean).to(torch.bfloat16)

    w = {"embed": mat(V, W, std=1 / scale), "side.embed": mat(V, len(config["layers"]) * side, std=1.0)}

    def add_norm(name):
        w[name], w[name + ".b"] = mat(W, std=0.3, mean=1.0), mat(W, std=0.2)
        w[name + ".alpha"] = mat(1, std=0.1, mean=0.6)[0]

    add_norm("final.norm")
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}", layer["mixer"]
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if layer.get("mlp") else ()):
            add_norm(f"{p}.{name}")
        if layer["type"] == "lightning":
            nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for name, rows in (("q", nk), ("k", nk), ("v", nv), ("g", nv)):
                w[f"{p}.mix.{name}"] = mat(rows, W)
            w[p + ".mix.o"], w[p + ".mix.norm"] = mat(W, nv), mat(nv, std=0.2, mean=1.0)
        else:
            a, r, q = m["left"], m["right"], p + ".mix.left"
            w[q + ".q"], w[q + ".k"] = mat(a["heads"] * a["dim"], W), mat(a["kv_heads"] * a["dim"], W)
            w[q + ".v"], w[q + ".o"] = mat(a["kv_heads"] * a["vdim"], W), mat(W, a["heads"] * a["vdim"])
            q, n, rank = p + ".mix.right", r["heads"] * r["dim"], 5 + 3 * i
            for s in "rkvg":
                w[f"{q}.{s}"] = mat(n, W)
            for s in "rkvgw":
                w[f"{q}.mu.{s}"] = mat(W, std=0.3, mean=0.5)
            w[q + ".w1"], w[q + ".w2"], w[q + ".w0"] = mat(rank, W), mat(n, rank, std=0.4), mat(n, std=2.0, mean=-2.0)
            w[q + ".u"], w[q + ".norm"], w[q + ".o"] = mat(r["heads"], r["dim"], std=0.5), mat(n, std=0.2, mean=1.0), mat(W, n)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            w[p + ".mlp.gate"], w[p + ".mlp.up"], w[p + ".mlp.down"] = mat(ff, W), mat(ff, W), mat(W, ff)
        w[p + ".side.gate"], w[p + ".side.proj"], w[p + ".side.norm"] = mat(side, W), mat(W, side), mat(W, std=0.2, mean=0.3)
    return {k: v.to(dtype) for k, v in w.items()}
