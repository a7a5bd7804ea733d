"""Fabulix on the GPU: every mechanism alone against the plain implementation (oracle/fabulix.py), then whole models in fp32
(tight) and bf16: prefill, portions, decoding through cache and state, reuse of both, generation, the command line and replay."""
import ctypes
import json
import os
import subprocess
import sys

import pytest
import torch

from fabulix_cases import CASES, case, dense, left, lightning, model, parallel, shapes_of
from oracle import fabulix as F

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]
ids_of = lambda p: str(p)[6:] if isinstance(p, torch.dtype) else str(p)   # noqa: E731


def pad64(n):
    return (n + 63) // 64 * 64


def gen(seed):
    return torch.Generator().manual_seed(seed)


def tokens_of(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=gen(seed)).tolist()


def padded(t, width, dtype):
    out = torch.zeros(*t.shape[:-1], width, dtype=dtype, device="cuda")
    out[..., :t.shape[-1]] = t.to(dtype)
    return out


def is32(dtype):
    return int(dtype == torch.float32)


# ---------------------------------------------------------------- attention: sink, rotation
def attn_spec(lft, out_scale=1.0):
    import cpmcu.C as C
    return C.LayerSpec(heads=lft["heads"], kv_heads=lft["kv_heads"], dim=lft["dim"], vdim=lft["vdim"], scale=lft["scale"], sink=1,
                       rot_dims=lft["rot"]["dims"], attn_scale=out_scale)


def run_attention(lft, q, k, v, splits, fp32, out_scale=1.0):
    """q [tq, H, d], k / v [keys, G, .] float tensors holding bf16 values; returns [tq, H * vdim] float."""
    import cpmcu.C as C
    dt = torch.float32 if fp32 else torch.bfloat16
    dk, dv = pad64(lft["dim"]), pad64(lft["vdim"])
    tq, keys = q.shape[0], k.shape[0]
    budget = (keys + 127) // 128 * 128
    kc = torch.zeros(budget, lft["kv_heads"], dk, dtype=dt, device="cuda")
    vc = torch.zeros(budget, lft["kv_heads"], dv, dtype=dt, device="cuda")
    kc[:keys, :, :lft["dim"]], vc[:keys, :, :lft["vdim"]] = k.to(dt), v.to(dt)
    kc[keys:], vc[keys:] = 3.0, 7.0          # rows of an earlier owner: nobody may see them
    qc = padded(q.cuda(), dk, dt)
    out = torch.zeros(tq, lft["heads"] * lft["vdim"], dtype=dt, device="cuda")
    sp = attn_spec(lft, out_scale)
    C.call("cpmcu_layer_attention", ctypes.byref(sp), qc.data_ptr(), kc.data_ptr(), vc.data_ptr(), budget, tq, keys, splits, int(fp32),
           out.data_ptr())
    return out.float().cpu()


def qkv(lft, tq, keys, seed=0):
    g = gen(seed)
    return [torch.randn(n, h, d, generator=g).bfloat16().float() for n, h, d in
            ((tq, lft["heads"], lft["dim"]), (keys, lft["kv_heads"], lft["dim"]), (keys, lft["kv_heads"], lft["vdim"]))]


ATTN_SHAPES = [left(5, 1, 64, 64, 8), left(6, 2, 40, 56, 8, scale=0.3), left(8, 1, 128, 64, 8), left(2, 2, 64, 128, 8), left(3, 3, 17, 3, 8)]


@pytest.mark.parametrize("lft", ATTN_SHAPES, ids=lambda m: "h%d_%d_d%d_%d" % (m["heads"], m["kv_heads"], m["dim"], m["vdim"]))
@pytest.mark.parametrize("tq,keys", [(1, 1), (1, 400), (2, 129), (70, 70), (150, 390)])
def test_attention_with_a_sink(lft, tq, keys):
    q, k, v = qkv(lft, tq, keys, seed=tq * 1000 + keys)
    ref = 0.7 * F.attention(q.double(), k.double(), v.double(), lft["scale"], keys - tq).float()
    assert (run_attention(lft, q, k, v, 0, True, 0.7) - ref).abs().max() < 2e-5
    for splits in ((0, 1, 4) if tq <= 64 else (0, 1)):
        assert (run_attention(lft, q, k, v, splits, False, 0.7) - ref).abs().max() < 0.03, splits


@pytest.mark.parametrize("splits,fp32", [(0, True), (1, False), (3, False)])
def test_sink_shows_at_every_size_of_the_scores(splits, fp32):
    """All scores of a row alike: the sink takes nearly everything of very negative ones and nothing of large ones."""
    lft = left(2, 1, 64, 64, 8, scale=1.0)
    for keys in (1, 7, 300):
        for size in (-9.0, -1.5, 0.0, 0.4, 5.0):
            q, k, v = qkv(lft, 2, keys + 1, seed=keys)
            q[:], k[:] = 0.0, 0.0
            q[:, :, 3], k[:, :, 3] = 4.0, size / 4
            v.abs_()
            ref = F.attention(q.double(), k.double(), v.double(), 1.0, keys - 1).float()
            got = run_attention(lft, q, k, v, splits, fp32)
            assert (got - ref).abs().max() <= (1e-5 if fp32 else 0.01) * (1e-3 + ref.abs().max()), (keys, size)
    q, k, v = qkv(lft, 1, 200, seed=3)
    q[:], k[:] = 0.0, 0.0
    q[:, :, 3], k[:, :, 3] = 16.0, -16.0                   # exp(-256): nothing but the sink is left
    assert (run_attention(lft, q, k, v, splits, fp32) == 0).all()


def test_far_key_stands_out_among_hundreds():
    lft = left(4, 2, 64, 64, 8, scale=1.0)
    for far in (0, 1, 127, 128, 255, 256, 899):
        q, k, v = qkv(lft, 1, 900, seed=far)
        k *= 0.05
        q[:] = 0.0
        q[0, 3, 9] = 8.0
        k[:, :, 9] = 0.0
        k[far, 1, 9] = 8.0
        for splits, fp32 in ((0, True), (1, False), (7, False)):
            assert (run_attention(lft, q, k, v, splits, fp32)[0, 192:] - v[far, 1]).abs().max() < 0.03, far


@pytest.mark.parametrize("lft", [left(6, 2, 40, 56, 16, base=300.0), left(3, 1, 9, 7, 6, base=20.0), left(4, 4, 128, 64, 128), left(2, 1, 48, 16, 40)],
                         ids=["h6", "odd", "whole", "part"])
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
@pytest.mark.parametrize("at", [0, 1, 777])
def test_rotation_and_append(lft, dtype, at):
    import cpmcu.C as C
    H, G, d, dv, rot = lft["heads"], lft["kv_heads"], lft["dim"], lft["vdim"], lft["rot"]
    rows, budget = 5, 896
    x = torch.randn(rows, H * d + G * (d + dv), generator=gen(5)).to(dtype)
    freq = (rot["base"] ** (-torch.arange(0, rot["dims"], 2, dtype=torch.float64) / rot["dims"])).float().cuda()
    q = torch.full((rows, H, pad64(d)), 5.0, dtype=dtype, device="cuda")
    kc, vc = (torch.zeros(budget, G, pad64(n), dtype=dtype, device="cuda") for n in (d, dv))
    xc, sp = x.cuda(), attn_spec(lft)
    C.call("cpmcu_layer_qkv_norm_append", ctypes.byref(sp), xc.data_ptr(), None, None, 0.0, freq.data_ptr(), rows, at, budget, is32(dtype),
           q.data_ptr(), kc.data_ptr(), vc.data_ptr())
    f = x.double()
    rq = F.rotate(f[:, :H * d].view(rows, H, d), at, rot["dims"], rot["base"])
    rk = F.rotate(f[:, H * d:(H + G) * d].view(rows, G, d), at, rot["dims"], rot["base"])
    tol = 2e-4 if dtype == torch.float32 else 0.03        # an angle of 777 has 6e-5 in its last bit
    assert (q[..., :d].cpu().double() - rq).abs().max() < tol and (kc[at:at + rows, :, :d].cpu().double() - rk).abs().max() < tol
    assert torch.equal(vc[at:at + rows, :, :dv].cpu(), x[:, (H + G) * d:].view(rows, G, dv))
    assert torch.equal(q[..., rot["dims"]:d].cpu(), x[:, :H * d].view(rows, H, d)[..., rot["dims"]:])
    assert (q[..., d:] == 0).all() and (kc[..., d:] == 0).all() and (kc[:at] == 0).all() and (kc[at + rows:] == 0).all()


# ---------------------------------------------------------------- recurrences
def rec_spec(kind, heads, dim, vdim, rank=0, scale=1.0):
    import cpmcu.C as C
    return C.LayerSpec(recurrence=C.REC_TIME_MIX if kind == "time mix" else C.REC_LIGHTNING, rec_heads=heads, rec_dim=dim, rec_vdim=vdim,
                       rec_rank=rank, rec_scale=scale)


def state_of(spec, fill=0.0):
    import cpmcu.C as C
    return torch.full((C.load().cpmcu_layer_scan_state_floats(ctypes.byref(spec)),), fill, device="cuda")


def rec_inputs(kind, heads, dim, vdim, rows, seed):
    """(r, k, v) as the kernel gets them, decays (time mix: with exact zeros and ones), bonus."""
    g = gen(seed)
    r, k, v = (torch.randn(rows, heads, n, generator=g).bfloat16().double() for n in (dim, dim, vdim))
    if kind == "time mix":
        w = torch.exp(-torch.exp(torch.randn(rows, heads, dim, generator=g) * 2.5 - 2)).float().double()
        w[:, :, 0], w[:, :, -1] = 1.0, 0.0
        return r, k, v, w, torch.randn(heads, dim, generator=g).bfloat16().double()
    return r, k, v, torch.tensor([(0.999, 0.02, 0.8, 1.0, 0.5)[h % 5] for h in range(heads)], dtype=torch.float64), None


def run_scan(kind, spec, r, k, v, w, u, state, position, dtype):
    import cpmcu.C as C
    rows = r.shape[0]
    rc, kc, vc = (x.reshape(rows, -1).to(dtype).cuda() for x in (r, k, v))
    wc = w.float().cuda().contiguous()
    uc = u.bfloat16().cuda() if u is not None else None
    out = torch.empty(rows, spec.rec_heads * spec.rec_vdim, device="cuda")
    mix = kind == "time mix"
    C.call("cpmcu_layer_scan", ctypes.byref(spec), rc.data_ptr(), kc.data_ptr(), vc.data_ptr(), wc.data_ptr() if mix else None,
           None if mix else wc.data_ptr(), uc.data_ptr() if mix else None, state.data_ptr(), rows, position, is32(dtype), out.data_ptr())
    return out.cpu().double().view(rows, spec.rec_heads, spec.rec_vdim)


def plain_scan(kind, r, k, v, w, u, S):
    if kind == "time mix":
        return F.time_mix_scan(r, k, v, w, u, S)
    return F.constant_decay_scan(F.silu(r), F.silu(k), F.silu(v), w, S)


SCANS = [("time mix", 3, 64, 64), ("time mix", 2, 32, 32), ("time mix", 1, 128, 128), ("time mix", 2, 200, 200), ("time mix", 3, 7, 7),
         ("lightning", 2, 32, 64), ("lightning", 3, 24, 40), ("lightning", 2, 128, 256), ("lightning", 1, 256, 24), ("lightning", 5, 5, 11),
         ("lightning", 2, 64, 300), ("lightning", 1, 1, 1)]


def tolerance(kind, ref, dtype):
    # bf16: the approximate exponential of lightning's silu
    return (1e-5 if dtype == torch.float32 or kind == "time mix" else 1e-4) * (1 + ref.abs().max())


@pytest.mark.parametrize("shape", SCANS, ids=lambda s: "%s_%d_%d_%d" % (s[0].replace(" ", ""), *s[1:]))
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
def test_recurrence_over_portions(shape, dtype):
    """Portions of every size between one token and several chunks, one after the other, against the token-by-token form; the
    first one begins at position 0, where whatever the state's memory holds counts as zero."""
    kind, heads, dim, vdim = shape
    spec = rec_spec(*shape)
    cuts = [1, 2, 64, 65, 7, 8, 9, 300, 63, 130, 1]
    total = sum(cuts)
    r, k, v, w, u = rec_inputs(kind, heads, dim, vdim, total, seed=dim + vdim)
    state, S, at = state_of(spec, 5.0), torch.zeros(heads, dim, vdim, dtype=torch.float64), 0
    for n in cuts:
        rows = slice(at, at + n)
        wr = w[rows] if kind == "time mix" else w
        ref, S = plain_scan(kind, r[rows], k[rows], v[rows], wr, u, S)
        got = run_scan(kind, spec, r[rows], k[rows], v[rows], wr, u, state, at, dtype)
        assert (got - ref).abs().max() < tolerance(kind, ref, dtype), (at, n)
        at += n


def test_recurrence_of_a_long_portion_and_many_heads():
    """More chunks than run at once, so that chunks get longer."""
    for kind, heads, dim, vdim in (("time mix", 24, 64, 64), ("lightning", 20, 64, 128)):
        spec = rec_spec(kind, heads, dim, vdim)
        r, k, v, w, u = rec_inputs(kind, heads, dim, vdim, 2600, seed=1)
        few = [0, 7, heads - 1]
        state = state_of(spec)
        got = run_scan(kind, spec, r, k, v, w, u, state, 0, torch.bfloat16)
        S = torch.zeros(len(few), dim, vdim, dtype=torch.float64)
        wf = w[:, few] if kind == "time mix" else w[few]
        ref, _ = plain_scan(kind, r[:, few], k[:, few], v[:, few], wf, u[few] if u is not None else None, S)
        assert (got[:, few] - ref).abs().max() < tolerance(kind, ref, torch.bfloat16)


@pytest.mark.parametrize("kind", ["time mix", "lightning"])
@pytest.mark.parametrize("lag", [1, 7, 8, 63, 64, 65, 128, 200, 511])
def test_one_far_token_shows_through_the_state(kind, lag):
    """All keys but one are zero: what a token reads is that key's value after `lag` decays."""
    heads, dim, vdim, total = 2, 32, 64, 520
    spec = rec_spec(kind, heads, dim, vdim)
    r, k, v, w, u = rec_inputs(kind, heads, dim, vdim, total, seed=9)
    src = total - 1 - lag
    k[:] = 0.0
    k[src, :, 4] = 30.0
    r[:] = 0.0
    r[-1, :, 4] = 2.0
    if kind == "time mix":
        w[:] = 0.995
    else:
        w = torch.tensor([0.995, 0.9], dtype=torch.float64)
    ref, _ = plain_scan(kind, r, k, v, w, u, torch.zeros(heads, dim, vdim, dtype=torch.float64))
    for cut in (total, src, src + 1, total - 1):              # in one portion, and with a portion's edge on either side
        state, got = state_of(spec), []
        for lo, hi in ((0, cut), (cut, total)):
            if hi > lo:
                wr = w[lo:hi] if kind == "time mix" else w
                got.append(run_scan(kind, spec, r[lo:hi], k[lo:hi], v[lo:hi], wr, u, state, lo, torch.bfloat16))
        got = torch.cat(got)[-1]
        assert (got - ref[-1]).abs().max() < 1e-4 * (1 + ref[-1].abs().max()), cut
    assert ref[-1, 0].abs().max() > 0.5


STEPS = [("time mix", 3, 64, 64, 16), ("time mix", 2, 32, 32, 70), ("time mix", 1, 128, 128, 5), ("time mix", 3, 7, 7, 33),
         ("lightning", 2, 32, 64, 0), ("lightning", 3, 24, 40, 0), ("lightning", 2, 128, 256, 0), ("lightning", 1, 256, 24, 0),
         ("lightning", 5, 5, 11, 0), ("lightning", 40, 16, 48, 0)]


@pytest.mark.parametrize("shape", STEPS, ids=lambda s: "%s_%d_%d_%d_%d" % (s[0].replace(" ", ""), *s[1:]))
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
def test_one_token_step(shape, dtype):
    """The step kernel token by token (first on a dirty state), then a portion of the ordinary kernel on the state it left."""
    import cpmcu.C as C
    kind, heads, dim, vdim, rank = shape
    spec = rec_spec(kind, heads, dim, vdim, rank, 0.7)
    mix, total, steps, eps = kind == "time mix", 40, 12, 1e-4
    r, k, v, w, u = rec_inputs(kind, heads, dim, vdim, total, seed=3)
    g = gen(4)
    inner = torch.randn(total, max(rank, 1), generator=g).bfloat16()
    w2, w0 = (torch.randn(heads * dim, max(rank, 1), generator=g) * 0.4).bfloat16(), (torch.randn(heads * dim, generator=g) * 2 - 1).bfloat16()
    gate, norm = torch.randn(total, heads * vdim, generator=g).bfloat16(), torch.randn(heads * vdim, generator=g).bfloat16()
    if mix:
        w = torch.exp(-torch.exp(torch.tanh(inner.double()) @ w2.double().T + w0.double())).view(total, heads, dim)
    S = torch.zeros(heads, dim, vdim, dtype=torch.float64)
    o, S_end = plain_scan(kind, r[:steps], k[:steps], v[:steps], w[:steps] if mix else w, u, S)
    flat = o.reshape(steps, -1)
    z = gate[:steps].double()
    if mix:
        ref = F.unit_rms(o, eps).reshape(steps, -1) * norm.double() * F.silu(z) * 0.7
    else:
        ref = F.unit_rms(flat, eps) * norm.double() / (1 + torch.exp(-z)) * 0.7
    state = state_of(spec, 4.0)
    w2c, w0c, nc = w2.cuda(), w0.cuda(), norm.cuda()
    uc = u.bfloat16().cuda() if mix else None
    dc = None if mix else w.float().cuda()
    for t in range(steps):
        rc, kc, vc, ic, gc = (x.reshape(-1).to(dtype).cuda() for x in (r[t], k[t], v[t], inner[t], gate[t]))
        out = torch.zeros(heads * vdim, dtype=dtype, device="cuda")
        C.call("cpmcu_layer_scan_step", ctypes.byref(spec), rc.data_ptr(), kc.data_ptr(), vc.data_ptr(), ic.data_ptr(), w2c.data_ptr(),
               w0c.data_ptr(), None if mix else dc.data_ptr(), uc.data_ptr() if mix else None, state.data_ptr(), nc.data_ptr(), gc.data_ptr(),
               eps, t, is32(dtype), out.data_ptr())
        err = (out.cpu().double() - ref[t]).abs().max()
        assert err < (2e-5 if dtype == torch.float32 else 0.01) * (1 + ref[t].abs().max()), t
    rest = slice(steps, total)
    ref2, _ = plain_scan(kind, r[rest], k[rest], v[rest], w[rest] if mix else w, u, S_end)
    got = run_scan(kind, spec, r[rest], k[rest], v[rest], w[rest] if mix else w, u, state, steps, dtype)
    assert (got - ref2).abs().max() < 3 * tolerance(kind, ref2, dtype)


@pytest.mark.parametrize("rank,channels", [(16, 256), (5, 77), (64, 300), (33, 1)])
@pytest.mark.parametrize("rows", [1, 5, 300])
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
def test_decays(rank, channels, rows, dtype):
    import cpmcu.C as C
    g = gen(rank + rows)
    x, w2 = torch.randn(rows, rank, generator=g).to(dtype), (torch.randn(channels, rank, generator=g) * 0.4).bfloat16()
    w0 = (torch.randn(channels, generator=g) * 3 - 1).bfloat16()
    out = torch.zeros(rows, channels, device="cuda")
    xc, w2c, w0c = x.cuda(), w2.cuda(), w0.cuda()
    C.call("cpmcu_layer_decay", xc.data_ptr(), w2c.data_ptr(), w0c.data_ptr(), rank, channels, rows, is32(dtype), out.data_ptr())
    ref = torch.exp(-torch.exp(torch.tanh(x.double()) @ w2.double().T + w0.double()))
    assert (out.cpu().double() - ref).abs().max() < 3e-6
    weights = {"p.w1": torch.eye(rank, dtype=torch.float64), "p.w2": w2.double(), "p.w0": w0.double()}
    assert torch.allclose(torch.exp(-torch.exp(F.log_log_decay(x.double(), weights, "p"))), ref)


@pytest.mark.parametrize("groups,group,silu", [(3, 64, 1), (5, 16, 1), (2, 40, 1), (3, 7, 1), (1, 256, 0), (1, 2048, 0), (1, 5000, 0), (1, 33, 0),
                                               (40, 128, 1), (1, 20000, 0)])
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
def test_norm_and_gate(groups, group, silu, dtype):
    import cpmcu.C as C
    rows, n, eps = 5, groups * group, 1e-2
    g = gen(n)
    o, w, gate = torch.randn(rows, n, generator=g) * 0.3, torch.randn(n, generator=g).bfloat16(), torch.randn(rows, n, generator=g).to(dtype)
    o[:, :group] *= 20                                   # one loud group
    out = torch.zeros(rows, n, dtype=dtype, device="cuda")
    oc, wc, gc = o.cuda(), w.cuda(), gate.cuda()
    C.call("cpmcu_layer_norm_gate", oc.data_ptr(), wc.data_ptr(), gc.data_ptr(), groups, group, silu, eps, 0.6, rows, is32(dtype), out.data_ptr())
    z = gate.double()
    ref = F.unit_rms(o.double().view(rows, groups, group), eps).reshape(rows, n) * w.double() * (F.silu(z) if silu else 1 / (1 + torch.exp(-z))) * 0.6
    assert (out.cpu().double() - ref).abs().max() < (1e-5 if dtype == torch.float32 else 0.01) * (1 + ref.abs().max())


# ---------------------------------------------------------------- row kernels
@pytest.mark.parametrize("width", [75, 200, 2048, 5000])
@pytest.mark.parametrize("rows", [1, 2, 3, 70, 300])
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
def test_dynamic_tanh_and_token_mixes(width, rows, dtype):
    import cpmcu.C as C
    ld, g = pad64(width), gen(width + rows)
    x = torch.randn(rows, width, generator=g) * 3
    w, b, mu = (torch.randn(*s, generator=g).bfloat16() for s in ((width,), (width,), (5, width)))
    before = torch.randn(width, generator=g)
    xc, wc, bc, muc = padded(x.cuda(), ld, torch.float32), padded(w.cuda(), ld, torch.bfloat16), padded(b.cuda(), ld, torch.bfloat16), padded(mu.cuda(), ld, torch.bfloat16)
    href = F.dynamic_tanh(x.double(), 0.4, w.double(), b.double())
    for position in (0, 9):
        prev = padded(before.cuda(), ld, torch.float32)
        h, mixes = torch.zeros(rows, ld, dtype=dtype, device="cuda"), torch.zeros(5, rows, ld, dtype=dtype, device="cuda")
        C.call("cpmcu_layer_tanh_norm", xc.data_ptr(), wc.data_ptr(), bc.data_ptr(), 0.4, muc.data_ptr(), prev.data_ptr(), rows, ld, position,
               is32(dtype), h.data_ptr(), mixes.data_ptr())
        shifted = torch.cat([before[None].double() * (position > 0), href[:-1]])
        mref = href + (shifted - href) * mu.double()[:, None]
        tol = 1e-5 if dtype == torch.float32 else 0.02
        assert (h[:, :width].cpu().double() - href).abs().max() < tol * (1 + href.abs().max())
        assert (mixes[..., :width].cpu().double() - mref).abs().max() < tol * (1 + mref.abs().max())
        assert (prev[:width].cpu().double() - href[-1]).abs().max() < 1e-5      # fp32 in both
        assert (h[:, width:] == 0).all() and (mixes[..., width:] == 0).all()


@pytest.mark.parametrize("limit,alpha", [(0.5, 1.702), (7.0, 1.702), (1.1, 0.9)])
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
def test_clamped_gate(limit, alpha, dtype):
    import cpmcu.C as C
    rows, ff = 9, 192
    gu = (torch.randn(rows, 2 * ff, generator=gen(1)) * 4).to(dtype)
    act, guc = torch.zeros(rows, ff, dtype=dtype, device="cuda"), gu.cuda()
    C.call("cpmcu_layer_clamped_gate", guc.data_ptr(), rows, ff, limit, alpha, is32(dtype), act.data_ptr())
    g, u = gu.double()[:, :ff].clamp(max=limit), gu.double()[:, ff:].clamp(-limit, limit)
    ref = g / (1 + torch.exp(-alpha * g)) * (u + 1)
    if alpha == 1.702:
        assert torch.allclose(ref, F.clamped_gate(gu.double()[:, :ff], gu.double()[:, ff:], limit))
    assert (act.cpu().double() - ref).abs().max() < (1e-5 if dtype == torch.float32 else 0.01) * (1 + ref.abs().max())


@pytest.mark.parametrize("width,dim", [(75, 3), (200, 12), (2048, 128), (384, 72), (1000, 300), (5000, 17)])
@pytest.mark.parametrize("dtype", DTYPES, ids=ids_of)
def test_side_input_of_one_row(width, dim, dtype):
    import cpmcu.C as C
    ld, layers, layer, vocab, eps = pad64(width), 3, 1, 11, 1e-3
    g = gen(width + dim)

    def mat(*s, std):
        return (torch.randn(*s, generator=g) * std).bfloat16()

    x, delta = torch.randn(1, width, generator=g) * 30, torch.randn(1, width, generator=g).to(dtype)
    w, b = mat(width, std=1.0), mat(width, std=0.3)
    wt = {"l1.side.gate": mat(dim, width, std=width ** -0.5 / 20), "l1.side.proj": mat(width, dim, std=dim ** -0.5), "l1.side.norm": mat(width, std=0.5)}
    table, tok = mat(vocab, layers * dim, std=1.0), 7
    ref = x.double() + F.dynamic_tanh(delta.double(), 0.8, w.double(), b.double())
    ref = ref + F.token_side(ref, table.double()[[tok], layer * dim:(layer + 1) * dim], {k: v.double() for k, v in wt.items()}, "l1", eps)
    xc, dc = padded(x.cuda(), ld, torch.float32), padded(delta.cuda(), ld, dtype)
    wc, bc, nc = (padded(t.cuda(), ld, torch.bfloat16) for t in (w, b, wt["l1.side.norm"]))
    gc, pc, tc, ic = wt["l1.side.gate"].cuda(), wt["l1.side.proj"].cuda(), table.cuda(), torch.tensor([tok], dtype=torch.int32, device="cuda")
    C.call("cpmcu_layer_side_step", xc.data_ptr(), dc.data_ptr(), wc.data_ptr(), bc.data_ptr(), 0.8, gc.data_ptr(), pc.data_ptr(), nc.data_ptr(),
           ic.data_ptr(), tc.data_ptr(), layers, layer, dim, vocab, width, ld, eps, is32(dtype))
    assert (xc[:, :width].cpu().double() - ref).abs().max() < (4e-5 if dtype == torch.float32 else 0.03)
    assert (xc[:, width:] == 0).all()


@pytest.mark.parametrize("n,N,N_s,K,rows", [(4, 96, 16, 256, 1), (4, 320, 33, 128, 2), (4, 200, 5, 64, 17), (3, 64, 0, 192, 70), (4, 130, 70, 320, 300),
                                            (1, 7, 3, 64, 700)])
def test_grouped_products(n, N, N_s, K, rows):
    import cpmcu.C as C
    g, parts = gen(N + rows), n + (1 if N_s else 0)
    x = torch.randn(parts * rows, K, generator=g).bfloat16()
    ws = [(torch.randn(N_s if i == n else N, K, generator=g) * K ** -0.5).bfloat16() for i in range(parts)]
    ldy = pad64(max(N, N_s))
    y = torch.full((parts * rows, ldy), 9.0, dtype=torch.bfloat16, device="cuda")
    xc, wc = x.cuda(), torch.cat([t.flatten() for t in ws]).cuda()
    C.call("cpmcu_grouped_linear", xc.data_ptr(), wc.data_ptr(), n, N, N_s, K, rows, ldy, y.data_ptr())
    for i, w in enumerate(ws):
        got = y[i * rows:(i + 1) * rows].cpu()
        ref = x[i * rows:(i + 1) * rows].double() @ w.double().T
        assert (got[:, :w.shape[0]].double() - ref).abs().max() < 0.03 and (got[:, w.shape[0]:] == 9.0).all()


# ---------------------------------------------------------------- whole models
def open_case(cfg, weights, dtype, chunk=128, max_tokens=1024, **kw):
    from cpmcu.fabulix import FabulixLLM
    os.environ["CPMCU_MAX_TOKENS"] = str(max_tokens)
    try:
        llm = FabulixLLM(config=cfg, shapes=shapes_of(weights), dtype=dtype, chunk_length=chunk, memory_limit=0.5, **kw)
        llm.init_storage()
    finally:
        os.environ["CPMCU_MAX_TOKENS"] = "4096"
    llm.load_state_dict_tensors(weights)
    return llm


def errors(got, ref):
    """Per-row error of logits: mean difference removed, RMS over the vocabulary, relative to the logits' spread."""
    d = got.double().cpu() - ref
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / ref.std()


def check(got, ref, dtype):
    e = errors(got, ref)
    if dtype == torch.float32:
        assert e.max() < 5e-5, e.max()
    else:
        assert e.median() < 0.03 and e.max() < 0.1, (e.median(), e.max())


@pytest.fixture(scope="module", params=[(n, d) for n in sorted(CASES) for d in DTYPES], ids=lambda p: "%s-%s" % (p[0], str(p[1])[6:]))
def loaded(request):
    import cpmcu.C as C
    name, dtype = request.param
    cfg = case(name)
    w = F.random_weights(cfg, seed=7)
    llm = open_case(cfg, w, dtype)
    toks = tokens_of(cfg, 420, seed=2)
    yield cfg, w, llm, dtype, toks, F.forward(cfg, w, toks)
    C.release()


def test_stream_after_every_layer(loaded):
    import cpmcu.C as C
    cfg, w, llm, dtype, toks, _ = loaded
    for n, first in ((60, 0), (1, 60)):               # a portion, then one decoded token
        seq, layers = F.Sequence(), []
        if first:
            F.forward(cfg, w, toks[:first], seq)
        F.forward(cfg, w, toks[first:first + n], seq, layers_out=layers)
        buf = torch.zeros(len(layers), n, cfg["width"], device="cuda")
        C.call("cpmcu_capture_layers", buf.data_ptr())
        try:
            llm.extend(toks[first:first + n], first, [0])
        finally:
            C.call("cpmcu_capture_layers", None)
        for i, x in enumerate(layers):
            err = (buf[i].cpu().double() - x).abs().max() / x.std()
            assert err < (1e-4 if dtype == torch.float32 else 0.2), (first, i, err)


def test_whole_prompt(loaded):
    _, _, llm, dtype, toks, ref = loaded
    check(llm.extend(toks, 0, range(len(toks))), ref, dtype)      # chunks of 128
    check(llm.extend(toks[:1], 0, [0]), ref[:1], dtype)


@pytest.mark.parametrize("cuts", [[2] * 30 + [60, 3, 2, 117], [1, 127, 1, 128, 2, 60], [63, 2, 64, 3, 65, 62], [65, 63, 129, 64], [8, 7, 9, 16, 15, 100]],
                         ids=["twos", "edges", "chunks", "tiles", "batches"])
def test_portions(loaded, cuts):
    _, _, llm, dtype, toks, ref = loaded
    got, at = [], 0
    for n in cuts:
        got.append(llm.extend(toks[at:at + n], at, list(range(n))))
        at += n
    check(torch.cat(got), ref[:at], dtype)


def test_token_by_token_and_long_decoding(loaded):
    _, _, llm, dtype, toks, ref = loaded
    got = [llm.extend(toks[:1], 0, [0])]
    for i in range(1, 300):
        got.append(llm.extend(toks[i:i + 1], i, [0]))
    check(torch.cat(got), ref[:300], dtype)


def test_decoding_behind_a_long_prompt(loaded):
    _, _, llm, dtype, toks, ref = loaded
    got = [llm.extend(toks[:350], 0, [349])]
    for i in range(350, 420):
        got.append(llm.extend(toks[i:i + 1], i, [0]))
    check(torch.cat(got), ref[349:420], dtype)


def test_wanted_places_come_in_the_order_asked_for(loaded):
    _, _, llm, dtype, toks, ref = loaded
    want = [200, 3, 3, 129, 0, 127, 128]
    check(llm.extend(toks[:201], 0, want), ref[want], dtype)
    assert llm.extend(toks[:5], 0, []).shape == (0, ref.shape[1])


def test_cache_and_state_are_used_again(loaded):
    cfg, w, llm, dtype, toks, _ = loaded
    other = tokens_of(cfg, 150, seed=9)

    def run():
        return torch.cat([llm.extend(other[:140], 0, [0, 70, 139]), llm.extend(other[140:141], 140, [0])])

    first = run()
    llm.extend(toks, 0, [])                                           # a longer request over the same rows and states
    assert torch.equal(first, run())
    llm.extend(toks[:1], 0, [])                                       # one that ends after a single token
    assert torch.equal(first, run())
    check(first, F.forward(cfg, w, other[:141])[[0, 70, 139, 140]], dtype)


def test_the_answer_does_not_depend_on_the_cut(loaded):
    _, _, llm, dtype, toks, _ = loaded
    a = llm.extend(toks[:200], 0, [199])
    llm.extend(toks[:198], 0, [])
    b = llm.extend(toks[198:200], 198, [1])
    llm.extend(toks[:199], 0, [])
    c = llm.extend(toks[199:200], 199, [0])
    tol = 2e-5 if dtype == torch.float32 else 0.06
    assert errors(b, a.double().cpu()).max() < tol and errors(c, a.double().cpu()).max() < tol


def test_greedy_generation(loaded):
    cfg, w, llm, dtype, toks, _ = loaded
    prompt = toks[:150]
    out, _, _ = llm.generate(torch.tensor(prompt, dtype=torch.int32, device="cuda"), 24)
    ref = F.forward(cfg, w, prompt + out)[len(prompt) - 1:-1]
    for i, tok in enumerate(out):
        assert float(ref[i].max() - ref[i, tok]) <= (1e-4 if dtype == torch.float32 else 0.2) * float(ref.std()), i
    if dtype == torch.float32:
        assert out == F.greedy(cfg, w, prompt, 24)
    streamed = [d["token"] for d in llm.generate(torch.tensor(prompt, dtype=torch.int32, device="cuda"), 24, use_stream=True)]
    assert streamed == out


def test_tokens_that_do_not_follow_the_state_are_refused(loaded):
    """The recurrent states hold one position: a pass begins there or at 0."""
    _, _, llm, dtype, toks, ref = loaded
    llm.extend(toks[:50], 0, [])
    with pytest.raises(RuntimeError, match="recurrent state"):
        llm.extend(toks[40:45], 40, [0])
    with pytest.raises(RuntimeError, match="recurrent state"):
        llm.extend(toks[50:51], 50, [0])                              # after an error only position 0 is open
    check(llm.extend(toks[:50], 0, [49]), ref[[49]], dtype)
    with pytest.raises(RuntimeError, match="recurrent state"):
        llm.extend(toks[60:61], 60, [0])
    check(llm.extend(toks[:50], 0, [49]), ref[[49]], dtype)


def test_capture_and_eager_decode_agree():
    import cpmcu.C as C
    cfg = case("mixed")
    w = F.random_weights(cfg, seed=1)
    outs = []
    for graph in (False, True):
        llm = open_case(cfg, w, torch.bfloat16, cuda_graph=graph)
        outs.append(llm.generate(torch.tensor(tokens_of(cfg, 50), dtype=torch.int32, device="cuda"), 40)[0])
        C.release()
    assert outs[0] == outs[1]


def test_weights_loaded_again_reach_the_captured_step():
    """alpha is an argument of captured kernels."""
    import cpmcu.C as C
    cfg = case("odd")
    w = F.random_weights(cfg, seed=1)
    llm, toks = open_case(cfg, w, torch.float32), tokens_of(cfg, 12)
    for alpha in (0.2, 0.9):
        w["l1.norm1.alpha"] = torch.tensor(alpha).bfloat16().double()
        w["final.norm.alpha"] = torch.tensor(alpha / 2).bfloat16().double()
        llm.load_state_dict_tensors({k: v for k, v in w.items() if k.endswith("alpha")})
        llm.extend(toks[:3], 0, [])
        got = torch.cat([llm.extend(toks[i:i + 1], i, [0]) for i in range(3, 12)])
        check(got, F.forward(cfg, w, toks)[3:], torch.float32)
    C.release()


def test_sampling_follows_the_seed():
    import cpmcu.C as C
    cfg = case("odd")
    w = F.random_weights(cfg, seed=1)
    outs = []
    for seed in (1, 1, 2):
        llm = open_case(cfg, w, torch.bfloat16, temperature=1.0, random_seed=seed)
        outs.append(llm.generate(torch.tensor(tokens_of(cfg, 20), dtype=torch.int32, device="cuda"), 30)[0])
        C.release()
    assert outs[0] == outs[1] != outs[2]


def test_models_with_one_kind_of_layer():
    """Only recurrences (no cache at all), and only parallel layers with a single head of width one group."""
    import cpmcu.C as C
    for cfg in (model(128, 90, [lightning(2, 16, 16, [0.9, 0.5], dense(64, 1.0)), lightning(1, 48, 8, [0.99])], side=64),
                model(64, 70, [parallel(left(1, 1, 64, 64, 64), 1, 64, mlp=dense(64, 1.0))], side=1, scale=1.0)):
        w = F.random_weights(cfg, seed=5)
        for dtype in DTYPES:
            llm = open_case(cfg, w, dtype)
            toks = tokens_of(cfg, 90, seed=4)
            got = [llm.extend(toks[:70], 0, list(range(70)))] + [llm.extend(toks[i:i + 1], i, [0]) for i in range(70, 90)]
            check(torch.cat(got), F.forward(cfg, w, toks), dtype)
            C.release()


def test_errors_are_reported():
    import cpmcu.C as C
    cfg = case("odd")
    w = F.random_weights(cfg, seed=1)
    llm = open_case(cfg, {k: v for k, v in w.items() if k != "l0.mix.right.mu.g"} | {"l0.mix.right.w1": w["l0.mix.right.w1"]}, torch.bfloat16, max_tokens=256)
    with pytest.raises(RuntimeError, match="l0.mix.right.mu.g"):
        llm.extend([1, 2], 0, [0])
    llm.load_state_dict_tensors({"l0.mix.right.mu.g": w["l0.mix.right.mu.g"]})
    ok = llm.extend([1, 2], 0, [1])
    with pytest.raises(RuntimeError, match="token id"):
        llm.extend([1, cfg["vocab"]], 0, [0])
    assert torch.equal(llm.extend([1, 2], 0, [1]), ok)
    with pytest.raises(ValueError):
        llm.extend([1] * 300, 0, [])
    for name in ("l0.mix.right.mu.x", "l0.mix.q", "l1.mix.left.q", "head", "l0.norm3", "l0.norm1.c"):
        with pytest.raises(RuntimeError, match="Unsupported name"):
            llm.load_state_dict_tensors({name: torch.zeros(4)})
    with pytest.raises(RuntimeError, match="drafter"):
        C.init_eagle_model(1, 2, 2, 4, 1)
    C.release()
    bad = case("odd")
    bad["layers"][0]["mixer"]["left"]["kv_heads"] = 2
    with pytest.raises(RuntimeError, match="layer 0"):
        open_case(bad, w, torch.bfloat16)
    bad = case("odd")
    bad["layers"][1]["mixer"]["dim"] = 257
    with pytest.raises(RuntimeError, match="layer 1"):
        open_case(bad, w, torch.bfloat16)


def write_checkpoint(mdir, cfg, w):
    from safetensors.torch import save_file
    mdir.mkdir()
    (mdir / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, str(mdir / "model.safetensors"))


def test_command_line(tmp_path):
    cfg = case("odd")
    w = F.random_weights(cfg, seed=12)
    write_checkpoint(tmp_path / "model", cfg, w)
    prompt = tokens_of(cfg, 40, seed=3)
    res = subprocess.run([sys.executable, "-m", "cpmcu", "--model", str(tmp_path / "model"), "--tokens", ",".join(map(str, prompt)), "--max-new", "12",
                          "--dtype", "float32", "--chunk-length", "64", "--max-tokens", "256"], capture_output=True, text=True, timeout=300,
                         env=dict(os.environ, PYTHONPATH=os.path.join(ROOT, "cpm.cu_b200")))
    assert res.returncode == 0, res.stderr[-2000:]
    assert [int(t) for t in res.stdout.strip().splitlines()[-1].split(",")] == F.greedy(cfg, w, prompt, 12)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(tmp_path, dtype):
    cfg = case("mixed")
    w = F.random_weights(cfg, seed=11)
    mdir, out = tmp_path / "model", tmp_path / "out"
    write_checkpoint(mdir, cfg, w)
    out.mkdir()
    toks, other = tokens_of(cfg, 80, seed=1), tokens_of(cfg, 9, seed=2)
    steps = [{"entries": [{"id": "x", "tokens": toks[:70], "want": [69, 0]}], "end": []},
             {"entries": [{"id": "x", "tokens": toks[70:71], "want": []}], "end": []},
             {"entries": [{"id": "x", "tokens": toks[71:72], "want": [0]}], "end": []},
             {"entries": [{"id": "x", "tokens": toks[72:], "want": [7, 1]}], "end": ["x"]},
             {"entries": [{"id": "y", "tokens": other, "want": [8]}], "end": ["y"]}]
    text = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(mdir), "--dtype", dtype, "--out", str(out), "--max-tokens", "80"],
                         input=text, capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == ["done %d" % i for i in range(5)]
    ref, ref_y = F.forward(cfg, w, toks), F.forward(cfg, w, other)
    for i, rows in ((0, ref[[69, 0]]), (2, ref[[71]]), (3, ref[[79, 73]]), (4, ref_y[[8]])):
        got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        check(got, rows, getattr(torch, dtype))
    assert not (out / "1.f32").exists()
