"""Fabulix without a GPU: the plain implementation's mechanisms on hand-made inputs, the config.json reader, the registry."""
import json
import math

import pytest
import torch

from fabulix_cases import CASES, case, dense, left, lightning, model, parallel, shapes_of
from oracle import fabulix as F

D = torch.float64


def t(*v):
    return torch.tensor(v, dtype=D)


def test_rotation_turns_the_first_half_against_the_second():
    x = torch.zeros(3, 1, 6, dtype=D)
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 5] = 1.0, 2.0, 7.0
    y = F.rotate(x, 4, 4, 100.0)                       # pairs (0, 2) and (1, 3) by p and p / 10; 4 and 5 stay
    for r in range(3):
        p = 4.0 + r
        ref = t(math.cos(p), -2 * math.sin(p / 10), math.sin(p), 2 * math.cos(p / 10), 0.0, 7.0)
        assert torch.allclose(y[r, 0], ref)
    q, k = torch.randn(1, 1, 8, dtype=D), torch.randn(1, 1, 8, dtype=D)
    near = (F.rotate(q, 9, 8, 50.0) * F.rotate(k, 2, 8, 50.0)).sum()
    assert torch.allclose(near, (F.rotate(q, 107, 8, 50.0) * F.rotate(k, 100, 8, 50.0)).sum())   # distances only


def test_sink_takes_its_share():
    p = F.sink_softmax(t(0.0, 0.0, float("-inf"))[None])
    assert torch.allclose(p, t(1 / 3, 1 / 3, 0.0)[None])
    assert F.sink_softmax(t(-50.0, -60.0)[None]).sum() < 1e-20
    assert torch.allclose(F.sink_softmax(t(800.0, 800.0)[None]), t(0.5, 0.5)[None])


def test_time_mix_gives_the_bonus_to_the_current_token_only():
    r = k = torch.ones(3, 1, 1, dtype=D)
    v = t(2.0, 3.0, 5.0).view(3, 1, 1)
    w = t(0.5, 0.1, 0.25).view(3, 1, 1)
    o, S = F.time_mix_scan(r, k, v, w, t(10.0).view(1, 1), torch.full((1, 1, 1), 8.0, dtype=D))
    # S: 8, 0.5 * 8 + 2 = 6, 0.1 * 6 + 3 = 3.6, 0.25 * 3.6 + 5 = 5.9; a token's own decay comes after its output
    assert torch.allclose(o.flatten(), t(8 + 20, 6 + 30, 3.6 + 50)) and torch.allclose(S.flatten(), t(5.9))


def test_lightning_reads_the_state_with_the_current_token():
    one = torch.ones(2, 2, 1, dtype=D)
    v = t(1.0, 4.0).view(2, 1, 1).expand(2, 2, 1)
    o, S = F.constant_decay_scan(one, one, v, t(0.5, 0.1), torch.full((2, 1, 1), 2.0, dtype=D))
    assert torch.allclose(o.view(2, 2), torch.stack([t(2.0, 1.2), t(5.0, 4.12)])) and torch.allclose(S.flatten(), t(5.0, 4.12))


def test_small_functions_by_hand():
    assert torch.allclose(F.dynamic_tanh(t(2.0), t(0.5), t(3.0), t(-1.0)), t(3 * math.tanh(1.0) - 1))
    g, u = t(5.0, -3.0, 0.5), t(-9.0, 9.0, 0.25)
    ref = [c / (1 + math.exp(-1.702 * c)) * (d + 1) for c, d in ((2.0, -2.0), (-3.0, 2.0), (0.5, 0.25))]   # the gate has no lower bound
    assert torch.allclose(F.clamped_gate(g, u, 2.0), t(*ref))
    assert torch.allclose(F.gelu_tanh(t(0.0, 1.0)), t(0.0, 0.5 * (1 + math.tanh(math.sqrt(2 / math.pi) * 1.044715))))
    assert torch.allclose(F.unit_rms(t(3.0, 4.0), 0.5), t(3.0, 4.0) / math.sqrt(13.0))
    assert torch.allclose(F.silu(t(1.0)), t(1 / (1 + math.exp(-1.0))))


@pytest.mark.parametrize("name", sorted(CASES))
def test_portions_equal_the_whole(name):
    cfg = case(name)
    w = F.random_weights(cfg, seed=3)
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = F.forward(cfg, w, toks)
    seq, parts, at = F.Sequence(), [], 0
    for n in (20, 2, 1, 1, 30, 6):
        parts.append(F.forward(cfg, w, toks[at:at + n], seq))
        at += n
    assert torch.allclose(torch.cat(parts), whole, atol=1e-9)
    assert whole.std() > 0.05 and (whole[5] - whole[40]).abs().max() > 0.1


def logit_errors(got, ref):
    d = got - ref
    return (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / ref.std()


def test_side_by_side_scales_and_the_far_past_show():
    """A wrong factor of either half, a lost state or a lost key changes the logits by far more than the tests let pass."""
    cfg = case("mixed")
    w = F.random_weights(cfg, seed=7)
    toks = torch.randint(0, cfg["vocab"], (200,), generator=torch.Generator().manual_seed(2)).tolist()
    ref = F.forward(cfg, w, toks)[-1:]
    for where, key in ((1, "left_scale"), (1, "right_scale"), (3, "left_scale"), (3, "right_scale")):
        bad = case("mixed")
        bad["layers"][where]["mixer"][key] *= 0.8
        assert logit_errors(F.forward(bad, w, toks)[-1:], ref).max() > 3e-3
    for changed in (0, 100, 190):
        assert logit_errors(F.forward(cfg, w, toks[:changed] + [(toks[changed] + 1) % 333] + toks[changed + 1:])[-1:], ref).max() > 1e-3


def test_first_token_has_nothing_before_it():
    cfg = case("odd")
    w = F.random_weights(cfg, seed=2)
    a, b = F.forward(cfg, w, [7]), F.forward(cfg, w, [3, 7])[1:]
    assert (a - b).abs().max() > 1e-2                         # token mixes, states and keys all see the 3


def test_reader_takes_every_size_from_the_configuration():
    import cpmcu.C as C
    from cpmcu.fabulix import layer_spec
    cfg = case("mixed")
    shapes = shapes_of(F.random_weights(cfg))
    a, b, c, d = [layer_spec(i, x, shapes) for i, x in enumerate(cfg["layers"])]
    assert (a.heads, a.recurrence, a.rec_heads, a.rec_dim, a.rec_vdim, a.ff) == (0, C.REC_LIGHTNING, 3, 24, 40, 0)
    assert (b.heads, b.kv_heads, b.dim, b.vdim, b.rot_dims, b.sink, b.window, b.kv_from) == (6, 2, 40, 56, 16, 1, 0, -1)
    assert (b.recurrence, b.rec_heads, b.rec_dim, b.rec_vdim, b.rec_rank, b.ff) == (C.REC_TIME_MIX, 5, 16, 16, 8, 100)
    for got, ref in ((b.scale, 0.21), (b.attn_scale, 0.7), (b.rec_scale, 1.3), (b.ff_limit, 0.8), (b.ff_alpha, 1.702), (b.bias_exp, 0.0)):
        assert abs(got - ref) < 1e-6
    assert c.ff == 72 and abs(c.ff_limit - 1.7) < 1e-6 and (d.ff, d.rec_rank, d.qk_norm, d.experts) == (0, 14, 0, 0)
    with pytest.raises(ValueError, match="shape"):
        layer_spec(1, cfg["layers"][1], {})
    with pytest.raises(ValueError, match="mixer"):
        layer_spec(0, {"type": "attention", "mixer": {}, "mlp": None}, {})
    with pytest.raises(ValueError, match="feed-forward"):
        layer_spec(0, lightning(1, 8, 8, [0.5], {"kind": "moe"}), {})


def unopened(cfg):
    from cpmcu.fabulix import FabulixLLM
    llm = FabulixLLM.__new__(FabulixLLM)
    torch.nn.Module.__init__(llm)
    llm._read_config(None, cfg, None)
    return llm


def test_constants_and_options_come_from_the_configuration():
    import cpmcu.C as C
    cfg = case("mixed")
    llm = unopened(cfg)
    assert llm.model_options() == dict(norm=C.NORM_DYNAMIC_TANH, embed_scale=5.0, tied_head=True, side_dim=12)
    c = llm.constants()
    assert sorted(c) == ["l0.mix.decay", "l1.mix.left.inv_freq", "l2.mix.decay", "l3.mix.left.inv_freq"]
    assert c["l0.mix.decay"].tolist() == [0.3, 0.999, 0.87]
    assert torch.allclose(c["l1.mix.left.inv_freq"], t(*[500.0 ** (-2 * i / 16) for i in range(8)]))
    assert unopened(model(64, 9, [], 4, scale=1.0)).constants() == {}


def test_registry_and_checkpoint_shapes(tmp_path):
    from cpmcu.fabulix import FabulixLLM
    from cpmcu.layered import checkpoint_shapes
    from cpmcu.models import model_class
    from safetensors.torch import save_file
    assert model_class({"architecture": "Fabulix"}) is FabulixLLM
    save_file({"a": torch.zeros(3, 4), "b": torch.zeros(())}, str(tmp_path / "model.safetensors"))
    assert checkpoint_shapes(str(tmp_path)) == {"a": (3, 4), "b": ()}


def test_random_weights_follow_the_shapes():
    cfg = model(64, 50, [parallel(left(2, 1, 8, 4, 8), 3, 10, mlp=dense(24, 1.0)), lightning(2, 6, 5, [0.5, 0.6])], side=4)
    w = F.random_weights(cfg)
    assert w["l0.mix.left.o"].shape == (64, 8) and w["l0.mix.right.w2"].shape == (30, 5) and w["l0.mix.right.u"].shape == (3, 10)
    assert w["side.embed"].shape == (50, 8) and w["l1.mix.o"].shape == (64, 10) and w["l0.norm2b.alpha"].shape == ()
    assert "l1.norm2" not in w and "l1.mlp.up" not in w and "head" not in w


def test_configurations_are_plain_json():
    for name in CASES:
        assert json.loads(json.dumps(case(name))) == case(name)
