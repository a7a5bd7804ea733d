"""Tipetar without a GPU: the plain implementation's mechanisms on hand-made inputs, the config.json reader, the model
registry and the trace runner's request handling."""
import math

import pytest
import torch

from oracle import tipetar as T
from tipetar_cases import CASES, attn, case, model, moe


def test_slopes_fall_by_powers_of_two():
    assert torch.allclose(T.distance_slopes(8), torch.tensor([2.0 ** -k for k in range(1, 9)], dtype=torch.float64))
    assert T.distance_slopes(4)[0] == 2.0 ** -2 and T.distance_slopes(16)[0] == 2.0 ** -0.5


def test_window_sees_itself_and_the_tokens_just_before():
    m = T.window_mask(1, 10, 9, 4)[0]
    assert m.tolist() == [False] * 6 + [True] * 4
    assert T.window_mask(1, 3, 2, 8)[0].all() and T.window_mask(2, 4, 2, None).tolist() == [[True, True, True, False], [True] * 4]


def test_norms_by_hand():
    x = torch.tensor([3.0, 4.0], dtype=torch.float64)
    r = math.sqrt(12.5 + 0.5)
    assert torch.allclose(T.norm_around_one(x, torch.tensor([0.0, 1.0]), 0.5), torch.tensor([3 / r, 8 / r], dtype=torch.float64))
    assert torch.allclose(T.norm_plain(x, torch.tensor([1.0, 2.0]), 0.5), torch.tensor([3 / r, 8 / r], dtype=torch.float64))


def test_choice_uses_the_correction_and_the_groups_but_the_weights_do_not():
    # scores by softmax: 0.4 0.3 0.2 0.1
    z = torch.log(torch.tensor([[0.4, 0.3, 0.2, 0.1]], dtype=torch.float64))
    r = {"experts": 4, "top": 2, "scale": 3.0}
    idx, w = T.route(z, None, r)
    assert idx.tolist() == [[0, 1]] and torch.allclose(w, torch.tensor([[12 / 7, 9 / 7]], dtype=torch.float64))
    # corrections make every choice score negative; the order turns round; groups of two, the better one is kept
    corr = torch.tensor([-2.0, -1.5, -1.2, -0.9], dtype=torch.float64)
    idx, w = T.route(z, corr, r)
    assert idx.tolist() == [[3, 2]] and torch.allclose(w, torch.tensor([[1.0, 2.0]], dtype=torch.float64))
    r["groups"] = {"count": 2, "keep": 1}
    idx, _ = T.route(z, torch.tensor([-1.0, -1.1, -0.2, -5.0], dtype=torch.float64), r)
    assert idx.tolist() == [[2, 3]]            # -5 is chosen: the other group counts as minus infinity, not as zero


def test_margin_is_the_closest_call():
    z = torch.log(torch.tensor([[0.4, 0.3, 0.2, 0.1]], dtype=torch.float64))
    assert abs(float(T.choice_margin(z, None, {"top": 2})) - 0.1 / 0.5) < 1e-3
    assert abs(float(T.choice_margin(z, None, {"top": 1, "groups": {"count": 2, "keep": 1}})) - 0.1 / 0.7) < 1e-3


@pytest.mark.parametrize("name", sorted(CASES))
def test_portions_equal_the_whole(name):
    cfg = case(name)
    w = T.random_weights(cfg, seed=3)
    toks = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(1)).tolist()
    whole = T.forward(cfg, w, toks)
    seq, parts, at = T.Sequence(), [], 0
    for n in (40, 2, 1, 1, 30, 16):
        parts.append(T.forward(cfg, w, toks[at:at + n], seq))
        at += n
    assert torch.allclose(torch.cat(parts), whole, atol=1e-9)


def test_reader_takes_every_size_from_the_configuration():
    from cpmcu.tipetar import layer_spec
    cfg = case("mixed")
    a, b, c, d = [layer_spec(i, x) for i, x in enumerate(cfg["layers"])]
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.kv_from, a.qk_norm, a.bias_exp) == (6, 2, 40, 56, 37, -1, 1, 8.0)
    assert abs(a.scale - 0.21) < 1e-7 and abs(a.router_scale - 1.7) < 1e-6
    assert (a.experts, a.identity, a.top, a.groups, a.keep_groups, a.expert_ff, a.shared_ff) == (5, 3, 3, 4, 2, 36, 100)
    assert b.kv_from == 0 and b.window == 61 and b.experts == b.identity == 0
    assert (c.groups, c.keep_groups, c.identity, c.shared_ff) == (1, 1, 0, 0)
    assert d.kv_from == 2 and d.shared_ff == 24
    free = layer_spec(0, {"type": "attention", "mixer": attn(2, 1, 16, 16, None), "mlp": None})
    assert free.window == 0
    with pytest.raises(ValueError):
        layer_spec(0, {"type": "recurrent", "mixer": {}, "mlp": None})
    with pytest.raises(ValueError):
        layer_spec(0, {"type": "attention", "mixer": attn(2, 1, 16, 16, 4), "mlp": {"kind": "dense"}})


def test_native_struct_matches_the_header():
    import os
    import re

    import cpmcu.C as C
    text = open(os.path.join(os.path.dirname(__file__), "..", "include", "cpmcu_b200.h")).read()
    body = re.sub(r"/\*.*?\*/", "", re.search(r"typedef struct \{(.*?)\} cpmcu_layer_spec;", text, re.S).group(1), flags=re.S)
    fields = []
    for kind, names in re.findall(r"(int|float)\s+([^;]+);", body):
        fields += [(n.strip(), kind) for n in names.split(",")]
    import ctypes
    assert [(n, "int" if t is ctypes.c_int else "float") for n, t in C.LayerSpec._fields_] == fields


def test_registry_picks_the_class_by_config():
    from cpmcu.llm import LLM
    from cpmcu.llm_w4a16_gptq_marlin import W4A16GPTQMarlinLLM
    from cpmcu.models import model_class
    from cpmcu.tipetar import TipetarLLM
    assert model_class({"architecture": "Tipetar"}) is TipetarLLM
    assert model_class({"architectures": ["LlamaForCausalLM"]}) is LLM
    assert model_class({"architectures": ["LlamaForCausalLM"], "quantization_config": {"bits": 4}}) is W4A16GPTQMarlinLLM


def test_random_weights_follow_the_shapes():
    cfg = model(64, 50, [(attn(2, 1, 8, 4, 3), moe(2, 1, 8, identity=1, shared=4)), (attn(2, 1, 8, 4, 9, kv_from=0), None)])
    w = T.random_weights(cfg)
    assert w["l0.mix.o"].shape == (64, 8) and w["l0.mlp.router"].shape == (3, 64) and w["l0.mlp.shared.up"].shape == (4, 64)
    assert "l1.mix.k" not in w and "l1.mix.k.norm" not in w and "l1.norm2" not in w and "l0.mlp.e2.gate" not in w


class FakeLLM:
    def __init__(self):
        import types
        self.config, self.calls = types.SimpleNamespace(vocab_size=10), []

    def extend(self, tokens, history, want):
        self.calls.append((list(tokens), history, list(want)))
        return torch.zeros(len(want), 10)


def test_trace_keeps_one_sequence_and_gives_it_back():
    from cpmcu.trace import Trace
    llm = FakeLLM()
    t = Trace(llm)
    assert t.step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": []}], "end": []}) is None
    assert t.step({"step": 1, "entries": [{"id": "a", "tokens": [4], "want": [0]}], "end": ["a"]}).shape == (1, 10)
    t.step({"step": 2, "entries": [{"id": "a", "tokens": [5], "want": [0]}], "end": []})
    assert llm.calls == [([1, 2, 3], 0, []), ([4], 3, [0]), ([5], 0, [0])]
    with pytest.raises(ValueError):
        t.step({"step": 3, "entries": [{"id": "b", "tokens": [5], "want": []}], "end": []})
    with pytest.raises(ValueError):
        t.step({"step": 4, "entries": [{"id": "a", "tokens": [10], "want": []}], "end": []})
