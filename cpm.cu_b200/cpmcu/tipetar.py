"""`TipetarLLM`: decoders of the Tipetar design, whose config.json lists every layer with its own sizes.

Per layer: softmax attention with a query / key norm over the whole projections, a distance bias instead of a rotation, a
sliding window and, in some layers, the keys and values of an earlier layer; then a mixture of experts with a shared
expert, identity experts and a grouped choice.  The norms sit on the sublayers' outputs and the residual stream is 32-bit.
Everything runs in the native engine as a layered model (`cpmcu_init_layered_model`); generation, sampling, chunking and the
cache are those of `LLM`.
"""
import json
import os
import types

import torch

from . import C
from .llm import LLM

BIAS_EXP = 8.0   # slope of head h of H: 2^(-8 (h + 1) / H)


def layer_spec(index, layer):
    """C.LayerSpec of one entry of config['layers']."""
    if layer["type"] != "attention":
        raise ValueError(f"layer {index}: unknown mixer '{layer['type']}'")
    mix, mlp = layer["mixer"], layer.get("mlp")
    kv_from = mix.get("kv_from")
    spec = C.LayerSpec(heads=mix["heads"], kv_heads=mix["kv_heads"], dim=mix["dim"], vdim=mix["vdim"], scale=mix["scale"],
                       window=(mix.get("mask") or {}).get("size") or 0, bias_exp=BIAS_EXP, qk_norm=1,
                       kv_from=-1 if kv_from is None else kv_from, groups=1, keep_groups=1, router_scale=1.0)
    if mlp is None:
        return spec
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {index}: unknown feed-forward '{mlp['kind']}'")
    router, groups = mlp["router"], mlp["router"].get("groups")
    spec.experts, spec.identity, spec.top = router["experts"], router.get("identity") or 0, router["top"]
    if groups:
        spec.groups, spec.keep_groups = groups["count"], groups["keep"]
    spec.router_scale = router.get("scale", 1.0)
    spec.expert_ff = mlp["expert"]["ff"]
    spec.shared_ff = mlp["shared"]["ff"] if mlp.get("shared") else 0
    return spec


class TipetarLLM(LLM):
    def __init__(self, path=None, cuda_graph=True, **kwargs):
        super().__init__(path, cuda_graph=cuda_graph, **kwargs)

    def _read_config(self, path, config, tokenizer):
        if config is None:
            with open(os.path.join(path, "config.json")) as f:
                config = json.load(f)
        self.tokenizer = tokenizer
        self.model_config = config
        self.config = types.SimpleNamespace(vocab_size=config["vocab"], hidden_size=config["width"],
                                            num_hidden_layers=len(config["layers"]), torch_dtype=torch.bfloat16)

    def _create_native(self, memory_limit, apply_sparse, sparse_args):
        if apply_sparse:
            raise ValueError("apply_sparse: block selection belongs to MiniCPM4 targets")
        cfg = self.model_config
        C.init_layered_model(memory_limit, cfg["vocab"], cfg["width"], cfg["norm"]["eps"], cfg.get("residual_mult", 1.0),
                             self.dtype_int, self.chunk_length, [layer_spec(i, x) for i, x in enumerate(cfg["layers"])])

    def _load(self, name, param, dtype=None, cls=None):
        # weights are bf16 whatever the activations are
        param = param.contiguous().to(torch.bfloat16)
        C.load_model(name, param.data_ptr())

    def load_from_hf(self):
        with torch.no_grad():
            self._load_from_ckpt(self.path)

    def load_state_dict_tensors(self, tensors, cls=None):
        with torch.no_grad():
            for name, param in tensors.items():
                self._load(name, param)
