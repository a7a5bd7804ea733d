"""`LayeredLLM`: base class of designs whose config.json lists every layer with its own sizes.

Such a model runs in the native engine as a layered model (`cpmcu_init_layered_model`); generation, sampling, chunking and
the cache are those of `LLM`.  A design supplies `layer_specs()`, and where it differs from the defaults `model_options()` and
`constants()`.
"""
import glob
import json
import os
import types

import torch

from . import C
from .llm import LLM


def checkpoint_shapes(path):
    """{tensor name: shape} of the safetensors files in a checkpoint directory, without reading the tensors."""
    from safetensors import safe_open
    shapes = {}
    for name in sorted(glob.glob(os.path.join(path, "*.safetensors"))):
        with safe_open(name, framework="pt") as f:
            for key in f.keys():
                shapes[key] = tuple(f.get_slice(key).get_shape())
    return shapes


class LayeredLLM(LLM):
    """`shapes`: {name: shape} for the sizes that only a tensor has; read from the checkpoint in `path` when not given."""

    def __init__(self, path=None, cuda_graph=True, shapes=None, **kwargs):
        self._given_shapes = shapes
        super().__init__(path, cuda_graph=cuda_graph, **kwargs)

    def _read_config(self, path, config, tokenizer):
        if config is None:
            with open(os.path.join(path, "config.json")) as f:
                config = json.load(f)
        self.tokenizer = tokenizer
        self.model_config = config
        self.config = types.SimpleNamespace(vocab_size=config["vocab"], hidden_size=config["width"],
                                            num_hidden_layers=len(config["layers"]), torch_dtype=torch.bfloat16)

    def layer_specs(self):
        """One C.LayerSpec per layer of `model_config`."""
        raise NotImplementedError

    def model_options(self):
        """Keyword arguments of `C.init_layered_model` beyond the sizes."""
        return {}

    def constants(self):
        """{name: fp32 tensor} the engine takes like weights but that the configuration gives."""
        return {}

    def shapes(self):
        if self._given_shapes is None:
            self._given_shapes = checkpoint_shapes(self.path) if self.path else {}
        return self._given_shapes

    def _create_native(self, memory_limit, apply_sparse, sparse_args):
        if apply_sparse:
            raise ValueError("apply_sparse: block selection belongs to MiniCPM4 targets")
        cfg = self.model_config
        C.init_layered_model(memory_limit, cfg["vocab"], cfg["width"], cfg["norm"]["eps"], cfg.get("residual_mult", 1.0),
                             self.dtype_int, self.chunk_length, self.layer_specs(), **self.model_options())

    def init_storage(self):
        super().init_storage()
        for name, value in self.constants().items():
            self._load(name, value, dtype=torch.float32)

    def _load(self, name, param, dtype=None, cls=None):
        # weights are bf16 whatever the activations are
        param = param.contiguous().to(dtype or torch.bfloat16)
        C.load_model(name, param.data_ptr())

    def load_from_hf(self):
        with torch.no_grad():
            self._load_from_ckpt(self.path)

    def load_state_dict_tensors(self, tensors, cls=None):
        with torch.no_grad():
            for name, param in tensors.items():
                self._load(name, param)
