"""`TipetarLLM`: decoders of the Tipetar design, whose config.json lists every layer with its own sizes.

Per layer: softmax attention with a query / key norm over the whole projections, a distance bias instead of a rotation, a
sliding window and, in some layers, the keys and values of an earlier layer; then a mixture of experts with a shared
expert, identity experts and a grouped choice.  The norms sit on the sublayers' outputs and the residual stream is 32-bit.
Everything runs in the native engine (`layered.py`).
"""
from . import C
from .layered import LayeredLLM

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


class TipetarLLM(LayeredLLM):
    def layer_specs(self):
        return [layer_spec(i, layer) for i, layer in enumerate(self.model_config["layers"])]
