"""`FabulixLLM`: decoders of the Fabulix design, whose config.json lists every layer with its own sizes.

A layer's mixer is lightning attention (a recurrence with one constant decay per head), or softmax attention with rotary
positions and a sink side by side with a time mix (a recurrence with decays per token and channel).  The norms are dynamic
tanh, before and after every sublayer; the feed-forward is a clamped gate; every layer adds an input of its own for each
token, and the head is the embedding table.
"""
import torch

from . import C
from .layered import LayeredLLM

GATE_ALPHA = 1.702   # y = g sigmoid(1.702 g) (u + 1)


def layer_spec(index, layer, shapes):
    """C.LayerSpec of one entry of config['layers']; `shapes` gives the inner width of a time mix's decay."""
    kind, mix, mlp = layer["type"], layer["mixer"], layer.get("mlp")
    if kind == "lightning":
        spec = C.LayerSpec(recurrence=C.REC_LIGHTNING, rec_heads=mix["heads"], rec_dim=mix["dim"], rec_vdim=mix["vdim"])
    elif kind == "parallel":
        left, right = mix["left"], mix["right"]
        rank = shapes.get(f"l{index}.mix.right.w1")
        if rank is None:
            raise ValueError(f"layer {index}: the shape of l{index}.mix.right.w1 is not known")
        spec = C.LayerSpec(heads=left["heads"], kv_heads=left["kv_heads"], dim=left["dim"], vdim=left["vdim"], scale=left["scale"],
                           sink=1, rot_dims=(left.get("rot") or {}).get("dims", 0), attn_scale=mix.get("left_scale", 1.0),
                           recurrence=C.REC_TIME_MIX, rec_heads=right["heads"], rec_dim=right["dim"], rec_vdim=right["dim"],
                           rec_rank=rank[0], rec_scale=mix.get("right_scale", 1.0))
    else:
        raise ValueError(f"layer {index}: unknown mixer '{kind}'")
    if mlp is not None:
        if mlp["kind"] != "dense":
            raise ValueError(f"layer {index}: unknown feed-forward '{mlp['kind']}'")
        spec.ff, spec.ff_limit, spec.ff_alpha = mlp["ff"], mlp["limit"], GATE_ALPHA
    return spec


class FabulixLLM(LayeredLLM):
    def layer_specs(self):
        return [layer_spec(i, layer, self.shapes()) for i, layer in enumerate(self.model_config["layers"])]

    def model_options(self):
        cfg = self.model_config
        return dict(norm=C.NORM_DYNAMIC_TANH, embed_scale=(cfg.get("embedding") or {}).get("scale", 1.0), tied_head=True,
                    side_dim=(cfg.get("token_side") or {}).get("dim", 0))

    def constants(self):
        out = {}
        for i, layer in enumerate(self.model_config["layers"]):
            mix = layer["mixer"]
            if layer["type"] == "lightning":
                decay = torch.as_tensor(mix["decay"], dtype=torch.float64)
                out[f"l{i}.mix.decay"] = decay.expand(mix["heads"])
            elif (mix["left"].get("rot") or {}).get("dims"):
                rot = mix["left"]["rot"]
                out[f"l{i}.mix.left.inv_freq"] = rot["base"] ** (-torch.arange(0, rot["dims"], 2, dtype=torch.float64) / rot["dims"])
        return out
