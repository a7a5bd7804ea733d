"""Small Tipetar configurations for the tests.  No two layers of a model are alike, and sizes that a model could happen to
have equal (head widths, windows, feed-forward widths, query and key heads) differ."""
import copy


def moe(experts, top, ff, identity=0, groups=None, scale=1.0, shared=None):
    router = {"experts": experts, "top": top, "scale": scale, "identity": identity}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router, "shared": {"ff": shared} if shared else None}


def attn(heads, kv_heads, dim, vdim, window, scale=None, kv_from=None):
    mix = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
           "mask": {"size": window} if window else None}
    if kv_from is not None:
        mix["kv_from"] = kv_from
    return mix


def model(width, vocab, layers, mult=0.7, eps=1e-5):
    return {"architecture": "Tipetar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


CASES = {
    # three query heads per key head, narrow heads, a layer without feed-forward that borrows layer 0's keys under
    # another window and scale, widths that are not multiples of 64
    "mixed": model(200, 333, [
        (attn(6, 2, 40, 56, 37, scale=0.21), moe(5, 3, 36, identity=3, groups=(4, 2), scale=1.7, shared=100)),
        (attn(6, 2, 40, 56, 61, scale=0.13, kv_from=0), None),
        (attn(4, 4, 64, 32, 130), moe(7, 2, 72, scale=0.6)),
        (attn(4, 4, 64, 32, 5, kv_from=2), moe(3, 4, 40, identity=5, shared=24)),
    ], mult=0.43, eps=1e-4),
    # 128-wide heads, one key head, a window of exactly one key tile, many experts
    "wide": model(384, 512, [
        (attn(8, 1, 128, 64, 128), moe(40, 6, 64, identity=8, groups=(6, 3), scale=2.5, shared=192)),
        (attn(2, 2, 64, 128, 300), moe(33, 5, 128)),
        (attn(8, 1, 128, 64, 200, kv_from=0), moe(10, 3, 48, identity=2, groups=(4, 1), shared=64)),
    ], mult=1.0),
    # head widths beyond the tensor-core kernel, no window
    "plain": model(320, 260, [
        (attn(4, 2, 136, 144, None, scale=0.05), moe(4, 2, 64, identity=4, groups=(2, 2), shared=96)),
        (attn(2, 1, 64, 192, 70), moe(6, 1, 80)),
    ], mult=0.9),
    # nothing divides anything
    "odd": model(75, 101, [
        (attn(3, 1, 9, 7, 11, scale=0.4), moe(3, 2, 13, identity=1, groups=(2, 1), scale=0.5, shared=5)),
        (attn(5, 5, 17, 3, 20), moe(5, 5, 21)),
        (attn(3, 1, 9, 7, 19, scale=0.2, kv_from=0), moe(2, 1, 30, identity=2, shared=66)),
    ], mult=1.3, eps=1e-3),
}


def case(name):
    return copy.deepcopy(CASES[name])
