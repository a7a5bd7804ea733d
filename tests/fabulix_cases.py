"""Small Fabulix configurations for the tests.  No two layers of a model are alike, and sizes that a model could happen to have
equal (head counts and widths, rotated dimensions, scales, limits, feed-forward widths) differ."""
import copy


def left(heads, kv_heads, dim, vdim, rot, scale=None, base=10000.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "rot": {"dims": rot, "base": base}}


def parallel(lft, heads, dim, left_scale=1.0, right_scale=1.0, mlp=None):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": lft, "right": {"heads": heads, "dim": dim}, "left_scale": left_scale, "right_scale": right_scale}}


def lightning(heads, dim, vdim, decay, mlp=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def model(width, vocab, layers, side, scale=3.0, eps=1e-5):
    return {"architecture": "Fabulix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "token_side": {"dim": side}, "layers": layers}


CASES = {
    # three query heads per key head, part of a head rotated, every kind of layer with and without feed-forward
    "mixed": model(200, 333, [
        lightning(3, 24, 40, [0.3, 0.999, 0.87]),
        parallel(left(6, 2, 40, 56, 16, scale=0.21, base=500.0), 5, 16, 0.7, 1.3, dense(100, 0.8)),
        lightning(2, 64, 32, [1.0, 0.95], dense(72, 1.7)),
        parallel(left(4, 4, 64, 96, 64, scale=0.13), 3, 40, 1.2, 0.6),
    ], side=12, scale=5.0, eps=1e-4),
    # 128-wide heads, one key head, recurrences as wide as one warp set takes, a wide side input
    "wide": model(384, 512, [
        parallel(left(8, 1, 128, 64, 128, base=1e6), 3, 128, 0.9, 1.1, dense(320, 2.0)),
        lightning(2, 128, 256, [0.97, 0.5], dense(192, 0.6)),
        parallel(left(2, 2, 96, 128, 80), 4, 64, 0.5, 0.8, dense(64, 1.1)),
        lightning(5, 32, 128, [0.999, 0.9, 0.8, 0.7, 0.01]),
    ], side=72, scale=11.0),
    # widths beyond the tensor-core attention and the one-token recurrence
    "plain": model(320, 260, [
        parallel(left(4, 2, 136, 144, 112, scale=0.05), 2, 160, 1.1, 0.4, dense(80, 0.9)),
        lightning(2, 200, 24, [0.92, 0.992]),
        parallel(left(2, 1, 64, 192, 32), 1, 256, 0.8, 0.9),
    ], side=20, scale=2.0),
    # nothing divides anything
    "odd": model(75, 101, [
        parallel(left(3, 1, 9, 7, 6, scale=0.4, base=37.0), 3, 7, 0.6, 1.4, dense(13, 0.7)),
        lightning(3, 5, 11, [0.6, 0.99, 0.2], dense(21, 1.3)),
        parallel(left(5, 5, 17, 3, 10), 2, 33, 1.5, 0.5, dense(66, 0.5)),
        lightning(1, 37, 1, [0.985]),
    ], side=3, scale=1.5, eps=1e-3),
}


def case(name):
    return copy.deepcopy(CASES[name])


def shapes_of(weights):
    return {k: tuple(v.shape) for k, v in weights.items()}
