"""The tests' own small configurations of the Ruzunex design, and weights for them.

They differ from one another in every size and in the order of the layers: one to five streams; convolutions of one to
five taps, of the sublayers' inputs and of the projections; query heads over fewer, as many and a single kv head; value
rows narrower than, as wide as and wider than key rows; rotated coordinates fewer than and equal to the head's, and
none; windows shorter than, equal to and longer than a cache page, down to one token; values mixed over layers of
different head counts, from a first mixing layer that is not the model's first, next to layers that do not mix;
recurrences whose value rows are narrower and wider than their key rows; one to four experts a token, one of two, and all
of them; dense feed-forwards and layers without one; the pair's constants equal, different and negative.  Matrices are
drawn wide so that weights are far from uniform."""
import copy

import torch


def window(heads, kv_heads, dim, vdim, size, v_mix=True, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
         "scale": scale if scale is not None else dim ** -0.5}
    if v_mix is not None:
        m["v_mix"] = v_mix
    return {"type": "attention", "mixer": m}


def pair(left, right, left_scale, right_scale):
    """left: (heads, kv heads, dim, vdim, taps, rotated, base[, scale]); right: (heads, dim, vdim)."""
    h, g, d, v, taps, rot, base = left[:7]
    return {"type": "parallel", "mixer": {
        "left": {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "conv": taps, "rot": {"base": base, "dims": rot},
                 "scale": left[7] if len(left) > 7 else d ** -0.5},
        "right": {"heads": right[0], "dim": right[1], "vdim": right[2]},
        "left_scale": left_scale, "right_scale": right_scale}}


def dense(layer, ff):
    layer = copy.deepcopy(layer)
    layer["mlp"] = None if ff is None else {"kind": "dense", "ff": ff}
    return layer


def moe(layer, experts, top, ff, limit):
    layer = copy.deepcopy(layer)
    layer["mlp"] = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    return layer


def model(vocab, width, eps, streams, taps, layers):
    return {"architecture": "Ruzunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "canon": {"taps": taps}, "layers": layers}


# odd sizes that no fast kernel takes; the first mixing layer is the third; three streams
A = model(97, 44, 1e-5, 3, 4,
          [moe(pair((6, 3, 10, 14, 2, 6, 300.0, 0.4), (3, 7, 9), 0.7, 1.3), 6, 2, 18, 1.2),
           dense(window(5, 5, 8, 6, 11, v_mix=False), 30),
           dense(window(4, 2, 12, 21, 9, scale=0.35), None),
           moe(window(6, 3, 6, 14, 30), 5, 3, 12, 0.8),
           dense(pair((2, 1, 14, 10, 5, 0, 50.0), (2, 12, 5), 1.1, -0.6), 26),
           dense(window(7, 1, 10, 42, 17), 22)])

# round sizes, which every fast kernel takes
B = model(256, 128, 1e-6, 4, 5,
          [dense(window(8, 4, 64, 64, 100), 128),
           moe(pair((8, 2, 64, 128, 4, 32, 10000.0), (2, 64, 64), 0.5, 1.5), 8, 2, 64, 1.25),
           moe(window(4, 2, 128, 128, 70), 16, 4, 64, 2.5),
           dense(pair((4, 4, 128, 64, 2, 128, 5000.0), (4, 128, 32), 1.0, 0.9), 256),
           dense(window(16, 2, 64, 128, 64), None)])

# what another model might make equal or one: one stream, one tap, a single head, a window of one token and of exactly a
# page, one expert of two, both constants one, a single mixing layer
C = model(50, 32, 1e-4, 1, 1,
          [dense(window(1, 1, 16, 8, 1, v_mix=None), 16),
           moe(pair((1, 1, 16, 8, 1, 16, 20.0), (1, 8, 16), 1.0, 1.0), 2, 1, 8, 1.0),
           dense(window(2, 1, 8, 24, 64), None),
           moe(pair((3, 1, 8, 8, 3, 2, 100.0), (2, 16, 16), 1.0, 1.0), 3, 3, 8, 4.0)])

# head sizes between the tensor-core kernel's tile sizes; five streams, two taps
D = model(300, 160, 1e-6, 5, 2,
          [moe(window(6, 2, 40, 80, 150), 8, 2, 32, 1.3),
           dense(pair((6, 3, 80, 112, 3, 40, 7000.0), (2, 96, 136), 0.9, 0.8), 96),
           dense(window(10, 5, 104, 32, 200), 64),
           moe(pair((2, 2, 72, 40, 6, 72, 500.0), (1, 24, 200), 1.2, 0.4), 4, 2, 64, 1.0)])

CONFIGS = {"A": (A, 41, 0.3), "B": (B, 42, 0.2), "C": (C, 43, 0.4), "D": (D, 44, 0.2)}


def build(name_or_cfg, seed=0, std=0.3, every_expert=False):
    """(typed configuration, weight store, the weights by name).  ``every_expert``: all experts a token instead of the
    best ones, with the same weights.  bfloat16 may pick another expert for a token whose best scores are nearly level,
    which moves that token by its whole size and, through keys and states, the tokens behind it: whole-model tests in
    bfloat16 run without the choice (the weighing, sorting and combining stay), float32 ones with it."""
    from supersonic_b200.config import config_from_dict
    from supersonic_b200.weights import random_store
    if isinstance(name_or_cfg, str):
        name_or_cfg, seed, std = CONFIGS[name_or_cfg]
    if every_expert:
        name_or_cfg = copy.deepcopy(name_or_cfg)
        for layer in name_or_cfg["layers"]:
            if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
                layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    cfg = config_from_dict(name_or_cfg)
    store = random_store(cfg, seed, std=std)
    plain = {n: store.get(n) for n in store.names()}
    return cfg, store, plain


def changed(plain, changes):
    """(weight store, weights by name) with some tensors replaced: ``changes`` maps names to tensors."""
    from supersonic_b200.weights import WeightStore
    t = dict(plain)
    for name, v in changes.items():
        t[name] = v.to(t[name].dtype)
    return WeightStore.from_tensors(t), t
