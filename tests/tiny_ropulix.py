"""The tests' own small configurations of the Ropulix design, and weights for them.

They differ from one another in every size and in the order of the layers: query heads over fewer, as many and a single
kv head; value rows narrower than, as wide as and wider than key rows; latents narrower and wider than what is made of
them; rotated parts of two coordinates and more; windows shorter than, equal to and longer than a cache page, down to one
token; latent layers that read an earlier one's rows with a shorter and with a longer window and with head counts, head
sizes and query latents of their own; recurrences of one to many blocks (of one channel, too) behind convolutions of one
to sixteen taps; one to four experts a token, one of one, and all of them; layers without a feed-forward.  Matrices are
drawn wide so that weights are far from uniform."""
import copy

import torch


def heads(n, kv, dim, vdim, size, scale=None):
    return {"type": "attention", "mixer": {"heads": n, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": size},
                                           "scale": scale if scale is not None else dim ** -0.5}}


def latent(n, dim, rot, vdim, rank, q_rank, size, base, scale=None):
    return {"type": "latent_attention", "mixer": {
        "heads": n, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "mask": {"size": size},
        "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else (dim + rot) ** -0.5}}


def reader(layers, j, size, **own):
    """A layer that reads layer j's rows, with a window (and heads, head sizes, a query latent) of its own."""
    layer = copy.deepcopy(layers[j])
    layer["mixer"].update(own, kv_from=j, mask={"size": size})
    return layer


def rglru(width, blocks, taps):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": taps}}


def moe(layer, experts=None, top=None, ff=None):
    layer = copy.deepcopy(layer)
    layer["mlp"] = None if experts is None else {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return layer


def model(vocab, width, eps, layers):
    return {"architecture": "Ropulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# odd sizes that no fast kernel takes; a reader with a longer window than its writer
_a = [moe(latent(6, 10, 6, 14, 22, 18, 9, 300.0, scale=0.4), 6, 2, 18), moe(rglru(30, 3, 4)), moe(heads(6, 3, 10, 14, 21, scale=0.5), 5, 3, 12)]
A = model(97, 44, 1e-5, _a + [moe(reader(_a, 0, 30, heads=4, dim=6, vdim=9, q_rank=26), 3, 1, 10), moe(heads(5, 5, 7, 6, 11)),
                              moe(rglru(21, 1, 2), 4, 2, 26)])

# round sizes, which every fast kernel takes; a reader with a shorter window than its writer
_b = [moe(rglru(128, 2, 4), 8, 2, 64), moe(latent(4, 64, 32, 64, 128, 96, 100, 10000.0), 8, 2, 128),
      moe(heads(8, 2, 64, 128, 70), 16, 4, 64)]
B = model(256, 128, 1e-6, _b + [moe(reader(_b, 1, 40, heads=2, dim=128, vdim=32), 4, 3, 192), moe(rglru(256, 4, 3)),
                                moe(heads(4, 4, 128, 64, 64, scale=0.2), 8, 1, 64)])

# what another model might make equal or one: one head, one tap, one block, blocks of one channel, a window of one token
# and of exactly a page, one expert of one, all experts
C = model(50, 32, 1e-4, [moe(latent(1, 1, 2, 8, 16, 8, 64, 20.0), 2, 1, 8), moe(rglru(16, 1, 1), 1, 1, 12), moe(heads(1, 1, 16, 8, 1)),
                         moe(rglru(8, 8, 16), 3, 3, 16), moe(latent(3, 8, 16, 8, 8, 32, 1, 500.0)), moe(heads(3, 1, 8, 8, 64), 4, 2, 8)])

# sizes between the tensor-core kernels' tiles; several readers of one entry, one right behind its writer
_d = [moe(latent(5, 40, 16, 48, 80, 72, 150, 7000.0), 8, 2, 40)]
D = model(300, 160, 1e-6, _d + [moe(reader(_d, 0, 64), 4, 2, 64), moe(rglru(200, 5, 5), 4, 2, 72), moe(heads(6, 2, 40, 80, 130)),
                                moe(reader(_d, 0, 200, heads=8, dim=24, vdim=16, q_rank=40), 8, 3, 32), moe(heads(10, 5, 104, 32, 200))])

CONFIGS = {"A": (A, 51, 0.3), "B": (B, 52, 0.12), "C": (C, 53, 0.4), "D": (D, 54, 0.2)}


def build(name_or_cfg, seed=0, std=0.3, every_expert=False):
    """(typed configuration, weight store, the weights by name).  ``every_expert``: all experts a token instead of the
    best ones, with the same weights.  bfloat16 may pick another expert for a token whose best logits are nearly level,
    which moves that token by its whole size and, through keys and states, the tokens behind it: whole-model tests in
    bfloat16 run without the choice (the weighing, sorting and combining stay), float32 ones with it."""
    from supersonic_b200.config import config_from_dict
    from supersonic_b200.weights import random_store
    if isinstance(name_or_cfg, str):
        name_or_cfg, seed, std = CONFIGS[name_or_cfg]
    if every_expert:
        name_or_cfg = copy.deepcopy(name_or_cfg)
        for layer in name_or_cfg["layers"]:
            if layer["mlp"] is not None:
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


def sharpened(name="A", sharp=2.0, every_expert=False):
    """(typed configuration, weight store, weights by name) with the scores' scales ``sharp`` times as large, so that a
    query's output stands on the few keys whose scores are high: a key more or less then moves the logits by far more than
    any tolerance."""
    d, seed, std = CONFIGS[name]
    d = copy.deepcopy(d)
    for layer in d["layers"]:
        if "scale" in layer["mixer"]:
            layer["mixer"]["scale"] *= sharp
    return build(d, seed, std, every_expert)


# Faults planted in the plain statement by name (weights of the experts that are all too large by one factor are not among
# them: the norm behind the experts takes the factor out), and changes of a layer that stand for one: (layer, key, value)
FAULTS = ("no_qk_norm", "no_gate", "head_order", "attention_window", "no_query_norm", "no_rotation", "latent_window",
          "no_latent_gate", "flipped_taps", "state_lost", "no_router_bias", "one_expert_more", "norm_before")
CHANGES = ((0, "mask", {"size": 8}), (2, "mask", {"size": 20}), (2, "mask", {"size": 22}), (3, "mask", {"size": 29}),
           (3, "mask", {"size": 31}), (4, "mask", {"size": 10}), (4, "mask", {"size": 12}), (3, "mask", {"size": 9}))


def changed_layer(cfg, layer, key, value):
    d = copy.deepcopy(cfg.to_dict())
    d["layers"][layer]["mixer"][key] = value
    return d
