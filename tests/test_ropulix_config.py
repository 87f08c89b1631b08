"""The Ropulix configuration on the CPU: its reader and refusals, the parts and the schedule it builds, what the cache is
asked for, and the plain statement's own masks, routing and recurrence."""
import copy

import pytest
import torch

import plain_ropulix as pr
import tiny_ropulix as tr
from supersonic_b200.cache import KvNeed, StateNeed
from supersonic_b200.config import ConfigError, config_from_dict, preset_config
from supersonic_b200.parts import MIXERS


def test_reads_and_writes_back():
    for name, (d, _, _) in tr.CONFIGS.items():
        cfg = config_from_dict(d)
        assert cfg.to_dict() == config_from_dict(cfg.to_dict()).to_dict(), name
        assert cfg.architectures == ["Ropulix"] and cfg.vocab_size == d["vocab"] and cfg.hidden_size == d["width"]
        assert cfg.num_hidden_layers == len(d["layers"])
    assert preset_config("ropulix-small").num_hidden_layers >= 4


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].update(type="mamba"), "not known"),
    (lambda d: d["layers"][2]["mixer"].update(heads=5), "kv heads"),
    (lambda d: d["layers"][2]["mixer"]["mask"].update(size=0), "positive"),
    (lambda d: d["layers"][2]["mixer"].pop("mask"), "missing"),
    (lambda d: d["layers"][2]["mixer"].update(kv_from=0), "only a layer of latent_attention"),
    (lambda d: d["layers"][1]["mixer"].update(blocks=4), "blocks"),
    (lambda d: d["layers"][1]["mixer"].update(conv=17), "taps"),
    (lambda d: d["layers"][0]["mixer"].pop("q_rank"), "missing"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=4), "rot.dims"),
    (lambda d: d["layers"][0]["mixer"].update(scale=0), "scale"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=4), "earlier layer"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=1), "keeps no latent rows"),
    (lambda d: d["layers"][3]["mixer"].update(kv_rank=20), "differs"),
    (lambda d: d["layers"][3]["mixer"]["rot"].update(base=5.0), "differs"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "experts a token"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "not known"),
    (lambda d: d["layers"][0]["mlp"].pop("expert"), "missing"),
    (lambda d: d.pop("norm"), "missing"),
])
def test_refusals(change, message):
    d = copy.deepcopy(tr.A)
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)


def test_parts_schedule_and_what_the_cache_is_asked_for():
    cfg = config_from_dict(tr.A)
    spec = cfg.build_spec()
    assert [(s.layer, s.cache, s.writes_cache) for s in spec.schedule] == \
        [(0, 0, True), (1, 1, True), (2, 2, True), (3, 0, False), (4, 4, True), (5, 5, True)]
    # the entry of layer 0 keeps rows for its reader's longer window; both say so
    assert cfg.cache_reach(0) == 30
    writer, reads = (MIXERS["latent_attention"].cache_need_from(spec.blocks[i].mixer.params) for i in (0, 3))
    assert writer == reads == KvNeed(1, 22 + 6, 30, value_dim=0)
    assert spec.blocks[0].mixer.params["window"] == 9 and spec.blocks[3].mixer.params["window"] == 30
    assert "dkv" in spec.blocks[0].mixer.weights and "dkv" not in spec.blocks[3].mixer.weights
    assert MIXERS["real_gated_recurrence"].cache_need_from(spec.blocks[1].mixer.params) == \
        {"state": StateNeed(30), "tail": StateNeed(3 * 30)}
    assert MIXERS["window_attention"].cache_need_from(spec.blocks[2].mixer.params) == KvNeed(3, 10, 21, value_dim=14)
    # the stream is read as it is: no norms in front, a rounded copy handed from stop to stop, none behind the last
    assert all(b.kind == "post_norm" and b.mixer_norm is None and b.feed_forward_norm is None for b in spec.blocks)
    assert [b.params["leaves_rounded"] for b in spec.blocks] == [True] * 5 + [False]
    assert spec.head.weights == spec.embedding.weights
    # several readers, one of them with a shorter window than the writer
    d = config_from_dict(tr.D)
    assert d.cache_reach(0) == 200 and [d.kv_source(i) for i in range(6)] == [0, 0, 2, 3, 0, 5]


def test_tensor_shapes_and_random_weights():
    cfg, store, plain = tr.build("A")
    shapes = cfg.tensor_shapes()
    assert set(shapes) == set(store.names())
    assert shapes["l0.mix.uq"] == [6 * 16, 18] and shapes["l0.mix.dkv"] == [28, 44] and shapes["l0.mix.g"] == [84, 44]
    assert "l3.mix.dkv" not in shapes and "l3.mix.dkv.norm" not in shapes and shapes["l3.mix.uk"] == [24, 22]
    assert shapes["l1.mix.ra"] == [3, 10, 10] and shapes["l1.mix.ri.b"] == [3, 10] and shapes["l1.mix.conv"] == [30, 4]
    assert shapes["l2.mix.g"] == [6, 44] and "l2.mix.q.norm" not in shapes
    assert "l1.norm2" not in shapes and cfg.ignorable_tensor("l1.norm2") and not cfg.ignorable_tensor("l2.norm2")
    assert shapes["l0.mlp.router.b"] == [6] and shapes["l0.mlp.e5.up"] == [18, 44] and "head" not in shapes
    decay = torch.exp(-8.0 * 0.5 * torch.log1p(torch.exp(plain["l1.mix.lam"].double())))
    assert float(decay.max()) > 0.9 and float(decay.min()) < 0.7         # channels that remember, and channels that forget


def test_plain_route_weighs_the_chosen_alone():
    cfg, _, plain = tr.build("A")
    h = torch.randn(40, 44, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    chosen, weight = pr.route(h, plain, "l0.mlp", 2)
    z = h @ plain["l0.mlp.router"].double().T + plain["l0.mlp.router.b"].double()
    for t in range(40):
        assert abs(sum(weight[t]) - 1.0) < 1e-12 and len(set(chosen[t])) == 2
        assert float(z[t, chosen[t]].min()) >= float(z[t].sort(descending=True).values[1]) - 1e-12
        assert abs(weight[t][0] / weight[t][1] - float(torch.exp(z[t, chosen[t][0]] - z[t, chosen[t][1]]))) < 1e-9


def test_plain_masks_and_recurrence():
    """A window of n tokens sees the token itself and the n - 1 before it; the model is causal; the recurrence's first
    token is like any other; a state decays and what enters it is scaled so that its size stays."""
    assert pr.in_window(5, 1) == [5] and pr.in_window(5, 3) == [3, 4, 5] and pr.in_window(1, 9) == [0, 1]
    cfg, _, plain = tr.build("C")
    toks = [3, 9, 27, 31, 4, 4, 18, 40, 2, 11]
    a, _ = pr.forward(tr.C, plain, toks)
    b, _ = pr.forward(tr.C, plain, toks[:6])
    assert float((a[:6] - b).abs().max()) < 1e-9
    x = torch.randn(9, 5, dtype=torch.float64)
    w, bias = torch.randn(5, 3, dtype=torch.float64), torch.randn(5, dtype=torch.float64)
    y = pr.causal_conv(x, w, bias)
    assert torch.allclose(y[0], bias + w[:, 2] * x[0])
    assert torch.allclose(y[4], bias + w[:, 0] * x[2] + w[:, 1] * x[3] + w[:, 2] * x[4])
    r = pr.turn(torch.ones(7, 2, 4, dtype=torch.float64), 4, 10.0)
    assert torch.allclose(r[0], torch.ones(2, 4, dtype=torch.float64)) and torch.allclose((r ** 2).sum(-1), torch.full((7, 2), 4.0, dtype=torch.float64))


def test_the_sharpened_weights_reveal_every_fault():
    """What the whole-model tests rest on: with these weights each planted fault, and a window one token longer or shorter,
    gives other logits at many positions, and a sequence that has lost its beginning gives others at its end."""
    cfg, _, plain = tr.sharpened("A")
    tokens = torch.randint(0, cfg.vocab, (200,), generator=torch.Generator().manual_seed(9)).tolist()
    ref = pr.forward(cfg.to_dict(), plain, tokens)[0]

    def error(got):
        return (got - ref[-got.shape[0]:]).pow(2).mean(-1).sqrt() / ref[-got.shape[0]:].std(-1)
    others = [(f, pr.forward(cfg.to_dict(), plain, tokens, {f})[0]) for f in tr.FAULTS]
    others += [(c, pr.forward(tr.changed_layer(cfg, *c), plain, tokens)[0]) for c in tr.CHANGES]
    for what, got in others:
        e = error(got)[40:]
        assert float((e > 0.02).double().mean()) > 0.4 and float(e.max()) > 0.3, what
    assert float(error(pr.forward(cfg.to_dict(), plain, tokens, {"first_token"})[0])[:40].median()) > 0.02
    assert float(error(pr.forward(cfg.to_dict(), plain, tokens[120:])[0])[-20:].min()) > 0.05
