"""The Ruzunex configuration on the CPU: its reader and refusals, the parts it builds, what the cache is asked for, and
the plain statement's own masks, mixing and routing."""
import copy

import pytest
import torch

import plain_ruzunex as pr
import tiny_ruzunex as tr
from supersonic_b200.config import ConfigError, config_from_dict


def test_reads_and_writes_back():
    for name, (d, _, _) in tr.CONFIGS.items():
        cfg = config_from_dict(d)
        assert cfg.to_dict() == config_from_dict(cfg.to_dict()).to_dict() == d, name
        assert cfg.architectures == ["Ruzunex"] and cfg.vocab_size == d["vocab"] and cfg.hidden_size == d["width"]
        assert cfg.num_hidden_layers == len(d["layers"])


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].update(type="mamba"), "not known"),
    (lambda d: d["layers"][1]["mixer"].update(heads=6), "kv heads"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(heads=5), "kv heads"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(conv=0), "taps"),
    (lambda d: d["layers"][0]["mixer"]["left"].pop("conv"), "missing"),
    (lambda d: d["layers"][0]["mixer"].pop("right_scale"), "missing"),
    (lambda d: d["layers"][0]["mixer"]["right"].update(dim=0), "positive"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), "positive"),
    (lambda d: d["layers"][3]["mixer"].update(vdim=13), "cannot be mixed"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "experts a token"),
    (lambda d: d["layers"][0]["mlp"]["expert"].pop("limit"), "missing"),
    (lambda d: d["layers"][1]["mlp"].update(kind="glu"), "not known"),
    (lambda d: d["canon"].update(taps=17), "taps"),
    (lambda d: d.update(streams=0), "positive"),
    (lambda d: d.update(streams=17), "streams"),
    (lambda d: d.pop("canon"), "missing"),
])
def test_refusals(change, message):
    d = copy.deepcopy(tr.A)
    change(d)
    with pytest.raises(ConfigError, match=message):
        config_from_dict(d)


def test_parts_and_what_the_cache_is_asked_for():
    from supersonic_b200.cache import KvNeed, StateNeed
    from supersonic_b200.engine.preflight import cache_needs
    cfg = config_from_dict(tr.A)
    spec = cfg.build_spec()
    assert [cfg.value_mix(i) for i in range(6)] == [None, None, "first", "later", None, "later"]
    assert [b.kind for b in spec.blocks] == ["hyper_connections"] * 6
    assert [b.params["last"] for b in spec.blocks] == [False] * 5 + [True]
    assert "vmix" in spec.blocks[3].mixer.weights and "vmix" not in spec.blocks[2].mixer.weights
    needs = cache_needs(spec)
    canon = StateNeed(3 * 44)
    assert needs[1] == {"mixer": KvNeed(5, 8, 11, value_dim=6), "conv0": canon, "conv1": canon}
    assert needs[2] == {"mixer": KvNeed(2, 12, 9, value_dim=21), "conv0": canon}            # no feed-forward
    assert needs[0]["mixer"] == {"left": {"tokens": KvNeed(3, 10, None, value_dim=14), "conv": StateNeed(60 + 30 + 42)},
                                 "right": StateNeed(3 * 7 * 9)}
    # one tap keeps nothing
    needs = cache_needs(config_from_dict(tr.C).build_spec())
    assert needs[0] == KvNeed(1, 16, 1, value_dim=8)
    assert needs[1] == {"left": KvNeed(1, 16, None, value_dim=8), "right": StateNeed(8 * 16)}


def test_tensor_shapes_and_random_weights():
    cfg, store, plain = tr.build("A")
    shapes = cfg.tensor_shapes()
    assert set(shapes) == set(store.names())
    assert shapes["l0.mix.left.q"] == [60, 44] and shapes["l0.mix.left.v.conv"] == [42, 2] and shapes["l0.mix.left.q.norm"] == [60]
    assert shapes["l0.mix.right.lower"] == [21] and shapes["l0.mix.right.norm"] == [9] and shapes["l0.mix.right.o"] == [44, 27]
    assert shapes["l3.mix.g"] == [84, 44] and shapes["l3.mix.q.norm"] == [6] and shapes["l3.mix.vmix"] == []
    assert "l1.mix.vmix" not in shapes and "l2.norm2" not in shapes and "l2.hc2.in" not in shapes and "l2.canon2" not in shapes
    assert shapes["l1.hc2.mix"] == [3, 3] and shapes["l0.canon1"] == [44, 4]
    assert cfg.ignorable_tensor("l1.mix.vmix") and cfg.ignorable_tensor("l2.hc2.mix") and not cfg.ignorable_tensor("l3.mix.vmix")
    assert not cfg.ignorable_tensor("l9.norm2") and not cfg.ignorable_tensor("lx.norm2")
    assert 0.0 <= float(plain["l0.mix.right.lower"].float().min()) and float(plain["l0.mix.right.lower"].float().max()) < 1.0


def test_plain_routes_by_softmax_and_renormalizes():
    cfg, _, plain = tr.build("A")
    h = torch.randn(40, 44, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    chosen, weight = pr.route(h, plain, "l3.mlp", tr.A["layers"][3]["mlp"]["router"])
    z = h @ plain["l3.mlp.router"].double().T
    for t in range(40):
        assert set(chosen[t]) == set(torch.topk(z[t], 3).indices.tolist()) and abs(sum(weight[t]) - 1.0) < 1e-9
        assert abs(weight[t][0] / weight[t][1] - float(torch.exp(z[t, chosen[t][0]] - z[t, chosen[t][1]]))) < 1e-6


def test_plain_masks_streams_and_recurrence():
    toks = [3, 9, 27, 31, 4, 4, 18, 40, 2, 11]
    for name in ("A", "C"):
        cfg, _, plain = tr.build(name)
        a, sums = pr.forward(cfg.to_dict(), plain, toks)
        b, _ = pr.forward(cfg.to_dict(), plain, toks[:6])
        assert float((a[:6] - b).abs().max()) < 1e-9                          # causal
        assert sums.shape == (len(cfg.layers), len(toks), cfg.width)
    # the mix matrix is indexed [from, to]; all streams are made from the old ones
    xs = torch.randn(2, 3, 5, dtype=torch.float64)
    y = torch.randn(3, 5, dtype=torch.float64)
    w = {"h.mix": torch.tensor([[1.0, 2.0], [3.0, 4.0]]), "h.out": torch.tensor([5.0, 6.0]), "h.in": torch.tensor([0.5, -1.0])}
    new = pr.write_streams(xs, y, w, "h")
    assert torch.allclose(new[0], xs[0] + 3 * xs[1] + 5 * y) and torch.allclose(new[1], 2 * xs[0] + 4 * xs[1] + 6 * y)
    assert torch.allclose(pr.read_streams(xs, w, "h"), 0.5 * xs[0] - xs[1])
    # a sink takes weight and gives no value; a bias of the distance prefers near keys
    v = torch.eye(2, dtype=torch.float64)
    assert torch.allclose(pr.weighted_sum(torch.zeros(2, dtype=F64), v, sink=0.0), torch.full((2,), 1 / 3, dtype=F64))
    assert pr.slope(0, 8) == 0.5 and pr.slope(7, 8) == 2.0 ** -8
    # what the gate forgets it writes: with constant values the state settles on them
    h = torch.ones(400, 4, dtype=F64)
    one = {"r.q": torch.eye(4), "r.f": torch.zeros(4, 4), "r.f.b": torch.zeros(4), "r.lower": torch.full((4,), 0.5),
           "r.v": torch.eye(4), "r.norm": torch.ones(4), "r.o": torch.eye(4)}
    out = pr.tied_recurrence(h, one, "r", {"heads": 1, "dim": 4, "vdim": 4}, 1e-12)
    assert torch.allclose(out, torch.ones(400, 4, dtype=F64))


F64 = torch.float64
