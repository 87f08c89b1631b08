"""The Ropulix design in the engine against the plain statement of it (``plain_ropulix``): every mechanism alone, the
kernels against one another, then whole models through the step function in every way of cutting and batching, and
generation through the entry point."""
import numpy as np
import pytest
import torch

import plain_ropulix as pr
import tiny_ropulix as tr

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def make_model(cfg, store, dtype, max_tokens=2048, **kw):
    from supersonic_b200.engine import Model
    return Model.from_config(cfg, store, dtype=dtype, device=DEV, max_tokens=max_tokens, **kw)


def run_in_portions(model, tokens, cuts):
    """Logits of every position [T, vocab] with the sequence fed in portions of the given sizes."""
    from supersonic_b200.engine import StepEntry
    slot, at, rows = model.open_sequence(), 0, []
    for n in cuts:
        rows.append(model.step([StepEntry(slot, tokens[at:at + n], list(range(n)))]).cpu())
        at += n
    assert at == len(tokens)
    model.close_sequence(slot)
    model.check_errors()
    return torch.cat(rows).double()


def position_errors(got, ref):
    return (got - ref).pow(2).mean(-1).sqrt() / ref.std(-1).clamp_min(1e-6)


def close(got, ref, dtype, what=""):
    """float32: a few units of float32 rounding of the logits' size.  bfloat16: the error's root mean square per
    position against the spread of that position's logits."""
    assert torch.isfinite(got).all(), what
    if dtype == torch.float32:
        assert float((got - ref).abs().max()) < 2e-4 * max(1.0, float(ref.abs().max())), what
    else:
        rel = position_errors(got, ref)
        assert float(rel.median()) < 0.05 and float(rel.max()) < 0.25, (what, rel.median(), rel.max())


def build_for(name, dtype):
    """float32 runs choose experts, bfloat16 ones take them all (see ``tiny_ropulix.build``)."""
    return tr.build(name, every_expert=dtype != torch.float32)


def tokens_of(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg.vocab, n).tolist()


def reference(cfg, plain, tokens):
    return pr.forward(cfg.to_dict(), plain, tokens)[0]


# ---- the parts alone ---------------------------------------------------------------------------------
def part_context(dtype, store, max_positions=600):
    from supersonic_b200.csrc.kernel_sets import kernel_set_for
    from supersonic_b200.parts import BuildContext, WeightAccess
    return BuildContext(torch.device(DEV), dtype, kernel_set_for(dtype), WeightAccess(store, DEV), max_positions)


def step_context(build, cache, entries):
    from supersonic_b200.engine import StepContext, pack_step
    starts = [cache.length(e.slot) for e in entries]
    batch = pack_step(entries, starts, DEV)
    for e in entries:
        cache.reserve(e.slot, len(e.tokens))
    cache.sync()
    return StepContext(batch, cache, build.kernels, build.dtype)


def mixers_alone(cfg, layers, store, dtype, xs, pieces):
    """What the mixers of ``layers`` add into zeroed streams for one sequence whose rows arrive in pieces, run one after the
    other within a step as layers are (a layer may read another one's cache entry), with rows ``xs[i]`` of their own."""
    from supersonic_b200.cache import SequenceCache
    from supersonic_b200.engine import StepEntry
    from supersonic_b200.parts import MIXERS, POSITION_ENCODINGS
    build = part_context(dtype, store)
    blocks = [cfg.build_spec().blocks[i] for i in layers]
    mixers = [MIXERS[b.mixer.kind](b.mixer.params, b.mixer.weights, build) for b in blocks]
    poss = [None if b.position is None else POSITION_ENCODINGS[b.position.kind](b.position.params, {}, build) for b in blocks]
    for m, b in zip(mixers, blocks):
        assert m.cache_need() == type(m).cache_need_from(b.mixer.params)
    needs = {i: m.cache_need() for i, m in zip(layers, mixers) if cfg.kv_source(i) == i}
    cache = SequenceCache(needs, 1024, 1024, dtype, DEV)
    slot, at, outs = cache.acquire(), 0, [[] for _ in layers]
    for n in pieces:
        ctx = step_context(build, cache, [StepEntry(slot, [0] * n)])
        for j, (i, mixer, pos) in enumerate(zip(layers, mixers, poss)):
            res = torch.zeros(n, xs[j].shape[1], device=DEV)
            mixer.forward(ctx, xs[j][at:at + n].to(DEV, dtype), res, cfg.kv_source(i), cfg.kv_source(i) == i, pos)
            outs[j].append(res.cpu())
        cache.advance(slot, n)
        at += n
    cache.check()
    return [torch.cat(o).double() for o in outs]


PIECES = [70, 2, 2, 59] + [1] * 17 + [90, 1, 1, 1, 2]      # crosses page borders; portions of two; token by token
LONG_PIECES = [300, 2] + [1] * 5 + [260, 1, 2]             # long enough for a recurrence that runs chunk-parallel


def rows_for(n, width, seed, dtype):
    return torch.randn(n, width, generator=torch.Generator().manual_seed(seed)).to(dtype)


def tolerance(dtype, ref, loose=0.04):
    return (1e-4 if dtype == torch.float32 else loose) * max(1.0, float(ref.abs().max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 2), ("A", 4), ("B", 2), ("B", 5), ("C", 2), ("C", 5), ("D", 3), ("D", 5)])
def test_window_attention_alone(dtype, name, layer):
    """Norms without a weight, windows of 1 to 200 tokens against pages of 64, a gate per head; value rows narrower and
    wider than key rows."""
    cfg, store, plain = tr.build(name)
    x = rows_for(sum(PIECES), cfg.width, layer, dtype)
    ref = pr.head_attention(x.double(), plain, f"l{layer}.mix", cfg.layers[layer]["mixer"], cfg.norm_eps)
    got, = mixers_alone(cfg, [layer], store, dtype, [x], PIECES)
    assert float((got - ref).abs().max()) < tolerance(dtype, ref)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layers", [("A", [0, 3]), ("B", [1, 3]), ("C", [0]), ("C", [4]), ("D", [0, 1, 4])])
def test_latent_attention_and_its_readers_alone(dtype, name, layers):
    """Queries through a latent, windows of 1 to 200 tokens, a gate per element; readers of the rows with shorter and longer
    windows, other heads and inputs of their own."""
    cfg, store, plain = tr.build(name)
    xs = [rows_for(sum(PIECES), cfg.width, 20 + i, dtype) for i in layers]
    rows = pr.latent_rows(xs[0].double(), plain, f"l{layers[0]}.mix", cfg.layers[layers[0]]["mixer"], cfg.norm_eps)
    got = mixers_alone(cfg, layers, store, dtype, xs, PIECES)
    for i, x, g in zip(layers, xs, got):
        ref = pr.latent_attention(x.double(), plain, f"l{i}.mix", cfg.layers[i]["mixer"], cfg.norm_eps, rows)
        assert float((g - ref).abs().max()) < tolerance(dtype, ref), i
        if dtype == torch.float32 and i != layers[0]:
            # a reader that saw other rows, or its own window one token off, would show
            m = dict(cfg.layers[i]["mixer"], mask={"size": cfg.layers[i]["mixer"]["mask"]["size"] + 1})
            off = pr.latent_attention(x.double(), plain, f"l{i}.mix", m, cfg.norm_eps, rows)
            assert float((off - ref).abs().max()) > 20 * tolerance(dtype, ref), i


@pytest.mark.parametrize("options", [{}, {"q_rank": 18}, {"gate": True}, {"q_rank": 18, "window": 7}, {"gate": True, "window": 7}])
def test_latent_attention_options_without_one_another(options):
    """A plain query projection beside a gate, a query latent without one, with and without a window, and a stop that reads
    rows which a mixer with keys of its own does not write."""
    from supersonic_b200.cache import SequenceCache
    from supersonic_b200.engine import StepEntry
    from supersonic_b200.parts import MIXERS, POSITION_ENCODINGS
    from supersonic_b200.weights import WeightStore
    g = torch.Generator().manual_seed(5)
    W, H, D, R, V, rank, qr = 24, 3, 8, 4, 6, 12, options.get("q_rank")
    shapes = {"dkv": (rank + R, W), "uk": (H * D, rank), "uv": (H * V, rank), "g": (H * V, W), "o": (W, H * V), "dkv.norm": (rank,)}
    shapes.update({"dq": (qr, W), "uq": (H * (D + R), qr), "dq.norm": (qr,)} if qr else {"q": (H * (D + R), W)})
    w = {f"m.{n}": torch.randn(s, generator=g) * 0.3 for n, s in shapes.items()}
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": rank, "mask": {"size": options.get("window") or 1 << 20},
         "scale": 0.4, "rot": {"base": 50.0, "dims": R}}
    # the plain statement has a latent and a gate always: the identity and a gate of one stand for their absence
    plain = dict(w)
    twist = {"no_query_norm"} if not qr else set()
    if not qr:
        plain.update({"m.dq": w["m.q"], "m.uq": torch.eye(H * (D + R))})
    if not options.get("gate"):
        twist.add("no_latent_gate")
    x = torch.randn(90, W, generator=g)
    ref = pr.latent_attention(x.double(), plain, "m", m, 1e-5, twist=twist)
    build = part_context(torch.float32, WeightStore.from_tensors(w))
    roles = {n.replace(".", "_"): f"m.{n}" for n in shapes}
    mixer = MIXERS["latent_attention"]({"hidden_size": W, "num_heads": H, "dim": D, "rot_dim": R, "value_dim": V, "kv_rank": rank,
                                        "scale": 0.4, "norm_eps": 1e-5, "window": options.get("window"), "q_rank": qr,
                                        "element_gate": bool(options.get("gate"))}, roles, build)
    pos = POSITION_ENCODINGS["rotary"]({"head_dim": R, "rotary_dim": R, "theta": 50.0, "max_positions": 1024, "scaling": None}, {}, build)
    cache = SequenceCache({0: mixer.cache_need()}, 256, 256, torch.float32, DEV)
    slot, at = cache.acquire(), 0
    for n in (65, 1, 1, 20, 3):
        ctx = step_context(build, cache, [StepEntry(slot, [0] * n)])
        for writes in (True, False):                     # the second stop reads what the first one wrote
            res = torch.zeros(n, W, device=DEV)
            mixer.forward(ctx, x[at:at + n].to(DEV), res, 0, writes, pos)
            assert float((res.cpu().double() - ref[at:at + n]).abs().max()) < 1e-4, (n, writes)
        cache.advance(slot, n)
        at += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 1), ("A", 5), ("B", 0), ("B", 4), ("C", 1), ("C", 3), ("D", 2)])
def test_recurrence_alone(dtype, name, layer):
    """Convolutions of 1 to 16 taps whose inputs cross portions of one and two tokens, one to eight blocks; then pieces long
    enough for the chunk-parallel form between single tokens, where a lost state would show."""
    cfg, store, plain = tr.build(name)
    m = cfg.layers[layer]["mixer"]
    for pieces in (PIECES, LONG_PIECES):
        x = rows_for(sum(pieces), cfg.width, layer, dtype)
        ref = pr.rglru(x.double(), plain, f"l{layer}.mix", m)
        got, = mixers_alone(cfg, [layer], store, dtype, [x], pieces)
        assert float((got - ref).abs().max()) < tolerance(dtype, ref), len(pieces)
    torn = pr.rglru(x[300:].double(), plain, f"l{layer}.mix", m)
    assert float((torn[:30] - ref[300:330]).abs().max()) > 5 * tolerance(dtype, ref, 0.01)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 2), ("A", 3), ("B", 1), ("B", 2), ("B", 5), ("C", 0), ("C", 1), ("C", 3), ("D", 4)])
def test_experts_alone(dtype, name, layer):
    """One to four experts of 1 to 16, and all of three: the sum added to a stream, and the choices a norm sums itself.
    Tokens whose last chosen and first left-out logits are level within bfloat16's rounding are left out there."""
    from supersonic_b200.cache import SequenceCache, StateNeed
    from supersonic_b200.engine import StepEntry
    from supersonic_b200.parts import FEED_FORWARDS
    cfg, store, plain = tr.build(name)
    spec = cfg.build_spec().blocks[layer].feed_forward
    build = part_context(dtype, store)
    ff = FEED_FORWARDS[spec.kind](spec.params, spec.weights, build)
    mlp = cfg.layers[layer]["mlp"]
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    for T in (83, 5):
        x = (torch.randn(T, cfg.width, generator=torch.Generator().manual_seed(layer)) * 2.0).to(dtype)
        ref = pr.experts(x.double(), plain, f"l{layer}.mlp", mlp)
        keep = torch.ones(T, dtype=torch.bool)
        if top < E:
            z = x.double() @ plain[f"l{layer}.mlp.router"].double().T + plain[f"l{layer}.mlp.router.b"].double()
            z = torch.sort(z, dim=-1, descending=True).values
            keep = (z[:, top - 1] - z[:, top]) > (1e-4 if dtype == torch.float32 else 0.05)
            assert int(keep.sum()) > 0.7 * T
        cache = SequenceCache({0: StateNeed(1)}, 256, 256, dtype, DEV)
        ctx = step_context(build, cache, [StepEntry(cache.acquire(), [0] * T)])
        res = torch.zeros(T, cfg.width, device=DEV)
        ff.forward(ctx, x.to(DEV), res)
        assert float((res.cpu().double() - ref)[keep].abs().max()) < tolerance(dtype, ref, 0.03)
        y, pw, n = ff.terms(ctx, x.to(DEV))
        own = (y.view(T, n, -1) * pw[:, :, None]).sum(1)
        assert float((own.cpu().double() - ref)[keep].abs().max()) < tolerance(dtype, ref, 0.03)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,experts,top,hidden,inter", [(1, 4, 2, 64, 64), (37, 8, 3, 128, 96), (700, 5, 2, 192, 200), (90, 1, 1, 64, 40),
                                                           (60, 6, 2, 44, 18), (1500, 16, 4, 256, 512), (300, 40, 6, 320, 136)])
def test_expert_products_with_the_activation_inside(dtype, rows, experts, top, hidden, inter):
    """The grouped products of both kernel sets, gathered, with the squared relu on their sums and stored in sorted order, and
    scattered into float32: experts that nobody chose, and one that everybody chose."""
    from supersonic_b200.csrc.kernel_sets import kernel_set_for
    from supersonic_b200.parts.experts import group_buffers
    k = kernel_set_for(dtype)
    g = torch.Generator().manual_seed(rows)
    x = torch.randn(rows, hidden, generator=g).to(dtype)
    w = (torch.randn(experts, inter, hidden, generator=g) * hidden ** -0.5).to(dtype)
    down = (torch.randn(experts, hidden, inter, generator=g) * inter ** -0.5).to(dtype)
    # expert 0 for every token; the last expert for none where there are enough others
    pool = max(experts - 1, top)
    chosen = torch.stack([torch.cat([torch.zeros(1, dtype=torch.long), 1 + torch.randperm(pool - 1, generator=g)[: top - 1]])
                          if top > 1 else torch.zeros(1, dtype=torch.long) for _ in range(rows)]).int()
    chosen = chosen[:, torch.randperm(top, generator=g)].contiguous()
    groups = group_buffers(k, rows, top, experts, hidden, inter, DEV)
    k.group_by_expert(chosen.to(DEV), experts, groups, x.to(DEV))
    z = torch.empty(rows * top, inter, dtype=dtype, device=DEV)
    k.expert_up(x.to(DEV), top, w.to(DEV), z, groups, "relu_squared")
    y = torch.full((rows * top, hidden), float("nan"), dtype=torch.float32, device=DEV)
    k.grouped_linear(z, False, top, down.to(DEV), y, True, groups)
    from supersonic_b200.csrc import ops
    ops.check_device_errors()
    order = groups["order"].cpu().long()
    assert sorted(order.tolist()) == list(range(rows * top))
    e = chosen.view(-1).long()
    tok = torch.arange(rows * top) // top
    ref = torch.empty(rows * top, inter, dtype=torch.float64)
    out = torch.empty(rows * top, hidden, dtype=torch.float64)
    for i in range(experts):
        at = (e == i).nonzero().view(-1)
        ref[at] = torch.relu(x[tok[at]].double() @ w[i].double().T) ** 2
        out[at] = ref[at].to(dtype).double() @ down[i].double().T
    assert float((z.cpu().double() - ref[order]).abs().max()) < (1e-5 if dtype == torch.float32 else 0.01) * float(ref.abs().max())
    assert float((y.cpu().double() - out).abs().max()) < (1e-5 if dtype == torch.float32 else 0.01) * float(out.abs().max())


@pytest.mark.parametrize("act", [None, ("clamped_swish", 0.75), ("gelu_tanh", 0.0)])
@pytest.mark.parametrize("tile_rows", [64, 128, 256])
def test_gated_expert_products_on_tcgen05(tile_rows, act):
    """Gate and up rows of an expert met inside the product, for every tile height: groups of one row, of whole tiles, of one
    row more and of none; widths that are not whole column tiles, an inner size that is not whole k-blocks."""
    from supersonic_b200.csrc import ops
    g = torch.Generator().manual_seed(tile_rows)
    sizes = [1, tile_rows, 0, tile_rows + 1, 3 * tile_rows - 5, 16, 17]
    E, P, K, I = len(sizes), sum(sizes), 136, 88
    expert_of = torch.cat([torch.full((n,), e, dtype=torch.int32) for e, n in enumerate(sizes)])[torch.randperm(P, generator=g)]
    x = (torch.randn(P, K, generator=g) * 1.5).bfloat16()
    w = (torch.randn(E, 2 * I, K, generator=g) * 0.15).bfloat16()
    mt = ops.expert_tiles_bound(P, E, tile_rows)
    groups = {k: torch.full((n,), -7, dtype=torch.int32, device=DEV) for k, n in
              (("offsets", E + 1), ("order", P), ("tile_expert", mt), ("tile_row0", mt), ("meta", 1))}
    rows = torch.empty(P, K, dtype=torch.bfloat16, device=DEV)
    ops.group_gather(expert_of.view(P, 1).to(DEV), E, tile_rows, groups["offsets"], groups["order"], groups["tile_expert"],
                     groups["tile_row0"], groups["meta"], x.to(DEV), rows)
    order = torch.sort(expert_of, stable=True).indices
    assert torch.equal(groups["order"].cpu().long(), order) and torch.equal(rows.cpu(), x[order])
    assert groups["offsets"].tolist() == [sum(sizes[:i]) for i in range(E + 1)]
    tiles = [(e, sum(sizes[:e]) + r) for e, n in enumerate(sizes) for r in range(0, n, tile_rows)]
    assert int(groups["meta"]) == len(tiles)
    assert list(zip(groups["tile_expert"].tolist(), groups["tile_row0"].tolist()))[: len(tiles)] == tiles
    groups.update(max_tiles=mt, tile_rows=tile_rows)
    out = torch.full((P, I), float("nan"), dtype=torch.bfloat16, device=DEV)
    ops.grouped_gemm_tc(rows, w.to(DEV), out, None, groups, ops.GG_SWIGLU, act)
    ops.check_device_errors()
    kind, limit = act or ("silu", 0.0)
    for i, p in enumerate(order.tolist()):
        h = w[expert_of[p]].double() @ x[p].double()
        gate, up = h[:I], h[I:]
        if kind == "clamped_swish":
            gate, up = gate.clamp(max=limit), up.clamp(-limit, limit) + 1.0
            gate = gate * pr.sigmoid(1.702 * gate)
        else:
            gate = pr.gelu(gate) if kind == "gelu_tanh" else gate * pr.sigmoid(gate)
        assert float((out[i].cpu().double() - gate * up).abs().max()) < 0.02 * max(1.0, float((gate * up).abs().max())), (i, p)


@pytest.mark.parametrize("experts,top", [(1, 1), (2, 1), (12, 3), (70, 5), (33, 33)])
def test_router_with_a_bias_alone(experts, top):
    """A bias decides the choice and enters the weights; renormalized, they are the softmax over the chosen logits alone."""
    from supersonic_b200.csrc import ops
    g = torch.Generator().manual_seed(4)
    T = 64
    z, bias = torch.randn(T, experts, generator=g) * 2.0, torch.randn(experts, generator=g) * 3.0
    z[5] = -bias                                          # all level
    z[6] += 300.0
    z[7] -= 300.0
    logits = torch.cat([z, torch.full((T, 3), 1e4)], dim=1).to(DEV)          # columns behind the experts do not count
    eo = torch.empty(T, top, dtype=torch.int32, device=DEV)
    pw = torch.empty(T, top, device=DEV)
    ops.route_softmax(logits, experts, True, 1.0, eo, pw, clear=True, bias=bias.to(DEV))
    assert bool((logits == 0).all())
    s = z + bias
    for t in range(T):
        idx = sorted(range(experts), key=lambda e: (-float(s[t, e]), e))[:top]
        assert eo[t].tolist() == idx
        assert float((pw[t].cpu().double() - torch.softmax(s[t, idx].double(), 0)).abs().max()) < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,top", [(44, 1), (46, 3), (256, 2), (1024, 6), (2048, 4), (4096, 2), (4100, 3)])
def test_joining_the_stream(dtype, width, top):
    """A branch and a sum of weighted choices, each through a norm into the stream, with the new stream rounded beside it;
    the branch is zero behind the read; a stream rounded by itself; embedding rows with and without a rounded copy."""
    from supersonic_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    T = 7
    x, br, w = torch.randn(T, width, generator=g), torch.randn(T, width, generator=g) * 3.0, torch.rand(width, generator=g) + 0.5
    y, pw = torch.randn(T * top, width, generator=g), torch.rand(T, top, generator=g)
    res, branch, nxt = x.to(DEV), br.to(DEV), torch.empty(T, width, dtype=dtype, device=DEV)
    ops.rms_add(res, branch, w.to(DEV), 1e-5, clear=True, next_out=nxt)
    ref = x.double() + pr.weighted_norm(br.double(), w.double(), 1e-5)
    assert float((res.cpu().double() - ref).abs().max()) < 1e-5 and float(branch.abs().max()) == 0.0
    assert torch.equal(nxt, res.to(dtype))
    v = (y.view(T, top, width).double() * pw[:, :, None].double()).sum(1)
    ref2 = ref + pr.weighted_norm(v, w.double(), 1e-5)
    for out in (nxt, None):
        again = res.clone()
        ops.combine_rms_add(again, y.to(DEV), pw.to(DEV), top, w.to(DEV), 1e-5, next_out=out)
        assert float((again.cpu().double() - ref2).abs().max()) < 1e-5
    assert torch.equal(nxt, again.to(dtype))
    ops.round_rows(res, nxt)
    assert torch.equal(nxt, res.to(dtype))
    table = torch.randn(20, width, generator=g).to(dtype).to(DEV)
    ids = torch.tensor([3, 0, 19, 3, 7, 7, 1], dtype=torch.int32, device=DEV)
    for scale in (1.0, 1.75):
        ops.embed(ids, table, res, scale, rounded=nxt)
        assert torch.equal(res, table[ids.long()].float() * scale) and torch.equal(nxt, res.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,K,N", [(5, 3, 24, 16), (70, 4, 128, 64), (300, 5, 80, 48), (33, 2, 20, 9), (129, 1, 64, 200),
                                     (1000, 3, 128, 256), (257, 16, 72, 33)])
def test_per_head_products_with_a_gate_inside(dtype, T, H, K, N):
    """out[t, h] = (W_h x[t, h]) * sigmoid(gate): inside the product where it takes the sizes, else behind it; without a gate
    from and into parts of wider heads."""
    from supersonic_b200.csrc.kernel_sets import kernel_set_for
    g = torch.Generator().manual_seed(T)
    x, w = torch.randn(T, H, K, generator=g).to(dtype), (torch.randn(H, N, K, generator=g) * K ** -0.5).to(dtype)
    rows = torch.randn(T, 3 + H * N, generator=g).to(dtype).to(DEV)           # the gate's columns sit inside wider rows
    out = torch.empty(T, H, N, dtype=dtype, device=DEV)
    kernel_set_for(dtype).head_linear(x.to(DEV), w.to(DEV), out, gate=rows[:, 3:])
    ref = torch.einsum("thk,hnk->thn", x.double(), w.double()) * pr.sigmoid(rows[:, 3:].cpu().double()).view(T, H, N)
    assert float((out.cpu().double() - ref).abs().max()) < (1e-5 if dtype == torch.float32 else 0.02) * max(1.0, float(ref.abs().max()))
    wide_x, wide_out = torch.full((T, H, K + 8), 9.0, dtype=dtype, device=DEV), torch.full((T, H, N + 5), 7.0, device=DEV)
    wide_x[:, :, :K] = x.to(DEV)
    kernel_set_for(dtype).head_linear(wide_x[:, :, :K], w.to(DEV), wide_out[:, :, :N])
    ref = torch.einsum("thk,hnk->thn", x.double(), w.double())
    assert float((wide_out[:, :, :N].cpu().double() - ref).abs().max()) < (1e-5 if dtype == torch.float32 else 1e-4) * max(1.0, float(ref.abs().max()))
    assert bool((wide_out[:, :, N:] == 7.0).all())
    from supersonic_b200.csrc import ops
    ops.check_device_errors()


@pytest.mark.parametrize("heads,rank,rot,window", [(4, 128, 32, 100), (5, 80, 16, 33), (16, 512, 64, 64), (1, 16, 16, 1), (8, 256, 32, 65),
                                                   (20, 64, 64, 128), (3, 48, 32, None)])
def test_latent_attention_kernels_agree_inside_windows(heads, rank, rot, window):
    """The tensor-core latent attention against the plain kernel in bfloat16: three sequences of unequal lengths as prompts
    that continue a cache and as decode steps (one and several parts a sequence), pages in a shuffled order.  Keys just
    inside and just outside the window of the last token are made to stand out."""
    from supersonic_b200.csrc import ops
    g = torch.Generator(device=DEV).manual_seed(rank)
    lens, new, pages_per, B, dk = [330, 64, 131], [170, 64, 1], 6, 3, rank + rot
    cache = (torch.randn(B * pages_per + 1, 1, 64, dk, device=DEV, generator=g) * 0.6).bfloat16()
    table = (torch.randperm(B * pages_per, device=DEV, generator=g).int() + 1).view(B, pages_per).contiguous()
    for decode in (False, True):
        n_new = [1] * B if decode else new
        T = sum(n_new)
        q = (torch.randn(T, heads * dk, device=DEV, generator=g) * 0.7).bfloat16()
        at = 0
        for b, (l, n) in enumerate(zip(lens, n_new)):
            at += n
            for j in ((l - window, l - window - 1) if window else (0,)):      # the last key inside, the first one outside
                if j >= 0:
                    cache[table[b, j // 64], 0, j % 64] = q[at - 1].view(heads, dk)[0] * 3.0
        cu = torch.tensor([0] + list(np.cumsum(n_new)), dtype=torch.int32, device=DEV)
        start = torch.tensor([l - n for l, n in zip(lens, n_new)], dtype=torch.int32, device=DEV)
        slots = torch.arange(B, dtype=torch.int32, device=DEV)
        pos = torch.cat([torch.arange(l - n, l, dtype=torch.int32) for l, n in zip(lens, n_new)]).to(DEV)
        slot_of = torch.cat([torch.full((n,), i, dtype=torch.int32) for i, n in enumerate(n_new)]).to(DEV)
        a, b = (torch.zeros(T, heads * rank, dtype=torch.bfloat16, device=DEV) for _ in range(2))
        ops.attention_plain(q, cache, None, pos, slot_of, table, a, heads, 1, dk, 6, window, dk ** -0.5, value_dim=rank)
        for splits in (1, 3) if decode else (1,):
            partial = torch.empty(T * heads * splits * (rank + 2), device=DEV) if splits > 1 else None
            ops.latent_attention_mma(q, cache, cu, start, slots, slot_of, table, b, None, max(n_new), heads, dk, rank, 6, window,
                                     dk ** -0.5, splits, partial)
            torch.cuda.synchronize()
            assert float((a.float() - b.float()).abs().max()) < 0.02 * max(1.0, float(a.float().abs().max())), (decode, splits)


# ---- whole models through the step function --------------------------------------------------------
def test_stream_after_every_layer():
    """float32: the stream after every layer, and the logits, against the plain statement."""
    from supersonic_b200.engine import StepEntry
    for name in ("A", "B", "C", "D"):
        cfg, store, plain = tr.build(name)
        model = make_model(cfg, store, torch.float32)
        tokens = tokens_of(cfg, 90, 3)
        ref, streams = pr.forward(cfg.to_dict(), plain, tokens)
        seen = []
        model.layer_probe = lambda stop, x: seen.append(x.cpu().double())
        slot = model.open_sequence()
        got = model.step([StepEntry(slot, tokens, list(range(len(tokens))))]).cpu().double()
        assert len(seen) == len(streams) == len(cfg.layers)
        for i, s in enumerate(seen):
            assert float((s - streams[i]).abs().max()) < 1e-4 * max(1.0, float(streams[i].abs().max())), (name, i)
        close(got, ref, torch.float32, name)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_portions_of_every_size_and_token_by_token(dtype, name):
    cfg, store, plain = build_for(name, dtype)
    model = make_model(cfg, store, dtype)
    T = 150
    tokens = tokens_of(cfg, T, 5)
    ref = reference(cfg, plain, tokens)
    for cuts in ([T], [64, 64, 22], [63, 2, 2, 61, 3, 7, 2, 10], [1] * 6 + [2] * 3 + [138], [100] + [1] * 50, [1] * T):
        close(run_in_portions(model, tokens, cuts), ref, dtype, (name, cuts))
    assert model.cache.slots.n_held == 0
    model.cache.check()


@pytest.mark.parametrize("kernels,deterministic", [("plain", False), (None, True)])
def test_other_kernel_sets_serve_the_design(kernels, deterministic):
    """bfloat16 on the plain kernels, and on the serving kernels without float atomics: there a sequence's logits are the
    same bits alone and in a batch."""
    from supersonic_b200.engine import StepEntry
    cfg, store, plain = tr.build("B", every_expert=True)
    model = make_model(cfg, store, torch.bfloat16, kernels=kernels, deterministic=deterministic)
    tokens, other = tokens_of(cfg, 130, 6), tokens_of(cfg, 40, 7)
    ref = reference(cfg, plain, tokens)
    alone = run_in_portions(model, tokens, [100] + [1] * 30)
    close(alone, ref, torch.bfloat16)
    a, b = model.open_sequence(), model.open_sequence()
    got = [model.step([StepEntry(b, other[:9], []), StepEntry(a, tokens[:100], list(range(100)))]).cpu()]
    for i in range(30):
        got.append(model.step([StepEntry(b, [other[9 + i]], [0]), StepEntry(a, [tokens[100 + i]], [0])]).cpu()[1:])
    got = torch.cat(got).double()
    close(got, ref, torch.bfloat16)
    if deterministic:
        assert torch.equal(got, alone)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_unequal_batches_against_each_alone_and_reused_slots(dtype, name):
    """Requests of 1 to 260 tokens start together and decode together, the short ones ending first; then other
    requests run in the slots, pages, convolution rows and states those gave back."""
    from supersonic_b200.engine import StepEntry
    cfg, store, plain = build_for(name, dtype)
    model = make_model(cfg, store, dtype, max_tokens=1024)
    for run, lens in enumerate(([1, 5, 64, 65, 131], [131, 2, 66], [260, 3, 195, 64], [7, 129, 64, 3])):
        decode = [3, 9, 14, 6, 11][: len(lens)]
        seqs = [tokens_of(cfg, n + d, 100 * run + i) for i, (n, d) in enumerate(zip(lens, decode))]
        refs = [reference(cfg, plain, s) for s in seqs]
        slots = [model.open_sequence() for _ in seqs]
        got = [[] for _ in seqs]
        rows = model.step([StepEntry(s, q[:n], list(range(n))) for s, q, n in zip(slots, seqs, lens)]).cpu().double()
        at = 0
        for i, n in enumerate(lens):
            got[i].append(rows[at:at + n])
            at += n
        for step in range(max(decode)):
            live = [i for i in range(len(seqs)) if step < decode[i]]
            rows = model.step([StepEntry(slots[i], [seqs[i][lens[i] + step]], [0]) for i in live]).cpu().double()
            for r, i in enumerate(live):
                got[i].append(rows[r:r + 1])
            for i in live:
                if step == decode[i] - 1:
                    model.close_sequence(slots[i])          # its slot, pages and state go back while the others go on
        for i in range(len(seqs)):
            close(torch.cat(got[i]), refs[i], dtype, (run, i))
        model.check_errors()
        assert model.cache.slots.n_held == 0
        model.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_window_edges_far_tokens_and_page_borders_show(dtype):
    """Weights under which a window one token off, a lost state or any other planted fault moves the logits by far more than
    the tolerance (``test_ropulix_config`` shows that they do); cuts at window edges (9, 11, 21, 30), one before and one
    behind them, at page borders (64, 128), the first tokens one by one, and decoding across all of these."""
    cfg, store, plain = tr.sharpened("A", every_expert=dtype != torch.float32)
    T = 330
    tokens = tokens_of(cfg, T, 9)
    ref = reference(cfg, plain, tokens)
    model = make_model(cfg, store, dtype)
    for cuts in ([T], [1, 1, 1, 1, 4, 1, 1, 1, 5, 1, 1, 12, 1, 1, 31, 1, 1, 62, 1, 1, 201],
                 [8, 2, 2, 8, 2, 6, 2, 34, 64] + [1] * 202, [256] + [1] * 74, [2] * 165):
        close(run_in_portions(model, tokens, cuts), ref, dtype, cuts)


def test_long_decoding_keeps_every_state():
    """400 tokens decoded one by one after a prompt of two, in float32: convolution inputs, states and the windows' pages
    are carried over hundreds of steps and several pages."""
    cfg, store, plain = tr.sharpened("D")
    model = make_model(cfg, store, torch.float32)
    tokens = tokens_of(cfg, 402, 21)
    close(run_in_portions(model, tokens, [2] + [1] * 400), reference(cfg, plain, tokens), torch.float32)


def test_a_long_step_in_chunks():
    """A step of more tokens than the budget runs as several."""
    from supersonic_b200.engine import StepEntry
    cfg, store, plain = tr.build("A")
    model = make_model(cfg, store, torch.float32, step_token_budget=50)
    tokens, other = tokens_of(cfg, 170, 8), tokens_of(cfg, 33, 9)
    a, b = model.open_sequence(), model.open_sequence()
    got = model.step([StepEntry(a, tokens, list(range(170))), StepEntry(b, other, list(range(33)))]).cpu().double()
    close(got[:170], reference(cfg, plain, tokens), torch.float32)
    close(got[170:], reference(cfg, plain, other), torch.float32)


def test_a_block_that_misses_its_rounded_stream_says_so():
    cfg, store, _ = tr.build("B")
    model = make_model(cfg, store, torch.bfloat16)
    from supersonic_b200.engine import StepEntry
    model.blocks[2].leaves = False
    slot = model.open_sequence()
    with pytest.raises(RuntimeError, match="rounded stream"):
        model.step([StepEntry(slot, [1, 2, 3], [2])])


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(dtype):
    """Prompts of unequal lengths in batches of three through ``Engine.generate`` (its scheduler, cache and
    sampler): the tokens are those the plain statement picks greedily, and in bfloat16 every picked token
    is the plain statement's first or close second choice."""
    from supersonic_b200.api import Engine
    cfg, store, plain = build_for("B", dtype)
    model = make_model(cfg, store, dtype, max_tokens=1024, max_seq_tokens=128)
    prompts = [tokens_of(cfg, n, 40 + n) for n in (1, 9, 64, 17, 70)]
    out = Engine(model).generate(prompts, max_new_tokens=20, temperature=0.0, ignore_eos=True, batch_size=3)
    assert [len(o) for o in out] == [20] * len(prompts)
    for prompt, new in zip(prompts, out):
        seq = list(prompt) + list(new)
        logits = reference(cfg, plain, seq)
        for i, tok in enumerate(new):
            row = logits[len(prompt) + i - 1]
            if dtype == torch.float32:
                assert tok == int(row.argmax())
            else:
                assert float(row.max() - row[tok]) < 0.1 * float(row.std())
    assert model.cache.slots.n_held == 0


def test_trace_replay_of_a_model_folder(tmp_path):
    """``bin/trace_run`` on a written folder: a batch of two prompts, decode steps, and a third request in a freed
    slot, logits against the plain statement; a second norm that a layer without a feed-forward never reads is passed
    over."""
    import json, os, subprocess, sys
    from supersonic_b200.weights import WeightStore, write_model_folder
    cfg, _, _ = tr.build("A")
    folder = write_model_folder(cfg, 3, str(tmp_path / "m"), std=0.3)
    st = WeightStore.from_dir(folder)
    plain = {n: st.get(n) for n in st.names()}
    a, b, c = tokens_of(cfg, 70, 1), tokens_of(cfg, 5, 2), tokens_of(cfg, 9, 3)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:3], "want": [2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[66:67], "want": [0]}, {"id": "b", "tokens": b[3:4], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[67:68], "want": [0]}, {"id": "b", "tokens": b[4:5], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[68:70], "want": [1]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "c", "tokens": c, "want": [8]}], "end": ["c"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    ra, rb, rc = (reference(cfg, plain, s) for s in (a, b, c))
    want = {0: torch.cat([ra[[0, 65]], rb[[2]]]), 1: ra[[66]], 2: torch.cat([ra[[67]], rb[[4]]]), 3: ra[[69]], 4: rc[[8]]}
    for i, ref in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg.vocab)).double()
        close(got, ref, torch.float32, i)
