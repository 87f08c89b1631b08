"""The Ruzunex design in the engine against the plain statement of it (``plain_ruzunex``): every mechanism alone, the
kernels against one another, then whole models through the step function in every way of cutting and batching, and
generation through the entry point."""
import copy

import numpy as np
import pytest
import torch

import plain_ruzunex as pr
import tiny_ruzunex as tr

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
    """float32 runs choose experts, bfloat16 ones take them all (see ``tiny_ruzunex.build``)."""
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


def mixers_alone(specs, store, dtype, xs, pieces):
    """What mixers add into zeroed streams for one sequence whose rows arrive in pieces.  ``specs``: (mixer spec,
    position spec) each, run one after the other within a step as layers are, with rows ``xs[i]`` of their own."""
    from supersonic_b200.cache import SequenceCache
    from supersonic_b200.engine import StepEntry
    from supersonic_b200.parts import MIXERS, POSITION_ENCODINGS
    build = part_context(dtype, store)
    mixers = [MIXERS[m.kind](m.params, m.weights, build) for m, _ in specs]
    poss = [None if p is None else POSITION_ENCODINGS[p.kind](p.params, {}, build) for _, p in specs]
    for m, (spec, _) in zip(mixers, specs):
        assert m.cache_need() == type(m).cache_need_from(spec.params)
    cache = SequenceCache({i: m.cache_need() for i, m in enumerate(mixers)}, 1024, 1024, dtype, DEV)
    slot, at, outs = cache.acquire(), 0, [[] for _ in specs]
    for n in pieces:
        ctx = step_context(build, cache, [StepEntry(slot, [0] * n)])
        for i, (mixer, pos) in enumerate(zip(mixers, poss)):
            res = torch.zeros(n, xs[i].shape[1], device=DEV)
            mixer.forward(ctx, xs[i][at:at + n].to(DEV, dtype), res, i, True, pos)
            outs[i].append(res.cpu())
        cache.advance(slot, n)
        at += n
    cache.check()
    return [torch.cat(o).double() for o in outs]


PIECES = [70, 2, 2, 59] + [1] * 17 + [90, 1, 1, 1, 2]      # crosses page borders; portions of two; token by token
LONG_PIECES = [300, 2] + [1] * 5 + [260, 1, 2]             # long enough for recurrences that run chunk-parallel


def rows_for(n, width, seed, dtype):
    return torch.randn(n, width, generator=torch.Generator().manual_seed(seed)).to(dtype)


def tolerance(dtype, ref, loose=0.04):
    return (1e-4 if dtype == torch.float32 else loose) * max(1.0, float(ref.abs().max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layers", [("A", [1]), ("A", [2, 3, 5]), ("B", [0, 2, 4]), ("C", [0]), ("C", [2]), ("D", [0, 2])])
def test_window_attention_with_bias_and_mixed_values_alone(dtype, name, layers):
    """Windows of 1 to 200 tokens against pages of 64, biases of one to sixteen heads, values mixed over two and three
    layers (of other head counts too), gates per element; value rows narrower and wider than key rows."""
    cfg, store, plain = tr.build(name)
    spec = cfg.build_spec()
    xs = [rows_for(sum(PIECES), cfg.width, 10 + i, dtype) for i in layers]
    got = mixers_alone([(spec.blocks[i].mixer, spec.blocks[i].position) for i in layers], store, dtype, xs, PIECES)
    first = None
    for n, (i, x, g) in enumerate(zip(layers, xs, got)):
        ref, own = pr.biased_attention(x.double(), plain, f"l{i}.mix", cfg.layers[i]["mixer"], cfg.norm_eps, first)
        if cfg.value_mix(i) == "first":
            first = own
        assert float((g - ref).abs().max()) < tolerance(dtype, ref), i


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 4), ("B", 1), ("B", 3), ("C", 1), ("C", 3), ("D", 1), ("D", 3)])
def test_attention_beside_recurrence_alone(dtype, name, layer):
    """Both halves of the pair, added with constants of their own: convolutions of 1 to 6 taps whose state crosses
    portions of one and two tokens, norms over the whole projection, rotation of all, some and none of a head's
    coordinates, factors and sinks per head; recurrences of 5 to 200 value columns a head."""
    cfg, store, plain = tr.build(name)
    block = cfg.build_spec().blocks[layer]
    x = rows_for(sum(PIECES), cfg.width, layer, dtype)
    ref = pr.side_by_side(x.double(), plain, f"l{layer}.mix", cfg.layers[layer]["mixer"], cfg.norm_eps)
    got, = mixers_alone([(block.mixer, block.position)], store, dtype, [x], PIECES)
    assert float((got - ref).abs().max()) < tolerance(dtype, ref)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 4), ("B", 3), ("D", 3)])
def test_recurrence_in_long_pieces(dtype, name, layer):
    """The recurrence alone over pieces long enough for its chunk-parallel form, between single tokens; lower bounds near
    one in some channels, so that what came hundreds of tokens before still counts."""
    cfg, store, plain = tr.build(name)
    low = plain[f"l{layer}.mix.right.lower"].float()
    low[::3] = 0.998
    store, plain = tr.changed(plain, {f"l{layer}.mix.right.lower": low})
    spec = cfg.build_spec().blocks[layer].mixer.params["right"]
    from supersonic_b200.config import PartSpec
    part = PartSpec(kind=spec["kind"], params=spec["params"], weights=spec["weights"])
    x = rows_for(sum(LONG_PIECES), cfg.width, layer, dtype)
    ref = cfg.layers[layer]["mixer"]["right_scale"] * \
        pr.tied_recurrence(x.double(), plain, f"l{layer}.mix.right", cfg.layers[layer]["mixer"]["right"], cfg.norm_eps)
    got, = mixers_alone([(part, None)], store, dtype, [x], LONG_PIECES)
    assert float((got - ref).abs().max()) < tolerance(dtype, ref)
    # a state that is lost at a piece's border shows
    torn = pr.tied_recurrence(x[300:].double(), plain, f"l{layer}.mix.right", cfg.layers[layer]["mixer"]["right"], cfg.norm_eps)
    assert float((torn[:40] * cfg.layers[layer]["mixer"]["right_scale"] - ref[300:340]).abs().max()) > 5 * tolerance(dtype, ref)


def test_tied_scan_forms_agree():
    """One walk, chunks in parallel, and one launch a token, in float32: the same recurrence, three sequences of unequal
    lengths (one of a single token) in shuffled slots, states left over from before, and a padding row."""
    from supersonic_b200.csrc import ops
    g = torch.Generator(device=DEV).manual_seed(3)
    H, d, dv = 3, 24, 40
    lens = [270, 1, 131]
    T, B = sum(lens), 3
    proj = torch.randn(T, H * (2 * d + dv), device=DEV, generator=g)
    bias, lower = torch.randn(H * d, device=DEV, generator=g), torch.rand(H * d, device=DEV, generator=g)
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32, device=DEV)
    slots = torch.tensor([4, 0, 2], dtype=torch.int32, device=DEV)
    state0 = torch.randn(6, H * d * dv, device=DEV, generator=g)
    runs = []
    for chunk in (0, 64, 128):
        state, out = state0.clone(), torch.zeros(T, H * dv, device=DEV)
        n = -(-max(lens) // chunk) if chunk else 0
        sums = torch.empty(B * n * H * d * dv, device=DEV) if chunk else None
        decays = torch.empty(B * n * H * d, device=DEV) if chunk else None
        ops.tied_scan(proj, 0, H * d, 2 * H * d, bias, lower, state, cu, slots, out, H, d, dv, chunk=chunk, max_new=max(lens),
                      sums=sums, decays=decays)
        runs.append((out, state))
    for out, state in runs[1:]:
        assert float((out - runs[0][0]).abs().max()) < 1e-4 * float(runs[0][0].abs().max())
        assert float((state - runs[0][1]).abs().max()) < 1e-4 * float(runs[0][1].abs().max())
    assert torch.equal(runs[0][1][[1, 3, 5]], state0[[1, 3, 5]])             # nobody else's state is touched
    # the head norm taken along
    w = torch.rand(dv, device=DEV, generator=g) + 0.5
    y = torch.zeros(T, H * dv, device=DEV)
    ops.tied_scan(proj, 0, H * d, 2 * H * d, bias, lower, state0.clone(), cu, slots, y, H, d, dv, norm_w=w, eps=1e-5)
    want = (pr.unit_rms(runs[0][0].cpu().double().reshape(T, H, dv), 1e-5) * w.cpu().double()).reshape(T, -1)
    assert float((y.cpu().double() - want).abs().max()) < 2e-4
    # token by token, with a padding row
    state = state0.clone()
    for i in range(lens[2]):
        row = torch.stack([proj[271 + i], proj[0]]).contiguous()
        y = torch.zeros(2, H * dv, device=DEV)
        ops.tied_step(row, 0, H * d, 2 * H * d, bias, lower, state, torch.tensor([0, 1, 2], dtype=torch.int32, device=DEV),
                      torch.tensor([2, -1], dtype=torch.int32, device=DEV), w, 1e-5, y, H, d, dv)
        want = pr.unit_rms(runs[0][0][271 + i].cpu().double().reshape(H, dv), 1e-5) * w.cpu().double()
        assert float((y[0].cpu().double() - want.reshape(-1)).abs().max()) < 2e-4 and float(y[1].abs().max()) == 0.0
    assert float((state[2] - runs[0][1][2]).abs().max()) < 1e-4 * float(runs[0][1].abs().max())
    assert torch.equal(state[[0, 1, 3, 4, 5]], state0[[0, 1, 3, 4, 5]])


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,bias,sink,gated", [
    (8, 4, 64, 64, 100, True, False, True), (16, 2, 64, 128, 70, True, False, True), (12, 3, 104, 32, 33, True, True, False),
    (8, 2, 96, 96, None, False, True, False), (4, 4, 128, 64, None, True, True, True), (6, 1, 40, 112, 1, True, False, True)])
def test_window_attention_kernels_agree_with_biases_sinks_and_gates(heads, kv_heads, dim, vdim, window, bias, sink, gated):
    """The tensor-core kernel against the plain one in bfloat16 with biases, factors and sinks per head and gates per
    element: three sequences of unequal lengths as prompts that continue a cache, and as decode steps, with pages in a
    shuffled order; the two differ by the rounding of the output alone."""
    from supersonic_b200.csrc import ops
    g = torch.Generator(device=DEV).manual_seed(dim + vdim)
    lens, new = [330, 64, 131], [170, 64, 1]
    pages_per, B = 6, 3
    kc = (torch.randn(B * pages_per + 1, kv_heads, 64, dim, device=DEV, generator=g) * 0.6).bfloat16()
    vc = (torch.randn(B * pages_per + 1, kv_heads, 64, vdim, device=DEV, generator=g) * 0.6).bfloat16()
    table = (torch.randperm(B * pages_per, device=DEV, generator=g).int() + 1).view(B, pages_per).contiguous()
    slopes = torch.tensor([pr.slope(h, heads) for h in range(heads)], device=DEV) if bias else None
    temp = torch.rand(heads, device=DEV, generator=g) + 0.5
    sinks = torch.randn(heads, device=DEV, generator=g) * 2.0 if sink else None
    for decode in (False, True):
        n_new = [1] * B if decode else new
        T = sum(n_new)
        q = (torch.randn(T, heads * (dim + vdim), device=DEV, generator=g) * 0.7).bfloat16()
        gate = q[:, heads * dim:] if gated else None
        cu = torch.tensor([0] + list(np.cumsum(n_new)), dtype=torch.int32, device=DEV)
        start = torch.tensor([l - n for l, n in zip(lens, n_new)], dtype=torch.int32, device=DEV)
        slots = torch.arange(B, dtype=torch.int32, device=DEV)
        pos = torch.cat([torch.arange(l - n, l, dtype=torch.int32) for l, n in zip(lens, n_new)]).to(DEV)
        slot_of = torch.cat([torch.full((n,), i, dtype=torch.int32) for i, n in enumerate(n_new)]).to(DEV)
        a, b = (torch.zeros(T, heads * vdim, dtype=torch.bfloat16, device=DEV) for _ in range(2))
        more = dict(gate=gate, gate_elems=gated, slopes=slopes, head_mul=temp)
        ops.window_attention_plain(q, kc, vc, table, None, pos, slot_of, a, heads, kv_heads, dim, vdim, 6, window, 0, 0,
                                   dim ** -0.5, None, sinks, None, None, False, 0.7, **more)
        ops.window_attention_mma(q, kc, vc, table, None, cu, start, slots, b, max(n_new), heads, kv_heads, dim, vdim, 6,
                                 window, 0, 0, dim ** -0.5, None, sinks, None, None, False, 0.7, **more)
        torch.cuda.synchronize()
        assert float((a.float() - b.float()).abs().max()) < 0.02 * max(1.0, float(a.float().abs().max())), decode


@pytest.mark.parametrize("channels,taps,behind", [(64, 2, 0), (1536, 3, 64), (2048, 4, 8), (200, 4, 24), (60, 3, 0), (64, 6, 8)])
def test_convolution_in_pieces_and_by_element(channels, taps, behind):
    """The convolution over sequences of 1 to 70 tokens with kept rows from before, in bfloat16 (16-byte pieces where the
    sizes allow it) against float64, and the rows kept for the next step; columns behind the channels pass through."""
    from supersonic_b200.csrc import ops
    g = torch.Generator().manual_seed(channels)
    lens = [1, 70, 2, 8, 33, 3]
    T, slots = sum(lens), [4, 0, 5, 2, 6, 1]
    x = torch.randn(T, channels + behind, generator=g).bfloat16()
    w, tail0 = torch.randn(channels, taps, generator=g), torch.randn(8, (taps - 1) * channels, generator=g)
    tail, out = tail0.to(DEV), torch.zeros(T, channels + behind, dtype=torch.bfloat16, device=DEV)
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32, device=DEV)
    ops.causal_conv(x.to(DEV), None, w.to(DEV), None, tail, cu, torch.tensor(slots, dtype=torch.int32, device=DEV), out, max(lens),
                    pass_cols=behind)
    at = 0
    for n, s in zip(lens, slots):
        rows = torch.cat([tail0[s].double().view(taps - 1, channels), x[at:at + n, :channels].double()])
        ref = pr.short_conv(rows, w.double())[taps - 1:]
        assert float((out[at:at + n, :channels].cpu().double() - ref).abs().max()) < 0.01 * float(ref.abs().max()) + 1e-3
        assert float((tail[s].cpu().double().view(taps - 1, channels) - rows[-(taps - 1):]).abs().max()) < 1e-6
        at += n
    assert torch.equal(out[:, channels:].cpu(), x[:, channels:]) and torch.equal(tail[[3, 7]].cpu(), tail0[[3, 7]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,streams,taps", [(50, 1, 4), (48, 1, 4), (64, 2, 1), (516, 2, 3), (2048, 2, 4), (4096, 2, 4), (50, 3, 2),
                                                (1032, 3, 2), (640, 4, 4), (64, 4, 5), (72, 6, 3), (40, 11, 2), (30, 16, 4)])
def test_streams_alone(dtype, width, streams, taps):
    """The pass between two sublayers: first read of equal streams, first write from them, write over the streams in
    place, the sum at the end; the branch is zero behind every read; the convolution behind the norm with its kept rows
    over single tokens, a padding row among them."""
    from supersonic_b200.csrc import ops
    g = torch.Generator().manual_seed(streams)
    T, W, S = 9, width, streams
    e, y1, y2 = (torch.randn(T, W, generator=g) for _ in range(3))
    w = {f"{p}.{r}": t for p in ("a", "b") for r, t in (("in", torch.randn(S, generator=g)), ("out", torch.randn(S, generator=g)),
                                                         ("mix", torch.randn(S, S, generator=g)))}
    nw = torch.randn(W, generator=g)
    d = {k: v.to(DEV) for k, v in w.items()}
    xs = torch.stack([e] * S).double()
    src = e.to(DEV).unsqueeze(0).contiguous()
    out = torch.empty(T, W, dtype=dtype, device=DEV)

    def norm(u):
        return pr.unit_rms(u, 1e-4) * nw.double()
    ops.stream_cross(src, S, d["a.in"], out, norm_weight=nw.to(DEV), eps=1e-4)
    ref = norm(pr.read_streams(xs, w, "a"))
    assert float((out.cpu().double() - ref).abs().max()) < tolerance(dtype, ref, 0.01)
    br, x = y1.to(DEV), torch.empty(S, T, W, device=DEV)
    ops.stream_cross(src, S, d["b.in"], out, br, d["a.mix"], d["a.out"], x, True, nw.to(DEV), 1e-4)
    xs = pr.write_streams(xs, y1.double(), w, "a")
    ref = norm(pr.read_streams(xs, w, "b"))
    assert float((out.cpu().double() - ref).abs().max()) < tolerance(dtype, ref, 0.01)
    assert float((x.cpu().double() - xs).abs().max()) < 1e-5 * float(xs.abs().max()) and float(br.abs().max()) == 0.0
    assert torch.equal(src[0].cpu(), e)
    # in place, with the convolution: one token each of nine sequences, the fourth a padding row
    br.copy_(y2)
    conv = torch.randn(W, taps, generator=g)
    slot = torch.tensor([3, 0, 9, -1, 5, 1, 2, 7, 8], dtype=torch.int32)
    tail0 = torch.randn(10, (taps - 1) * W, generator=g)
    tail = tail0.to(DEV)
    ops.stream_cross(x, S, d["a.in"], out, br, d["b.mix"], d["b.out"], x, True, nw.to(DEV), 1e-4, conv.T.contiguous().to(DEV), tail,
                     slot.to(DEV))
    xs = pr.write_streams(xs, y2.double(), w, "b")
    n = norm(pr.read_streams(xs, w, "a"))
    for t in range(T):
        if slot[t] < 0:
            continue
        rows = torch.cat([tail0[slot[t]].double().view(taps - 1, W), n[t:t + 1]])
        ref = pr.short_conv(rows, conv.double())[-1]
        assert float((out[t].cpu().double() - ref).abs().max()) < tolerance(dtype, ref, 0.01)
        assert torch.allclose(tail[slot[t]].cpu().double().view(taps - 1, W), rows[1:], rtol=0, atol=1e-4 * float(rows.abs().max()))
    assert torch.equal(tail[[4, 6]].cpu(), tail0[[4, 6]])
    total = torch.empty(T, W, device=DEV)
    br.copy_(y1)
    ops.stream_cross(x, S, None, total, br, d["a.mix"], d["a.out"], None, True)
    ref = pr.write_streams(xs, y1.double(), w, "a").sum(0)
    assert float((total.cpu().double() - ref).abs().max()) < 2e-5 * float(ref.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,layer", [("A", 0), ("A", 1), ("A", 3), ("B", 1), ("B", 2), ("B", 3), ("C", 1), ("C", 3), ("D", 3)])
def test_feed_forwards_alone(dtype, name, layer):
    """The gated unit with gelu (inputs on both sides of zero), and experts: one to four of 2 to 16, and all of three.
    Tokens whose last chosen and first left-out scores are level within bfloat16's rounding are left out there."""
    from supersonic_b200.cache import SequenceCache, StateNeed
    from supersonic_b200.engine import StepEntry
    from supersonic_b200.parts import FEED_FORWARDS
    cfg, store, plain = tr.build(name)
    spec = cfg.build_spec().blocks[layer].feed_forward
    build = part_context(dtype, store)
    ff = FEED_FORWARDS[spec.kind](spec.params, spec.weights, build)
    mlp = cfg.layers[layer]["mlp"]
    x = (torch.randn(83, cfg.width, generator=torch.Generator().manual_seed(layer)) * 2.0).to(dtype)
    ref = pr.feed_forward(x.double(), plain, f"l{layer}.mlp", mlp)
    keep = torch.ones(83, dtype=torch.bool)
    if mlp["kind"] == "moe" and mlp["router"]["top"] < mlp["router"]["experts"]:
        z = torch.sort(x.double() @ plain[f"l{layer}.mlp.router"].double().T, dim=-1, descending=True).values
        keep = (z[:, mlp["router"]["top"] - 1] - z[:, mlp["router"]["top"]]) > (1e-4 if dtype == torch.float32 else 0.05)
        assert int(keep.sum()) > 60
    cache = SequenceCache({0: StateNeed(1)}, 256, 256, dtype, DEV)
    ctx = step_context(build, cache, [StepEntry(cache.acquire(), [0] * 83)])
    res = torch.zeros(83, cfg.width, device=DEV)
    ff.forward(ctx, x.to(DEV), res)
    assert float((res.cpu().double() - ref)[keep].abs().max()) < tolerance(dtype, ref, 0.03)


@pytest.mark.parametrize("rows", [1, 40, 128, 200, 1500])
def test_gelu_unit_inside_the_products(rows):
    """The serving set's products that end in the gated unit's inner step against product, then activation, of the plain
    set, for the gelu form: far from zero on both sides as well."""
    from supersonic_b200.csrc import ops
    from supersonic_b200.csrc.fast_sets import FastKernels
    from supersonic_b200.csrc.kernel_sets import PlainKernels
    g = torch.Generator().manual_seed(rows)
    K, I = 192, 160
    x = (torch.randn(rows, K, generator=g) * 3.0).bfloat16().to(DEV)
    gate, up = ((torch.randn(I, K, generator=g) * 0.2).bfloat16().to(DEV) for _ in range(2))
    outs = []
    for ks in (FastKernels(), PlainKernels()):
        w, layout = ks.pack_gate_up(gate, up)
        out = torch.empty(rows, I, dtype=torch.bfloat16, device=DEV)
        ks.gate_up_swiglu(x, w, layout, out, act=("gelu_tanh", 0.0))
        outs.append(out.float().cpu())
    ops.check_device_errors()
    ref = (pr.gelu_tanh(x.double().cpu() @ gate.double().cpu().T) * (x.double().cpu() @ up.double().cpu().T)).float()
    for out in outs:
        assert torch.isfinite(out).all() and float((out - ref).abs().max()) < 0.02 * float(ref.abs().max())


@pytest.mark.parametrize("experts,top", [(1, 1), (2, 1), (12, 3), (70, 5), (33, 33)])
def test_router_alone(experts, top):
    """Softmax over all experts, the best of them, weights that sum to one; level scores go to the lower index; logits
    far from zero; without renormalizing, the scores themselves times a constant."""
    from supersonic_b200.csrc import ops
    g = torch.Generator().manual_seed(4)
    T = 64
    z = torch.randn(T, experts, generator=g) * 2.0
    z[5] = 0.0                                            # all level
    z[6] += 300.0
    z[7] -= 300.0
    logits = torch.cat([z, torch.full((T, 3), 1e4)], dim=1).to(DEV)          # columns behind the experts do not count
    s = torch.softmax(z.double(), dim=-1)
    for renorm in (True, False):
        eo = torch.empty(T, top, dtype=torch.int32, device=DEV)
        pw = torch.empty(T, top, device=DEV)
        ops.route_softmax(logits, experts, renorm, 1.0 if renorm else 2.5, eo, pw, clear=not renorm)
        assert bool((logits == 0).all()) == (not renorm)         # cleared behind the read, if asked
        for t in range(T):
            idx = sorted(range(experts), key=lambda e: (-float(z[t, e]), e))[:top]
            assert eo[t].tolist() == idx
            want = s[t, idx] / s[t, idx].sum() if renorm else s[t, idx] * 2.5
            assert float((pw[t].cpu().double() - want).abs().max()) < 1e-5


# ---- whole models through the step function --------------------------------------------------------
def test_stream_after_every_layer():
    """float32: the sum of the streams after every layer, and the logits, against the plain statement."""
    from supersonic_b200.engine import StepEntry
    for name in ("A", "B", "C", "D"):
        cfg, store, plain = tr.build(name)
        model = make_model(cfg, store, torch.float32)
        tokens = tokens_of(cfg, 90, 3)
        ref, sums = pr.forward(cfg.to_dict(), plain, tokens)
        seen = []
        model.layer_probe = lambda stop, x: seen.append(x.cpu().double())
        slot = model.open_sequence()
        got = model.step([StepEntry(slot, tokens, list(range(len(tokens))))]).cpu().double()
        assert len(seen) == len(sums) == len(cfg.layers)
        for i, s in enumerate(seen):
            assert float((s - sums[i]).abs().max()) < 1e-4 * max(1.0, float(sums[i].abs().max())), (name, i)
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


def sharpened(name="A", sharp=6.0, dtype=torch.float32):
    """The configuration's weights changed so that faults show: the weights of the norms of q are scaled up, so that a
    query's output stands on the few keys whose scores are high: a key more or less then moves the logits by far more
    than any tolerance."""
    cfg, store, plain = build_for(name, dtype)
    changes = {n: t.float() * sharp for n, t in plain.items() if n.endswith(".q.norm")}
    store, plain = tr.changed(plain, changes)
    return cfg, store, plain


def _variant(cfg, layer, path, value):
    d = copy.deepcopy(cfg.to_dict())
    at = d["layers"][layer]
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    return d


@pytest.mark.parametrize("dtype", DTYPES)
def test_window_edges_far_tokens_sinks_streams_and_page_borders_show(dtype):
    # bfloat16 takes the edges with milder weights: a softmax that stands on one key turns the rounding of a score
    # into another key, which says nothing about the masks
    cfg, store, plain = sharpened("A", 6.0 if dtype == torch.float32 else 2.0, dtype)
    T = 330
    tokens = tokens_of(cfg, T, 9)
    ref = reference(cfg, plain, tokens)
    if dtype == torch.float32:
        # the test is sharp: a window one token longer or shorter, other values mixed in, a sublayer's input without its
        # convolution, a mix matrix read the other way round, sinks left out, factors left out, an expert more, the
        # halves' constants exchanged, taps in the other order: each gives other logits at most positions ...
        def differs(d, w, share):
            other = position_errors(pr.forward(d, w, tokens)[0], ref)
            return float((other[40:] > 0.02).double().mean()) > share and float(other[40:].median()) > 0.01
        for layer, path, value in ((1, ("mixer", "mask", "size"), 10), (1, ("mixer", "mask", "size"), 12),
                                   (2, ("mixer", "mask", "size"), 8), (3, ("mixer", "mask", "size"), 29),
                                   (3, ("mixer", "mask", "size"), 31), (5, ("mixer", "mask", "size"), 16),
                                   (5, ("mixer", "mask", "size"), 18), (3, ("mixer", "v_mix"), False),
                                   (0, ("mlp", "router", "top"), 3), (0, ("mixer", "left_scale"), 1.3),
                                   (0, ("mixer", "left", "rot", "dims"), 8)):
            assert differs(_variant(cfg, layer, path, value), plain, 0.3), (layer, path, value)
        for change in ({"l1.canon1": plain["l1.canon1"] * 0}, {"l3.canon2": plain["l3.canon2"] * 0},
                       {"l1.hc1.mix": plain["l1.hc1.mix"].T}, {"l3.hc2.mix": plain["l3.hc2.mix"].T},
                       {"l0.mix.left.sink": plain["l0.mix.left.sink"] * 0 - 60.0},
                       {"l0.mix.left.temp": plain["l0.mix.left.temp"] * 0 + 1.0},
                       {"l0.mix.right.lower": plain["l0.mix.right.lower"] * 0},
                       {"l0.mix.left.v.conv": plain["l0.mix.left.v.conv"].flip(1)},
                       {"l3.mix.vmix": plain["l3.mix.vmix"] * 0}):
            assert differs(cfg.to_dict(), dict(plain, **change), 0.3), list(change)
    # ... and a sequence that has lost what came 200 and more positions before gives other logits at its end
    tail = position_errors(pr.forward(cfg.to_dict(), plain, tokens[200:])[0], ref[200:])
    assert float(tail[-30:].min()) > (0.05 if dtype == torch.float32 else 0.02)
    model = make_model(cfg, store, dtype)
    # cuts at window edges (9, 11, 17, 30), one before and one behind them, at page borders (64, 128), the first tokens
    # one by one, and decoding across all of these
    for cuts in ([T], [1, 1, 1, 1, 4, 1, 1, 1, 5, 1, 1, 12, 1, 1, 31, 1, 1, 62, 1, 1, 201],
                 [8, 2, 2, 4, 2, 10, 2, 34, 64] + [1] * 202, [256] + [1] * 74, [2] * 165):
        close(run_in_portions(model, tokens, cuts), ref, dtype, cuts)


def test_long_decoding_keeps_every_state():
    """400 tokens decoded one by one after a prompt of two, in float32: the convolutions' rows, the recurrences' states
    and the windows' pages are carried over hundreds of steps and several pages."""
    cfg, store, plain = sharpened("D", 3.0)
    model = make_model(cfg, store, torch.float32)
    tokens = tokens_of(cfg, 402, 21)
    close(run_in_portions(model, tokens, [2] + [1] * 400), reference(cfg, plain, tokens), torch.float32)


def test_a_long_step_in_chunks():
    """A step of more tokens than the budget runs as several; values mixed from an earlier layer are those of the
    piece's own tokens."""
    from supersonic_b200.engine import StepEntry
    cfg, store, plain = tr.build("A")
    model = make_model(cfg, store, torch.float32, step_token_budget=50)
    tokens, other = tokens_of(cfg, 170, 8), tokens_of(cfg, 33, 9)
    a, b = model.open_sequence(), model.open_sequence()
    got = model.step([StepEntry(a, tokens, list(range(170))), StepEntry(b, other, list(range(33)))]).cpu().double()
    close(got[:170], reference(cfg, plain, tokens), torch.float32)
    close(got[170:], reference(cfg, plain, other), torch.float32)


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
    slot, logits against the plain statement."""
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
