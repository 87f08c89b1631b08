"""Block arrangements.  ``pre_norm``: h += mixer(norm(h)); h += feed_forward(norm(h)),
the residual stream kept and summed in float32 (crates/runner/src/prefill_engine.rs:1116-1222).
``sandwich``: h += norm_b(mixer(norm_a(h))); h += norm_d(feed_forward(norm_c(h))): a sublayer's result passes a
norm of its own before it joins the stream.
``post_norm``: h += norm_b(mixer(h)); h += norm_d(feed_forward(h)): the sublayers read the stream as it is.
``parallel``: h += mixer(n) + feed_forward(n) with the one n = norm(h), or with a norm each (both of the
same h); optionally the mixer's input is mixed with the previous token's (token shift), and optionally the
layer is followed by a learned weighted sum over the results of all layers so far.
``hyper_connections``: several residual streams; a sublayer reads a weighted sum of them and its result is written into
all of them, which are mixed with one another at the same time."""
from __future__ import annotations

import torch

from ..cache import StateNeed
from ..csrc.kernel_sets import NormedInput
from .registry import register_block


@register_block("pre_norm")
class PreNormBlock:
    """Interface of a block: ``forward(ctx, residual, cache_id, writes_cache)`` updates the
    float32 residual stream ``[T, hidden]`` in place."""

    def __init__(self, mixer, feed_forward, mixer_norm, feed_forward_norm, position):
        self.mixer, self.feed_forward = mixer, feed_forward
        self.mixer_norm, self.feed_forward_norm = mixer_norm, feed_forward_norm
        self.position = position

    @staticmethod
    def _give(x, part):
        """Parts that set ``takes_lazy_input`` get the norm unapplied (a NormedInput) so that
        their kernels may fold it in; all others get the normed activations."""
        return x if getattr(part, "takes_lazy_input", False) else x.tensor()

    def forward(self, ctx, residual, cache_id, writes_cache):
        x = NormedInput(ctx, residual, self.mixer_norm)
        ctx.stage = "mixer"           # names the running part for stage timings; nothing depends on it
        self.mixer.forward(ctx, self._give(x, self.mixer), residual, cache_id, writes_cache, self.position)
        if self.feed_forward is None:
            return
        x2 = NormedInput(ctx, residual, self.feed_forward_norm)
        ctx.stage = "feed_forward"
        self.feed_forward.forward(ctx, self._give(x2, self.feed_forward), residual)


@register_block("sandwich")
class SandwichBlock:
    """x <- x + norm_1b(mixer(norm_1(x))), then x <- x + norm_2b(feed_forward(norm_2(x))): RMS norms before and
    behind each sublayer (the feed-forward may be absent).

    ``params``: ``size``, ``eps``, ``unit_offset`` (the norms behind the sublayers multiply by 1 + w); tensors
    ``mixer_out`` and ``feed_forward_out`` [size].  The sublayers add their products into a float32 row of zeros per
    token (one buffer for the whole step, which the kernel that norms it and adds it to the stream zeroes again
    behind its read); the same kernel takes the feed-forward's entry norm of the new stream, where that is an RMS
    norm, so that between the two sublayers the stream is read once."""

    def __init__(self, mixer, feed_forward, mixer_norm, feed_forward_norm, position, params=None, weights=None, build=None):
        self.mixer, self.feed_forward = mixer, feed_forward
        self.mixer_norm, self.feed_forward_norm, self.position = mixer_norm, feed_forward_norm, position
        params, weights = params or {}, weights or {}
        self.size, self.eps = int(params["size"]), float(params["eps"])
        offset = 1.0 if params.get("unit_offset") else 0.0

        def multiplier(role):
            w = build.weights.stored(weights[role]).float()
            if tuple(w.shape) != (self.size,):
                raise ValueError(f"{weights[role]} has shape {tuple(w.shape)}, expected ({self.size},)")
            return (w + offset).contiguous()
        self.mixer_out = multiplier("mixer_out")
        self.feed_forward_out = multiplier("feed_forward_out") if feed_forward is not None else None
        self.dtype = build.dtype
        self.fused_entry = feed_forward is not None and getattr(feed_forward_norm, "fusable_rms", False)

    _give = staticmethod(PreNormBlock._give)

    def forward(self, ctx, residual, cache_id, writes_cache):
        branch = ctx.streams
        if not (isinstance(branch, torch.Tensor) and branch.shape == residual.shape and branch.dtype == torch.float32):
            branch = ctx.streams = torch.zeros_like(residual)         # zero again behind every use
        x = NormedInput(ctx, residual, self.mixer_norm)
        ctx.stage = "mixer"
        self.mixer.forward(ctx, self._give(x, self.mixer), branch, cache_id, writes_cache, self.position)
        if self.feed_forward is None:
            ctx.kernels.rms_add(residual, branch, self.mixer_out, self.eps, clear=True)
            return
        ctx.stage = "feed_forward"
        if self.fused_entry:
            x2 = torch.empty(residual.shape, dtype=self.dtype, device=residual.device)
            ctx.kernels.rms_add(residual, branch, self.mixer_out, self.eps, clear=True, next_norm=self.feed_forward_norm,
                                next_out=x2)
        else:
            ctx.kernels.rms_add(residual, branch, self.mixer_out, self.eps, clear=True)
            x2 = self._give(NormedInput(ctx, residual, self.feed_forward_norm), self.feed_forward)
        self.feed_forward.forward(ctx, x2, branch)
        ctx.kernels.rms_add(residual, branch, self.feed_forward_out, self.eps, clear=True)


@register_block("post_norm")
class PostNormBlock:
    """x <- x + norm_1(mixer(x)), then x <- x + norm_2(feed_forward(x)): RMS norms behind the sublayers alone, which read
    the stream itself (the feed-forward may be absent).

    ``params``: ``size``, ``eps``, ``takes_rounded``, ``leaves_rounded``; tensors ``mixer_out`` and ``feed_forward_out``
    [size].  The stream is float32.  Where the activations are too, the sublayers read it in place; else they read a
    rounded copy, which the kernel that adds a normed result to the stream writes in the same pass.  ``takes_rounded``: the
    stop before this one (a block of this kind with ``leaves_rounded``, or an embedding with it) left the copy of the
    stream in ``ctx.carried``; without it the block rounds the stream itself.  As in a sandwich, the sublayers' products
    add into a float32 row of zeros per token, which the norm zeroes again behind its read; a feed-forward that ends in a
    weighted sum over its choices (``terms``) hands the norm the choices instead, and its result is never stored."""

    ENTRY = "rounded_stream"

    def __init__(self, mixer, feed_forward, mixer_norm, feed_forward_norm, position, params=None, weights=None, build=None):
        if mixer_norm is not None or feed_forward_norm is not None:
            raise ValueError("post_norm: the sublayers read the stream itself, without a norm in front of them")
        self.mixer, self.feed_forward, self.position = mixer, feed_forward, position
        self.size, self.eps = int(params["size"]), float(params["eps"])
        self.takes, self.leaves = bool(params.get("takes_rounded")), bool(params.get("leaves_rounded"))

        def multiplier(role):
            w = build.weights.stored(weights[role]).float().contiguous()
            if tuple(w.shape) != (self.size,):
                raise ValueError(f"{weights[role]} has shape {tuple(w.shape)}, expected ({self.size},)")
            return w
        self.mixer_out = multiplier("mixer_out")
        self.feed_forward_out = multiplier("feed_forward_out") if feed_forward is not None else None
        self.dtype = build.dtype

    def forward(self, ctx, residual, cache_id, writes_cache):
        k = ctx.kernels
        branch = ctx.streams
        if not (isinstance(branch, torch.Tensor) and branch.shape == residual.shape and branch.dtype == torch.float32):
            branch = ctx.streams = torch.zeros_like(residual)         # zero again behind every use
        rounds = self.dtype != residual.dtype

        def copy(wanted):
            return torch.empty(residual.shape, dtype=self.dtype, device=residual.device) if rounds and wanted else None
        x = residual
        if rounds:
            x = ctx.carried.pop(self.ENTRY, None) if self.takes else None
            if self.takes and (x is None or x.shape != residual.shape):
                raise RuntimeError("post_norm: the stop before this one left no rounded stream")
            if x is None:
                x = copy(True)
                k.round_rows(residual, x)
        ff = self.feed_forward
        ctx.stage = "mixer"
        self.mixer.forward(ctx, x, branch, cache_id, writes_cache, self.position)
        nxt = copy(ff is not None or self.leaves)
        k.rms_add(residual, branch, self.mixer_out, self.eps, clear=True, next_out=nxt)
        if ff is not None:
            x = residual if nxt is None else nxt
            ctx.stage = "feed_forward"
            nxt = copy(self.leaves)
            if getattr(ff, "sums_choices", False):
                y, pair_weight, top = ff.terms(ctx, x)
                k.combine_rms_add(residual, y, pair_weight, top, self.feed_forward_out, self.eps, next_out=nxt)
            else:
                ff.forward(ctx, x, branch)
                k.rms_add(residual, branch, self.feed_forward_out, self.eps, clear=True, next_out=nxt)
        if self.leaves and rounds:
            ctx.carried[self.ENTRY] = nxt


@register_block("parallel")
class ParallelBlock:
    """x <- x + mixer(n) + feed_forward(n), n = norm(x): one norm, read by both sublayers (the
    feed-forward may be absent).  With a second norm: x <- x + mixer(norm_1(x)) + feed_forward(norm_2(x)), both
    norms taken of the x that enters the layer.

    ``params["token_shift"] = {"size": width}`` with the tensor ``shift`` [width]: the mixer reads
    n_t + (n_(t-1) - n_t) * shift instead of n_t, where n_(t-1) is the previous token's normed row as it was
    before this replacement (zeros for a sequence's first token).  The last row of a step is kept per
    sequence: the block then asks the cache for ``{"mixer": the mixer's need, "shift": a row of width
    floats}``, and the mixer gets the cache id ``(cache_id, "mixer")``.

    ``params["depth_average"] = {"index": i, "layers": L}`` adds a weighted sum over depth.  Call R_0 what the
    embedding gives and R_(n+1) = s_n + mixer(norm(s_n)) + feed_forward(norm(s_n)) the raw result of layer n,
    where s_n is the stream that enters it; then s_(i+1) = sum_{j = 0 .. i+1} a_i[j] R_j with layer i's own
    i + 2 numbers a_i (``depth_weights``).  The R_j of a step are planes of one float32 stack ``ctx.streams``
    [L + 2, T, width]: plane i + 1 holds s_i, the sublayers add into it in place (which makes it R_(i+1)), and
    the weighted sum is written into plane i + 2, which the block returns as the stream from then on.
    """

    def __init__(self, mixer, feed_forward, mixer_norm, feed_forward_norm, position, params=None,
                 weights=None, build=None):
        self.mixer, self.feed_forward, self.mixer_norm, self.position = mixer, feed_forward, mixer_norm, position
        self.feed_forward_norm = feed_forward_norm
        self.shift = (params or {}).get("token_shift")
        if self.shift is not None:
            self.shift_size = int(self.shift["size"])
            mu = build.weights.stored(weights["shift"]).float().reshape(1, -1).contiguous()
            if tuple(mu.shape) != (1, self.shift_size):
                raise ValueError(f"{weights['shift']} has shape {tuple(mu.shape[1:])}, expected ({self.shift_size},)")
            self.shift_mu = mu
        self.depth = (params or {}).get("depth_average")
        if self.depth is not None:
            self.index, self.layers = int(self.depth["index"]), int(self.depth["layers"])
            w = build.weights.stored(weights["depth_weights"]).float().contiguous()
            if tuple(w.shape) != (self.index + 2,):
                raise ValueError(f"{weights['depth_weights']} has shape {tuple(w.shape)}, expected ({self.index + 2},)")
            self.depth_weights = w
            self.one = torch.ones(1, dtype=torch.float32, device=build.device)

    _give = staticmethod(PreNormBlock._give)

    def cache_need(self):
        """What the block's stop of the schedule keeps per sequence: the mixer's need, and with token shift a
        row of its own beside it."""
        need = self.mixer.cache_need()
        if self.shift is None:
            return need
        return {"mixer": need, "shift": StateNeed(self.shift_size)}

    @staticmethod
    def cache_need_from(params, mixer_need):
        shift = (params or {}).get("token_shift")
        return mixer_need if shift is None else {"mixer": mixer_need, "shift": StateNeed(int(shift["size"]))}

    def forward(self, ctx, residual, cache_id, writes_cache):
        if self.depth is not None:
            if self.index == 0:
                T, width = residual.shape
                ctx.streams = torch.empty((self.layers + 2, T, width), dtype=torch.float32, device=residual.device)
                ctx.kernels.stream_mix(residual.unsqueeze(0), self.one, 1, ctx.streams[0])
                ctx.kernels.stream_mix(residual.unsqueeze(0), self.one, 1, ctx.streams[1])
            elif ctx.streams is None:
                raise RuntimeError("a depth-averaging layer ran before the first one of its step")
            residual = ctx.streams[self.index + 1]
        fused = self.shift is not None and hasattr(self.mixer_norm, "with_shift") and \
            (self.feed_forward is None or type(self.feed_forward_norm) is type(self.mixer_norm))
        if fused:
            # both norms and the shift read the entering stream once (a norm kind that offers this form)
            if not writes_cache:
                raise ValueError("a block with token shift keeps state: its stop must write its cache entry")
            ctx.stage = "mixer"
            mixed, n2 = self.mixer_norm.with_shift(ctx, residual, self.shift_mu, ctx.cache.state((cache_id, "shift")),
                                                   self.feed_forward_norm if self.feed_forward is not None else None)
            self.mixer.forward(ctx, mixed, residual, (cache_id, "mixer"), writes_cache, self.position)
            if self.feed_forward is not None:
                ctx.stage = "feed_forward"
                self.feed_forward.forward(ctx, n2, residual)
            return self._after(ctx)
        x = NormedInput(ctx, residual, self.mixer_norm)
        x2 = x
        if self.feed_forward is not None and self.feed_forward_norm is not None:
            # the second norm reads the stream as it enters the layer: taken before the mixer adds to it
            x2 = NormedInput(ctx, residual, self.feed_forward_norm)
            x2.tensor()
        ctx.stage = "mixer"
        if self.shift is not None:
            if not writes_cache:
                raise ValueError("a block with token shift keeps state: its stop must write its cache entry")
            n = x.tensor()
            mixed = torch.empty((1,) + tuple(n.shape), dtype=n.dtype, device=n.device)
            ctx.kernels.shift_mix(n, self.shift_mu, ctx.cache.state((cache_id, "shift")), ctx.batch, mixed)
            self.mixer.forward(ctx, mixed[0], residual, (cache_id, "mixer"), writes_cache, self.position)
        else:
            self.mixer.forward(ctx, self._give(x, self.mixer), residual, cache_id, writes_cache, self.position)
        if self.feed_forward is not None:
            ctx.stage = "feed_forward"
            self.feed_forward.forward(ctx, self._give(x2, self.feed_forward), residual)
        return self._after(ctx)

    def _after(self, ctx):
        if self.depth is None:
            return None
        out = ctx.streams[self.index + 2]
        ctx.kernels.stream_mix(ctx.streams, self.depth_weights, self.index + 2, out)
        return out


class _Streams:
    """The residual streams within one step: ``x`` [streams, T, width], or [1, T, width] while all of them still equal the
    embedding's output; ``branch`` [T, width], which sublayers add into; ``write``, the (mix, out) of the last sublayer
    whose result still waits in the branch (None: nothing waits)."""

    def __init__(self, embedded):
        self.x, self.branch, self.write = embedded.unsqueeze(0), torch.zeros_like(embedded), None


@register_block("hyper_connections")
class HyperConnectionBlock:
    """Residual streams x_1 .. x_S, all equal to the embedding's output at the start.  For each of the two sublayers

        u = sum_s in[s] x_s,    n = norm(u),    h = n + conv(n),    y = sublayer(h)
        x_t <- sum_s mix[s, t] x_s + out[t] y        (all streams at once from the old ones; mix is [from, to])

    with conv a causal convolution over time on each channel, conv(n)_t = sum_j w[:, j] n_(t - taps + 1 + j), whose last
    taps - 1 inputs are per-sequence state of the block, one row for each sublayer.  Behind the last layer the stream is
    the sum of the streams.

    ``params``: ``size``, ``streams``, ``taps`` (0: no convolution), ``last`` (the layer that sums the streams); tensors per
    sublayer ``s`` in ``mixer``, ``ff``: ``<s>_in`` [S], ``<s>_mix`` [S, S], ``<s>_out`` [S], with a convolution ``<s>_conv``
    [size, taps].  A sublayer's write waits until the next one's read: both are one pass over the streams, which also
    takes the norm (and, in steps of one token a sequence, the convolution).  1 is added to the convolution's last tap
    when the part is built, so that n + conv(n) is one convolution."""

    def __init__(self, mixer, feed_forward, mixer_norm, feed_forward_norm, position, params=None, weights=None, build=None):
        self.mixer, self.feed_forward = mixer, feed_forward
        self.mixer_norm, self.feed_forward_norm, self.position = mixer_norm, feed_forward_norm, position
        self.size, self.streams = int(params["size"]), int(params["streams"])
        self.taps, self.last = int(params.get("taps") or 0), bool(params.get("last"))
        from ..csrc.ops import CONV_MAX_TAPS, STREAMS_MAX
        if not 1 <= self.streams <= STREAMS_MAX or not 0 <= self.taps <= CONV_MAX_TAPS:
            raise ValueError(f"hyper_connections: {self.streams} streams (1 to {STREAMS_MAX}), {self.taps} taps (0 to {CONV_MAX_TAPS})")
        S = self.streams

        def stored(role, shape):
            t = build.weights.stored(weights[role]).float().contiguous()
            if tuple(t.shape) != shape:
                raise ValueError(f"{weights[role]} has shape {tuple(t.shape)}, expected {shape}")
            return t
        self.reads, self.writes, self.convs = [], [], []
        for sub, norm in (("mixer", mixer_norm), ("ff", feed_forward_norm))[: 1 if feed_forward is None else 2]:
            if not getattr(norm, "fusable_rms", False):
                raise ValueError("hyper_connections: the norm behind a read of the streams is an RMS norm")
            self.reads.append(stored(f"{sub}_in", (S,)))
            self.writes.append((stored(f"{sub}_mix", (S, S)), stored(f"{sub}_out", (S,))))
            if self.taps:
                w = stored(f"{sub}_conv", (self.size, self.taps)).clone()
                w[:, -1] += 1.0
            else:
                w = torch.ones((self.size, 1), dtype=torch.float32, device=build.device)
            self.convs.append((w, w.T.contiguous()))        # by channel, for prompts; by tap, for single tokens
        self.dtype = build.dtype

    @staticmethod
    def _needs(mixer_need, size, taps, sublayers):
        if taps < 2:
            return mixer_need
        return {"mixer": mixer_need, **{f"conv{i}": StateNeed((taps - 1) * size) for i in range(sublayers)}}

    def cache_need(self):
        return self._needs(self.mixer.cache_need(), self.size, self.taps, len(self.reads))

    @staticmethod
    def cache_need_from(params, mixer_need):
        return HyperConnectionBlock._needs(mixer_need, int(params["size"]), int(params.get("taps") or 0),
                                           2 if params.get("feed_forward", True) else 1)

    def _enter(self, ctx, st, i, norm, cache_id):
        """Finish the write that waits, read the streams for sublayer i, norm and convolve."""
        T, dev = st.branch.shape[0], st.branch.device
        h = torch.empty((T, self.size), dtype=self.dtype, device=dev)
        dst = None
        if st.write is not None:
            # written over the old streams, except where those are the one row all of them equal
            dst = st.x if st.x.shape[0] == self.streams and self.streams > 1 else \
                torch.empty((self.streams, T, self.size), dtype=torch.float32, device=dev)
        tail = ctx.cache.state((cache_id, f"conv{i}")) if self.taps > 1 else None
        ctx.kernels.stream_enter(st.x, self.streams, self.reads[i], st.branch, st.write, dst, norm, self.convs[i], tail,
                                 ctx.batch, h)
        if dst is not None:
            st.x = dst
        st.write = self.writes[i]
        return h

    def forward(self, ctx, residual, cache_id, writes_cache):
        if not writes_cache:
            raise ValueError("hyper_connections: the block keeps state: its stop must write its cache entry")
        if not isinstance(ctx.streams, _Streams):
            ctx.streams = _Streams(residual)
        st = ctx.streams
        ctx.stage = "mixer"
        h = self._enter(ctx, st, 0, self.mixer_norm, cache_id)
        self.mixer.forward(ctx, h, st.branch, (cache_id, "mixer") if self.taps > 1 else cache_id, writes_cache, self.position)
        if self.feed_forward is not None:
            ctx.stage = "feed_forward"
            h = self._enter(ctx, st, 1, self.feed_forward_norm, cache_id)
            self.feed_forward.forward(ctx, h, st.branch)
        return self._sum(ctx, st) if self.last else None

    def _sum(self, ctx, st, clear=True):
        out = torch.empty_like(st.branch)
        ctx.kernels.stream_sum(st.x, self.streams, st.branch, st.write, out, clear)
        return out

    def stream_view(self, ctx, residual):
        """The stream behind this layer, for probes: the sum of the streams with the waiting write applied."""
        return residual if self.last else self._sum(ctx, ctx.streams, clear=False)
