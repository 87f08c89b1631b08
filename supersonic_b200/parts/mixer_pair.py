"""Two mixers side by side: both read the same input, and their results are joined as

    result = scale * (rms(left) * w_left + rms(right) * w_right)

with the root mean square taken over the model width (eps inside the root) and a weight vector each, or, with
``join`` = ``"add"``, added as they are, result = left + right, each half with the constant factor its own parameters
give it (``out_scale``): both then add straight into the stream.  Halves that keep their products apart from what lies
between (``splits_products``) share them: one product over the input rows of both, one over the concatenated heads.
Either half is any registered mixer; each keeps what it needs in the cache under the pair's id
(``(cache_id, "left")`` and ``(cache_id, "right")``), and each gets the position encoding only if it asks for it.
"""
from __future__ import annotations

import torch

from .registry import MIXERS, BuildContext, lookup, register_mixer


@register_mixer("mixer_pair")
class MixerPair:
    """params: ``hidden_size``, ``join`` (``"normed"``, the default, or ``"add"``), for normed halves ``norm_eps`` and ``scale``
    (default 1/2), ``left`` and ``right``: each ``{"kind", "params", "weights", "position": bool}``; weights, for normed
    halves: ``left_out``, ``right_out`` [hidden]."""

    def __init__(self, params, weights, build: BuildContext):
        self.hidden, self.join = int(params["hidden_size"]), params.get("join") or "normed"
        if self.join not in ("normed", "add"):
            raise ValueError(f"mixer_pair: join {self.join!r} is not known ('normed' or 'add')")
        self.halves = []
        for side in ("left", "right"):
            sub = params[side]
            self.halves.append((side, lookup(MIXERS, sub["kind"], "mixer")(sub["params"], sub["weights"], build),
                                bool(sub.get("position", False))))
        self.shared = self.join == "add" and all(getattr(m, "splits_products", False) for _, m, _ in self.halves)
        if self.shared:
            (_, left, _), (_, right, _) = self.halves
            self.in_cols, self.out_cols = left.in_weight.shape[0], left.out_weight.shape[1]
            self.w_in = torch.cat([left.in_weight, right.in_weight], dim=0).contiguous()
            self.w_o = torch.cat([left.out_weight, right.out_weight], dim=1).contiguous()
            self.dtype = build.dtype
            # the halves keep views: nothing is held twice
            left.share_products(self.w_in[: self.in_cols], self.w_o[:, : self.out_cols])
            right.share_products(self.w_in[self.in_cols:], self.w_o[:, self.out_cols:])
        if self.join == "add":
            return
        self.eps, self.scale = float(params["norm_eps"]), float(params.get("scale", 0.5))
        self.out_w = [build.weights.stored(weights[s + "_out"]).float().contiguous() for s in ("left", "right")]
        for s, t in zip(("left_out", "right_out"), self.out_w):
            if tuple(t.shape) != (self.hidden,):
                raise ValueError(f"{weights[s]} has shape {tuple(t.shape)}, expected ({self.hidden},)")

    def cache_need(self):
        return {side: mixer.cache_need() for side, mixer, _ in self.halves}

    @staticmethod
    def cache_need_from(params):
        needs = {}
        for side in ("left", "right"):
            hook = getattr(lookup(MIXERS, params[side]["kind"], "mixer"), "cache_need_from", None)
            needs[side] = hook(params[side]["params"]) if hook is not None else None
        return needs

    @staticmethod
    def activation_elements(params) -> int:
        total = 0 if params.get("join") == "add" else 4 * int(params["hidden_size"])
        for side in ("left", "right"):
            hook = getattr(lookup(MIXERS, params[side]["kind"], "mixer"), "activation_elements", None)
            total += int(hook(params[side]["params"])) if hook is not None else 4 * int(params["hidden_size"])
        return total

    def forward(self, ctx, x, residual, cache_id, writes_cache, position):
        x = x.tensor() if hasattr(x, "tensor") else x
        if self.shared:
            T, dev, k = ctx.batch.n_tokens, residual.device, ctx.kernels
            proj = torch.empty((T, self.w_in.shape[0]), dtype=self.dtype, device=dev)
            k.linear(x, self.w_in, proj)
            heads = torch.empty((T, self.w_o.shape[1]), dtype=self.dtype, device=dev)
            for (side, mixer, wants_position), p, h in zip(self.halves, (proj[:, : self.in_cols], proj[:, self.in_cols:]),
                                                           (heads[:, : self.out_cols], heads[:, self.out_cols:])):
                mixer.inner(ctx, p, h, (cache_id, side), writes_cache, position if wants_position else None)
            k.linear(heads, self.w_o, residual, accumulate=True)
            return
        if self.join == "add":
            for side, mixer, wants_position in self.halves:
                mixer.forward(ctx, x, residual, (cache_id, side), writes_cache, position if wants_position else None)
            return
        outs = []
        for side, mixer, wants_position in self.halves:
            # a half adds into what it is given: a zeroed stream of its own
            out = torch.zeros_like(residual)
            mixer.forward(ctx, x, out, (cache_id, side), writes_cache, position if wants_position else None)
            outs.append(out)
        ctx.kernels.rms_pair_add(residual, outs[0], self.out_w[0], outs[1], self.out_w[1], self.eps, self.scale)
