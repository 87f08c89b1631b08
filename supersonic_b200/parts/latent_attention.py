"""The latent-attention mixer: causal softmax attention that caches one low-rank row per token.

In equations, for a token at position p with normed input h, per head g of H:

    u_g = Wq_g h                       split as u_g = [a_g (dim) | b_g (rot_dim)]
    y   = Wdkv h                       split as y   = [y_lat (kv_rank) | y_rot (rot_dim)]
    c   = rms(y_lat) * w_norm          the latent row of the token
    r   = rot_p(y_rot),  b'_g = rot_p(b_g)      rotation by the position encoding the mixer is given
    K_g(j) = [Wuk_g c_j | r_j],   V_g(j) = Wuv_g c_j          for every earlier or equal position j
    s_gj = ([a_g | b'_g] . K_g(j)) * scale
    out_g = sum_j exp(s_gj) V_g(j) / (sum_j exp(s_gj) + exp(sink_g))       (without a sink: the plain softmax)
    result = Wo [out_1 ... out_H]

Options, each usable without the others:

* ``q_rank``: the queries go through a latent of their own, u = Wuq (rms(Wdq h) * w_qnorm).
* ``window`` W: position p sees the positions j with p - W < j <= p.
* ``element_gate``: the concatenated heads are multiplied by sigmoid(Wg h) element by element.
* ``own_kv`` = False: the mixer has no Wdkv; its stop of the schedule reads the rows [c_j | r_j] another layer wrote,
  with its own queries, Wuk, Wuv, window and gate.  ``cache_window``: how far back the cache entry keeps tokens, where
  a reader of the entry has a longer window.

The cache holds [c_j | r_j] per token, whatever H is.  K and V are never formed: since
a_g . (Wuk_g c_j) = (Wuk_g^T a_g) . c_j, the query is moved into the latent space once
(a'_g = Wuk_g^T a_g), the score is a'_g . c_j + b'_g . r_j, the probabilities weight the c_j
themselves, and Wuv_g is applied to that one sum per query.  A cached token then costs a head
2 kv_rank + rot_dim multiply-adds and no matrix product.
"""
from __future__ import annotations

import torch

from ..cache import PAGE_SHIFT, KvNeed
from .registry import BuildContext, register_mixer


@register_mixer("latent_attention")
class LatentAttention:
    """params: ``hidden_size``, ``num_heads``, ``dim``, ``rot_dim``, ``value_dim``, ``kv_rank``, ``scale``,
    ``norm_eps``, ``window`` (None = all earlier keys), ``q_rank`` (None), ``element_gate`` (False), ``own_kv`` (True),
    ``cache_window`` (None); weights: ``q`` or (with a query latent) ``dq``, ``dq_norm``, ``uq``; ``dkv``, ``dkv_norm``
    (keys of its own), ``uk``, ``uv``, ``o``, with a gate ``g`` [heads x value_dim, hidden], and optionally ``sink``.  The
    position encoding it is given rotates the ``rot_dim`` parts."""

    takes_lazy_input = True

    def __init__(self, params, weights, build: BuildContext):
        self.hidden, self.H = int(params["hidden_size"]), int(params["num_heads"])
        self.dim, self.rot, self.vdim = int(params["dim"]), int(params["rot_dim"]), int(params["value_dim"])
        self.rank = int(params["kv_rank"])
        self.q_rank = int(params["q_rank"]) if params.get("q_rank") else None
        self.scale, self.eps = float(params["scale"]), float(params["norm_eps"])
        self.window = params.get("window")
        self.own_kv, self.element_gate = bool(params.get("own_kv", True)), bool(params.get("element_gate", False))
        self.cache_window = self._reach(self.window, params.get("cache_window"))
        w, dt = build.weights, build.dtype
        H, d, r, dv, rank = self.H, self.dim, self.rot, self.vdim, self.rank
        want = {"uk": (H * d, rank), "uv": (H * dv, rank), "o": (self.hidden, H * dv)}
        if self.q_rank:
            want.update(dq=(self.q_rank, self.hidden), uq=(H * (d + r), self.q_rank))
        else:
            want["q"] = (H * (d + r), self.hidden)
        if self.own_kv:
            want["dkv"] = (rank + r, self.hidden)
        if self.element_gate:
            want["g"] = (H * dv, self.hidden)
        got = {role: w.as_dtype(weights[role], dt) for role in want}
        for role, n in (("dq_norm", self.q_rank), ("dkv_norm", rank if self.own_kv else None)):
            if n:
                t = w.stored(weights[role])
                got[role], want[role] = t.float() if dt == torch.float32 else t, (n,)
        for role, shape in want.items():
            if tuple(got[role].shape) != shape:
                raise ValueError(f"{weights[role]} has shape {tuple(got[role].shape)}, expected {shape}")
        # one product over [queries or their latent | low-rank row | gate]; a stop that reads another stop's rows
        # projects [queries or their latent | gate]
        head = got["dq" if self.q_rank else "q"]
        self.q_cols = head.shape[0]
        tail = [got["g"]] if self.element_gate else []
        pad = (-(head.shape[0] + sum(t.shape[0] for t in tail) + (rank + r if self.own_kv else 0))) % 8 if tail else 0
        if pad:                                  # rows of the product's result stay a multiple of 8 wide
            tail.append(torch.zeros((pad, self.hidden), dtype=dt, device=head.device))
        if self.own_kv:
            self.w_in = torch.cat([head, got["dkv"]] + tail, dim=0).contiguous()
            self.w_q = self.w_in[: self.q_cols] if not tail else None       # with a gate: built if such a stop ever runs
            self._tail = [self.w_in[self.q_cols + rank + r:]]
        else:
            self.w_in = None
            self.w_q = torch.cat([head] + tail, dim=0).contiguous()
        self.w_uq, self.q_norm_w = got.get("uq"), got.get("dq_norm")
        self.norm_w = got.get("dkv_norm", got.get("dq_norm"))      # without rows of its own nothing is normed with it
        if self.norm_w is None:
            self.norm_w = torch.ones(rank, dtype=dt, device=build.device)
        # Wuk_g^T [rank, dim] per head carries a plain query into the latent space; Wuv_g [vdim, rank] carries
        # the summed latent out of it
        self.w_absorb = torch.empty((H, rank, d), dtype=dt, device=got["uk"].device)      # (a copy whose strides hold for d = 1 too)
        self.w_absorb.copy_(got["uk"].view(H, d, rank).transpose(1, 2))
        self.w_uv = got["uv"].view(H, dv, rank).contiguous()
        self.w_o = got["o"]
        self.sinks = None
        if weights.get("sink"):
            self.sinks = w.stored(weights["sink"]).float().contiguous()
            if tuple(self.sinks.shape) != (H,):
                raise ValueError(f"{weights['sink']} has shape {tuple(self.sinks.shape)}, expected ({H},)")
        self.dtype = dt

    @staticmethod
    def _reach(window, cache_window):
        """How far back the cache entry keeps tokens."""
        return None if not window else max(int(window), int(cache_window or 0))

    def cache_need(self):
        return KvNeed(1, self.rank + self.rot, self.cache_window, value_dim=0)

    @staticmethod
    def cache_need_from(params):
        return KvNeed(1, int(params["kv_rank"]) + int(params["rot_dim"]),
                      LatentAttention._reach(params.get("window"), params.get("cache_window")), value_dim=0)

    @staticmethod
    def activation_elements(params) -> int:
        """Elements per token while the part runs: the projected row, the latent-space queries, the summed
        latents and the heads' outputs."""
        H, rank, r = int(params["num_heads"]), int(params["kv_rank"]), int(params["rot_dim"])
        more = int(params.get("q_rank") or 0) + (H * int(params["value_dim"]) if params.get("element_gate") else 0)
        return H * (int(params["dim"]) + r) + rank + r + H * (2 * rank + r) + H * int(params["value_dim"]) + more

    def forward(self, ctx, x, residual, cache_id, writes_cache, position):
        if position is None or not hasattr(position, "rotary_tables"):
            raise ValueError("latent attention needs a rotary position encoding for its rotated parts")
        if writes_cache and not self.own_kv:
            raise ValueError("latent attention: a mixer without rows of its own cannot write a cache entry")
        H, d, r, dv, rank = self.H, self.dim, self.rot, self.vdim, self.rank
        T, dev, k = ctx.batch.n_tokens, residual.device, ctx.kernels
        cache, _, table, _ = ctx.cache.kv(cache_id)
        weight = self.w_in if writes_cache else self._read_weight()
        c_off = self.q_cols
        g_off = c_off + (rank + r if writes_cache else 0)
        proj = torch.empty((T, weight.shape[0]), dtype=self.dtype, device=dev)
        k.linear(x, weight, proj)
        position.check_range(ctx.batch)
        q_abs = torch.empty((T, H * (rank + r)), dtype=self.dtype, device=dev)
        queries = proj
        if self.q_rank:
            # the query latent's norm and the cache row before the queries exist, their rotated parts behind them
            k.latent_prepare(proj, c_off, None, self.norm_w, self.eps, position, ctx.batch, table, cache, 0, d, r, rank,
                             PAGE_SHIFT, writes_cache, q_latent=(0, self.q_rank, self.q_norm_w))
            queries = torch.empty((T, H * (d + r)), dtype=self.dtype, device=dev)
            k.linear(proj[:, : self.q_rank], self.w_uq, queries)
            writes_cache = False                 # the row is there
        k.latent_prepare(queries, c_off, q_abs, self.norm_w, self.eps, position, ctx.batch, table, cache, H, d, r, rank,
                         PAGE_SHIFT, writes_cache)
        k.head_linear(queries[:, : H * (d + r)].view(T, H, d + r)[:, :, :d], self.w_absorb,
                      q_abs.view(T, H, rank + r)[:, :, :rank])
        latent = torch.empty((T, H * rank), dtype=self.dtype, device=dev)
        k.latent_attention(q_abs, cache, ctx.batch, table, latent, H, rank, r, PAGE_SHIFT, self.window, self.scale, self.sinks)
        heads = torch.empty((T, H * dv), dtype=self.dtype, device=dev)
        if self.element_gate:
            k.head_linear(latent.view(T, H, rank), self.w_uv, heads.view(T, H, dv), gate=proj[:, g_off: g_off + H * dv])
        else:
            k.head_linear(latent.view(T, H, rank), self.w_uv, heads.view(T, H, dv))
        k.linear(heads, self.w_o, residual, accumulate=True)

    def _read_weight(self):
        """[queries or their latent | gate] for a stop that reads another stop's rows."""
        if self.w_q is None:
            self.w_q = torch.cat([self.w_in[: self.q_cols]] + self._tail, dim=0).contiguous()
        return self.w_q
