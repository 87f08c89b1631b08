"""Typed configuration of the ``Ropulix`` architecture.

Its config.json is nested.  Top level: ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list with one entry per layer:
``type`` (``attention``, ``rglru`` or ``latent_attention``), ``mixer`` (that mixer's sizes and constants) and ``mlp`` (null or
``{"kind": "moe", "router": {"experts", "top"}, "expert": {"ff"}}``).

``build_spec`` turns that into parts.  A layer is a ``post_norm`` block: mixer and feed-forward read the stream itself, and
each result passes an RMS norm (``norm1``, ``norm2``) before it joins the stream.  The mixers:

* ``attention``: a ``window_attention`` without rotation inside a sliding window ``mask.size``: q and k divided by their root
  mean square per head (a norm without a weight), a sigmoid gate per head;
* ``rglru``: a ``real_gated_recurrence``;
* ``latent_attention``: a ``latent_attention`` inside a sliding window, queries through a latent of ``q_rank``, a sigmoid gate
  per element of the heads.  With ``kv_from``: j the layer has no key and value projection; its stop of the schedule
  reads layer j's cache entry.

The feed-forward is ``experts`` without gates (squared relu) behind a ``softmax`` router with a bias, whose weights are
renormalized over the chosen experts.  The head is the embedding's table.  Tensor names: ``embed``, ``final.norm`` and per
layer i ``l<i>.norm1``, ``norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``.  The design has no position limit; the cache bounds a
sequence.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

import torch

from .base import BlockSpec, ConfigError, ModelSpec, PartSpec, ScheduleEntry
from .kilisun import NO_POSITION_LIMIT, _number
from .ronelorn import _need, _positive
from .ruzunex import _heads, _taps

ARCHITECTURE = "Ropulix"
MIXERS = ("attention", "rglru", "latent_attention")


def _window(m, where: str) -> None:
    _need(m, ("mask",), where)
    _need(m["mask"], ("size",), where + ".mask")
    _positive(m["mask"], ("size",), where + ".mask")


@dataclass(frozen=True)
class RopulixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[Dict[str, Any]] = field(default_factory=list)
    eos_token_ids: List[int] = field(default_factory=list)
    model_type: str = "ropulix"

    # ---- reading -----------------------------------------------------
    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "RopulixConfig":
        _need(d, ("vocab", "width", "layers", "norm"), "config.json")
        _need(d["norm"], ("eps",), "norm")
        _positive(d, ("vocab", "width"), "config.json")
        eos = d.get("eos_token_id")
        cfg = RopulixConfig(
            vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]), layers=copy.deepcopy(list(d["layers"])),
            eos_token_ids=[] if eos is None else [int(eos)] if isinstance(eos, int) else [int(e) for e in eos])
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if not self.layers:
            raise ConfigError("layers must name at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            m, kind, at = layer["mixer"], layer["type"], where + ".mixer"
            if kind == "attention":
                _heads(m, at)
                _window(m, at)
            elif kind == "rglru":
                _need(m, ("width", "blocks", "conv"), at)
                _positive(m, ("width", "blocks"), at)
                _taps(m, "conv", at)
                if m["width"] % m["blocks"]:
                    raise ConfigError(f"{at}: {m['width']} channels in {m['blocks']} blocks")
            elif kind == "latent_attention":
                self._validate_latent(i, m, at)
            else:
                raise ConfigError(f"{where}.type {kind!r} is not known (known: {list(MIXERS)})")
            if kind != "latent_attention" and m.get("kv_from") is not None:
                raise ConfigError(f"{at}.kv_from: only a layer of latent_attention reads another layer's rows")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
                raise ConfigError(f"{where}.mlp.kind {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not known (known: 'moe')")
            _need(mlp, ("router", "expert"), where + ".mlp")
            _need(mlp["router"], ("experts", "top"), where + ".mlp.router")
            _positive(mlp["router"], ("experts", "top"), where + ".mlp.router")
            if mlp["router"]["top"] > mlp["router"]["experts"]:
                raise ConfigError(f"{where}.mlp.router: {mlp['router']['top']} experts a token of {mlp['router']['experts']}")
            _need(mlp["expert"], ("ff",), where + ".mlp.expert")
            _positive(mlp["expert"], ("ff",), where + ".mlp.expert")
        for e in self.eos_token_ids:
            if not 0 <= e < self.vocab:
                raise ConfigError(f"eos_token_id {e} is outside the vocabulary")

    def _validate_latent(self, i: int, m, at: str) -> None:
        _need(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot"), at)
        _positive(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"), at)
        _number(m, "scale", at)
        _window(m, at)
        _need(m["rot"], ("base", "dims"), at + ".rot")
        _number(m["rot"], "base", at + ".rot")
        if m["rot"]["dims"] != m["rot_dim"] or m["rot_dim"] % 2:
            raise ConfigError(f"{at}: the rotated part turns as a whole: rot.dims {m['rot']['dims']!r} must equal rot_dim "
                              f"{m['rot_dim']!r}, an even number")
        src = m.get("kv_from")
        if src is None:
            return
        if not isinstance(src, int) or isinstance(src, bool) or not 0 <= src < i:
            raise ConfigError(f"{at}.kv_from must name an earlier layer, got {src!r}")
        other = self.layers[src]
        if other["type"] != "latent_attention" or other["mixer"].get("kv_from") is not None:
            raise ConfigError(f"{at}.kv_from names layer {src}, which keeps no latent rows of its own")
        if any(other["mixer"][k] != m[k] for k in ("kv_rank", "rot_dim")) or other["mixer"]["rot"] != m["rot"]:
            raise ConfigError(f"{at}.kv_from names layer {src}, whose kv_rank, rot_dim or rotation differs")

    # ---- writing -----------------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": ARCHITECTURE, "layers": copy.deepcopy(self.layers), "norm": {"eps": self.norm_eps},
                             "vocab": self.vocab, "width": self.width}
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- what other parts of the framework ask ---------------------------------------
    @property
    def architectures(self) -> List[str]:
        return [ARCHITECTURE]

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        return NO_POSITION_LIMIT

    def kv_source(self, i: int) -> int:
        """The layer whose cache entry layer i reads (itself unless it says ``kv_from``)."""
        src = self.layers[i]["mixer"].get("kv_from")
        return i if src is None else int(src)

    def cache_reach(self, i: int) -> int:
        """How far back the cache entry of latent layer i keeps tokens: the longest window among the layers that read it."""
        return max(int(l["mixer"]["mask"]["size"]) for j, l in enumerate(self.layers)
                   if l["type"] == "latent_attention" and self.kv_source(j) == i)

    # ---- the architecture as parts ----------------------------------
    def _mixer(self, i: int):
        W, eps = self.width, self.norm_eps
        layer, p = self.layers[i], f"l{i}.mix"
        m = layer["mixer"]
        if layer["type"] == "attention":
            return PartSpec(kind="window_attention", params={
                "hidden_size": W, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "dim": m["dim"],
                "value_dim": m["vdim"], "scale": float(m["scale"]), "norm_eps": eps, "qk_norm": "head",
                "window": int(m["mask"]["size"]), "head_gate": True}, weights={r: f"{p}.{r}" for r in ("q", "k", "v", "g", "o")}), None
        if layer["type"] == "rglru":
            weights = {r: f"{p}.{r}" for r in ("y", "x", "conv", "ra", "ri", "lam", "o")}
            weights.update({f"{r}_bias": f"{p}.{r}.b" for r in ("y", "x", "conv", "ra", "ri")})
            return PartSpec(kind="real_gated_recurrence", params={
                "hidden_size": W, "width": m["width"], "blocks": m["blocks"], "taps": m["conv"]}, weights=weights), None
        src = self.kv_source(i)
        weights = {r: f"{p}.{r}" for r in ("dq", "uq", "uk", "uv", "g", "o")}
        weights["dq_norm"] = f"{p}.dq.norm"
        if src == i:
            weights.update(dkv=f"{p}.dkv", dkv_norm=f"{p}.dkv.norm")
        mixer = PartSpec(kind="latent_attention", params={
            "hidden_size": W, "num_heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "value_dim": m["vdim"],
            "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": float(m["scale"]), "norm_eps": eps,
            "window": int(m["mask"]["size"]), "cache_window": self.cache_reach(src), "element_gate": True, "own_kv": src == i},
            weights=weights)
        position = PartSpec(kind="rotary", params={
            "head_dim": m["rot_dim"], "rotary_dim": m["rot"]["dims"], "theta": float(m["rot"]["base"]),
            "max_positions": NO_POSITION_LIMIT, "pairing": "halves", "scaling": None})
        return mixer, position

    def _feed_forward(self, i: int) -> Optional[PartSpec]:
        mlp, p = self.layers[i].get("mlp"), f"l{i}.mlp"
        if mlp is None:
            return None
        E = int(mlp["router"]["experts"])
        weights = {"weight": f"{p}.router", "bias": f"{p}.router.b"}
        for e in range(E):
            weights.update({f"{r}.{e}": f"{p}.e{e}.{r}" for r in ("up", "down")})
        return PartSpec(kind="experts", params={
            "hidden_size": self.width, "n_experts": E, "top": int(mlp["router"]["top"]), "expert_size": mlp["expert"]["ff"],
            "gated": False, "activation": "relu_squared", "shared": None, "router": {"kind": "softmax", "renormalize": True}},
            weights=weights)

    def build_spec(self) -> ModelSpec:
        W, n = self.width, len(self.layers)
        blocks = []
        for i in range(n):
            mixer, position = self._mixer(i)
            ff = self._feed_forward(i)
            weights = {"mixer_out": f"l{i}.norm1"}
            if ff is not None:
                weights["feed_forward_out"] = f"l{i}.norm2"
            blocks.append(BlockSpec(kind="post_norm", mixer=mixer, feed_forward=ff, mixer_norm=None, feed_forward_norm=None,
                                    position=position, weights=weights, params={
                                        "size": W, "eps": self.norm_eps, "takes_rounded": True, "leaves_rounded": i < n - 1}))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=W, max_positions=NO_POSITION_LIMIT,
            embedding=PartSpec(kind="embedding", params={"vocab_size": self.vocab, "hidden_size": W, "leaves_rounded": True},
                               weights={"weight": "embed"}),
            blocks=blocks,
            schedule=[ScheduleEntry(layer=i, cache=self.kv_source(i), writes_cache=self.kv_source(i) == i) for i in range(n)],
            final_norm=PartSpec(kind="rmsnorm", params={"size": W, "eps": self.norm_eps}, weights={"weight": "final.norm"}),
            head=PartSpec(kind="linear_head", params={"vocab_size": self.vocab, "hidden_size": W}, weights={"weight": "embed"}),
            stop_token_ids=list(self.eos_token_ids))
        spec.validate()
        return spec

    def tensor_shapes(self) -> Dict[str, List[int]]:
        W = self.width
        shapes: Dict[str, List[int]] = {"embed": [self.vocab, W], "final.norm": [W]}
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}", layer["mixer"]
            q = p + ".mix"
            shapes[f"{p}.norm1"] = [W]
            if layer["type"] == "attention":
                H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
                shapes[f"{q}.q"], shapes[f"{q}.k"], shapes[f"{q}.v"] = [H * D, W], [G * D, W], [G * V, W]
                shapes[f"{q}.g"], shapes[f"{q}.o"] = [H, W], [W, H * V]
            elif layer["type"] == "rglru":
                C, nb = m["width"], m["blocks"]
                for r in ("y", "x"):
                    shapes[f"{q}.{r}"], shapes[f"{q}.{r}.b"] = [C, W], [C]
                shapes[f"{q}.conv"], shapes[f"{q}.conv.b"], shapes[f"{q}.lam"] = [C, m["conv"]], [C], [C]
                for r in ("ra", "ri"):
                    shapes[f"{q}.{r}"], shapes[f"{q}.{r}.b"] = [nb, C // nb, C // nb], [nb, C // nb]
                shapes[f"{q}.o"] = [W, C]
            else:
                H, D, R, V, rank, qr = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
                shapes[f"{q}.dq"], shapes[f"{q}.dq.norm"], shapes[f"{q}.uq"] = [qr, W], [qr], [H * (D + R), qr]
                if self.kv_source(i) == i:
                    shapes[f"{q}.dkv"], shapes[f"{q}.dkv.norm"] = [rank + R, W], [rank]
                shapes[f"{q}.uk"], shapes[f"{q}.uv"] = [H * D, rank], [H * V, rank]
                shapes[f"{q}.g"], shapes[f"{q}.o"] = [H * V, W], [W, H * V]
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            shapes[f"{p}.norm2"] = [W]
            for e in range(mlp["router"]["experts"]):
                shapes[f"{p}.mlp.e{e}.up"], shapes[f"{p}.mlp.e{e}.down"] = [mlp["expert"]["ff"], W], [W, mlp["expert"]["ff"]]
            shapes[f"{p}.mlp.router"], shapes[f"{p}.mlp.router.b"] = [mlp["router"]["experts"], W], [mlp["router"]["experts"]]
        return shapes

    def ignorable_tensor(self, name: str) -> bool:
        """Stored tensors that this configuration never reads: the second norm of a layer without a feed-forward."""
        head, _, rest = name.partition(".")
        return rest == "norm2" and head[:1] == "l" and head[1:].isdigit() and int(head[1:]) < len(self.layers) \
            and self.layers[int(head[1:])].get("mlp") is None

    def is_norm_tensor(self, name: str) -> bool:
        return name.rsplit(".", 1)[-1] in ("norm", "norm1", "norm2")

    def special_random_tensor(self, name: str, seed: int, device, std: float) -> Optional[torch.Tensor]:
        """Random values for what is neither a matrix nor a norm weight: biases of the matrices' spread (so that they do not
        drown what the matrices say of a token), gate matrices and convolution taps of order one over their fan-in's root,
        decay rates that keep a state for a few to a few hundred tokens."""
        from ..weights.random_fill import fnv1a64
        shape = self.tensor_shapes()[name]
        g = torch.Generator().manual_seed((seed * 0x9E3779B1 + fnv1a64(name)) % (1 << 62))
        last = name.rsplit(".", 1)[-1]
        if last == "b":
            t = std * torch.randn(shape, generator=g)
        elif last == "lam":
            t = -1.0 - 5.0 * torch.rand(shape, generator=g)
        elif last in ("conv", "ra", "ri"):
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
        else:
            return None
        return t.to(torch.bfloat16).contiguous().to(device)

    def parameter_count(self) -> int:
        total = 0
        for shape in self.tensor_shapes().values():
            n = 1
            for s in shape:
                n *= s
            total += n
        return total
