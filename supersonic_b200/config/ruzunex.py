"""Typed configuration of the ``Ruzunex`` architecture.

Its config.json is nested.  Top level: ``vocab``, ``width``, ``norm.eps``, ``canon.taps``, ``streams`` and ``layers``, a list
with one entry per layer: ``type`` (``attention`` or ``parallel``), ``mixer`` (that mixer's sizes and constants) and ``mlp``
(null, ``{"kind": "dense", "ff"}`` or ``{"kind": "moe", "router": {"experts", "top"}, "expert": {"ff", "limit"}}``).

``build_spec`` turns that into parts.  A layer is a ``hyper_connections`` block: ``streams`` residual streams, of which
each sublayer reads a weighted sum (``hc1.in``, ``hc2.in``) through an RMS norm and a short causal convolution
(``canon1``, ``canon2``), and into which its result is written (``hc1.out``) while the streams are mixed (``hc1.mix``).
The mixers:

* ``attention``: a ``window_attention`` inside a sliding window ``mask.size`` without rotation: norms of q and k per head, a
  bias that grows with the distance, values mixed with those of the first layer that says ``v_mix``, a sigmoid gate
  per element of the heads;
* ``parallel``: a ``mixer_pair`` whose halves are added, each times a constant of its own (``left_scale``,
  ``right_scale``): a ``window_attention`` over all earlier tokens (convolutions of ``conv`` taps behind the projections of
  q, k and v, norms over the whole projection, the first ``rot.dims`` coordinates rotated, a factor per head on the
  scores, a learned sink per head), and an ``hgrn2`` recurrence.

The feed-forward is a gated unit with gelu (``swiglu`` with ``activation``), or ``experts`` with the clamped activation
behind a ``softmax`` router whose weights are renormalized.  Tensor names: ``embed``, ``final.norm``, ``head`` and per layer i
``l<i>.norm1``, ``norm2``, ``canon1``, ``canon2``, ``hc1.*``, ``hc2.*``, ``l<i>.mix.*``, ``l<i>.mlp.*``.  The design has no position
limit; the cache bounds a sequence.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

import torch

from .base import BlockSpec, ConfigError, ModelSpec, PartSpec, default_schedule
from .kilisun import GATE_SLOPE_ACTIVATION, NO_POSITION_LIMIT, _number
from .ronelorn import _need, _positive

ARCHITECTURE = "Ruzunex"
MIXERS = ("attention", "parallel")
MAX_TAPS = 16
MAX_STREAMS = 16


def _taps(d, key: str, where: str) -> None:
    v = d[key]
    if isinstance(v, bool) or not isinstance(v, int) or not 1 <= v <= MAX_TAPS:
        raise ConfigError(f"{where}.{key} must be 1 to {MAX_TAPS} taps, got {v!r}")


def _heads(m, where: str) -> None:
    _need(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
    _positive(m, ("heads", "kv_heads", "dim", "vdim"), where)
    _number(m, "scale", where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: {m['heads']} heads over {m['kv_heads']} kv heads")


@dataclass(frozen=True)
class RuzunexConfig:
    vocab: int
    width: int
    norm_eps: float
    taps: int
    streams: int
    layers: List[Dict[str, Any]] = field(default_factory=list)
    eos_token_ids: List[int] = field(default_factory=list)
    model_type: str = "ruzunex"

    # ---- reading -----------------------------------------------------
    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "RuzunexConfig":
        _need(d, ("vocab", "width", "layers", "norm", "canon", "streams"), "config.json")
        _need(d["norm"], ("eps",), "norm")
        _need(d["canon"], ("taps",), "canon")
        _taps(d["canon"], "taps", "canon")
        _positive(d, ("vocab", "width", "streams"), "config.json")
        eos = d.get("eos_token_id")
        cfg = RuzunexConfig(
            vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float(d["norm"]["eps"]), taps=int(d["canon"]["taps"]),
            streams=int(d["streams"]), layers=copy.deepcopy(list(d["layers"])),
            eos_token_ids=[] if eos is None else [int(eos)] if isinstance(eos, int) else [int(e) for e in eos])
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.norm_eps > 0:
            raise ConfigError("norm.eps must be positive")
        if self.streams > MAX_STREAMS:
            raise ConfigError(f"streams must be 1 to {MAX_STREAMS}, got {self.streams}")
        if not self.layers:
            raise ConfigError("layers must name at least one layer")
        mixed = None
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            m, kind = layer["mixer"], layer["type"]
            if kind == "attention":
                _heads(m, where + ".mixer")
                _need(m, ("mask",), where + ".mixer")
                _need(m["mask"], ("size",), where + ".mixer.mask")
                _positive(m["mask"], ("size",), where + ".mixer.mask")
                if m.get("v_mix"):
                    values = m["kv_heads"] * m["vdim"]
                    if mixed is not None and values != mixed:
                        raise ConfigError(f"{where}.mixer: {values} values a token cannot be mixed with {mixed}")
                    mixed = values
            elif kind == "parallel":
                _need(m, ("left", "right", "left_scale", "right_scale"), where + ".mixer")
                for s in ("left_scale", "right_scale"):
                    _number(m, s, where + ".mixer", positive=False)
                left, right = m["left"], m["right"]
                _heads(left, where + ".mixer.left")
                _need(left, ("conv", "rot"), where + ".mixer.left")
                _taps(left, "conv", where + ".mixer.left")
                _need(left["rot"], ("base", "dims"), where + ".mixer.left.rot")
                dims = left["rot"]["dims"]
                if not isinstance(dims, int) or isinstance(dims, bool) or dims < 0 or dims % 2 or dims > left["dim"]:
                    raise ConfigError(f"{where}.mixer.left.rot.dims must be even and at most dim, got {dims!r}")
                _number(left["rot"], "base", where + ".mixer.left.rot")
                _need(right, ("heads", "dim", "vdim"), where + ".mixer.right")
                _positive(right, ("heads", "dim", "vdim"), where + ".mixer.right")
            else:
                raise ConfigError(f"{where}.type {kind!r} is not known (known: {list(MIXERS)})")
            self._validate_mlp(layer.get("mlp"), where + ".mlp")
        for e in self.eos_token_ids:
            if not 0 <= e < self.vocab:
                raise ConfigError(f"eos_token_id {e} is outside the vocabulary")

    @staticmethod
    def _validate_mlp(mlp, where: str) -> None:
        if mlp is None:
            return
        kind = mlp.get("kind") if isinstance(mlp, dict) else None
        if kind == "dense":
            _need(mlp, ("ff",), where)
            _positive(mlp, ("ff",), where)
        elif kind == "moe":
            _need(mlp, ("router", "expert"), where)
            _need(mlp["router"], ("experts", "top"), where + ".router")
            _positive(mlp["router"], ("experts", "top"), where + ".router")
            if mlp["router"]["top"] > mlp["router"]["experts"]:
                raise ConfigError(f"{where}.router: {mlp['router']['top']} experts a token of {mlp['router']['experts']}")
            _need(mlp["expert"], ("ff", "limit"), where + ".expert")
            _positive(mlp["expert"], ("ff",), where + ".expert")
            _number(mlp["expert"], "limit", where + ".expert")
        else:
            raise ConfigError(f"{where}.kind {kind!r} is not known (known: 'dense', 'moe')")

    # ---- writing -----------------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": ARCHITECTURE, "canon": {"taps": self.taps}, "layers": copy.deepcopy(self.layers),
                             "norm": {"eps": self.norm_eps}, "streams": self.streams, "vocab": self.vocab,
                             "width": self.width}
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

    def value_mix(self, i: int) -> Optional[str]:
        """``"first"`` for the first layer whose values are mixed into later ones, ``"later"`` for the layers that mix them
        in, None for all others."""
        mixing = [j for j, l in enumerate(self.layers) if l["type"] == "attention" and l["mixer"].get("v_mix")]
        return None if i not in mixing else "first" if i == mixing[0] else "later"

    # ---- the architecture as parts ----------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec(kind="rmsnorm", params={"size": self.width, "eps": self.norm_eps}, weights={"weight": name})

    def _mixer(self, i: int):
        W, eps = self.width, self.norm_eps
        layer, p = self.layers[i], f"l{i}.mix"
        m = layer["mixer"]

        def attention(m_, p_, **more):
            params = {"hidden_size": W, "num_heads": m_["heads"], "num_kv_heads": m_["kv_heads"], "dim": m_["dim"],
                      "value_dim": m_["vdim"], "scale": float(m_["scale"]), "norm_eps": eps, **more}
            return params, {**{r: f"{p_}.{r}" for r in ("q", "k", "v", "o")}, "q_norm": f"{p_}.q.norm", "k_norm": f"{p_}.k.norm"}
        if layer["type"] == "attention":
            mix = self.value_mix(i)
            params, weights = attention(m, p, qk_norm="head", window=int(m["mask"]["size"]), distance_bias="geometric",
                                        element_gate=True, value_mix=mix)
            weights["g"] = f"{p}.g"
            if mix == "later":
                weights["vmix"] = f"{p}.vmix"
            return PartSpec(kind="window_attention", params=params, weights=weights), None
        left, right, lp, rp = m["left"], m["right"], p + ".left", p + ".right"
        rot = left["rot"]
        position = None
        if rot["dims"] > 0:
            position = PartSpec(kind="rotary", params={
                "head_dim": left["dim"], "rotary_dim": rot["dims"], "theta": float(rot["base"]),
                "max_positions": NO_POSITION_LIMIT, "pairing": "halves", "scaling": None})
        params, weights = attention(left, lp, qk_norm="row", window=None, conv=int(left["conv"]), conv_values=True,
                                    head_scale=True, sink="learned", out_scale=float(m["left_scale"]))
        weights.update({f"{r}_conv": f"{lp}.{r}.conv" for r in "qkv"}, temp=f"{lp}.temp", sink=f"{lp}.sink")
        halves = {
            "left": {"kind": "window_attention", "position": True, "params": params, "weights": weights},
            "right": {"kind": "hgrn2", "position": False,
                      "params": {"hidden_size": W, "num_heads": right["heads"], "dim": right["dim"], "value_dim": right["vdim"],
                                 "norm_eps": eps, "out_scale": float(m["right_scale"])},
                      "weights": {**{r: f"{rp}.{r}" for r in ("q", "f", "v", "lower", "norm", "o")}, "f_bias": f"{rp}.f.b"}}}
        # the halves' tensors once more under the pair's own names: what counts weights reads them there
        names = {f"{side}.{role}": name for side, half in halves.items() for role, name in half["weights"].items()}
        return PartSpec(kind="mixer_pair", params={"hidden_size": W, "join": "add", **halves}, weights=names), position

    def _feed_forward(self, i: int) -> Optional[PartSpec]:
        mlp, p, W = self.layers[i].get("mlp"), f"l{i}.mlp", self.width
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec(kind="swiglu", params={"hidden_size": W, "intermediate_size": mlp["ff"],
                                                   "activation": {"kind": "gelu_tanh"}},
                            weights={"gate": f"{p}.gate", "up": f"{p}.up", "down": f"{p}.down"})
        E = int(mlp["router"]["experts"])
        weights = {"weight": f"{p}.router"}
        for e in range(E):
            weights.update({f"{r}.{e}": f"{p}.e{e}.{r}" for r in ("gate", "up", "down")})
        return PartSpec(kind="experts", params={
            "hidden_size": W, "n_experts": E, "top": int(mlp["router"]["top"]), "expert_size": mlp["expert"]["ff"],
            "activation": {"kind": GATE_SLOPE_ACTIVATION, "limit": float(mlp["expert"]["limit"])}, "shared": None,
            "router": {"kind": "softmax", "renormalize": True}}, weights=weights)

    def build_spec(self) -> ModelSpec:
        W = self.width
        blocks = []
        for i in range(len(self.layers)):
            p = f"l{i}"
            mixer, position = self._mixer(i)
            ff = self._feed_forward(i)
            weights = {}
            for n, sub in ((1, "mixer"), (2, "ff"))[: 1 if ff is None else 2]:
                weights.update({f"{sub}_{r}": f"{p}.hc{n}.{r}" for r in ("in", "mix", "out")})
                weights[f"{sub}_conv"] = f"{p}.canon{n}"
            blocks.append(BlockSpec(
                kind="hyper_connections", mixer=mixer, feed_forward=ff, mixer_norm=self._norm(f"{p}.norm1"),
                feed_forward_norm=None if ff is None else self._norm(f"{p}.norm2"), position=position,
                params={"size": W, "streams": self.streams, "taps": self.taps, "feed_forward": ff is not None,
                        "last": i == len(self.layers) - 1}, weights=weights))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=W, max_positions=NO_POSITION_LIMIT,
            embedding=PartSpec(kind="embedding", params={"vocab_size": self.vocab, "hidden_size": W}, weights={"weight": "embed"}),
            blocks=blocks, schedule=default_schedule(len(self.layers)), final_norm=self._norm("final.norm"),
            head=PartSpec(kind="linear_head", params={"vocab_size": self.vocab, "hidden_size": W}, weights={"weight": "head"}),
            stop_token_ids=list(self.eos_token_ids))
        spec.validate()
        return spec

    def tensor_shapes(self) -> Dict[str, List[int]]:
        W, S = self.width, self.streams
        shapes: Dict[str, List[int]] = {"embed": [self.vocab, W], "final.norm": [W], "head": [self.vocab, W]}

        def sublayer(p, n):
            shapes[f"{p}.norm{n}"], shapes[f"{p}.canon{n}"] = [W], [W, self.taps]
            shapes[f"{p}.hc{n}.in"], shapes[f"{p}.hc{n}.out"], shapes[f"{p}.hc{n}.mix"] = [S], [S], [S, S]

        def attention(q, m):
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            shapes[f"{q}.q"], shapes[f"{q}.k"], shapes[f"{q}.v"], shapes[f"{q}.o"] = [H * D, W], [G * D, W], [G * V, W], [W, H * V]
            return H, G, D, V
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}", layer["mixer"]
            q = p + ".mix"
            sublayer(p, 1)
            if layer["type"] == "attention":
                H, G, D, V = attention(q, m)
                shapes[f"{q}.q.norm"], shapes[f"{q}.k.norm"], shapes[f"{q}.g"] = [D], [D], [H * V, W]
                if m.get("v_mix"):
                    shapes[f"{q}.vmix"] = []
            else:
                left, right = m["left"], m["right"]
                H, G, D, V = attention(q + ".left", left)
                lp, rp = q + ".left", q + ".right"
                for r, n in (("q", H * D), ("k", G * D), ("v", G * V)):
                    shapes[f"{lp}.{r}.conv"] = [n, left["conv"]]
                shapes[f"{lp}.q.norm"], shapes[f"{lp}.k.norm"] = [H * D], [G * D]
                shapes[f"{lp}.temp"], shapes[f"{lp}.sink"] = [H], [H]
                HD, HV = right["heads"] * right["dim"], right["heads"] * right["vdim"]
                shapes[f"{rp}.q"], shapes[f"{rp}.f"], shapes[f"{rp}.v"], shapes[f"{rp}.o"] = [HD, W], [HD, W], [HV, W], [W, HV]
                shapes[f"{rp}.f.b"], shapes[f"{rp}.lower"], shapes[f"{rp}.norm"] = [HD], [HD], [right["vdim"]]
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            sublayer(p, 2)
            f = p + ".mlp"

            def unit(prefix, ff):
                shapes[f"{prefix}.gate"], shapes[f"{prefix}.up"], shapes[f"{prefix}.down"] = [ff, W], [ff, W], [W, ff]
            if mlp["kind"] == "dense":
                unit(f, mlp["ff"])
            else:
                for e in range(mlp["router"]["experts"]):
                    unit(f"{f}.e{e}", mlp["expert"]["ff"])
                shapes[f"{f}.router"] = [mlp["router"]["experts"], W]
        return shapes

    def ignorable_tensor(self, name: str) -> bool:
        """Stored tensors that this configuration never reads: the second sublayer's in a layer without one, and a
        mixing share in a layer that does not mix."""
        head, _, rest = name.partition(".")
        if not (head[:1] == "l" and head[1:].isdigit() and int(head[1:]) < len(self.layers)):
            return False
        layer = self.layers[int(head[1:])]
        if layer.get("mlp") is None and (rest in ("norm2", "canon2") or rest.startswith("hc2.")):
            return True
        return rest == "mix.vmix" and layer["type"] == "attention" and not layer["mixer"].get("v_mix")

    def is_norm_tensor(self, name: str) -> bool:
        return name.rsplit(".", 1)[-1] in ("norm", "norm1", "norm2")

    def special_random_tensor(self, name: str, seed: int, device, std: float) -> Optional[torch.Tensor]:
        """Random values for what is neither a matrix nor a norm weight: stream weights whose streams stay of one size,
        convolution taps and mixing shares below one, lower bounds and gate offsets that keep a state for a few to a few
        hundred tokens, score factors near one, sinks of order one."""
        from ..weights.random_fill import fnv1a64
        shape = self.tensor_shapes()[name]
        g = torch.Generator().manual_seed((seed * 0x9E3779B1 + fnv1a64(name)) % (1 << 62))
        last, two = name.rsplit(".", 1)[-1], ".".join(name.rsplit(".", 2)[-2:])
        S = self.streams
        if two in ("hc1.in", "hc2.in"):
            t = 1.0 / S + 0.2 * torch.randn(shape, generator=g)
        elif two in ("hc1.out", "hc2.out"):
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif two in ("hc1.mix", "hc2.mix"):
            t = 0.8 * torch.eye(S) + 0.2 / S + 0.1 * torch.randn(shape, generator=g)
        elif last in ("canon1", "canon2"):
            t = 0.3 * torch.randn(shape, generator=g)
        elif last == "conv":
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif last == "vmix":
            t = 0.2 + 0.6 * torch.rand(shape, generator=g)
        elif last == "temp":
            t = 0.7 + 0.6 * torch.rand(shape, generator=g)
        elif last == "sink":
            t = torch.randn(shape, generator=g)
        elif two == "f.b":
            t = 1.0 + torch.randn(shape, generator=g)
        elif last == "lower":
            t = 0.98 * torch.rand(shape, generator=g)
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
