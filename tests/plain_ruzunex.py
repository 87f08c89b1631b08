"""A plain, slow statement of the Ruzunex design in float64 on the CPU: one function per mechanism, one sequence at a
time, every query and every recurrent step a turn of a Python loop.  It shares no code with the library: the tests
compare the library's kernels, cache and step function against it.

``weights`` maps tensor names to tensors, ``config`` is the dictionary of a config.json.  Every function takes a
whole sequence ``[T, ...]`` and starts from empty state; ``forward`` returns the logits of every position and the
stream (the sum of the streams) after every layer.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def _w(weights, name):
    return weights[name].to(F)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def short_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                y[t] += w[:, j] * u[src]
    return y


def with_conv(h, w):
    """What a sublayer reads: its input and a short convolution of it over time."""
    return h + short_conv(h, w)


def turn(x, dims, base):
    """x [T, heads, d]: the first ``dims`` coordinates turned by the row's position, i with i + dims / 2."""
    if not dims:
        return x
    half = dims // 2
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    angle = torch.arange(x.shape[0], dtype=F)[:, None] * freq[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def weighted_sum(scores, values, sink=None):
    """Softmax of the scores [n] over the values [n, v]; a sink joins the denominator alone."""
    m = float(scores.max()) if sink is None else max(float(scores.max()), float(sink))
    e = torch.exp(scores - m)
    total = e.sum() + (0.0 if sink is None else math.exp(float(sink) - m))
    return (e @ values) / total


def mixed_values(v, first, lam):
    """The values of a mixing layer behind the first one (element by element of a token's values, whatever the heads)."""
    return (1.0 - lam) * v + lam * first.reshape(v.shape)


def biased_attention(h, weights, p, m, eps, first_values=None):
    """The mixer ``attention``: a sliding window, a bias that falls with the distance, norms per head, values mixed
    with those of the first mixing layer (None: this is that layer, or it does not mix), an output gate per element.
    Returns the result and the layer's own values as projected."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = unit_rms((h @ _w(weights, f"{p}.q").T).reshape(T, H, D), eps) * _w(weights, f"{p}.q.norm")
    k = unit_rms((h @ _w(weights, f"{p}.k").T).reshape(T, G, D), eps) * _w(weights, f"{p}.k.norm")
    own = (h @ _w(weights, f"{p}.v").T).reshape(T, G, V)
    v = own if first_values is None else mixed_values(own, first_values, _w(weights, f"{p}.vmix").reshape(()))
    gate = sigmoid(h @ _w(weights, f"{p}.g").T)                          # [T, H * V]
    out = torch.zeros((T, H, V), dtype=F)
    for i in range(T):
        vis = [j for j in range(i + 1) if i - j < m["mask"]["size"]]
        away = torch.tensor([float(i - j) for j in vis], dtype=F)
        for a in range(H):
            g = a // (H // G)
            s = (k[vis, g] @ q[i, a]) * m["scale"] - slope(a, H) * away
            out[i, a] = weighted_sum(s, v[vis, g])
    return (out.reshape(T, -1) * gate) @ _w(weights, f"{p}.o").T, own


def sink_attention(h, weights, p, m, eps):
    """The left half of ``parallel``: short convolutions behind all three projections, a norm over the whole
    projection, rotation, a factor per head on the scores, causal softmax with a learned sink per head."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (short_conv(h @ _w(weights, f"{p}.{r}").T, _w(weights, f"{p}.{r}.conv")) for r in "qkv")
    q = unit_rms(q, eps) * _w(weights, f"{p}.q.norm")
    k = unit_rms(k, eps) * _w(weights, f"{p}.k.norm")
    q = turn(q.reshape(T, H, D), m["rot"]["dims"], m["rot"]["base"])
    k = turn(k.reshape(T, G, D), m["rot"]["dims"], m["rot"]["base"])
    v = v.reshape(T, G, V)
    temp, sink = _w(weights, f"{p}.temp"), _w(weights, f"{p}.sink")
    out = torch.zeros((T, H, V), dtype=F)
    for i in range(T):
        for a in range(H):
            g = a // (H // G)
            s = (k[: i + 1, g] @ q[i, a]) * m["scale"] * temp[a]
            out[i, a] = weighted_sum(s, v[: i + 1, g], sink=sink[a])
    return out.reshape(T, -1) @ _w(weights, f"{p}.o").T


def tied_recurrence(h, weights, p, m, eps):
    """The right half of ``parallel``: a matrix state per head whose forget gate also says what is written."""
    H, D, V = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(h @ _w(weights, f"{p}.q").T).reshape(T, H, D)
    v = (h @ _w(weights, f"{p}.v").T).reshape(T, H, V)
    low = _w(weights, f"{p}.lower")
    f = low + (1.0 - low) * sigmoid(h @ _w(weights, f"{p}.f").T + _w(weights, f"{p}.f.b"))
    f = f.reshape(T, H, D)
    S = torch.zeros((H, D, V), dtype=F)
    out = torch.zeros((T, H, V), dtype=F)
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return (unit_rms(out, eps) * _w(weights, f"{p}.norm")).reshape(T, -1) @ _w(weights, f"{p}.o").T


def side_by_side(h, weights, p, m, eps):
    """The mixer ``parallel``."""
    return m["left_scale"] * sink_attention(h, weights, f"{p}.left", m["left"], eps) \
        + m["right_scale"] * tied_recurrence(h, weights, f"{p}.right", m["right"], eps)


def gelu_unit(h, weights, p):
    """The dense feed-forward: down(gelu(gate) up)."""
    return (gelu_tanh(h @ _w(weights, f"{p}.gate").T) * (h @ _w(weights, f"{p}.up").T)) @ _w(weights, f"{p}.down").T


def clamped_unit(h, weights, p, limit):
    """An expert: g = min(gate, limit), u = clamp(up, +-limit), down(g sigmoid(1.702 g) (u + 1))."""
    g = torch.clamp(h @ _w(weights, f"{p}.gate").T, max=limit)
    u = torch.clamp(h @ _w(weights, f"{p}.up").T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ _w(weights, f"{p}.down").T


def route(h, weights, p, r):
    """Per token the experts with the largest softmax scores, and their scores divided by their sum."""
    s = torch.softmax(h @ _w(weights, f"{p}.router").T, dim=-1)
    chosen, weight = [], []
    for t in range(h.shape[0]):
        idx = sorted(range(r["experts"]), key=lambda e: (-float(s[t, e]), e))[: r["top"]]
        total = sum(float(s[t, e]) for e in idx) + 1e-20
        chosen.append(idx)
        weight.append([float(s[t, e]) / total for e in idx])
    return chosen, weight


def experts(h, weights, p, mlp):
    chosen, weight = route(h, weights, p, mlp["router"])
    out = torch.zeros((h.shape[0], _w(weights, f"{p}.e0.down").shape[0]), dtype=F)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weight[t]):
            out[t] += w * clamped_unit(h[t:t + 1], weights, f"{p}.e{e}", mlp["expert"]["limit"])[0]
    return out


def feed_forward(h, weights, p, mlp):
    return gelu_unit(h, weights, p) if mlp["kind"] == "dense" else experts(h, weights, p, mlp)


def read_streams(xs, weights, p):
    """u = sum_s in[s] x_s; xs [S, T, width]."""
    return torch.einsum("s,stw->tw", _w(weights, f"{p}.in"), xs)


def write_streams(xs, y, weights, p):
    """x_t <- sum_s mix[s, t] x_s + out[t] y, all from the old streams."""
    return torch.einsum("st,snw->tnw", _w(weights, f"{p}.mix"), xs) + _w(weights, f"{p}.out")[:, None, None] * y


def forward(config, weights, tokens):
    """(logits [T, vocab], the sum of the streams after every layer [layers, T, width])."""
    eps = config["norm"]["eps"]
    x = _w(weights, "embed")[torch.as_tensor(tokens)]
    xs = torch.stack([x] * config["streams"])
    first, sums = None, []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = with_conv(unit_rms(read_streams(xs, weights, f"{p}.hc1"), eps) * _w(weights, f"{p}.norm1"), _w(weights, f"{p}.canon1"))
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = biased_attention(h, weights, f"{p}.mix", m, eps, first if mixes else None)
            if mixes and first is None:
                first = own
        else:
            y = side_by_side(h, weights, f"{p}.mix", m, eps)
        xs = write_streams(xs, y, weights, f"{p}.hc1")
        if layer.get("mlp") is not None:
            h = with_conv(unit_rms(read_streams(xs, weights, f"{p}.hc2"), eps) * _w(weights, f"{p}.norm2"), _w(weights, f"{p}.canon2"))
            xs = write_streams(xs, feed_forward(h, weights, f"{p}.mlp", layer["mlp"]), weights, f"{p}.hc2")
        sums.append(xs.sum(0))
    logits = (unit_rms(xs.sum(0), eps) * _w(weights, "final.norm")) @ _w(weights, "head").T
    return logits, torch.stack(sums)
