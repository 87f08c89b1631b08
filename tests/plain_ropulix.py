"""A plain, slow statement of the Ropulix design in float64 on the CPU: one function per mechanism, one sequence at a
time, every query a Python loop over what it may see.  It shares no code with the library: the tests compare the
library's kernels, cache and step function against it.

``weights`` maps tensor names to tensors, ``config`` is the dictionary of a config.json.  Every function takes a whole
sequence ``[T, ...]`` and starts from empty state; ``forward`` returns the logits of every position and the stream after
every layer.  ``twist`` (a set of names) plants a mistake: what a test uses to show that its weights would reveal one.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def _w(weights, name):
    return weights[name].to(F)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def weighted_norm(x, w, eps):
    return unit_rms(x, eps) * w


def in_window(i, size):
    """The positions a query at i sees: itself and the size - 1 before it."""
    return [j for j in range(i + 1) if i - j < size]


def softmax_sum(scores, values):
    return torch.softmax(scores, dim=0) @ values


def turn(x, dims, base):
    """x [T, ..., d]: the first ``dims`` coordinates turned by the row's position, coordinate i with i + dims / 2."""
    half = dims // 2
    angle = torch.arange(x.shape[0], dtype=F)[:, None] * torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c, s = torch.cos(angle).reshape(shape), torch.sin(angle).reshape(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def head_attention(h, weights, p, m, eps, twist=()):
    """The mixer ``attention``: no positions, q and k of unit root mean square per head, a window, one gate per head."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ _w(weights, f"{p}.q").T).reshape(T, H, D)
    k = (h @ _w(weights, f"{p}.k").T).reshape(T, G, D)
    v = (h @ _w(weights, f"{p}.v").T).reshape(T, G, V)
    if "no_qk_norm" not in twist:
        q, k = unit_rms(q, eps), unit_rms(k, eps)
    gate = sigmoid(h @ _w(weights, f"{p}.g").T)
    if "no_gate" in twist:
        gate = torch.ones_like(gate)
    size = m["mask"]["size"] + (1 if "attention_window" in twist else 0)
    out = torch.zeros((T, H, V), dtype=F)
    for i in range(T):
        vis = in_window(i, size)
        for a in range(H):
            g = a % G if "head_order" in twist else a // (H // G)
            out[i, a] = softmax_sum((k[vis, g] @ q[i, a]) * m["scale"], v[vis, g]) * gate[i, a]
    return out.reshape(T, -1) @ _w(weights, f"{p}.o").T


def latent_rows(h, weights, p, m, eps):
    """What a latent layer keeps of every token: the normed latent [T, kv_rank] and the turned key part [T, rot_dim]."""
    y = h @ _w(weights, f"{p}.dkv").T
    R = m["kv_rank"]
    return weighted_norm(y[:, :R], _w(weights, f"{p}.dkv.norm"), eps), turn(y[:, R:], m["rot"]["dims"], m["rot"]["base"])


def latent_attention(h, weights, p, m, eps, rows=None, twist=()):
    """The mixer ``latent_attention``, keys and values written out per head; ``rows``: another layer's (latent, key part)."""
    H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    T = h.shape[0]
    c, kr = latent_rows(h, weights, p, m, eps) if rows is None else rows
    cq = h @ _w(weights, f"{p}.dq").T
    if "no_query_norm" not in twist:
        cq = weighted_norm(cq, _w(weights, f"{p}.dq.norm"), eps)
    q = (cq @ _w(weights, f"{p}.uq").T).reshape(T, H, D + R)
    qu, qr = q[..., :D], turn(q[..., D:], m["rot"]["dims"], m["rot"]["base"])
    if "no_rotation" in twist:
        qr = q[..., D:]
    ku = (c @ _w(weights, f"{p}.uk").T).reshape(T, H, D)
    v = (c @ _w(weights, f"{p}.uv").T).reshape(T, H, V)
    size = m["mask"]["size"] + (1 if "latent_window" in twist else 0)
    out = torch.zeros((T, H, V), dtype=F)
    for i in range(T):
        vis = in_window(i, size)
        for a in range(H):
            s = (ku[vis, a] @ qu[i, a] + kr[vis] @ qr[i, a]) * m["scale"]
            out[i, a] = softmax_sum(s, v[vis, a])
    gate = sigmoid(h @ _w(weights, f"{p}.g").T)
    if "no_latent_gate" in twist:
        gate = torch.ones_like(gate)
    return (out.reshape(T, -1) * gate) @ _w(weights, f"{p}.o").T


def causal_conv(x, w, bias):
    """x [T, C], w [C, taps] (the last column is the current token's): zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = bias.expand(T, -1).clone()
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                y[t] += w[:, j] * x[src]
    return y


def rglru(h, weights, p, m, twist=()):
    """The mixer ``rglru``: a gelu branch times a gated linear recurrence behind a short convolution."""
    T, C, nb = h.shape[0], m["width"], m["blocks"]
    bs = C // nb
    y = gelu(h @ _w(weights, f"{p}.y").T + _w(weights, f"{p}.y.b"))
    x = h @ _w(weights, f"{p}.x").T + _w(weights, f"{p}.x.b")
    w = _w(weights, f"{p}.conv")
    u = causal_conv(x, w.flip(1) if "flipped_taps" in twist else w, _w(weights, f"{p}.conv.b"))
    ub = u.reshape(T, nb, bs)

    def gate(name):
        z = torch.einsum("tbi,boi->tbo", ub, _w(weights, f"{p}.{name}")) + _w(weights, f"{p}.{name}.b")
        return sigmoid(z.reshape(T, C))
    r, i = gate("ra"), gate("ri")
    lam = _w(weights, f"{p}.lam")
    log_a = -8.0 * r * torch.log1p(torch.exp(lam))
    S, out = torch.zeros(C, dtype=F), torch.zeros((T, C), dtype=F)
    for t in range(T):
        share = torch.sqrt(-torch.expm1(2.0 * log_a[t]))
        if t == 0 and "first_token" in twist:
            share = torch.ones_like(share)
        if "state_lost" in twist and t == T // 2:
            S = torch.zeros(C, dtype=F)
        S = torch.exp(log_a[t]) * S + share * i[t] * u[t]
        out[t] = S
    return (out * y) @ _w(weights, f"{p}.o").T


def route(h, weights, p, top, twist=()):
    """Per token the experts with the largest logits, and the softmax over those logits alone."""
    z = h @ _w(weights, f"{p}.router").T
    if "no_router_bias" not in twist:
        z = z + _w(weights, f"{p}.router.b")
    chosen, weight = [], []
    for t in range(h.shape[0]):
        idx = sorted(range(z.shape[1]), key=lambda e: (-float(z[t, e]), e))[:top]
        over = z[t] if "softmax_over_all" in twist else z[t, idx]
        share = torch.exp(z[t, idx] - over.max()) / torch.exp(over - over.max()).sum()
        chosen.append(idx)
        weight.append(share.tolist())
    return chosen, weight


def expert(h, weights, p):
    return torch.relu(h @ _w(weights, f"{p}.up").T) ** 2 @ _w(weights, f"{p}.down").T


def experts(h, weights, p, mlp, twist=()):
    chosen, weight = route(h, weights, p, mlp["router"]["top"] + (1 if "one_expert_more" in twist else 0), twist)
    out = torch.zeros((h.shape[0], _w(weights, f"{p}.e0.down").shape[0]), dtype=F)
    for e in range(mlp["router"]["experts"]):
        rows = [t for t in range(h.shape[0]) if e in chosen[t]]
        if rows:
            share = torch.tensor([weight[t][chosen[t].index(e)] for t in rows], dtype=F)
            out[rows] += share[:, None] * expert(h[rows], weights, f"{p}.e{e}")
    return out


def forward(config, weights, tokens, twist=()):
    """(logits [T, vocab], the stream after every layer [layers, T, width])."""
    eps = config["norm"]["eps"]
    x = _w(weights, "embed")[torch.as_tensor(tokens)]
    kept, streams = {}, []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = unit_rms(x, eps) if "norm_before" in twist else x
        if layer["type"] == "attention":
            y = head_attention(h, weights, f"{p}.mix", m, eps, twist)
        elif layer["type"] == "rglru":
            y = rglru(h, weights, f"{p}.mix", m, twist)
        else:
            src = m.get("kv_from")
            if src is None:
                src = i
                kept[i] = latent_rows(h, weights, f"{p}.mix", m, eps)
            y = latent_attention(h, weights, f"{p}.mix", m, eps, kept[src], twist)
        x = x + weighted_norm(y, _w(weights, f"{p}.norm1"), eps)
        if layer.get("mlp") is not None:
            x = x + weighted_norm(experts(x, weights, f"{p}.mlp", layer["mlp"], twist), _w(weights, f"{p}.norm2"), eps)
        streams.append(x.clone())
    return weighted_norm(x, _w(weights, "final.norm"), eps) @ _w(weights, "embed").T, torch.stack(streams)
