"""Plain, slow implementation of the Sikalorn design: whole sequences, no cache, one function per mechanism.

Written from the design's equations on a raw config dict and a dict of tensors. It shares no code with skein_b200: it is
what the framework's operators, cache and scheduler are compared with. Everything runs in the dtype of `x` (the tests use
float64 or float32); weights are cast to it where they are used. Recurrences go one token at a time.
"""
from __future__ import annotations

import math

import torch


def rms(v, eps):
    """v divided by its root mean square over the last dimension."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def causal_conv(h, w, b=None):
    """out[t, c] = b[c] + sum_j w[c, j] * h[t - taps + 1 + j, c], zeros before the start. h [T, C], w [C, taps]."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for t in range(T):
        if b is not None:
            out[t] += b
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def rotate_half(v, positions, dims, base, factor):
    """Pairs (i, i + dims / 2) of the first `dims` coordinates turned by position * base^(-2i / dims) / factor. v [..., T, D]."""
    out = v.clone()
    n = dims // 2
    for i in range(n):
        a = positions.to(torch.float64) * (base ** (-2.0 * i / dims) / factor)
        c, s = torch.cos(a).to(v.dtype), torch.sin(a).to(v.dtype)
        u, w = v[..., i], v[..., n + i]
        out[..., i] = u * c - w * s
        out[..., n + i] = w * c + u * s
    return out


def windowed_attention(h, m, W, eps):
    """Grouped-query attention over a sliding window; query and key norm over all heads at once, before the rotation."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot, size = m["rot"], m["mask"]["size"]
    pos = torch.arange(T)
    q = (rms(h @ W("q").T, eps) * W("q.norm")).view(T, H, D)
    k = (rms(h @ W("k").T, eps) * W("k.norm")).view(T, G, D)
    v = (h @ W("v").T).view(T, G, V)
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    back = pos[:, None] - pos[None, :]
    visible = (back >= 0) & (back < size)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        qn = rotate_half(q[:, n], pos, rot["dims"], rot["base"], factor)
        kn = rotate_half(k[:, g], pos, rot["dims"], rot["base"], factor)
        s = (qn @ kn.T) * m["scale"]
        out[:, n] = torch.softmax(s.masked_fill(~visible, -math.inf), dim=-1) @ v[:, g]
    return out.reshape(T, H * V) @ W("o").T


def state_space(h, m, W, eps):
    """Mamba-2: one scalar decay per head and token, inputs scaled by the step size, a skip D x, gate before the norm."""
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    p = h @ W("in").T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, W("conv"), W("conv.b")))
    x = xbc[:, :inner].view(T, H, V)
    B = xbc[:, inner:inner + G * N].view(T, G, N).repeat_interleave(H // G, dim=1)
    C = xbc[:, inner + G * N:].view(T, G, N).repeat_interleave(H // G, dim=1)
    dt = softplus(dt + W("dt_bias"))
    decay = torch.exp(-torch.exp(W("A_log")) * dt)
    S = torch.zeros(H, N, V, dtype=h.dtype)
    y = torch.zeros(T, H, V, dtype=h.dtype)
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnv,hn->hv", S, C[t]) + W("D")[:, None] * x[t]
    y = (y.reshape(T, inner) * silu(z)).view(T, m["norm_groups"], -1)
    return (rms(y, eps).reshape(T, inner) * W("norm")) @ W("o").T


def two_mixers(h, m, W, eps):
    left = windowed_attention(h, m["left"], lambda n: W("left." + n), eps)
    right = state_space(h, m["right"], lambda n: W("right." + n), eps)
    return m["left_scale"] * left + m["right_scale"] * right


def unit(v):
    return v / torch.sqrt((v * v).sum(-1, keepdim=True) + 1e-6)


def gated_delta(h, m, W, eps):
    """Gated delta rule: the state decays, then what it holds for k is replaced by v to the degree beta."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ W("q").T, W("q.conv"))).view(T, G, D)
    k = silu(causal_conv(h @ W("k").T, W("k.conv"))).view(T, G, D)
    v = silu(causal_conv(h @ W("v").T, W("v.conv"))).view(T, H, V)
    q = (unit(q) * D ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(k).repeat_interleave(H // G, dim=1)
    beta = sigmoid(h @ W("b").T)
    g = torch.exp(-torch.exp(W("A_log")) * softplus(h @ W("a").T + W("dt_bias")))
    S = torch.zeros(H, D, V, dtype=h.dtype)
    o = torch.zeros(T, H, V, dtype=h.dtype)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    o = rms(o, eps) * W("norm") * silu(h @ W("g").T).view(T, H, V)
    return o.reshape(T, H * V) @ W("o").T


def lightning(h, m, W, eps):
    """Linear attention with one fixed decay per head."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ W(n).T) for n in ("q", "k", "v"))
    q, k, v = q.view(T, H, D), k.view(T, H, D), v.view(T, H, V)
    decay = torch.tensor(m["decay"], dtype=h.dtype)
    S = torch.zeros(H, D, V, dtype=h.dtype)
    o = torch.zeros(T, H, V, dtype=h.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    o = rms(o.reshape(T, H * V), eps) * W("norm") * sigmoid(h @ W("g").T)
    return o @ W("o").T


MIXERS = {"parallel": two_mixers, "delta": gated_delta, "lightning": lightning}


def squared_relu_ff(h, W):
    return torch.clamp(h @ W("up").T, min=0) ** 2 @ W("down").T


def layer_runs(cfg):
    """(layer, pass) in the order they run; pass is None outside the loop."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(cfg, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence. layers_out: a list that receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    T = lambda name: tensors[name].to(dtype)        # noqa: E731
    norm = lambda x, n: dynamic_tanh(x, T(n + ".alpha"), T(n), T(n + ".b"))        # noqa: E731
    x0 = x = T("embed")[torch.as_tensor(tokens).long()]
    for i, t in layer_runs(cfg):
        layer = cfg["layers"][i]
        if t is not None and i == cfg["loop"]["start"]:
            x = torch.cat([x, x0], dim=-1) @ T("loop.in").T + T("loop.step")[t]
        h = norm(x, f"l{i}.norm1")
        y = MIXERS[layer["type"]](h, layer["mixer"], lambda n: T(f"l{i}.mix.{n}"), eps)        # noqa: B023
        if layer["mlp"] is not None:
            y = y + squared_relu_ff(h, lambda n: T(f"l{i}.mlp.{n}"))        # noqa: B023
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ T("head").T
