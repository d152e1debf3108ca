"""Plain, slow implementation of the Barorax design: whole sequences, no cache, one function per mechanism.

Written from the design's equations on a raw config dict and a dict of tensors. It shares no code with skein_b200: it is
what the framework's operators, cache and scheduler are compared with. Everything runs in the dtype of `x` (the tests use
float64 or float32); weights are cast to it where they are used. The recurrence goes one token at a time.
"""
from __future__ import annotations

import math

import torch


def rms(v, eps):
    """v divided by its root mean square over the last dimension."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_pairs(v, positions, dims, base):
    """Pairs (2i, 2i + 1) of the first `dims` coordinates turned by position * base^(-2i / dims). v [T, D]."""
    out = v.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(v.dtype), torch.sin(a).to(v.dtype)
        u, w = v[:, 2 * i], v[:, 2 * i + 1]
        out[:, 2 * i] = u * c - w * s
        out[:, 2 * i + 1] = w * c + u * s
    return out


def softmax_map(q, k, v, scale, visible, sink=False):
    """One attention map: q, k [T, D], v [T, V], visible [T, T]. With `sink` the weights' denominator has one more term, exp(0)."""
    s = ((q @ k.T) * scale).masked_fill(~visible, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    if sink:
        total = total + torch.exp(-top)
    return (e / total) @ v


def difference_weight(m, W):
    return torch.exp((W("lq1") * W("lk1")).sum()) - torch.exp((W("lq2") * W("lk2")).sum()) + m["diff"]


def differential_attention(h, m, W, eps):
    """Two maps per head over the same values, the second subtracted with a weight; head norm; output gate."""
    T, H, G, D, V, rot = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    pos = torch.arange(T)
    q = (h @ W("q").T).view(T, H, 2, D)
    k = (h @ W("k").T).view(T, G, 2, D)
    v = (h @ W("v").T).view(T, G, V)
    causal = pos[None, :] <= pos[:, None]
    lam = difference_weight(m, W)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        a = [softmax_map(rotate_pairs(q[:, n, j], pos, rot["dims"], rot["base"]), rotate_pairs(k[:, g, j], pos, rot["dims"], rot["base"]),
                         v[:, g], m["scale"], causal) for j in (0, 1)]
        out[:, n] = rms(a[0] - lam * a[1], eps) * (1.0 - m["diff"])
    return (out.reshape(T, H * V) * sigmoid(h @ W("g").T)) @ W("o").T


def chunked_attention(h, m, W, eps):
    """Causal attention inside chunks counted from position 0; unit root mean square of rotated queries and keys; a sink."""
    T, H, G, D, V, rot, size = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"], m["mask"]["size"]
    pos = torch.arange(T)
    q, k, v = (h @ W("q").T).view(T, H, D), (h @ W("k").T).view(T, G, D), (h @ W("v").T).view(T, G, V)
    visible = (pos[None, :] <= pos[:, None]) & (pos[None, :] // size == pos[:, None] // size)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        qn = rms(rotate_pairs(q[:, n], pos, rot["dims"], rot["base"]), eps)
        kn = rms(rotate_pairs(k[:, g], pos, rot["dims"], rot["base"]), eps)
        out[:, n] = softmax_map(qn, kn, v[:, g], m["scale"], visible, sink=True)
    return out.reshape(T, H * V) @ W("o").T


def causal_conv(x, w, b):
    """out[t, c] = b[c] + sum_j w[c, j] * x[t - taps + 1 + j, c], zeros before the start. x [T, C], w [C, taps]."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        out[t] = b
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out


def selective_scan(x, dt, A, B, C, D):
    """Diagonal recurrence per channel and state dimension. x, dt [T, I]; A [I, N]; B, C [T, N]; D [I]."""
    S = torch.zeros_like(A)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba(h, m, W, eps):
    I, N, R = m["inner"], m["state"], m["dt_rank"]
    p = h @ W("in").T
    x, z = p[:, :I], p[:, I:]
    x = silu(causal_conv(x, W("conv"), W("conv.b")))
    p = x @ W("x").T
    dt = softplus(p[:, :R] @ W("dt").T + W("dt.b"))
    y = selective_scan(x, dt, -torch.exp(W("A_log")), p[:, R:R + N], p[:, R + N:], W("D"))
    return (y * silu(z)) @ W("o").T


MIXERS = {"attention": differential_attention, "attention_2": chunked_attention, "mamba1": mamba}


def gated_unit(h, W):
    return (silu(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


def choose_experts(s, top, count, keep):
    """Indices of the `top` largest scores among the best `keep` of `count` groups of neighbours; a group counts its two best."""
    per = s.shape[0] // count
    groups = s.view(count, per)
    worth = [sum(sorted(g.tolist(), reverse=True)[:2]) for g in groups]
    kept = sorted(range(count), key=lambda g: (-worth[g], g))[:keep]
    allowed = [e for e in range(s.shape[0]) if e // per in kept]
    return sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]


def routed_experts(h, ml, W):
    r = ml["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = sigmoid(h @ W("router").T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose_experts(s[t], r["top"], groups["count"], groups["keep"])
        total = sum(s[t, e] for e in ids) + 1e-20
        for e in ids:
            out[t] += r["scale"] * s[t, e] / total * gated_unit(h[t:t + 1], lambda n: W(f"e{e}.{n}"))[0]        # noqa: B023
    if ml.get("shared"):
        out = out + gated_unit(h, lambda n: W("shared." + n))
    return out


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
    norm = lambda x, n: rms(x, eps) * T(n)        # noqa: E731
    x = T("embed")[torch.as_tensor(tokens).long()]
    for i, t in layer_runs(cfg):
        layer = cfg["layers"][i]
        if t is not None and i == cfg["loop"]["start"]:
            x = x + T("loop.step")[t]
        x = x + MIXERS[layer["type"]](norm(x, f"l{i}.norm1"), layer["mixer"], lambda n: T(f"l{i}.mix.{n}"), eps)        # noqa: B023
        if layer["mlp"] is not None:
            x = x + routed_experts(norm(x, f"l{i}.norm2"), layer["mlp"], lambda n: T(f"l{i}.mlp.{n}"))        # noqa: B023
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ T("head").T
