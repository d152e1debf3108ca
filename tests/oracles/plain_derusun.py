"""Plain, slow implementation of the Derusun design: whole sequences, no cache, one function per mechanism.

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


def grouped_norm(x, w, groups, eps):
    """Every one of `groups` equal parts of a row divided by its own root mean square; one weight per element."""
    T, C = x.shape
    return rms(x.view(T, groups, C // groups), eps).reshape(T, C) * w


def token_shift(h, mix):
    """h + (the previous token's h - h) * mix, element by element; zeros before the first token."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mix


def depth_average(outputs, weights):
    """Weighted sum of the embedding output and every layer's result so far."""
    return sum(weights[j] * x for j, x in enumerate(outputs))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def unit(v):
    return v / torch.sqrt((v * v).sum(-1, keepdim=True) + 1e-6)


def causal_conv(x, w):
    """out[t, c] = sum_j w[c, j] * x[t - taps + 1 + j, c], zeros before the start. x [T, C], w [C, taps]."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out


def delta_rule(q, k, v, beta, g):
    """Per head a state [D, V] whose rows decay by g; what it holds for k is then replaced by v to the degree beta; read with q.
    q, k, g [T, H, D]; v [T, H, V]; beta [T, H]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o


def channel_decay(h, W, heads):
    """One decay per head and key channel."""
    a = (h @ W("a1").T) @ W("a2").T + W("dt_bias")
    return torch.exp(-torch.exp(W("A_log"))[None, :, None] * softplus(a).view(h.shape[0], heads, -1))


def channel_delta(h, m, W, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ W("q").T, W("q.conv"))).view(T, G, D)
    k = silu(causal_conv(h @ W("k").T, W("k.conv"))).view(T, G, D)
    v = silu(causal_conv(h @ W("v").T, W("v.conv"))).view(T, H, V)
    q = (unit(q) * D ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(k).repeat_interleave(H // G, dim=1)
    o = delta_rule(q, k, v, sigmoid(h @ W("b").T), channel_decay(h, W, H))
    gate = sigmoid((h @ W("g1").T) @ W("g2").T).view(T, H, V)
    return (rms(o, eps) * W("norm") * gate).reshape(T, H * V) @ W("o").T


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


def sink_softmax(s, visible, sink):
    """Weights of the visible scores; the denominator has one more term, exp(sink)."""
    s = s.masked_fill(~visible, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h, m, W, eps):
    T, H, D, R, V, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ W("q").T).view(T, H, D + R)
    ckr = h @ W("dkv").T
    c = rms(ckr[:, :K], eps) * W("dkv.norm")
    kr = rotate_pairs(ckr[:, K:], pos, m["rot"]["dims"], m["rot"]["base"])
    kn, v = (c @ W("uk").T).view(T, H, D), (c @ W("uv").T).view(T, H, V)
    causal = pos[None, :] <= pos[:, None]
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        qr = rotate_pairs(q[:, n, D:], pos, m["rot"]["dims"], m["rot"]["base"])
        s = (q[:, n, :D] @ kn[:, n].T + qr @ kr.T) * m["scale"]
        out[:, n] = sink_softmax(s, causal, W("sink")[n]) @ v[:, n]
    return out.reshape(T, H * V) @ W("o").T


def visible_keys(T, size, keep):
    """Position i sees the last `size` positions, its own included, and the sequence's first `keep`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep))


def attention_values(h, W):
    return h @ W("v").T + W("v.b")


def mixed_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, m, W, eps, v_first=None):
    """v_first: values [T, G V] of the first layer that mixes values, None in that layer and without mixing."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ W("q").T + W("q.b")).view(T, H, D), eps) * W("q.norm")
    k = rms((h @ W("k").T + W("k.b")).view(T, G, D), eps) * W("k.norm")
    v = attention_values(h, W)
    if v_first is not None:
        v = mixed_values(v, v_first, W("vmix"))
    v = v.view(T, G, V)
    visible = visible_keys(T, m["mask"]["size"], m["mask"].get("keep_first", 0))
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        s = m["softcap"] * torch.tanh((q[:, n] @ k[:, g].T) * m["scale"] / m["softcap"])
        out[:, n] = sink_softmax(s, visible, W("sink")[n]) @ v[:, g]
    return out.reshape(T, H * V) @ W("o").T


def clamped_unit(h, limit, W):
    g = torch.clamp(h @ W("gate").T, max=limit)
    u = torch.clamp(h @ W("up").T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W("down").T


def forward(cfg, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence. layers_out: a list that receives the stream behind every layer, averaged over depth."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    T = lambda name: tensors[name].to(dtype)        # noqa: E731
    norm = lambda x, n: grouped_norm(x, T(n), groups, eps)        # noqa: E731
    x = T("embed")[torch.as_tensor(tokens).long()]
    outputs, v_first = [x], None
    for i, layer in enumerate(cfg["layers"]):
        W = lambda n: T(f"l{i}.mix.{n}")        # noqa: B023, E731
        m, h = layer["mixer"], token_shift(norm(x, f"l{i}.norm1"), T(f"l{i}.shift"))
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y = attention(h, m, W, eps, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = attention_values(h, W)
        else:
            y = {"channel_delta": channel_delta, "latent_attention": latent_attention}[layer["type"]](h, m, W, eps)
        x = x + y
        if layer["mlp"] is not None:
            x = x + clamped_unit(norm(x, f"l{i}.norm2"), layer["mlp"]["limit"], lambda n: T(f"l{i}.mlp.{n}"))        # noqa: B023
        outputs.append(x)
        x = depth_average(outputs, T(f"l{i}.dwa"))
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ T("head").T
