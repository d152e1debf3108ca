"""Plain, slow implementation of the Zarorax design: whole sequences, no cache, one function per mechanism.

Written from the design's equations on a raw config dict and a dict of tensors. It shares no code with skein_b200: it is
what the framework's operators, cache and scheduler are compared with. Everything runs in the dtype of `x` (the tests use
float64 or float32); weights are cast to it where they are used.
"""
from __future__ import annotations

import math

import torch


def rms(v, eps):
    """v divided by its root mean square over the last dimension."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def scalar_norm(v, g, eps):
    """RMS norm whose gain is one number for all coordinates."""
    return rms(v, eps) * g


def vector_norm(v, w, eps):
    return rms(v, eps) * w


def causal_conv(h, w):
    """out[t, c] = sum_j w[c, j] * h[t - taps + 1 + j, c], zeros before the start. h [T, C], w [C, taps]."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def rotate_interleaved(v, positions, dims, base):
    """Pairs (2i, 2i + 1) of the first `dims` coordinates turned by position * base^(-2i / dims). v [..., T, D]."""
    out = v.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(v.dtype), torch.sin(a).to(v.dtype)
        u, w = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = u * c - w * s
        out[..., 2 * i + 1] = w * c + u * s
    return out


def latent_attention(h, m, W, eps, gated, q_latent):
    """h [T, C]; m: the mixer's sizes; W(name): its tensors. Keys and values are expanded per head from the latent."""
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    if q_latent:
        q = vector_norm(h @ W("dq").T, W("dq.norm"), eps) @ W("uq").T
    else:
        q = h @ W("q").T
    q = q.view(T, H, D + R)
    ckr = h @ W("dkv").T
    c = vector_norm(ckr[:, :K], W("dkv.norm"), eps)
    k_rot = rotate_interleaved(ckr[:, K:], pos, m["rot"]["dims"], m["rot"]["base"])
    k = (c @ W("uk").T).view(T, H, D)
    v = (c @ W("uv").T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    for n in range(H):
        q_rot = rotate_interleaved(q[:, n, D:], pos, m["rot"]["dims"], m["rot"]["base"])
        s = (q[:, n, :D] @ k[:, n].T + q_rot @ k_rot.T) * m["scale"]
        out[:, n] = torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1) @ v[:, n]
    out = out.reshape(T, H * V)
    if gated:
        out = out * torch.sigmoid(h @ W("g").T)
    return out @ W("o").T


def poly_norm(z, act, eps):
    a, b, c, e = (act[i] for i in range(4))
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense_ff(h, W, eps):
    return poly_norm(h @ W("up").T, W("act"), eps) @ W("down").T


def route(z, top, groups=None):
    """Router logits [E] of one token -> (chosen experts, their weights): softmax over all experts, only the best `keep`
    groups eligible, weights not renormalised."""
    s = torch.softmax(z, dim=-1)
    E = z.shape[0]
    allowed = torch.ones(E, dtype=torch.bool)
    if groups:
        per = E // groups["count"]
        best = s.view(groups["count"], per).max(dim=1).values
        kept = torch.topk(best, groups["keep"]).indices
        allowed[:] = False
        for g in kept.tolist():
            allowed[g * per:(g + 1) * per] = True
    chosen = torch.topk(s.masked_fill(~allowed, -1.0), top).indices
    return chosen, s[chosen]


def expert_ff(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def moe_ff(h, mlp, W):
    z = h @ W("router").T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, ws = route(z[t], mlp["router"]["top"], mlp["router"].get("groups"))
        for e, w in zip(ids.tolist(), ws):
            out[t] += w * expert_ff(h[t], W(f"e{e}.gate"), W(f"e{e}.up"), W(f"e{e}.down"), mlp["expert"]["limit"])
    return out


def forward(cfg, tensors, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence. layers_out: a list that receives the residual stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    T = lambda name: tensors[name].to(dtype)        # noqa: E731
    x = T("embed")[torch.as_tensor(tokens).long()]
    for i, layer in enumerate(cfg["layers"]):
        j = layer.get("weights_of")
        j = i if j is None else j
        mix = lambda n: T(f"l{j}.mix.{n}")          # noqa: E731
        ff = lambda n: T(f"l{j}.mlp.{n}")           # noqa: E731
        h = x + causal_conv(x, T(f"l{j}.canon1"))
        y = latent_attention(h, layer["mixer"], mix, eps, gated=layer["type"] == "latent_attention_2",
                             q_latent=layer["type"] == "latent_attention")
        x = scalar_norm(alpha * x + y, T(f"l{j}.norm1"), eps)
        if layer["mlp"] is not None:
            y = dense_ff(x, ff, eps) if layer["mlp"]["kind"] == "dense" else moe_ff(x, layer["mlp"], ff)
            x = scalar_norm(alpha * x + y, T(f"l{j}.norm2"), eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return scalar_norm(x, T("final.norm"), eps) @ T("head").T
