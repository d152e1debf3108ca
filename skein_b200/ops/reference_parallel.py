"""Plain PyTorch form of the operators of parallel layers, sliding-window attention and recurrences (ops/parallel.py,
ops/recurrent.py): 32-bit math, results in the activation type."""
from __future__ import annotations

import torch

from .reference_latent import rotate_pairs


def residual_tanh(x, y, bias, norm, dtype):
    a = sum(t.float() for t in (x, y, bias) if t is not None)
    if norm is None:
        return a, a.to(dtype)
    return a, (torch.tanh(norm.alpha * a) * norm.w + norm.b).to(dtype)


def gated_norm(o, gate, w, groups, eps, gate_first, silu, scale):
    T, n = o.shape
    v, z = o.float(), gate.float()
    g = torch.nn.functional.silu(z) if silu else torch.sigmoid(z)
    if gate_first:
        v = v * g
    v = v.view(T, groups, -1)
    v = (v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, n) * w.repeat(n // w.shape[0])
    return ((v if gate_first else v * g) * scale).to(o.dtype)


def _rotate(x, cos_sin, dims):
    half = dims // 2
    c, s = cos_sin[:, None, :half, 0], cos_sin[:, None, :half, 1]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def _pages(cache, K, ps, D, V):
    """(keys [pages, K, ps, D], values [pages, K, ps, V]) views of a cache."""
    n = K * ps * D
    return cache[:, :n].view(-1, K, ps, D), cache[:, n:].view(-1, K, ps, V)


def window_append(q, k, v, q_norm, k_norm, spec, cos_sin, positions, seq_of_token, block_table, cache, page_size, eps):
    keys, vals = _pages(cache, spec.kv_heads, page_size, spec.dim, spec.vdim)
    T = q.shape[0]
    for t in range(T):
        pos = int(positions[t])
        if pos < 0:
            continue
        cs = cos_sin[pos:pos + 1]
        unit = lambda z, w: z.float() / torch.sqrt(z.float().pow(2).mean() + eps) * w        # noqa: E731
        q[t] = _rotate(unit(q[t], q_norm).view(1, spec.heads, -1), cs, spec.rot_dims).reshape(-1).to(q.dtype)
        page = int(block_table[int(seq_of_token[t]) if seq_of_token is not None else t, pos // page_size])
        keys[page, :, pos % page_size] = _rotate(unit(k[t], k_norm).view(1, spec.kv_heads, -1), cs, spec.rot_dims)[0].to(cache.dtype)
        vals[page, :, pos % page_size] = v[t].view(spec.kv_heads, -1)


def head_append(q, k, v, spec, cos_sin, positions, seq_of_token, block_table, cache, page_size, eps, w=None, mix=None):
    D, W = spec.dim, spec.key_width
    keys, vals = _pages(cache, spec.kv_heads, page_size, W, spec.vdim)

    def turn(z, cs, bias, norm):
        z = z.float()
        if bias is not None:
            z = z + bias
        z = z.view(-1, D)
        if norm is not None:
            z = z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps) * norm
        if cs is None:
            pass
        elif spec.interleaved:
            z = torch.cat([rotate_pairs(z[:, :spec.rot_dims], cs), z[:, spec.rot_dims:]], dim=1)
        else:
            z = _rotate(z[None], cs, spec.rot_dims)[0]
        return z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps) if spec.unit else z
    for t in range(q.shape[0]):
        pos = int(positions[t])
        if pos < 0:
            continue
        cs = cos_sin[pos:pos + 1] if cos_sin is not None else None
        qb, kb, vb = (w.q_bias, w.k_bias, w.v_bias) if spec.bias else (None, None, None)
        qn, kn = (w.q_norm, w.k_norm) if spec.head_norm else (None, None)
        q[t] = turn(q[t], cs, qb, qn).reshape(-1).to(q.dtype)
        page = int(block_table[int(seq_of_token[t]) if seq_of_token is not None else t, pos // page_size])
        keys[page, :, pos % page_size] = turn(k[t], cs, kb, kn).view(spec.kv_heads, W).to(cache.dtype)
        x = v[t].float() + (vb if vb is not None else 0.0)
        if mix is not None and mix.keep:
            mix.v_first[t] = x.to(v.dtype)
        elif mix is not None:
            x = (1.0 - w.vmix) * x + w.vmix * mix.v_first[t].float()
        vals[page, :, pos % page_size] = x.to(cache.dtype).view(spec.kv_heads, -1)


def window_attn_rows(q, spec, positions, seq_of_token, block_table, cache, page_size, out_scale, mix=None):
    H, D, V, M = spec.heads, spec.dim, spec.vdim, spec.maps
    keys, vals = _pages(cache, spec.kv_heads, page_size, spec.key_width, V)
    T, G = q.shape[0], spec.heads // spec.kv_heads
    out = torch.zeros(T, H * V, dtype=q.dtype)
    for t in range(T):
        pos = int(positions[t])
        if pos < 0:
            continue
        lo = pos // spec.chunk * spec.chunk if spec.chunk else max(0, pos - spec.window + 1) if spec.window else 0
        kept = min(spec.keep_first, lo) if spec.window else 0
        js = torch.cat([torch.arange(kept), torch.arange(lo, pos + 1)])
        pages = block_table[int(seq_of_token[t]) if seq_of_token is not None else t][js // page_size].long()
        k = keys[pages, :, js % page_size].float().view(-1, spec.kv_heads, M, D).repeat_interleave(G, dim=1)
        v = vals[pages, :, js % page_size].float().repeat_interleave(G, dim=1)
        s = torch.einsum("hmd,jhmd->hmj", q[t].float().view(H, M, D), k) * spec.scale
        if spec.softcap:
            s = spec.softcap * torch.tanh(s / spec.softcap)
        if spec.sink:
            s = torch.cat([s, torch.zeros(H, M, 1)], dim=-1)
        if spec.head_sink:
            s = torch.cat([s, mix.sinks.view(H, 1, 1).expand(H, M, 1)], dim=-1)
        p = torch.softmax(s, dim=-1)[..., :len(js)]
        a = torch.einsum("hmj,jhv->hmv", p, v)
        o = a[:, 0]
        if spec.diff is not None:
            o = a[:, 0] - mix.lam * a[:, 1]
            o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + mix.eps) * (1.0 - spec.diff)
        o = o.reshape(-1)
        if mix is not None and mix.gate is not None:
            o = o * torch.sigmoid(mix.gate[t].float())
        out[t] = (o * out_scale).to(q.dtype)
    return out


def rec_chunk(row, cols, spec, w, state, positions, slots, q_start, q_len, step=None):
    H, G, D, V, taps = spec.heads, spec.groups, spec.dim, spec.vdim, spec.taps
    dt = row.dtype
    out = torch.zeros(row.shape[0], H * V, dtype=dt)
    for s in range(q_len.shape[0]):
        t0, n = int(q_start[s]), int(q_len[s])
        if n < 1 or int(positions[t0]) < 0:
            continue
        pos0, slot = int(positions[t0]), int(slots[s])
        r = row[t0:t0 + n].float()
        x = torch.cat([r[:, cols.q:cols.q + G * D], r[:, cols.k:cols.k + G * D], r[:, cols.v:cols.v + H * V]], dim=1)
        if spec.conv_channels:
            prev = torch.zeros(taps - 1, x.shape[1])
            for j in range(1, taps):
                if pos0 - j >= 0:
                    prev[taps - 1 - j] = state.tail[slot, (pos0 - j) % taps].float()
            full = torch.cat([prev, x])
            if state.tail is not None:
                for j in range(max(0, n - taps + 1), n):
                    state.tail[slot, (pos0 + j) % taps] = x[j].to(state.tail.dtype)
            x = sum(w.conv[j] * full[j:j + n] for j in range(taps)) + (w.conv_b if w.conv_b is not None else 0.0)
        x = torch.nn.functional.silu(x).to(dt).float()
        q, k, v = x[:, :G * D].view(n, G, D), x[:, G * D:2 * G * D].view(n, G, D), x[:, 2 * G * D:].view(n, H, V)
        if spec.corrects:
            q, k = (z / torch.sqrt(z.pow(2).sum(-1, keepdim=True) + 1e-6) for z in (q, k))
            q = q * D ** -0.5
        q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
        if spec.kind == "lightning":
            g, coef = (w.neg_decay.exp() if w.decay is None else w.decay).expand(n, H), torch.ones(n, H)
        elif spec.kind == "channel_delta":
            a = torch.nn.functional.softplus(step[t0:t0 + n] + w.dt_bias, threshold=60.0).view(n, H, D)
            g, coef = (w.neg_decay[:, None] * a).exp(), torch.sigmoid(r[:, cols.b:cols.b + H])
        else:
            step = torch.nn.functional.softplus(r[:, cols.a:cols.a + H] + w.dt_bias, threshold=60.0)
            g = (w.neg_decay * step).exp()
            coef = torch.sigmoid(r[:, cols.b:cols.b + H]) if spec.kind == "delta" else step
        S = state.mat[slot].clone() if pos0 > 0 else torch.zeros(H, D, V)
        for t in range(n):
            S = g[t].view(H, -1, 1) * S
            u = v[t] - torch.einsum("hdv,hd->hv", S, k[t]) if spec.corrects else v[t]
            S = S + k[t][:, :, None] * (coef[t][:, None] * u)[:, None, :]
            o = torch.einsum("hdv,hd->hv", S, q[t])
            if w.skip is not None:
                o = o + w.skip[:, None] * v[t]
            out[t0 + t] = o.reshape(-1).to(dt)
        state.mat[slot] = S
    return out
