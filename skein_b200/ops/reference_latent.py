"""Plain PyTorch reference of the operators in ops/latent.py (post-norm blocks of latent attention): the implementation on
CPU-only machines. Same shapes and conventions; sums, norms, rotation and softmax in fp32, results in the activation type.
"""
from __future__ import annotations

import torch


def _rows_of(block_table, seq, positions, page_size):
    """(page, slot) of each absolute position of a sequence."""
    pages = block_table[seq].long()[positions // page_size]
    return pages, positions % page_size


def conv_input(x, conv, tail, positions, seq_of_token, q_start, block_table, page_size, dtype, write_tail):
    T, C = x.shape
    taps = conv.shape[0]
    R = tail.shape[1] if tail is not None else 0
    xr = x.to(dtype).float()
    h = x.clone()
    for t in range(T):
        pos = int(positions[t])
        seq = int(seq_of_token[t]) if seq_of_token is not None else t
        first = int(q_start[seq]) if q_start is not None else t
        h[t] += conv[taps - 1] * xr[t]
        for j in range(1, taps):
            q = pos - j
            if q < 0:
                break
            if t - j >= first:
                v = xr[t - j]
            else:
                page, slot = int(block_table[seq, q // page_size]), q % page_size
                v = tail[page, slot % R].float()
            h[t] += conv[taps - 1 - j] * v
        if write_tail and pos >= 0 and R:
            tail[int(block_table[seq, pos // page_size]), (pos % page_size) % R] = x[t].to(dtype)
    return h.to(dtype)


def post_norm(x, y, alpha, gain, eps, row_idx=None, row_w=None):
    v = alpha * x
    if y is not None:
        if row_idx is None:
            v = v + y.float()
        else:
            for j in range(row_idx.shape[1]):
                v = v + row_w[:, j:j + 1].float() * y.float()[row_idx[:, j].long()]
    return v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps) * gain


def rms_rows(v, w, eps):
    v = v.float()
    return v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps) * w


def rotate_pairs(v, cs):
    """v [..., rot] with cs [..., rot/2, 2] broadcastable: neighbouring dimensions turned together."""
    u, w = v.float()[..., 0::2], v.float()[..., 1::2]
    c, s = cs[..., 0], cs[..., 1]
    return torch.stack([u * c - w * s, w * c + u * s], dim=-1).flatten(-2)


def latent_append(proj, off_kv, q_norm, kv_norm, rot, cos_sin, positions, seq_of_token, block_table, cache, eps, x, tail, seq_lens, taps):
    """Returns the normed query latent (or None); writes the cache rows and, with x, the convolution's tail rows."""
    T, K = proj.shape[0], kv_norm.shape[0]
    ps = cache.shape[1]
    cq = rms_rows(proj[:, :q_norm.shape[0]], q_norm, eps).to(proj.dtype) if q_norm is not None else None
    c = rms_rows(proj[:, off_kv:off_kv + K], kv_norm, eps)
    kr = rotate_pairs(proj[:, off_kv + K:off_kv + K + rot], cos_sin[positions.long().clamp(min=0)])
    rows = torch.cat([c, kr], dim=1).to(proj.dtype)
    R = tail.shape[1] if tail is not None else 0
    for t in range(T):
        pos = int(positions[t])
        if pos < 0:
            continue
        seq = int(seq_of_token[t]) if seq_of_token is not None else t
        page, slot = int(block_table[seq, pos // ps]), pos % ps
        cache[page, slot] = rows[t]
        if x is not None and R and (pos >= int(seq_lens[seq]) - (taps - 1) or slot >= ps - (taps - 1)):
            tail[page, slot % R] = x[t].to(tail.dtype)
    return cq


def latent_attention_rows(q_abs, q, D, rot, scale, cos_sin, positions, seq_of_token, block_table, cache, sinks=None):
    """q_abs [T, H, K]; q [T, H, D + rot] (rotated part not yet rotated). Returns [T, H, K]."""
    T, H, K = q_abs.shape
    ps = cache.shape[1]
    qr = rotate_pairs(q[..., D:], cos_sin[positions.long().clamp(min=0)].unsqueeze(1)).to(q.dtype).float()
    out = torch.zeros(T, H, K, dtype=q_abs.dtype)
    ctx = {}
    for t in range(T):
        pos = int(positions[t])
        if pos < 0:
            continue
        seq = int(seq_of_token[t]) if seq_of_token is not None else t
        n = pos + 1
        if seq not in ctx or ctx[seq].shape[0] < n:
            upto = int(positions[seq_of_token == seq].max()) + 1 if seq_of_token is not None else n
            pages = block_table[seq, :(upto + ps - 1) // ps].long()
            ctx[seq] = cache[pages].reshape(-1, cache.shape[2]).float()
        kv = ctx[seq][:n]
        s = (q_abs[t].float() @ kv[:, :K].t() + qr[t] @ kv[:, K:].t()) * scale
        if sinks is not None:
            s = torch.cat([s, sinks[:, None]], dim=-1)
        out[t] = (torch.softmax(s, dim=-1)[:, :n] @ kv[:, :K]).to(out.dtype)
    return out


def head_linear(x, x_cols, w, gate=None):
    """Per-head product: x [T, >= H * x_cols] read in blocks of x_cols columns (the first K of each), w [H, F, K] -> [T, H * F]."""
    H, F, K = w.shape
    xs = torch.stack([x[:, h * x_cols:h * x_cols + K] for h in range(H)]).float()
    y = torch.einsum("htk,hfk->thf", xs, w.float()).reshape(x.shape[0], H * F)
    if gate is not None:
        y = y * torch.sigmoid(gate.float())
    return y.to(x.dtype)


def poly_norm(z, act, eps):
    z = z.float()
    n = lambda v: v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)     # noqa: E731
    return act[0] * n(z) + act[1] * n(z ** 2) + act[2] * n(z ** 3) + act[3]


def clamped_glu(g, u, limit, slope):
    g, u = g.float().clamp(max=limit), u.float().clamp(-limit, limit)
    return g * torch.sigmoid(slope * g) * (u + 1.0)


def select_grouped(logits, top, groups, keep):
    """(ids int32 [T, top], weights fp32): softmax over all experts, best `keep` of the `groups` eligible, not renormalised."""
    T, E = logits.shape
    s = torch.softmax(logits.float(), dim=-1)
    z = logits.float()
    if keep < groups:
        best = z.view(T, groups, E // groups).amax(-1)
        kept = torch.sort(best, dim=-1, descending=True, stable=True).indices[:, :keep]
        ok = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, kept, True)
        z = z.masked_fill(~ok.repeat_interleave(E // groups, dim=1), float("-inf"))
    ids = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :top]
    return ids.to(torch.int32), s.gather(1, ids)
