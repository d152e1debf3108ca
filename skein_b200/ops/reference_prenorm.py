"""Plain PyTorch form of the operators of pre-norm layers and of the selective scan (ops/prenorm.py, ops/selective.py): 32-bit math,
results in the activation type."""
from __future__ import annotations

import torch


def add_norm(x, y, row_idx, row_w, step, gain, eps, dtype):
    a = x
    if y is not None:
        a = a + sum(row_w[:, j:j + 1] * y.float()[row_idx[:, j].long()] for j in range(row_idx.shape[1]))
    if step is not None:
        a = a + step
    return a, None if gain is None else (a / torch.sqrt(a.pow(2).mean(-1, keepdim=True) + eps) * gain).to(dtype)


def depth_norm(terms, weights, gain, groups, eps, dtype, x_out, shift, inp, slots, decode):
    x = terms[0] if weights is None else sum(weights[j] * terms[j] for j in range(terms.shape[0]))
    if x_out is not None:
        x_out.copy_(x)
    T, C = x.shape
    v = x.view(T, groups, C // groups)
    h = (v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, C) * gain
    if shift is None:
        return h.to(dtype)
    out = h.clone()
    n = inp.seq_lens.shape[0]
    starts, lens = (range(n), [1] * n) if decode else (inp.q_start.tolist(), inp.q_len.tolist())
    for s, (t0, m) in enumerate(zip(starts, lens)):
        if m < 1 or int(inp.positions[t0]) < 0:
            continue
        before = shift.state[int(slots[s])].clone() if int(inp.positions[t0]) > 0 else torch.zeros(C)
        for t in range(t0, t0 + m):
            out[t] = h[t] + (before - h[t]) * shift.mix
            before = h[t]
        shift.state[int(slots[s])] = before
    return out.to(dtype)


def select(logits, f):
    """(ids int32 [T, top], weights fp32) by the rule of `f`."""
    T, E = logits.shape
    s = torch.sigmoid(logits) if f.score == "sigmoid" else torch.softmax(logits, dim=-1)
    z = s
    if f.keep < f.groups:
        best = s.view(T, f.groups, E // f.groups)
        best = best.topk(min(f.group_best, best.shape[-1]), dim=-1).values.sum(-1)
        kept = torch.sort(best, dim=-1, descending=True, stable=True).indices[:, :f.keep]
        ok = torch.zeros(T, f.groups, dtype=torch.bool).scatter_(1, kept, True)
        z = s.masked_fill(~ok.repeat_interleave(E // f.groups, dim=1), -1.0)
    ids = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :f.top]
    w = s.gather(1, ids)
    if f.renorm:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return ids.to(torch.int32), w * f.scale


# ---- selective scan ---------------------------------------------------------------------------------------------------
def short_conv(x, taps, w, state, positions, slots, q_start, q_len):
    """Convolution and silu of portions (rows q_start[s] .. of sequence s); the state's last inputs are left alone (scan writes them)."""
    out = torch.zeros(x.shape, dtype=x.dtype)
    for s in range(q_len.shape[0]):
        t0, n = int(q_start[s]), int(q_len[s])
        if n < 1 or int(positions[t0]) < 0:
            continue
        pos0, slot = int(positions[t0]), int(slots[s])
        prev = torch.zeros(taps - 1, x.shape[1])
        for j in range(1, taps):
            if pos0 - j >= 0:
                prev[taps - 1 - j] = state.tail[slot, (pos0 - j) % taps].float()
        full = torch.cat([prev, x[t0:t0 + n].float()])
        out[t0:t0 + n] = torch.nn.functional.silu(sum(w.conv[j] * full[j:j + n] for j in range(taps)) + w.conv_b).to(x.dtype)
    return out


def scan(xc, proj, dt, x, z, out, spec, w, state, positions, slots, q_start, q_len):
    N, taps = spec.state, spec.taps
    b0 = (spec.dt_rank + 7) // 8 * 8
    c0 = b0 + (N + 7) // 8 * 8
    for s in range(q_len.shape[0]):
        t0, n = int(q_start[s]), int(q_len[s])
        if n < 1 or int(positions[t0]) < 0:
            continue
        pos0, slot = int(positions[t0]), int(slots[s])
        S = state.mat[slot].clone() if pos0 > 0 else torch.zeros_like(state.mat[slot])
        step = torch.nn.functional.softplus(dt[t0:t0 + n] + w.dt_bias, threshold=60.0)
        u = xc[t0:t0 + n].float()
        for t in range(n):
            p = proj[t0 + t].float()
            S = torch.exp(step[t] * w.neg_a) * S + (step[t] * u[t]) * p[b0:b0 + N, None]
            y = p[c0:c0 + N] @ S + w.skip * u[t]
            out[t0 + t] = (y * torch.nn.functional.silu(z[t0 + t].float())).to(out.dtype)
        state.mat[slot] = S
        if state.tail is not None:
            for j in range(max(0, n - taps + 1), n):
                state.tail[slot, (pos0 + j) % taps] = x[t0 + j].to(state.tail.dtype)
