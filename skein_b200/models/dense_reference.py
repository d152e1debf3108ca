"""Straight-line, cache-free PyTorch implementation of the same decoder math (fp32 compute on bf16
weights), independent of the operator interface. It follows the HuggingFace Mixtral / Llama
modelling code step by step (RMSNorm -> attention with NeoX RoPE and causal mask -> residual ->
RMSNorm -> top-k softmax-routed SwiGLU experts or SwiGLU MLP -> residual) and serves as the
"HF-style" oracle of the parity gate and of the graph tests, in the role of the reference's Python
subprocess oracle (crates/skein_parity/reference/verify_reference.py).
"""
from __future__ import annotations

import math

import torch

from ..ops.reference import rope_inv_freq
from .config import ModelConfig
from .decoder import ModelWeights


def _rms(x, g, eps):
    xf = x.float()
    return (xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)) * g.float()


def _rope(x, pos, theta, scaling=None):
    # x: [T, heads, D]
    D = x.shape[-1]
    half = D // 2
    inv = rope_inv_freq(D, theta, scaling).to(x.device)
    ang = pos.double().unsqueeze(1) * inv.unsqueeze(0)
    cos, sin = ang.cos().float().unsqueeze(1), ang.sin().float().unsqueeze(1)
    x0, x1 = x[..., :half], x[..., half:]
    return torch.cat([x0 * cos - x1 * sin, x1 * cos + x0 * sin], dim=-1)


@torch.no_grad()
def forward_full(cfg: ModelConfig, w: ModelWeights, token_ids: torch.Tensor, capture_hidden: list | None = None):
    """Full-sequence forward of ONE sequence (unsharded weights). Returns fp32 logits [T, V]."""
    if cfg.is_parallel:
        return _forward_parallel(cfg, w, token_ids, capture_hidden)
    if cfg.is_shifted:
        return _forward_shifted(cfg, w, token_ids, capture_hidden)
    if cfg.is_prenorm:
        return _forward_prenorm(cfg, w, token_ids, capture_hidden)
    if cfg.is_layered:
        return _forward_layered(cfg, w, token_ids, capture_hidden)
    T = token_ids.shape[0]
    H, D, Hq, Hkv = cfg.hidden_size, cfg.head_dim, cfg.num_heads, cfg.num_kv_heads
    x = w.embed[token_ids.long()].float()
    pos = torch.arange(T, device=x.device)
    mask = torch.triu(torch.full((T, T), float("-inf"), device=x.device), diagonal=1)
    for lw in w.layers:
        h = _rms(x, lw.attn_norm, cfg.rms_norm_eps)
        qkv = h @ lw.wqkv.float().t()
        if getattr(lw, "bqkv", None) is not None:
            qkv = qkv + lw.bqkv.float()
        q = _rope(qkv[:, :Hq * D].view(T, Hq, D), pos, cfg.rope_theta, cfg.rope_scaling)
        k = _rope(qkv[:, Hq * D:(Hq + Hkv) * D].view(T, Hkv, D), pos, cfg.rope_theta, cfg.rope_scaling)
        v = qkv[:, (Hq + Hkv) * D:].view(T, Hkv, D)
        G = Hq // Hkv
        k = k.repeat_interleave(G, dim=1)
        v = v.repeat_interleave(G, dim=1)
        s = torch.einsum("qhd,khd->hqk", q, k) / math.sqrt(D) + mask
        a = torch.einsum("hqk,khd->qhd", torch.softmax(s, dim=-1), v).reshape(T, Hq * D)
        x = x + a @ lw.wo.float().t()
        h = _rms(x, lw.ffn_norm, cfg.rms_norm_eps)
        # a Decoder on the same weights may have re-laid the expert matrices tile by tile: read the logical view
        w13 = lw.w13.unpack() if hasattr(lw.w13, "unpack") else lw.w13
        w2 = lw.w2.unpack() if hasattr(lw.w2, "unpack") else lw.w2
        if cfg.is_moe:
            logits = h @ lw.router.float().t()
            probs = torch.softmax(logits, dim=-1)
            topv, topi = probs.topk(cfg.top_k, dim=-1)
            topv = topv / topv.sum(-1, keepdim=True)
            y = torch.zeros_like(x)
            I = w13.shape[1] // 2
            for e in range(cfg.num_experts):
                sel = (topi == e)
                rows = sel.any(-1).nonzero().squeeze(-1)
                if rows.numel() == 0:
                    continue
                he = h[rows]
                g = he @ w13[e, :I].float().t()
                u = he @ w13[e, I:].float().t()
                o = (torch.nn.functional.silu(g) * u) @ w2[e].float().t()
                y[rows] += o * (topv[rows] * sel[rows].float()).sum(-1, keepdim=True)
            x = x + y
        else:
            I = w13.shape[0] // 2
            g = h @ w13[:I].float().t()
            u = h @ w13[I:].float().t()
            x = x + (torch.nn.functional.silu(g) * u) @ w2.float().t()
        if capture_hidden is not None:
            capture_hidden.append(x.clone())
    h = _rms(x, w.final_norm, cfg.rms_norm_eps)
    return h @ w.lm_head.float().t()


def _forward_layered(cfg, w, token_ids, capture_hidden):
    """The same for designs that list their layers (post-norm blocks of latent attention), keys and values expanded per head."""
    from .layered import GLU_SLOPE, RoutedFFSpec
    T, eps = token_ids.shape[0], cfg.rms_norm_eps
    unit = lambda v: v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)      # noqa: E731
    x = w.embed[token_ids.long()].float()
    pos = torch.arange(T, device=x.device)
    mask = torch.triu(torch.full((T, T), float("-inf"), device=x.device), diagonal=1)

    def rotate(v, base):        # neighbouring pairs
        n = v.shape[-1]
        ang = pos.double()[:, None] * base ** (-torch.arange(0, n, 2, device=x.device).double() / n)
        c, s = ang.cos().float(), ang.sin().float()
        if v.dim() == 3:
            c, s = c[:, None], s[:, None]
        return torch.stack([v[..., 0::2] * c - v[..., 1::2] * s, v[..., 1::2] * c + v[..., 0::2] * s], dim=-1).flatten(-2)

    for sp, lw in zip(cfg.layers, w.layers):
        m, mw = sp.mixer, lw.mixer
        H, D, V, K = m.heads, m.dim, m.vdim, m.kv_rank
        taps = lw.conv.shape[0]
        h = x + sum(lw.conv[j] * torch.nn.functional.pad(x, (0, 0, taps - 1 - j, 0))[:T] for j in range(taps))
        z = h @ mw.w_in.float().t()
        q = z[:, :m.q_width] if not m.q_rank else (unit(z[:, :m.q_rank]) * mw.q_norm) @ mw.w_uq.float().t()
        q = q.view(T, H, D + m.rot_dim)
        c = unit(z[:, mw.off_kv:mw.off_kv + K]) * mw.kv_norm
        kr = rotate(z[:, mw.off_kv + K:mw.off_kv + K + m.rot_dim], m.rope_base)
        kv = c @ mw.w_ukv.float().t()
        k, v = kv[:, :H * D].view(T, H, D), kv[:, H * D:].view(T, H, V)
        s = (torch.einsum("qhd,khd->hqk", q[..., :D], k) + torch.einsum("qhr,kr->hqk", rotate(q[..., D:], m.rope_base), kr)) * m.scale
        o = torch.einsum("hqk,khv->qhv", torch.softmax(s + mask, dim=-1), v).reshape(T, H * V)
        if m.gated:
            o = o * torch.sigmoid(z[:, mw.off_gate:mw.off_gate + H * V])
        x = unit(cfg.post_alpha * x + o @ mw.wo.float().t()) * lw.norm1
        if isinstance(sp.mlp, RoutedFFSpec):
            f = sp.mlp
            sc = torch.softmax(x @ lw.router.float().t(), dim=-1)
            best = sc.view(T, f.groups, -1).amax(-1).topk(f.keep, dim=-1).indices
            ok = torch.zeros(T, f.groups, dtype=torch.bool, device=x.device).scatter_(1, best, True).repeat_interleave(f.experts // f.groups, dim=1)
            ids = sc.masked_fill(~ok, -1.0).topk(f.top, dim=-1).indices
            y = torch.zeros_like(x)
            for e in range(f.experts):
                rows = (ids == e).any(-1).nonzero().squeeze(-1)
                if rows.numel():
                    g, u = (x[rows] @ lw.w13[e].float().t()).chunk(2, dim=1)
                    g, u = g.clamp(max=f.limit), u.clamp(-f.limit, f.limit)
                    y[rows] += sc[rows, e:e + 1] * ((g * torch.sigmoid(GLU_SLOPE * g) * (u + 1)) @ lw.w2[e].float().t())
        elif sp.mlp is not None:
            z = x @ lw.w_up.float().t()
            y = (lw.act[0] * unit(z) + lw.act[1] * unit(z ** 2) + lw.act[2] * unit(z ** 3) + lw.act[3]) @ lw.w2.float().t()
        if sp.mlp is not None:
            x = unit(cfg.post_alpha * x + y) * lw.norm2
        if capture_hidden is not None:
            capture_hidden.append(x.clone())
    return (unit(x) * w.final_norm) @ w.lm_head.float().t()


def _forward_parallel(cfg, w, token_ids, capture_hidden):
    """The same for parallel layers: attention by a full mask, recurrences one token at a time, no state kept."""
    from .parallel_layers import LayerLayout, WindowAttnSpec
    T, C, eps = token_ids.shape[0], cfg.hidden_size, cfg.rms_norm_eps
    unit = lambda v: v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)      # noqa: E731
    norm = lambda v, n: torch.tanh(n.alpha * v) * n.w + n.b                       # noqa: E731
    act = torch.nn.functional
    x0 = x = w.embed[token_ids.long()].float()
    pos = torch.arange(T, device=x.device)
    back = pos[:, None] - pos[None, :]

    def attention(a, aw, z, at):
        q, k, v = (z[:, at[n]:at[n] + rows] for n, rows in a.sections())
        inv = a.rope_base ** (-torch.arange(0, a.rot_dims, 2, device=x.device).double() / max(a.rot_dims, 1)) / a.rope_factor
        ang = pos.double()[:, None] * inv
        c, s = ang.cos().float()[:, None], ang.sin().float()[:, None]
        n = a.rot_dims // 2
        turn = lambda t: torch.cat([t[..., :n] * c - t[..., n:2 * n] * s, t[..., n:2 * n] * c + t[..., :n] * s, t[..., 2 * n:]], dim=-1)   # noqa: E731
        q = turn((unit(q) * aw.q_norm).view(T, a.heads, a.dim))
        k = turn((unit(k) * aw.k_norm).view(T, a.kv_heads, a.dim)).repeat_interleave(a.heads // a.kv_heads, dim=1)
        v = v.view(T, a.kv_heads, a.vdim).repeat_interleave(a.heads // a.kv_heads, dim=1)
        seen = (back >= 0) & (back < a.window) if a.window else back >= 0
        s = (torch.einsum("qhd,khd->hqk", q, k) * a.scale).masked_fill(~seen, float("-inf"))
        return torch.einsum("hqk,khv->qhv", torch.softmax(s, dim=-1), v).reshape(T, -1)

    def recurrence(r, rw, z, at):
        H, G, D, V = r.heads, r.groups, r.dim, r.vdim
        if r.kind == "ssd":
            v0 = at["conv"]
            cols = (v0 + H * V + G * D, v0 + H * V, v0)
        else:
            cols = (at["q"], at["k"], at["v"])
        u = torch.cat([z[:, c0:c0 + n] for c0, n in zip(cols, (G * D, G * D, H * V))], dim=1)
        if r.conv_channels:
            u = sum(rw.conv[j] * act.pad(u, (0, 0, r.taps - 1 - j, 0))[:T] for j in range(r.taps)) + (rw.conv_b if rw.conv_b is not None else 0.0)
        u = act.silu(u)
        q, k, v = u[:, :G * D].view(T, G, D), u[:, G * D:2 * G * D].view(T, G, D), u[:, 2 * G * D:].view(T, H, V)
        if r.kind == "delta":
            q, k = (t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6) for t in (q, k))
            q = q * D ** -0.5
        q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
        if r.kind == "lightning":
            g, coef = rw.decay.expand(T, H), torch.ones(T, H, device=x.device)
        else:
            a0 = at["dt" if r.kind == "ssd" else "a"]
            step = act.softplus(z[:, a0:a0 + H] + rw.dt_bias)
            g = (rw.neg_decay * step).exp()
            coef = torch.sigmoid(z[:, at["b"]:at["b"] + H]) if r.kind == "delta" else step
        S, out = torch.zeros(H, D, V, device=x.device), []
        for t in range(T):
            S = g[t][:, None, None] * S
            d = v[t] - torch.einsum("hdv,hd->hv", S, k[t]) if r.kind == "delta" else v[t]
            S = S + k[t][:, :, None] * (coef[t][:, None] * d)[:, None]
            out.append(torch.einsum("hdv,hd->hv", S, q[t]) + (rw.skip[:, None] * v[t] if rw.skip is not None else 0.0))
        o = torch.stack(out)
        if r.kind == "ssd":
            o = o.reshape(T, -1) * act.silu(z[:, at["z"]:at["z"] + H * V])
            return unit(o.view(T, r.norm_groups, -1)).reshape(T, -1) * rw.norm
        gate = z[:, at["g"]:at["g"] + H * V]
        if r.kind == "delta":
            return (unit(o) * rw.norm).reshape(T, -1) * act.silu(gate)
        return unit(o.reshape(T, -1)) * rw.norm * torch.sigmoid(gate)

    for sp, lw in zip(cfg.layers, w.layers):
        lay = LayerLayout(sp)
        if sp.loop_pass is not None:
            x = torch.cat([x, x0], dim=1) @ w.loop.w_in.float().t() + w.loop.step[sp.loop_pass]
        z = torch.zeros(T, lay.width, device=x.device)
        z[:, lay.in_first:] = norm(x, lw.norm) @ lw.w_in.float().t()
        z[:, lay.ff:lay.ff + lay.ff_cols] = z[:, lay.ff:lay.ff + lay.ff_cols].clamp(min=0).square()
        for sec in lay.parts:
            f, mw = (attention, lw.attn) if isinstance(sec.spec, WindowAttnSpec) else (recurrence, lw.rec)
            z[:, sec.out:sec.out + sec.spec.out_width] = sec.scale * f(sec.spec, mw, z, sec.col)
        x = x + z[:, :lay.out_cols] @ lw.w_out.float().t()
        if capture_hidden is not None:
            capture_hidden.append(x.clone())
    return norm(x, w.final_norm) @ w.lm_head.float().t()


def _forward_prenorm(cfg, w, token_ids, capture_hidden):
    """The same for pre-norm layers: attention by a full mask, the scan one token at a time, every expert over all tokens that chose it."""
    from .parallel_layers import LayerLayout, SelectiveSpec, up8
    T, eps = token_ids.shape[0], cfg.rms_norm_eps
    unit = lambda v: v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)      # noqa: E731
    act = torch.nn.functional
    x = w.embed[token_ids.long()].float()
    pos = torch.arange(T, device=x.device)

    def attention(a, aw, z, at):
        H, G, M, D = a.heads, a.kv_heads, a.maps, a.dim
        q, k, v = (z[:, at[n]:at[n] + rows] for n, rows in a.sections()[:3])
        n = a.rot_dims
        ang = pos.double()[:, None] * (a.rope_base ** (-torch.arange(0, n, 2, device=x.device).double() / max(n, 1)) / a.rope_factor)
        c, s = ang.cos().float()[:, None], ang.sin().float()[:, None]

        def turn(t):
            if a.interleaved:
                u, y = t[..., 0:n:2], t[..., 1:n:2]
                r = torch.stack([u * c - y * s, y * c + u * s], dim=-1).flatten(-2)
            else:
                u, y = t[..., :n // 2], t[..., n // 2:n]
                r = torch.cat([u * c - y * s, y * c + u * s], dim=-1)
            t = torch.cat([r, t[..., n:]], dim=-1)
            return unit(t) if a.unit else t
        q = turn(q.reshape(T, H * M, D)).view(T, H, M, D)
        k = turn(k.reshape(T, G * M, D)).view(T, G, M, D).repeat_interleave(H // G, dim=1)
        v = v.reshape(T, G, a.vdim).repeat_interleave(H // G, dim=1)
        back = pos[:, None] - pos[None, :]
        seen = back >= 0
        if a.chunk:
            seen = seen & (pos[:, None] // a.chunk == pos[None, :] // a.chunk)
        if a.window:
            seen = seen & (back < a.window)
        sc = (torch.einsum("qhmd,khmd->hmqk", q, k) * a.scale).masked_fill(~seen, float("-inf"))
        if a.sink:
            sc = torch.cat([sc, torch.zeros_like(sc[..., :1])], dim=-1)
        o = torch.einsum("hmqk,khv->mqhv", torch.softmax(sc, dim=-1)[..., :T], v)
        o = o[0] if M == 1 else unit(o[0] - aw.lam * o[1]) * (1.0 - a.diff)
        o = o.reshape(T, -1)
        return o * torch.sigmoid(z[:, at["g"]:at["g"] + a.out_width]) if a.gated else o

    def scan(m, sw, z, at):
        N = m.state
        u = z[:, at["x"]:at["x"] + m.inner]
        u = act.silu(sum(sw.conv[j] * act.pad(u, (0, 0, m.taps - 1 - j, 0))[:T] for j in range(m.taps)) + sw.conv_b)
        p = u @ sw.w_x.float().t()
        b0, c0 = up8(m.dt_rank), up8(m.dt_rank) + up8(N)
        dt = act.softplus(p[:, :sw.w_dt.shape[1]] @ sw.w_dt.float().t() + sw.dt_bias)
        S, ys = torch.zeros(N, m.inner, device=x.device), []
        for t in range(T):
            S = torch.exp(dt[t] * sw.neg_a) * S + (dt[t] * u[t]) * p[t, b0:b0 + N, None]
            ys.append(p[t, c0:c0 + N] @ S + sw.skip * u[t])
        return torch.stack(ys) * act.silu(z[:, at["z"]:at["z"] + m.inner])

    def glu(h, w13, w2):
        g, u = (h @ w13.float().t()).chunk(2, dim=1)
        return (act.silu(g) * u) @ w2.float().t()

    for sp, lw in zip(cfg.layers, w.layers):
        lay, f = LayerLayout(sp, ff=False), sp.mlp
        if sp.loop_pass is not None:
            x = x + w.loop.step[sp.loop_pass]
        z = torch.zeros(T, lay.width, device=x.device)
        z[:, lay.in_first:] = (unit(x) * lw.norm1) @ lw.w_in.float().t()
        sec = lay.parts[0]
        o = scan(sp.mixer, lw.scan, z, sec.col) if isinstance(sp.mixer, SelectiveSpec) else attention(sp.mixer, lw.attn, z, sec.col)
        x = x + act.pad(o, (0, lay.out_cols - o.shape[1])) @ lw.w_out.float().t()
        if f is not None:
            h = unit(x) * lw.norm2
            s = h @ lw.router.float().t()
            s = torch.sigmoid(s) if f.score == "sigmoid" else torch.softmax(s, dim=-1)
            grouped = s.view(T, f.groups, -1)
            best = grouped.topk(min(f.group_best, grouped.shape[-1]), dim=-1).values.sum(-1).topk(f.keep, dim=-1).indices
            ok = torch.zeros(T, f.groups, dtype=torch.bool, device=x.device).scatter_(1, best, True).repeat_interleave(f.experts // f.groups, dim=1)
            top, ids = s.masked_fill(~ok, -1.0).topk(f.top, dim=-1)
            top = (top / (top.sum(-1, keepdim=True) + 1e-20) if f.renorm else top) * f.scale
            y = glu(h, lw.shared13, lw.shared2) if f.shared_ff else torch.zeros_like(x)
            for e in range(f.experts):
                rows, slot = (ids == e).nonzero(as_tuple=True)
                if rows.numel():
                    y[rows] += top[rows, slot, None] * glu(h[rows], lw.w13[e], lw.w2[e])
            x = x + y
        if capture_hidden is not None:
            capture_hidden.append(x.clone())
    return (unit(x) * w.final_norm) @ w.lm_head.float().t()


def _forward_shifted(cfg, w, token_ids, capture_hidden):
    """The same for shifted pre-norm layers: attention by a full mask, keys and values of latent attention expanded, the recurrence one token
    at a time."""
    from .layered import GLU_SLOPE, LatentMixerSpec
    from .parallel_layers import LayerLayout, RecurrentSpec
    act, eps, T = torch.nn.functional, cfg.rms_norm_eps, token_ids.shape[0]
    unit = lambda v: v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)      # noqa: E731
    norm = lambda v, g: unit(v.view(T, cfg.norm_groups, -1)).reshape(T, -1) * g  # noqa: E731
    xs = [w.embed[token_ids.long()].float()]
    pos = torch.arange(T, device=xs[0].device)
    back = pos[:, None] - pos[None, :]
    v_first = None

    def softmax_values(sc, seen, sinks, v):
        sc = torch.cat([sc.masked_fill(~seen, float("-inf")), sinks[:, None, None].expand(-1, T, 1)], dim=-1)
        return torch.einsum("hqk,khv->qhv", torch.softmax(sc, dim=-1)[..., :T], v).reshape(T, -1)

    def latent(m, lw, z, at):
        mw = lw.latent
        ang = pos.double()[:, None] * m.rope_base ** (-torch.arange(0, m.rot_dim, 2, device=pos.device).double() / m.rot_dim)
        turn = lambda t: torch.view_as_real(torch.complex(t[..., 0::2], t[..., 1::2])                 # noqa: E731
                                            * torch.polar(torch.ones_like(ang), ang).to(torch.complex64)[:, None]).flatten(-2)
        q = z[:, at["q"]:at["q"] + m.q_width].reshape(T, m.heads, -1)
        ckr = z[:, at["dkv"]:at["dkv"] + m.cache_width]
        kr = turn(ckr[:, None, m.kv_rank:])[:, 0]
        kv = (unit(ckr[:, :m.kv_rank]) * mw.kv_norm) @ mw.w_ukv.float().t()
        k, v = kv[:, :m.heads * m.dim].view(T, m.heads, -1), kv[:, m.heads * m.dim:].view(T, m.heads, -1)
        sc = (torch.einsum("qhd,khd->hqk", q[..., :m.dim], k) + torch.einsum("qhd,kd->hqk", turn(q[..., m.dim:]), kr)) * m.scale
        return softmax_values(sc, back >= 0, mw.sinks, v)

    def attention(a, lw, z, at):
        nonlocal v_first
        aw = lw.attn
        q, k, v = (z[:, at[n]:at[n] + rows] + b for (n, rows), b in zip(a.sections(), (aw.q_bias, aw.k_bias, aw.v_bias)))
        q = unit(q.reshape(T, a.heads, -1)) * aw.q_norm
        k = (unit(k.reshape(T, a.kv_heads, -1)) * aw.k_norm).repeat_interleave(a.heads // a.kv_heads, dim=1)
        if a.v_mix and v_first is None:
            v_first = v
        elif a.v_mix:
            v = torch.lerp(v, v_first, aw.vmix)
        v = v.reshape(T, a.kv_heads, -1).repeat_interleave(a.heads // a.kv_heads, dim=1)
        seen = back >= 0
        if a.window:
            seen = seen & ((back < a.window) | (pos[None, :] < a.keep_first))
        sc = torch.einsum("qhd,khd->hqk", q, k) * a.scale
        return softmax_values(a.softcap * torch.tanh(sc / a.softcap) if a.softcap else sc, seen, aw.sinks, v)

    def recurrence(r, lw, z, at):
        rw, H, G, D, V = lw.rec, r.heads, r.groups, r.dim, r.vdim
        u = torch.cat([z[:, at[n]:at[n] + rows] for n, rows in r.sections()[:3]], dim=1)
        u = act.silu(sum(rw.conv[j] * act.pad(u, (0, 0, r.taps - 1 - j, 0))[:T] for j in range(r.taps)))
        q, k, v = u[:, :G * D].view(T, G, D), u[:, G * D:2 * G * D].view(T, G, D), u[:, 2 * G * D:].view(T, H, V)
        q, k = ((t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)).repeat_interleave(H // G, dim=1) for t in (q, k))
        behind = lambda n, wt: z[:, at[n]:at[n] + wt.shape[1]] @ wt.float().t()       # noqa: E731
        g = (rw.neg_decay[:, None] * act.softplus(behind("a1", rw.w_decay) + rw.dt_bias).view(T, H, D)).exp()
        beta = torch.sigmoid(z[:, at["b"]:at["b"] + H])
        S, out = torch.zeros(H, D, V, device=z.device), []
        for t in range(T):
            S = g[t][:, :, None] * S
            S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t])))[:, None]
            out.append(torch.einsum("hdv,hd->hv", S, q[t]) * D ** -0.5)
        return (unit(torch.stack(out)) * rw.norm).reshape(T, -1) * torch.sigmoid(behind("g1", rw.w_gate))

    x = xs[0]
    for sp, lw in zip(cfg.layers, w.layers):
        lay = LayerLayout(sp, ff=False)
        h = norm(x, lw.norm1)
        h = torch.lerp(h, act.pad(h, (0, 0, 1, 0))[:T], lw.shift)
        z = torch.zeros(T, lay.width, device=x.device)
        z[:, lay.in_first:] = h @ lw.w_in.float().t()
        f = latent if isinstance(sp.mixer, LatentMixerSpec) else recurrence if isinstance(sp.mixer, RecurrentSpec) else attention
        o = f(sp.mixer, lw, z, lay.parts[0].col)
        x = x + act.pad(o, (0, lay.out_cols - o.shape[1])) @ lw.w_out.float().t()
        if sp.mlp is not None:
            g, u = (norm(x, lw.norm2) @ lw.dense13.float().t()).chunk(2, dim=1)
            g, u = g.clamp(max=sp.mlp.limit), u.clamp(-sp.mlp.limit, sp.mlp.limit)
            x = x + (g * torch.sigmoid(GLU_SLOPE * g) * (u + 1.0)) @ lw.dense2.float().t()
        xs.append(x)
        x = torch.einsum("j,jtc->tc", lw.depth, torch.stack(xs))
        if capture_hidden is not None:
            capture_hidden.append(x.clone())
    return norm(x, w.final_norm) @ w.lm_head.float().t()
