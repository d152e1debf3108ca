"""Sizes and kernel tables of pre-norm designs for utils/design_bench.py: differential and chunked attention, the selective scan and the
routed feed-forward, beside a Mixtral-shaped block of the same width, query heads and experts. The scan's like kernel is the state-space
recurrence of the framework's other recurrent design at the same width."""
from __future__ import annotations

import torch

from .. import ops
from ..models import config as mc
from ..models.layered import RoutedFFSpec, unroll_loop
from ..models.parallel_layers import LayerLayout, RecurrentSpec, SelectiveSpec, SelectiveWeights, WindowAttnSpec, up8
from ..ops import parallel as par, prenorm as pre, recurrent as rec, reference as ref, selective as sel
from .design_bench_parallel import _columns, _i32, _rec_weights, _Step
from .microbench import _bf

SIZES = ("scan-2k", "scan-4k")
CHUNK = 1024


def size_config(name: str):
    """(design's configuration, closest uniform configuration): scan, differential, scan, chunked."""
    C, H, ff, E, top, groups, keep, shared = {"scan-2k": (2048, 16, 1408, 64, 6, 8, 3, 2816), "scan-4k": (4096, 32, 7168, 16, 2, 4, 2, 7168)}[name]
    diff = WindowAttnSpec(H, H // 4, 64, 128, 64 ** -0.5, 64, 5e5, kind="attention", row_norm=False, interleaved=True, diff=0.8, gated=True)
    chunk = WindowAttnSpec(H, H // 4, 128, 128, 128 ** -0.5, 128, 1e4, kind="attention_2", chunk=CHUNK, row_norm=False, interleaved=True, unit=True, sink=True)
    scan = SelectiveSpec(2 * C, 16, C // 16, 4)
    f = RoutedFFSpec(ff, None, E, top, groups, keep, score="sigmoid", group_best=2, renorm=True, scale=2.0, shared_ff=shared)
    new = mc.ModelConfig.layered("Barorax", unroll_loop([(m, f) for m in (scan, diff, scan, chunk)], None), width=C, vocab=32000, max_pos=8192,
                                 name=f"barorax-{name}")
    near = mc.ModelConfig(architecture="MixtralForCausalLM", hidden_size=C, intermediate_size=ff, num_layers=new.num_layers, num_heads=H,
                          num_kv_heads=H // 4, head_dim=128, vocab_size=32000, num_experts=E, top_k=top, max_position_embeddings=8192, name=f"mixtral-{name}")
    return new, near


def describe(new) -> dict:
    f = new.layers[0].mlp
    return {"width": new.hidden_size, "layers": [l.mixer.kind for l in new.layers], "chunk": CHUNK, "experts": f.experts, "top": f.top, "ff": f.ff, "shared": f.shared_ff}


def _mixers(new):
    return new.layers[0].mixer, new.layers[1].mixer, new.layers[3].mixer


def _like_ssd(new):
    return RecurrentSpec("ssd", new.hidden_size // 64, 1, 128, 64, 4, 8)


def _scan_weights(m):
    f = lambda *s: torch.randn(*s, device="cuda")          # noqa: E731
    return SelectiveWeights(None, None, conv=f(m.taps, m.inner) * 0.5, conv_b=f(m.inner) * 0.1, dt_bias=f(m.inner) - 3, neg_a=-f(m.state, m.inner).exp(), skip=f(m.inner))


def _scan_args(m, T):
    row = _bf(T, 2 * m.inner, std=1.0)
    cols = sum(up8(r) for _, r in m.x_sections())
    return row[:, :m.inner], row[:, m.inner:], _bf(T, m.inner, std=1.0), _bf(T, cols, std=1.0), torch.randn(T, m.inner, device="cuda"), _bf(T, m.inner)


def _product(T, F, K, f32=False, back=False):
    def make():
        x, w = _bf(T, K, std=1.0), _bf(F, K)
        if back:
            r = torch.zeros(T, F, device="cuda")
            return lambda: ops.linear(x, w, out=r, residual=r, out_f32=True), (w.numel() + x.numel()) * 2 + T * F * 8, 2 * T * F * K
        return lambda: ops.linear(x, w, out_f32=f32), (w.numel() + x.numel()) * 2 + T * F * (4 if f32 else 2), 2 * T * F * K
    return make


def _pair(T, F, K):
    def make():
        x, w = _bf(T, K, std=1.0), _bf(2 * F, K)
        return lambda: ops.swiglu_linear(x, w), (w.numel() + x.numel() + T * F) * 2, 4 * T * F * K
    return make


def _products(new, near, T):
    """The products of every kind of layer. Small ones (the scan's inputs) beside the like model's output projection."""
    C, Hq, Hkv = new.hidden_size, near.num_heads, near.num_kv_heads
    out = []
    for name, i in (("scan", 0), ("differential", 1), ("chunked", 3)):
        lay = LayerLayout(new.layers[i], ff=False)
        out += [(f"{name}: product in", _product(T, lay.in_rows, C), _product(T, (Hq + 2 * Hkv) * 128, C)),
                (f"{name}: product out + residual", _product(T, C, lay.out_cols, back=True), _product(T, C, Hq * 128))]
    m, f = new.layers[0].mixer, new.layers[0].mlp
    out += [("scan: product of B, C, step bottleneck", _product(T, sum(up8(r) for _, r in m.x_sections()), m.inner), _product(T, C, Hq * 128)),
            ("scan: product of step sizes", _product(T, m.inner, up8(m.dt_rank), f32=True), _product(T, C, Hq * 128)),
            ("shared expert: gate / up", _pair(T, f.shared_ff, C), _product(T, (Hq + 2 * Hkv) * 128, C)),
            ("shared expert: down + residual", _product(T, C, f.shared_ff, back=True), _product(T, C, Hq * 128))]

    def experts(down):
        def make():
            per = max(1, T * f.top // f.experts)
            cnt = torch.full((f.experts,), per, dtype=torch.int32, device="cuda")
            off = (torch.arange(f.experts + 1, device="cuda") * per).to(torch.int32)
            Fo, K = (C, f.ff) if down else (2 * f.ff, C)
            xs, w = _bf(f.experts * per, K, std=1.0), _bf(f.experts, Fo, K)
            cols = Fo if down else f.ff
            return (lambda: ops.grouped_linear(xs, w, cnt, off, swiglu=not down), (w.numel() + xs.numel() + f.experts * per * cols) * 2,
                    2 * f.experts * per * Fo * K)
        return make
    return out + [("experts gate / up", experts(False), experts(False)), ("experts down", experts(True), experts(True))]


def _norm_kernels(new, T, decode):
    C, f = new.hidden_size, new.layers[0].mlp
    k = f.top

    def summed(n):
        def make():
            x, y, g = torch.randn(T, C, device="cuda"), _bf(T * k, C, std=1.0), torch.ones(C, device="cuda")
            idx, w = torch.randperm(T * k, device="cuda").to(torch.int32).view(T, k), torch.rand(T, k, device="cuda")
            args = (y, idx, w) if n else (None, None, None)
            return lambda: pre.add_norm(x, *args, gain=g, eps=1e-5), T * C * (6 + (4 + 2 * k if n else 0)), 8 * T * C
        return make

    def summed_like(n):
        def make():
            r, y, g = _bf(T, C, std=1.0), _bf(1, T * max(1, n), C, std=1.0), _bf(C)
            idx = torch.randperm(T * n, device="cuda").to(torch.int32).view(T, n) if n else None
            w = torch.rand(T, n, device="cuda") if n else None
            return lambda: ops.reduce_residual_rmsnorm(r, y, g, 1e-5, idx, w), T * C * (6 + 2 * max(1, n)), 8 * T * C
        return make

    def route():
        wg = _bf(f.experts, C)
        if decode:
            x, g = torch.randn(T, C, device="cuda"), torch.ones(C, device="cuda")
            return lambda: pre.norm_route(x, g, 1e-5, wg, f), T * C * (6 + 2 * k) + 2 * f.experts * C, 2 * T * f.experts * C
        x = _bf(T, C, std=1.0)
        return lambda: pre.route(x, wg, f), T * C * 2 * (2 + 2 * k), 2 * T * f.experts * C

    def route_like():
        wg = _bf(f.experts, C)
        if decode:
            r, y, g = _bf(T, C, std=1.0), _bf(1, T, C, std=1.0), _bf(C)
            return lambda: ops.reduce_norm_route(r, y, g, 1e-5, wg, k), T * C * (8 + 2 * k) + 2 * f.experts * C, 2 * T * f.experts * C
        x = _bf(T, C, std=1.0)

        def fn():
            r = ops.route(x, wg, k)
            return ops.gather_rows(x, r[5])
        return fn, T * C * 2 * (2 + 2 * k), 2 * T * f.experts * C
    out = [("expert sum + norm", summed(True), summed_like(k)), ("norm + router + scatter" if decode else "router + gather", route, route_like)]
    return out if decode else out + [("norm", summed(False), summed_like(0))]


def decode_kernels(new, near, B=64, ctx=640):
    """(name, new op, like op): each op is a function returning (launch, bytes, flops)."""
    m, diff, chunk = _mixers(new)
    Hq, Hkv = near.num_heads, near.num_kv_heads
    pos1 = lambda n: torch.full((B,), n - 1, dtype=torch.int32, device="cuda")      # noqa: E731

    def paged(n, ps):
        nb = (n + ps - 1) // ps
        return torch.arange(B * nb, dtype=torch.int32, device="cuda").view(B, nb), B * nb

    def attn(a, n):
        def make():
            bt, pages = paged(n, 64)
            cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda").normal_()
            q, out, gate = _bf(B, a.heads * 128, std=1.0), _bf(B, a.heads * 128), _bf(B, a.heads * 128, std=1.0)
            inp = _Step(False, positions=pos1(n), seq_of_token=None, block_table=bt, seq_lens=pos1(n) + 1)
            mix = par.HeadMix(torch.tensor([0.5], device="cuda"), gate if a.gated else None, 1e-5)
            keys = n - (n - 1) // a.chunk * a.chunk if a.chunk else n
            return lambda: par.window_attn(q, a, inp, cache, 64, out, 1.0, mix), B * keys * 2 * a.kv_heads * 256, 4 * B * a.maps * a.heads * keys * 128
        return make

    def attn_like(n):
        def make():
            bt, pages = paged(n, 16)
            kv, q, lens = _bf(pages, 2, Hkv, 16, 128, std=1.0), _bf(B, Hq * 128, std=1.0), pos1(n) + 1
            return lambda: ops.attn_decode(q, kv, bt, lens, Hq, Hkv, 128, ctx_hint=n), B * n * 2 * Hkv * 256, 4 * B * Hq * n * 128
        return make

    def append(a):
        def make():
            bt, pages = paged(ctx, 64)
            cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda")
            row, t = _bf(B, (a.heads + 2 * a.kv_heads) * 128, std=1.0), ref.rope_cos_sin_table(ctx + 8, a.rot_dims, 1e4, "cuda")
            q, k, v = row.split([a.heads * 128, a.kv_heads * 128, a.kv_heads * 128], dim=1)
            pos = pos1(ctx)
            return (lambda: par.head_append(q, k, v, a, t, pos, None, bt, cache, 64, 1e-5), B * (2 * a.heads + 4 * a.kv_heads) * 256, B * a.heads * 1024)
        return make

    def append_like():
        bt, pages = paged(ctx, 16)
        qkv, kv, t = _bf(B, (Hq + 2 * Hkv) * 128, std=1.0), _bf(pages, 2, Hkv, 16, 128), ref.rope_cos_sin_table(ctx + 8, 128, 1e4, "cuda")
        pos = pos1(ctx)
        return lambda: ops.rope_kv_append(qkv, pos, None, bt, t, kv, Hq, Hkv, 128), B * (2 * Hq + 4 * Hkv) * 256, B * Hq * 512

    def conv():
        w, st, inp = _scan_weights(m), sel.ScanState.make(m, B, torch.bfloat16, "cuda"), _Step(False, positions=pos1(ctx), seq_lens=pos1(ctx) + 1)
        x, slots = _scan_args(m, B)[0], torch.arange(B, dtype=torch.int32, device="cuda")
        return lambda: sel.short_conv(x, m, w, st, inp, slots, True), B * m.inner * 2 * (2 + m.taps) + m.inner * 4 * (m.taps + 1), 10 * B * m.inner

    def step():
        w, st, inp = _scan_weights(m), sel.ScanState.make(m, B, torch.bfloat16, "cuda"), _Step(False, positions=pos1(ctx), seq_lens=pos1(ctx) + 1)
        x, z, xc, proj, dt, out = _scan_args(m, B)
        slots = torch.arange(B, dtype=torch.int32, device="cuda")
        by = B * (8 * m.state_elems + m.inner * 10) + 4 * m.state_elems
        return lambda: sel.scan(xc, proj, dt, x, z, out, m, w, st, inp, slots, True), by, 6 * B * m.state_elems

    def step_like():
        r = _like_ssd(new)
        col, width = _columns(r)
        row, w, st = _bf(B, width, std=1.0), _rec_weights(r), rec.RecState.make(r, B, torch.bfloat16, "cuda")
        cols, pos, slots = rec.RecColumns.of(r, col), pos1(ctx), torch.arange(B, dtype=torch.int32, device="cuda")
        by = B * (8 * r.state_elems + 2 * (r.conv_channels * (1 + r.conv_rows) + r.out_width * 2))
        return lambda: rec.rec_step(row, cols, r, w, st, pos, slots), by, 6 * B * r.state_elems

    def norm_like():
        C = new.hidden_size
        r, y, g = _bf(B, C, std=1.0), _bf(1, B, C, std=1.0), _bf(C)
        return lambda: ops.reduce_residual_rmsnorm(r, y, g, 1e-5), B * C * 8, 6 * B * C
    return [("differential attention, difference, norm, gate", attn(diff, ctx), attn_like(ctx)),
            ("differential attention, 4096 tokens", attn(diff, 4096), attn_like(4096)),
            ("chunked attention, one chunk", attn(chunk, ctx), attn_like(ctx)),
            ("chunked attention, 4096 tokens, chunk 1024", attn(chunk, 4096), attn_like(1024)),
            ("differential: rotation + append", append(diff), append_like), ("chunked: rotation, unit heads + append", append(chunk), append_like),
            ("scan: convolution", conv, norm_like), ("scan: step", step, step_like)] + _norm_kernels(new, B, True) + _products(new, near, B)


def prefill_kernels(new, near, S=4, L=2048):
    T = S * L
    m, diff, chunk = _mixers(new)
    Hq, Hkv = near.num_heads, near.num_kv_heads
    start, qlen = _i32([s * L for s in range(S)]), _i32([L] * S)
    pos, sot = _i32(list(range(L)) * S), _i32([s for s in range(S) for _ in range(L)])
    slots = torch.arange(S, dtype=torch.int32, device="cuda")
    t_like = ref.rope_cos_sin_table(L, 128, 1e4, "cuda")

    def paged(ps):
        nb = (L + ps - 1) // ps
        return torch.arange(S * nb, dtype=torch.int32, device="cuda").view(S, nb), S * nb

    def step():
        return _Step(True, positions=pos, seq_of_token=sot, block_table=paged(64)[0], seq_lens=qlen, q_start=start, q_len=qlen, max_q_len=L)

    def attn(a):
        def make():
            cache = par.window_cache(paged(64)[1], 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda").normal_()
            q, out, gate, inp = _bf(T, a.heads * 128, std=1.0), _bf(T, a.heads * 128), _bf(T, a.heads * 128, std=1.0), step()
            mix = par.HeadMix(torch.tensor([0.5], device="cuda"), gate if a.gated else None, 1e-5)
            w = a.chunk or L
            pairs = S * (L // w) * (w * (w + 1) // 2)
            by = ((3 if a.gated else 2) * q.numel() + T * 2 * a.kv_heads * 128) * 2
            return lambda: par.window_attn(q, a, inp, cache, 64, out, 1.0, mix), by, 2 * a.heads * a.maps * (a.dim + a.vdim) * pairs
        return make

    def attn_like(w):
        def make():
            bt, pages = paged(16)
            kv, q = _bf(pages, 2, Hkv, 16, 128, std=1.0), _bf(T, Hq * 128, std=1.0)
            if w < L:      # prompts of the chunk's length: the same number of (query, key) pairs
                n = T // w
                st, ln = _i32([s * w for s in range(n)]), _i32([w] * n)
                bw = torch.arange(n * (w // 16), dtype=torch.int32, device="cuda").view(n, w // 16)
                return (lambda: ops.attn_prefill(q, kv, bw, st, ln, ln, w, Hq, Hkv, 128), (2 * q.numel() + T * 2 * Hkv * 128) * 2,
                        4 * Hq * 128 * n * w * (w + 1) // 2)
            return (lambda: ops.attn_prefill(q, kv, bt, start, qlen, qlen, L, Hq, Hkv, 128), (2 * q.numel() + T * 2 * Hkv * 128) * 2,
                    4 * Hq * 128 * S * L * (L + 1) // 2)
        return make

    def append(a):
        def make():
            bt, pages = paged(64)
            cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda")
            row, t = _bf(T, (a.heads + 2 * a.kv_heads) * 128, std=1.0), ref.rope_cos_sin_table(L, a.rot_dims, 1e4, "cuda")
            q, k, v = row.split([a.heads * 128, a.kv_heads * 128, a.kv_heads * 128], dim=1)
            return (lambda: par.head_append(q, k, v, a, t, pos, sot, bt, cache, 64, 1e-5), T * (2 * a.heads + 4 * a.kv_heads) * 256, T * a.heads * 1024)
        return make

    def append_like():
        bt, pages = paged(16)
        qkv, kv = _bf(T, (Hq + 2 * Hkv) * 128, std=1.0), _bf(pages, 2, Hkv, 16, 128)
        return lambda: ops.rope_kv_append(qkv, pos, sot, bt, t_like, kv, Hq, Hkv, 128), T * (2 * Hq + 4 * Hkv) * 256, T * Hq * 512

    def conv():
        w, st, inp, x = _scan_weights(m), sel.ScanState.make(m, S, torch.bfloat16, "cuda"), step(), _scan_args(m, T)[0]
        return lambda: sel.short_conv(x, m, w, st, inp, slots, False), T * m.inner * 4, 10 * T * m.inner

    def scan(L2):
        def make():
            w, st = _scan_weights(m), sel.ScanState.make(m, T // L2, torch.bfloat16, "cuda")
            n = T // L2
            inp = _Step(True, positions=_i32(list(range(L2)) * n), seq_of_token=_i32([s for s in range(n) for _ in range(L2)]), seq_lens=_i32([L2] * n),
                        q_start=_i32([s * L2 for s in range(n)]), q_len=_i32([L2] * n), max_q_len=L2)
            x, z, xc, proj, dt, out = _scan_args(m, T)
            sl = torch.arange(n, dtype=torch.int32, device="cuda")
            by = T * m.inner * 10 + T * proj.shape[1] * 2 + 8 * n * m.state_elems
            return lambda: sel.scan(xc, proj, dt, x, z, out, m, w, st, inp, sl, False), by, 6 * T * m.state_elems
        return make

    def ssd(only):
        def make():
            r = _like_ssd(new)
            col, width = _columns(r)
            row, w, st = _bf(T, width, std=1.0), _rec_weights(r), rec.RecState.make(r, S, torch.bfloat16, "cuda")
            run = rec.ChunkRun(row, rec.RecColumns.of(r, col), r, w, st, pos, slots, sot, start, qlen, L)
            run.prep()
            qkv, out = 2 * r.groups * r.dim + r.out_width, r.out_width
            fl = T * r.heads * (4 * r.dim * r.vdim + 64 * (r.dim + r.vdim))
            by = T * (qkv + out) * 2 + T * r.heads * 8 + 8 * S * r.state_elems
            return (run.prep, T * qkv * 4, 16 * T * qkv) if only == "prep" else (run.walk, by, fl)
        return make
    return [("differential attention, difference, norm, gate", attn(diff), attn_like(L)), ("chunked attention", attn(chunk), attn_like(CHUNK)),
            ("differential: rotation + append", append(diff), append_like), ("chunked: rotation, unit heads + append", append(chunk), append_like),
            ("scan: convolution", conv, ssd("prep")), ("scan: recurrence", scan(L), ssd("walk")),
            ("scan: recurrence, one prompt of 8192", scan(T), ssd("walk"))] + _norm_kernels(new, T, False) + _products(new, near, T)
