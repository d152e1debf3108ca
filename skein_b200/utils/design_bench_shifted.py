"""Sizes and kernel tables of shifted pre-norm designs for utils/design_bench.py, beside a Llama-shaped model of the same width, heads and
feed-forward. Kernels that such a model does not have stand beside those of the framework's other designs at the same size: the delta rule
with a decay per head, latent attention without a sink, the norms and products of the uniform block."""
from __future__ import annotations

import torch

from .. import ops
from ..models import config as mc
from ..models.layered import GLU_SLOPE, DenseFFSpec, LatentMixerSpec, unroll_loop
from ..models.parallel_layers import LayerLayout, RecurrentSpec, RecurrentWeights, WindowAttnSpec, WindowAttnWeights
from ..ops import latent as lat, parallel as par, prenorm as pre, recurrent as rec, reference as ref
from .design_bench_parallel import _columns, _i32, _rec_weights, _Step
from .design_bench_prenorm import _product
from .microbench import _bf

SIZES = ("shift-2k", "shift-4k")
WINDOW, KEEP = 1024, 64


def size_config(name: str):
    """(design's configuration, closest uniform configuration): delta rule, window, delta rule, latent attention."""
    C, H, ff = {"shift-2k": (2048, 16, 8192), "shift-4k": (4096, 32, 14336)}[name]
    r = RecurrentSpec("channel_delta", H, H, 128, 128, 4, decay_rank=128, gate_rank=128)
    a = WindowAttnSpec(H, H // 4, 128, 128, 128 ** -0.5, 0, 1e4, window=WINDOW, kind="attention", row_norm=False, bias=True, head_norm=True, softcap=50.0,
                       keep_first=KEEP, head_sink=True, v_mix=True)
    m = LatentMixerSpec("latent_attention", H, 128, 64, 128, 512, 5e5, 192 ** -0.5, sink=True)
    new = mc.ModelConfig.layered("Derusun", unroll_loop([(x, DenseFFSpec(ff, 7.0)) for x in (r, a, r, m)], None), width=C, vocab=32000, max_pos=8192,
                                 name=f"derusun-{name}", groups=2)
    near = mc.ModelConfig(architecture="LlamaForCausalLM", hidden_size=C, intermediate_size=ff, num_layers=new.num_layers, num_heads=H,
                          num_kv_heads=H // 4, head_dim=128, vocab_size=32000, num_experts=0, top_k=0, max_position_embeddings=8192, name=f"llama-{name}")
    return new, near


def describe(new) -> dict:
    return {"width": new.hidden_size, "layers": [l.mixer.kind for l in new.layers], "window": WINDOW, "keep_first": KEEP, "norm_groups": new.norm_groups}


def _mixers(new):
    return new.layers[0].mixer, new.layers[1].mixer, new.layers[3].mixer


def _like_delta(r):
    return RecurrentSpec("delta", r.heads, r.groups, r.dim, r.vdim, r.taps)


def _channel_weights(r):
    f = lambda *s: torch.randn(*s, device="cuda")          # noqa: E731
    return RecurrentWeights(norm=torch.ones(r.vdim, device="cuda"), neg_decay=-torch.rand(r.heads, device="cuda") * 0.5, dt_bias=f(r.heads * r.dim) - 3,
                            conv=f(r.taps, r.conv_channels).bfloat16().float() * 0.5)


def _rec_case(r, T, slots):
    col, width = _columns(r)
    w = _channel_weights(r) if r.kind == "channel_delta" else _rec_weights(r)
    step = torch.randn(T, r.heads * r.dim, device="cuda") if r.kind == "channel_delta" else None
    return _bf(T, width, std=1.0), rec.RecColumns.of(r, col), w, rec.RecState.make(r, slots, torch.bfloat16, "cuda"), step


def _pair(T, F, K, glu):
    def make():
        x, w = _bf(T, K, std=1.0), _bf(2 * F, K)
        return lambda: ops.swiglu_linear(x, w, glu=glu), (w.numel() + x.numel() + T * F) * 2, 4 * T * F * K
    return make


def _products(new, near, T):
    C, Hq, Hkv, ff = new.hidden_size, near.num_heads, near.num_kv_heads, near.intermediate_size
    qkv, o = _product(T, (Hq + 2 * Hkv) * 128, C), _product(T, C, Hq * 128)
    out = []
    for name, i in (("delta rule", 0), ("window", 1), ("latent", 3)):
        lay = LayerLayout(new.layers[i], ff=False)
        out += [(f"{name}: product in", _product(T, lay.in_rows, C), qkv), (f"{name}: product out + residual", _product(T, C, lay.out_cols, back=True), o)]
    r = new.layers[0].mixer
    return out + [("delta rule: product of the decays, 32-bit", _product(T, r.heads * r.dim, r.decay_rank, f32=True), o),
                  ("delta rule: product of the gate", _product(T, r.out_width, r.gate_rank), o),
                  ("clamped gate / up", _pair(T, ff, C, (7.0, GLU_SLOPE)), _pair(T, ff, C, None)),
                  ("down + residual", _product(T, C, ff, back=True), _product(T, C, ff))]


def _norm_like(C, T):
    def make():
        r, y, g = _bf(T, C, std=1.0), _bf(1, T, C, std=1.0), _bf(C)
        return lambda: ops.reduce_residual_rmsnorm(r, y, g, 1e-5), T * C * 8, 6 * T * C
    return make


def _norms(new, T, inp, slots, decode):
    C = new.hidden_size

    def depth(n):
        def make():
            x, w, g, xo = torch.randn(n, T, C, device="cuda"), torch.ones(n, device="cuda"), torch.ones(C, device="cuda"), torch.empty(T, C, device="cuda")
            sh = pre.TokenShift(torch.full((C,), 0.5, device="cuda"), torch.zeros(slots.shape[0], C, device="cuda"))
            S = slots.shape[0]
            return (lambda: pre.depth_norm(x, w, g, new.norm_groups, 1e-5, torch.bfloat16, xo, sh, inp, slots, decode),
                    T * C * (4 * n + 6) + S * C * 8, T * C * (2 * n + 8))
        return make

    def plain():
        x, g = torch.randn(1, T, C, device="cuda"), torch.ones(C, device="cuda")
        return lambda: pre.depth_norm(x, None, g, new.norm_groups, 1e-5, torch.bfloat16), T * C * 6, 5 * T * C
    like = _norm_like(C, T)
    return [("depth average of 3, norm, shift", depth(3), like), ("depth average of 24, norm, shift", depth(24), like), ("norm in groups", plain, like)]


def decode_kernels(new, near, B=64, ctx=640):
    """(name, new op, like op): each op is a function returning (launch, bytes, flops)."""
    r, a, m = _mixers(new)
    Hq, Hkv = near.num_heads, near.num_kv_heads
    H, D, R, V, K = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
    pos1 = lambda n: torch.full((B,), n - 1, dtype=torch.int32, device="cuda")      # noqa: E731
    slots = torch.arange(B, dtype=torch.int32, device="cuda")

    def paged(n, ps):
        nb = (n + ps - 1) // ps
        return torch.arange(B * nb, dtype=torch.int32, device="cuda").view(B, nb), B * nb

    def attn(n):
        def make():
            bt, pages = paged(n, 64)
            cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda").normal_()
            q, out = _bf(B, a.heads * 128, std=1.0), _bf(B, a.heads * 128)
            inp, mix = _Step(False, positions=pos1(n), seq_of_token=None, block_table=bt, seq_lens=pos1(n) + 1), par.HeadMix(sinks=torch.zeros(a.heads, device="cuda"))
            keys = min(n, a.window + a.keep_first)
            return lambda: par.window_attn(q, a, inp, cache, 64, out, 1.0, mix), B * keys * 2 * a.kv_heads * 256, 4 * B * a.heads * keys * 128
        return make

    def attn_like(n):
        def make():
            bt, pages = paged(n, 16)
            kv, q, lens = _bf(pages, 2, Hkv, 16, 128, std=1.0), _bf(B, Hq * 128, std=1.0), pos1(n) + 1
            return lambda: ops.attn_decode(q, kv, bt, lens, Hq, Hkv, 128, ctx_hint=n), B * n * 2 * Hkv * 256, 4 * B * Hq * n * 128
        return make

    def append():
        bt, pages = paged(ctx, 64)
        cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda")
        n = a.heads * 128, a.kv_heads * 128, a.kv_heads * 128
        q, k, v = _bf(B, sum(n), std=1.0).split(n, dim=1)
        f = lambda k: torch.ones(k, device="cuda")      # noqa: E731
        w = WindowAttnWeights(q_norm=f(128), k_norm=f(128), q_bias=f(n[0]), k_bias=f(n[1]), v_bias=f(n[2]), vmix=f(1))
        pos, mix = pos1(ctx), par.ValueMix(_bf(B, n[2]), False)
        return (lambda: par.head_append(q, k, v, a, None, pos, None, bt, cache, 64, 1e-5, w, mix), B * (2 * n[0] + 2 * n[1] + 3 * n[2]) * 2, 8 * B * n[0])

    def append_like():
        bt, pages = paged(ctx, 16)
        qkv, kv, t = _bf(B, (Hq + 2 * Hkv) * 128, std=1.0), _bf(pages, 2, Hkv, 16, 128), ref.rope_cos_sin_table(ctx + 8, 128, 1e4, "cuda")
        pos = pos1(ctx)
        return lambda: ops.rope_kv_append(qkv, pos, None, bt, t, kv, Hq, Hkv, 128), B * (2 * Hq + 4 * Hkv) * 256, B * Hq * 512

    def step(spec):
        def make():
            row, cols, w, st, a_in = _rec_case(spec, B, B)
            pos, out = pos1(ctx), _bf(B, spec.out_width)
            gate = rec.HeadGate(w.norm[:spec.vdim], _bf(B, spec.out_width, std=1.0), out, 1e-5, sigmoid=spec.kind == "channel_delta")
            by = B * (8 * spec.state_elems + 2 * (spec.conv_channels * (1 + spec.conv_rows) + spec.out_width * 2) + (4 * spec.heads * spec.dim if a_in is not None else 0))
            return lambda: rec.rec_step(row, cols, spec, w, st, pos, slots, gate, a_in), by, 6 * B * spec.state_elems
        return make

    def latent(n, sinks):
        def make():
            bt, pages = paged(n, 64)
            cache, q, qa, pos = _bf(pages, 64, K + R, std=1.0), _bf(B, H * (D + R), std=1.0), _bf(B, H * K, std=0.1), pos1(n)
            cs, s = ref.rope_cos_sin_table(n + 8, R, 1e4, "cuda"), torch.zeros(H, device="cuda") if sinks else None
            return (lambda: lat.latent_attn_rows(qa, q, H, D, R, m.scale, cs, pos, None, bt, cache, n, sinks=s), B * n * (K + R) * 2 + 2 * B * H * K * 2,
                    2 * B * H * n * (2 * K + R))
        return make

    def latent_append(strided):
        def make():
            bt, pages = paged(ctx, 64)
            proj, cache = _bf(B, H * (D + R) + K + R + (H * V if strided else 0), std=1.0), _bf(pages, 64, K + R)
            pos, kn, cs = pos1(ctx), torch.ones(K, device="cuda"), ref.rope_cos_sin_table(ctx + 8, R, 1e4, "cuda")
            return lambda: lat.latent_append(proj, H * (D + R), None, kn, R, cs, pos, None, bt, cache, 1e-5), B * (K + R) * 4, 4 * B * K
        return make

    def head(cols, F, Kk, back):
        def make():
            x, w = _bf(B, H * cols, std=1.0), _bf(H, F, Kk)
            out = _bf(B, 2 * H * F)[:, :H * F] if back else None
            return lambda: lat.head_linear(x, cols, w, out=out), (w.numel() + x.numel() + B * H * F) * 2, 2 * B * H * F * Kk
        return make
    inp = _Step(False, positions=pos1(ctx), seq_of_token=None, seq_lens=pos1(ctx) + 1)
    return [("window attention, all keys in the window", attn(ctx), attn_like(ctx)), ("window attention, 4096 tokens", attn(4096), attn_like(WINDOW + KEEP)),
            ("window: bias, norm, mixing, append", append, append_like), ("delta rule: step, norm, gate", step(r), step(_like_delta(r))),
            ("latent attention, 640 tokens", latent(ctx, True), latent(ctx, False)), ("latent attention, 4096 tokens", latent(4096, True), latent(4096, False)),
            ("latent: append", latent_append(True), latent_append(False)), ("latent: queries through the key expansion", head(D + R, K, D, False), head(D + R, K, D, False)),
            ("latent: values from the latents", head(K, V, K, True), head(K, V, K, False))] + _norms(new, B, inp, slots, True) + _products(new, near, B)


def prefill_kernels(new, near, S=4, L=2048):
    T = S * L
    r, a, m = _mixers(new)
    Hq, Hkv = near.num_heads, near.num_kv_heads
    H, D, R, V, K = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
    start, qlen = _i32([s * L for s in range(S)]), _i32([L] * S)
    pos, sot = _i32(list(range(L)) * S), _i32([s for s in range(S) for _ in range(L)])
    slots = torch.arange(S, dtype=torch.int32, device="cuda")
    t_like, pairs = ref.rope_cos_sin_table(L, 128, 1e4, "cuda"), S * L * (L + 1) // 2

    def paged(ps):
        nb = (L + ps - 1) // ps
        return torch.arange(S * nb, dtype=torch.int32, device="cuda").view(S, nb), S * nb

    def step_inputs():
        return _Step(True, positions=pos, seq_of_token=sot, block_table=paged(64)[0], seq_lens=qlen, q_start=start, q_len=qlen, max_q_len=L)

    def attn(spec):
        def make():
            cache = par.window_cache(paged(64)[1], 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda").normal_()
            q, out, inp, mix = _bf(T, a.heads * 128, std=1.0), _bf(T, a.heads * 128), step_inputs(), par.HeadMix(sinks=torch.zeros(a.heads, device="cuda"))
            w = WINDOW
            seen = S * (w * (w + 1) // 2 + (L - w) * w + sum(min(spec.keep_first, max(0, i - w + 1)) for i in range(L)))
            return lambda: par.window_attn(q, spec, inp, cache, 64, out, 1.0, mix), (2 * q.numel() + T * 2 * a.kv_heads * 128) * 2, 4 * a.heads * 128 * seen
        return make

    def append():
        bt, pages = paged(64)
        cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda")
        n = a.heads * 128, a.kv_heads * 128, a.kv_heads * 128
        q, k, v = _bf(T, sum(n), std=1.0).split(n, dim=1)
        f = lambda k: torch.ones(k, device="cuda")      # noqa: E731
        w = WindowAttnWeights(q_norm=f(128), k_norm=f(128), q_bias=f(n[0]), k_bias=f(n[1]), v_bias=f(n[2]), vmix=f(1))
        mix = par.ValueMix(_bf(T, n[2]), False)
        return (lambda: par.head_append(q, k, v, a, None, pos, sot, bt, cache, 64, 1e-5, w, mix), T * (2 * n[0] + 2 * n[1] + 3 * n[2]) * 2, 8 * T * n[0])

    def append_like():
        bt, pages = paged(16)
        qkv, kv = _bf(T, (Hq + 2 * Hkv) * 128, std=1.0), _bf(pages, 2, Hkv, 16, 128)
        return lambda: ops.rope_kv_append(qkv, pos, sot, bt, t_like, kv, Hq, Hkv, 128), T * (2 * Hq + 4 * Hkv) * 256, T * Hq * 512

    def chunk(spec, only):
        def make():
            row, cols, w, st, a_in = _rec_case(spec, T, S)
            run = rec.ChunkRun(row, cols, spec, w, st, pos, slots, sot, start, qlen, L, step=a_in)
            run.prep()
            qkv, out = 2 * spec.groups * spec.dim + spec.out_width, spec.out_width
            fl = T * spec.heads * (6 * spec.dim * spec.vdim + 128 * (spec.dim + spec.vdim))
            by = T * (qkv + out) * 2 + T * spec.heads * 8 + 8 * S * spec.state_elems + (T * spec.heads * spec.dim * 4 if a_in is not None else 0)
            return (run.prep, T * qkv * 4, 16 * T * qkv) if only == "prep" else (run.walk, by, fl)
        return make

    def gnorm(silu):
        def make():
            o, g, out, w = _bf(T, r.out_width, std=1.0), _bf(T, r.out_width, std=1.0), _bf(T, r.out_width), torch.ones(r.vdim, device="cuda")
            return lambda: par.gated_norm(o, g, w, out, r.heads, 1e-5, False, silu), T * r.out_width * 6, 10 * T * r.out_width
        return make

    def latent(sinks):
        def make():
            q, dense, kv = _bf(T, H * (D + R), std=1.0), _bf(T, K + R, std=1.0), _bf(T, H * (D + V), std=1.0)
            s = torch.zeros(H, device="cuda") if sinks else None
            return (lambda: lat.latent_attn_prefill(q, H, D, R, V, m.scale, dense, kv, start, qlen, qlen, start, L, sinks=s),
                    (q.numel() + kv.numel() + T * R + T * H * V) * 2, 2 * H * (D + R + V) * pairs)
        return make

    def latent_append(strided):
        def make():
            bt, pages = paged(64)
            proj, cache, dn = _bf(T, H * (D + R) + K + R + (H * V if strided else 0), std=1.0), _bf(pages, 64, K + R), _bf(T, K + R)
            kn, cs = torch.ones(K, device="cuda"), ref.rope_cos_sin_table(L, R, 1e4, "cuda")
            return lambda: lat.latent_append(proj, H * (D + R), None, kn, R, cs, pos, sot, bt, cache, 1e-5, dense=dn, dense_start=start), T * (K + R) * 6, 4 * T * K
        return make

    def rope(strided):
        def make():
            q, cs = _bf(T, H * (D + R) + (K + R + H * V if strided else 0), std=1.0), ref.rope_cos_sin_table(L, R, 1e4, "cuda")
            return lambda: lat.rope_rows(q, H, D, R, cs, pos), T * H * R * 4, T * H * R * 3
        return make
    plain = WindowAttnSpec(a.heads, a.kv_heads, 128, 128, a.scale, 0, 1e4, window=WINDOW)
    expand = _product(T, H * (D + V), K)
    return [("window attention", attn(a), attn(plain)), ("window: bias, norm, mixing, append", append, append_like),
            ("delta rule: convolution, silu, gates", chunk(r, "prep"), chunk(_like_delta(r), "prep")), ("delta rule: recurrence", chunk(r, "walk"), chunk(_like_delta(r), "walk")),
            ("delta rule: norm, gate", gnorm(False), gnorm(True)), ("latent attention", latent(True), latent(False)), ("latent: append", latent_append(True), latent_append(False)),
            ("latent: query rotation", rope(True), rope(False)), ("latent: key / value expansion", expand, expand)] \
        + _norms(new, T, step_inputs(), slots, False) + _products(new, near, T)
