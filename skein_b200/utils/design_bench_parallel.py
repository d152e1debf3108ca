"""Sizes and kernel tables of parallel-layer designs for utils/design_bench.py: window attention, recurrences and the two products of
a layer, beside a Llama-shaped block of the same width, query heads and feed-forward size."""
from __future__ import annotations

import torch

from .. import ops
from ..models import config as mc
from ..models.layered import DenseFFSpec, unroll_loop
from ..models.parallel_layers import LayerLayout, MixerPairSpec, RecurrentSpec, RecurrentWeights, TanhNorm, WindowAttnSpec
from ..ops import parallel as par
from ..ops import recurrent as rec
from ..ops import reference as ref
from .microbench import _bf

SIZES = ("width-2k", "width-4k")


class _Step:
    """What the operators read of a step's inputs."""

    def __init__(self, prefill, **kw):
        self.is_prefill, self.ctx_hint = prefill, 1024
        self.__dict__.update(kw)


def size_config(name: str):
    """(design's configuration, closest uniform configuration): delta, pair, lightning, pair; the middle two layers run twice."""
    C, H, ff = {"width-2k": (2048, 16, 8192), "width-4k": (4096, 32, 14336)}[name]
    pair = MixerPairSpec(WindowAttnSpec(H, H // 4, 128, 128, 128 ** -0.5, 128, 5e5, 2.0, 1024), RecurrentSpec("ssd", 2 * H, 1, 128, 64, 4, 8), 0.7, 0.7)
    delta = RecurrentSpec("delta", H, H // 2, 128, 128, 4)
    light = RecurrentSpec("lightning", H, H, 128, 128, decay=tuple(1 - 2.0 ** -(2 + 6 * i / (H - 1)) for i in range(H)))
    specs = [(delta, DenseFFSpec(ff)), (pair, DenseFFSpec(ff)), (light, DenseFFSpec(ff)), (pair, DenseFFSpec(ff))]
    loop = (1, 3, 2)
    new = mc.ModelConfig.layered("Sikalorn", unroll_loop(specs, loop), width=C, vocab=32000, max_pos=8192, name=f"sikalorn-{name}", loop=loop)
    near = mc.ModelConfig(architecture="LlamaForCausalLM", hidden_size=C, intermediate_size=ff, num_layers=new.num_layers, num_heads=H,
                          num_kv_heads=H // 4, head_dim=128, vocab_size=32000, num_experts=0, top_k=0, max_position_embeddings=8192, name=f"llama-{name}")
    return new, near


def describe(new) -> dict:
    return {"width": new.hidden_size, "layer_runs": [l.mixer.kind for l in new.layers], "window": 1024}


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _rec_weights(r):
    H, ch = r.heads, r.conv_channels
    f = lambda *s: torch.randn(*s, device="cuda")          # noqa: E731
    w = RecurrentWeights(norm=torch.ones(r.vdim if r.kind == "delta" else r.out_width, device="cuda"), neg_decay=-torch.rand(H, device="cuda") * 0.1)
    if r.kind != "lightning":
        w.conv, w.dt_bias = f(r.taps, ch).bfloat16().float() * 0.5, f(H) - 3
    if r.kind == "ssd":
        w.conv_b, w.skip = f(ch) * 0.1, f(H)
    return w


def _columns(r):
    col, at = {}, 0
    for n, rows in r.sections():
        col[n] = at
        at += (rows + 7) // 8 * 8
    return col, at


def _mixers(new):
    pair = new.layers[1].mixer
    return pair.left, {"delta rule": new.layers[0].mixer, "state space": pair.right, "lightning": new.layers[2].mixer}


def decode_kernels(new, near, B=64, ctx=640):
    """(name, new op, like op): each op is a function returning (launch, bytes, flops)."""
    C = new.hidden_size
    a, recs = _mixers(new)
    Hq, Hkv = near.num_heads, near.num_kv_heads
    pos1 = lambda n: torch.full((B,), n - 1, dtype=torch.int32, device="cuda")      # noqa: E731

    def paged(n, ps):
        nb = (n + ps - 1) // ps
        return torch.arange(B * nb, dtype=torch.int32, device="cuda").view(B, nb), B * nb

    def attn(n):
        def make():
            bt, pages = paged(n, 64)
            cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda").normal_()
            q, out = _bf(B, a.heads * 128, std=1.0), _bf(B, a.heads * 128)
            inp = _Step(False, positions=pos1(n), seq_of_token=None, block_table=bt, seq_lens=pos1(n) + 1)
            keys = min(n, a.window)
            return lambda: par.window_attn(q, a, inp, cache, 64, out), B * keys * 2 * a.kv_heads * 256, 4 * B * a.heads * keys * 128
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
        row, t = _bf(B, (a.heads + 2 * a.kv_heads) * 128, std=1.0), ref.rope_cos_sin_table(ctx + 8, 128, 1e4, "cuda")
        q, k, v = row.split([a.heads * 128, a.kv_heads * 128, a.kv_heads * 128], dim=1)
        qn, kn, pos = torch.ones(a.heads * 128, device="cuda"), torch.ones(a.kv_heads * 128, device="cuda"), pos1(ctx)
        return (lambda: par.window_append(q, k, v, qn, kn, a, t, pos, None, bt, cache, 64, 1e-5), B * (2 * a.heads + 4 * a.kv_heads) * 256,
                B * a.heads * 1024)

    def append_like():
        bt, pages = paged(ctx, 16)
        qkv, kv, t = _bf(B, (Hq + 2 * Hkv) * 128, std=1.0), _bf(pages, 2, Hkv, 16, 128), ref.rope_cos_sin_table(ctx + 8, 128, 1e4, "cuda")
        pos = pos1(ctx)
        return lambda: ops.rope_kv_append(qkv, pos, None, bt, t, kv, Hq, Hkv, 128), B * (2 * Hq + 4 * Hkv) * 256, B * Hq * 512

    def step(r):
        def make():
            col, width = _columns(r)
            row, w, st = _bf(B, width, std=1.0), _rec_weights(r), rec.RecState.make(r, B, torch.bfloat16, "cuda")
            cols, pos, slots, out = rec.RecColumns.of(r, col), pos1(ctx), torch.arange(B, dtype=torch.int32, device="cuda"), _bf(B, r.out_width)
            gate = rec.HeadGate(w.norm, row[:, col["g"]:col["g"] + r.out_width], out, 1e-5) if r.kind == "delta" else None
            by = B * (8 * r.state_elems + 2 * (r.conv_channels * (1 + r.conv_rows) + r.out_width * 2))
            return lambda: rec.rec_step(row, cols, r, w, st, pos, slots, gate), by, 6 * B * r.state_elems
        return make

    def gnorm(r):
        def make():
            o, g, w, out = _bf(B, r.out_width, std=1.0), _bf(B, r.out_width, std=1.0), torch.ones(r.out_width, device="cuda"), _bf(B, r.out_width)
            return (lambda: par.gated_norm(o, g, w, out, r.norm_groups, 1e-5, r.kind == "ssd", r.kind == "ssd"), B * r.out_width * 6 + r.out_width * 4,
                    10 * B * r.out_width)
        return make

    def norm():
        x, n = torch.randn(B, C, device="cuda"), TanhNorm(*(torch.ones(k, device="cuda") for k in (1, C, C)))
        return lambda: par.residual_tanh(x, norm=n, want_x=False), B * C * 6 + C * 8, 12 * B * C

    def norm_like():
        r, y, g = _bf(B, C, std=1.0), _bf(1, B, C, std=1.0), _bf(C)
        return lambda: ops.reduce_residual_rmsnorm(r, y, g, 1e-5), B * C * 8, 6 * B * C

    out = [("attention, all keys in the window", attn(ctx), attn_like(ctx)), ("attention, 4096 tokens, window 1024", attn(4096), attn_like(1024)),
           ("norm + rotation + append", append, append_like)]
    for name, r in recs.items():
        out.append((f"{name}: step" + (" + gated norm" if r.kind == "delta" else ""), step(r), attn_like(ctx)))
        if r.kind != "delta":
            out.append((f"{name}: gated norm", gnorm(r), norm_like))
    out.append(("tanh norm", norm, norm_like))
    return out + [(n, p, q) for n, p, q in _products(new, near, B)]


def _products(new, near, T):
    """The two products of every kind of layer and the loop's."""
    C = new.hidden_size
    Hq, Hkv = near.num_heads, near.num_kv_heads

    def plain(F, K):
        def make():
            x, w = _bf(T, K, std=1.0), _bf(F, K)
            return lambda: ops.linear(x, w), (w.numel() + x.numel() + T * F) * 2, 2 * T * F * K
        return make

    def product(F, K, relu, back):
        def make():
            x, w = _bf(T, K, std=1.0), _bf(F, K)
            if back:
                r = torch.zeros(T, F, device="cuda")
                return lambda: ops.linear(x, w, out=r, residual=r, out_f32=True), (w.numel() + x.numel()) * 2 + T * F * 8, 2 * T * F * K
            return lambda: ops.linear(x, w, relu2_cols=relu), (w.numel() + x.numel() + T * F) * 2, 2 * T * F * K
        return make
    out = []
    for name, i in (("delta", 0), ("pair", 1), ("lightning", 2)):
        lay = LayerLayout(new.layers[i])
        out.append((f"{name}: product in", product(lay.in_rows, C, lay.ff_cols, False), plain((Hq + 2 * Hkv) * 128, C)))
        out.append((f"{name}: product out + residual", product(C, lay.out_cols, 0, True), plain(C, near.intermediate_size)))
    out.append(("loop: product", plain(C, 2 * C), plain(C, Hq * 128)))
    return out


def prefill_kernels(new, near, S=4, L=2048):
    C, T = new.hidden_size, S * L
    a, recs = _mixers(new)
    Hq, Hkv = near.num_heads, near.num_kv_heads
    start, qlen = _i32([s * L for s in range(S)]), _i32([L] * S)
    pos, sot = _i32(list(range(L)) * S), _i32([s for s in range(S) for _ in range(L)])
    t_like = ref.rope_cos_sin_table(L, 128, 1e4, "cuda")

    def paged(ps):
        nb = (L + ps - 1) // ps
        return torch.arange(S * nb, dtype=torch.int32, device="cuda").view(S, nb), S * nb

    def attn():
        bt, pages = paged(64)
        cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda").normal_()
        q, out = _bf(T, a.heads * 128, std=1.0), _bf(T, a.heads * 128)
        inp = _Step(True, positions=pos, seq_of_token=sot, block_table=bt, seq_lens=qlen, q_start=start, q_len=qlen, max_q_len=L)
        w = min(a.window, L)
        pairs = S * (w * (w + 1) // 2 + (L - w) * w)
        return lambda: par.window_attn(q, a, inp, cache, 64, out), (2 * q.numel() + T * 2 * a.kv_heads * 128) * 2, 4 * a.heads * 128 * pairs

    def attn_like():
        bt, pages = paged(16)
        kv, q = _bf(pages, 2, Hkv, 16, 128, std=1.0), _bf(T, Hq * 128, std=1.0)
        return (lambda: ops.attn_prefill(q, kv, bt, start, qlen, qlen, L, Hq, Hkv, 128), (2 * q.numel() + T * 2 * Hkv * 128) * 2,
                4 * Hq * 128 * S * L * (L + 1) // 2)

    def append():
        bt, pages = paged(64)
        cache = par.window_cache(pages, 64, a.kv_heads, 128, 128, torch.bfloat16, "cuda")
        row = _bf(T, (a.heads + 2 * a.kv_heads) * 128, std=1.0)
        q, k, v = row.split([a.heads * 128, a.kv_heads * 128, a.kv_heads * 128], dim=1)
        qn, kn = torch.ones(a.heads * 128, device="cuda"), torch.ones(a.kv_heads * 128, device="cuda")
        return (lambda: par.window_append(q, k, v, qn, kn, a, t_like, pos, sot, bt, cache, 64, 1e-5), T * (2 * a.heads + 4 * a.kv_heads) * 256,
                T * a.heads * 1024)

    def append_like():
        bt, pages = paged(16)
        qkv, kv = _bf(T, (Hq + 2 * Hkv) * 128, std=1.0), _bf(pages, 2, Hkv, 16, 128)
        return lambda: ops.rope_kv_append(qkv, pos, sot, bt, t_like, kv, Hq, Hkv, 128), T * (2 * Hq + 4 * Hkv) * 256, T * Hq * 512

    def chunk(r, only):
        def make():
            col, width = _columns(r)
            row, w, st = _bf(T, width, std=1.0), _rec_weights(r), rec.RecState.make(r, S, torch.bfloat16, "cuda")
            run = rec.ChunkRun(row, rec.RecColumns.of(r, col), r, w, st, pos, torch.arange(S, dtype=torch.int32, device="cuda"), sot, start, qlen, L)
            run.prep()
            qkv, out = 2 * r.groups * r.dim + r.out_width, r.out_width
            # what the recurrence itself needs: q, k, v, the gates in, the read-outs and states out. Products over chunks of 64 tokens:
            # read-out and update of the state, scores and their use, and the correction's three
            fl = T * r.heads * (4 * r.dim * r.vdim + 64 * (r.dim + r.vdim)
                                + ((2 * r.dim * r.vdim + 64 * (r.dim + r.vdim)) if r.kind == "delta" else 0))
            by = T * (qkv + out) * 2 + T * r.heads * 8 + 8 * S * r.state_elems
            return (run.prep, T * qkv * 4, 16 * T * qkv) if only == "prep" else (run.walk, by, fl)
        return make

    def gnorm(r):
        def make():
            o, g, out = _bf(T, r.out_width, std=1.0), _bf(T, r.out_width, std=1.0), _bf(T, r.out_width)
            groups = {"delta": r.heads, "ssd": r.norm_groups, "lightning": 1}[r.kind]
            w = torch.ones(r.vdim if r.kind == "delta" else r.out_width, device="cuda")
            return lambda: par.gated_norm(o, g, w, out, groups, 1e-5, r.kind == "ssd", r.kind != "lightning"), T * r.out_width * 6, 10 * T * r.out_width
        return make

    def norm():
        x, n = torch.randn(T, C, device="cuda"), TanhNorm(*(torch.ones(k, device="cuda") for k in (1, C, C)))
        return lambda: par.residual_tanh(x, norm=n, want_x=False), T * C * 6, 12 * T * C

    def norm_like():
        r, y, g = _bf(T, C, std=1.0), _bf(1, T, C, std=1.0), _bf(C)
        return lambda: ops.reduce_residual_rmsnorm(r, y, g, 1e-5), T * C * 8, 6 * T * C

    out = [("attention, window 1024", attn, attn_like), ("norm + rotation + append", append, append_like)]
    for name, r in recs.items():
        out += [(f"{name}: convolution, silu, gates", chunk(r, "prep"), append_like), (f"{name}: recurrence", chunk(r, "walk"), attn_like),
                (f"{name}: gated norm", gnorm(r), norm_like)]
    out.append(("tanh norm", norm, norm_like))
    return out + _products(new, near, T)
