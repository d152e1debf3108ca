"""Throughput and per-kernel rooflines of a design that lists its layers, beside the closest uniform family at equal size.

    python bench.py --design zarorax                    # one JSON object per size; also: sikalorn, barorax, derusun
    python -m skein_b200.utils.design_bench --design sikalorn --only kernels --size width-2k

Weights are random. Each size is a few layers of a real model's width; the closest model has the same width, number of layers,
query heads, experts and feed-forward size (a Mixtral-shaped block for routed layers, a Llama-shaped one for dense layers).
Decode: 64 sequences, context 512 and growing, captured steps with device-side token feedback; prefill: 8192 prompt tokens per
step. Kernel times are CUDA-event medians with cold L2 (decode-sized launches back to back inside a graph over rotating
operand copies, prefill-sized ones with an L2 flush in between); `far` is how many times longer a kernel takes than its
roofline, and `ratio` that of the new kernel over that of the like kernel of the closest model.
"""
from __future__ import annotations

import argparse
import json
import sys

import torch

from .. import ops
from ..models import config as mc
from ..models.decoder import Decoder, random_weights
from ..models.layered import DenseFFSpec, LatentMixerSpec, LayerSpec, RoutedFFSpec
from ..ops import latent as lat
from ..ops import reference as ref
from ..runtime.runner import ModelRunner
from . import design_bench_parallel as parallel, design_bench_prenorm as prenorm, design_bench_shifted as shifted
from .microbench import _bf, peaks, timeit, timeit_graph


def size_config(name: str, layers: int = 4):
    """(design's configuration, closest uniform configuration)"""
    C, H, q_rank, ff = {"moe-2k": (2048, 16, 1024, 1408), "moe-4k": (4096, 32, 1536, 14336), "dense-4k": (4096, 32, 1536, 14336)}[name]
    a = LatentMixerSpec("latent_attention_2", heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=512, rope_base=1e4, scale=192 ** -0.5, gated=True)
    b = LatentMixerSpec("latent_attention", heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=512, rope_base=1e4, scale=192 ** -0.5, q_rank=q_rank)
    if name == "dense-4k":
        mlp, E, top = DenseFFSpec(ff), 0, 0
    else:
        E, top, groups, keep = (64, 6, 8, 3) if name == "moe-2k" else (8, 2, 4, 2)
        mlp = RoutedFFSpec(ff, 7.0, E, top, groups, keep)
    new = mc.ModelConfig.layered("Zarorax", tuple(LayerSpec(b if i % 2 else a, mlp) for i in range(layers)), width=C, vocab=32000, taps=4,
                                 alpha=2.0, max_pos=8192, name=f"zarorax-{name}")
    near = mc.ModelConfig(architecture="MixtralForCausalLM" if E else "LlamaForCausalLM", hidden_size=C, intermediate_size=ff, num_layers=layers,
                          num_heads=H, num_kv_heads=max(1, H // 4), head_dim=128, vocab_size=32000, num_experts=E, top_k=top,
                          max_position_embeddings=8192, name=("mixtral" if E else "llama") + f"-{name}")
    return new, near


def throughput(cfg, B=64, prompt=512, steps=64, warmup=8, repeats=3, prompts_per_chunk=16):
    """Device-timed decode and prefill tokens/s of a model with random weights."""
    dev = torch.device("cuda")
    w = random_weights(cfg, mc.ParallelLayout(), dev, seed=0)
    ps = cfg.default_page_size
    blocks = (prompt + steps + warmup + ps) // ps + 1
    dec = Decoder(cfg, w, num_pages=B * blocks + 1, max_pos=prompt + steps + warmup + 64, state_slots=B)
    run = ModelRunner(dec, blocks, ctx_hint=prompt + steps // 2)
    g = torch.Generator().manual_seed(1)
    prompts = torch.randint(0, cfg.vocab_size, (B, prompt), generator=g).tolist()
    tables = [list(range(1 + s * blocks, 1 + (s + 1) * blocks)) for s in range(B)]
    first = []
    for c in range(0, B, prompts_per_chunk):
        first += run.prefill([(prompts[s], tables[s], 0, s) for s in range(c, min(B, c + prompts_per_chunk))])
    inp, _ = run._prefill_inputs([(prompts[s], tables[s], 0, s) for s in range(prompts_per_chunk)], None)
    ev = lambda: torch.cuda.Event(enable_timing=True)      # noqa: E731
    pf = []
    for _ in range(repeats + 2):
        s, e = ev(), ev()
        torch.cuda.synchronize()
        s.record()
        dec.forward_logits(inp)
        e.record()
        torch.cuda.synchronize()
        pf.append(s.elapsed_time(e))
    bk = run.bucket(B)
    run._ensure_graph(bk, True)
    times = []
    for _ in range(repeats):
        run.load_decode_inputs(bk, first, [prompt] * B, [prompt + 1] * B, tables)
        bk.dev_in.copy_(bk.host_in)
        for _ in range(warmup):
            run.decode_loop_step(bk)
        torch.cuda.synchronize()
        s, e = ev(), ev()
        s.record()
        for _ in range(steps):
            run.decode_loop_step(bk)
        e.record()
        torch.cuda.synchronize()
        times.append(s.elapsed_time(e) / steps)
    ops.workspace().check_status()
    ms, pms = sorted(times)[len(times) // 2], sorted(pf)[len(pf) // 2]
    from ..ops import _lib
    l0 = _lib.launches()
    run._decode_body(bk, False)
    return {"model": cfg.name, "layers": cfg.num_layers, "params_m": round(cfg.param_count() / 1e6, 1), "decode_ms_per_step": round(ms, 4),
            "decode_tokens_per_s": round(B / ms * 1e3), "prefill_ms": round(pms, 3), "kernels_per_step": _lib.launches() - l0,
            "prefill_tokens_per_s": round(prompts_per_chunk * prompt / pms * 1e3)}


# ---- kernels ----------------------------------------------------------------------------------------------------------
def _paged(B, ctx, ps):
    nb = (ctx + ps - 1) // ps
    return torch.arange(B * nb, dtype=torch.int32, device="cuda").view(B, nb), B * nb


def _pos(B, ctx):
    return torch.full((B,), ctx - 1, dtype=torch.int32, device="cuda")


def decode_kernels(new, near, B=64, ctx=640):
    """(name, new op, like op): each op is a function returning (launch, bytes, flops)."""
    C, m = new.hidden_size, new.layers[0].mixer
    H, D, R, V, K = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
    f32 = lambda *s: torch.randn(*s, device="cuda")          # noqa: E731
    cs = ref.rope_cos_sin_table(ctx + 8, R, 1e4, "cuda")
    one = torch.ones(1, device="cuda")

    def attn():
        bt, n = _paged(B, ctx, 64)
        cache, q, qa, pos = _bf(n, 64, K + R, std=1.0), _bf(B, H * (D + R), std=1.0), _bf(B, H * K, std=0.1), _pos(B, ctx)
        return (lambda: lat.latent_attn_rows(qa, q, H, D, R, m.scale, cs, pos, None, bt, cache, ctx),
                B * ctx * (K + R) * 2 + 2 * B * H * K * 2, 2 * B * H * ctx * (2 * K + R))

    def attn_like():
        Hq, Hkv = near.num_heads, near.num_kv_heads
        bt, n = _paged(B, ctx, 16)
        kv, q, lens = _bf(n, 2, Hkv, 16, 128, std=1.0), _bf(B, Hq * 128, std=1.0), torch.full((B,), ctx, dtype=torch.int32, device="cuda")
        return lambda: ops.attn_decode(q, kv, bt, lens, Hq, Hkv, 128, ctx_hint=ctx), B * ctx * 2 * Hkv * 256, 4 * B * Hq * ctx * 128

    def head(cols, F, Kk, gated):
        x, w = _bf(B, H * cols, std=1.0), _bf(H, F, Kk)
        gate = _bf(B, H * F, std=1.0) if gated else None
        return lambda: lat.head_linear(x, cols, w, gate), (w.numel() + x.numel() + B * H * F * (2 if gated else 1)) * 2, 2 * B * H * F * Kk

    def dense(F, Kk):
        x, w = _bf(B, Kk, std=1.0), _bf(F, Kk)
        return lambda: ops.linear(x, w), (w.numel() + x.numel() + B * F) * 2, 2 * B * F * Kk

    def norm(conv):
        x, y, w = f32(B, C), _bf(B, C, std=1.0), f32(4, C)
        bt, n = _paged(B, ctx, 64)
        tail, pos = _bf(n, 4, C, std=1.0), _pos(B, ctx)
        st = lat.ConvState(w, tail, 64) if conv else None
        return (lambda: lat.post_norm(x, y, 3.0, one, 1e-5, conv=st, positions=pos, block_table=bt),
                B * C * (12 + (8 if conv else 0)) + (16 * C if conv else 0), 10 * B * C)

    def norm_like():
        r, y, g = _bf(B, C, std=1.0), _bf(1, B, C, std=1.0), _bf(C)
        return lambda: ops.reduce_residual_rmsnorm(r, y, g, 1e-5), B * C * 8, 6 * B * C

    def append():
        bt, n = _paged(B, ctx, 64)
        proj, cache, pos, kn = _bf(B, H * (D + R) + K + R, std=1.0), _bf(n, 64, K + R), _pos(B, ctx), torch.ones(K, device="cuda")
        return lambda: lat.latent_append(proj, H * (D + R), None, kn, R, cs, pos, None, bt, cache, 1e-5), B * (K + R) * 4, 4 * B * K

    def append_like():
        Hq, Hkv = near.num_heads, near.num_kv_heads
        bt, n = _paged(B, ctx, 16)
        qkv, kv, pos, t = _bf(B, (Hq + 2 * Hkv) * 128, std=1.0), _bf(n, 2, Hkv, 16, 128), _pos(B, ctx), ref.rope_cos_sin_table(ctx + 8, 128, 1e4, "cuda")
        return lambda: ops.rope_kv_append(qkv, pos, None, bt, t, kv, Hq, Hkv, 128), B * (2 * Hq + 4 * Hkv) * 256, B * Hq * 512

    out = [("attention", attn, attn_like),
           ("queries through the key expansion", lambda: head(D + R, K, D, False), lambda: dense(K * H * D // C, C)),
           ("values from the latents, gated", lambda: head(K, V, K, True), lambda: dense(K * H * V // C, C)),
           ("input projection", lambda: dense(H * (D + R) + K + R + H * V, C), lambda: dense((near.num_heads + 2 * near.num_kv_heads) * 128, C)),
           ("norm", lambda: norm(False), norm_like), ("norm + next convolution", lambda: norm(True), norm_like), ("append", append, append_like)]
    mlp = new.layers[0].mlp
    if isinstance(mlp, RoutedFFSpec):
        E, k, Fe = mlp.experts, mlp.top, mlp.ff

        def route():
            x, y, wg = f32(B, C), _bf(B, C, std=1.0), _bf(E, C)
            return lambda: lat.post_norm_route(x, y, 3.0, one, 1e-5, wg, k, mlp.groups, mlp.keep), B * C * (10 + 2 * k) + 2 * E * C, 2 * B * E * C

        def route_like():
            r, y, g, wg = _bf(B, C, std=1.0), _bf(1, B, C, std=1.0), _bf(C), _bf(E, C)
            return lambda: ops.reduce_norm_route(r, y, g, 1e-5, wg, k), B * C * (8 + 2 * k) + 2 * E * C, 2 * B * E * C

        def experts(glu):
            per = max(1, B * k // E)
            cnt = torch.full((E,), per, dtype=torch.int32, device="cuda")
            off = (torch.arange(E + 1, device="cuda") * per).to(torch.int32)
            xs, w = _bf(E * per, C, std=1.0), _bf(E, 2 * Fe, C)
            return (lambda: ops.grouped_linear(xs, w, cnt, off, swiglu=True, glu=glu), (w.numel() + xs.numel() + E * per * Fe) * 2,
                    4 * E * per * Fe * C)
        out += [("norm + router + scatter", route, route_like), ("experts gate/up", lambda: experts((7.0, 1.702)), lambda: experts(None))]
    else:
        def poly():
            z, act = _bf(B, mlp.ff, std=1.0), torch.ones(4, device="cuda")
            return lambda: lat.poly_norm(z, act, 1e-5), B * mlp.ff * 4, 12 * B * mlp.ff

        def poly_like():
            r, g = _bf(B, mlp.ff, std=1.0), _bf(mlp.ff)
            return lambda: ops.rmsnorm(r, g, 1e-5), B * mlp.ff * 6, 6 * B * mlp.ff
        out.append(("polynomial activation", poly, poly_like))
    return out


def prefill_kernels(new, near, S=4, L=2048):
    C, m = new.hidden_size, new.layers[0].mixer
    H, D, R, V, K = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
    T = S * L
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")      # noqa: E731
    start, qlen = i32([s * L for s in range(S)]), i32([L] * S)
    pos, sot = i32(list(range(L)) * S), i32([s for s in range(S) for _ in range(L)])
    f32 = lambda *s: torch.randn(*s, device="cuda")                        # noqa: E731
    cs = ref.rope_cos_sin_table(L, R, 1e4, "cuda")
    cs_like = ref.rope_cos_sin_table(L, 128, 1e4, "cuda")
    one = torch.ones(1, device="cuda")
    Hq, Hkv = near.num_heads, near.num_kv_heads
    pairs = S * L * (L + 1) // 2

    def attn():
        q, dense, kv, gate = _bf(T, H * (D + R), std=1.0), _bf(T, K + R, std=1.0), _bf(T, H * (D + V), std=1.0), _bf(T, H * V, std=1.0)
        return (lambda: lat.latent_attn_prefill(q, H, D, R, V, m.scale, dense, kv, start, qlen, qlen, start, L, gate),
                (q.numel() + kv.numel() + T * R + 2 * gate.numel()) * 2, 2 * H * (D + R + V) * pairs)

    def attn_like():
        bt, n = _paged(S, L, 16)
        kv, q = _bf(n, 2, Hkv, 16, 128, std=1.0), _bf(T, Hq * 128, std=1.0)
        return lambda: ops.attn_prefill(q, kv, bt, start, qlen, qlen, L, Hq, Hkv, 128), (2 * q.numel() + T * 2 * Hkv * 128) * 2, 4 * Hq * 128 * pairs

    def dense(F, Kk):
        x, w = _bf(T, Kk, std=1.0), _bf(F, Kk)
        return lambda: ops.linear(x, w), (w.numel() + x.numel() + T * F) * 2, 2 * T * F * Kk

    def append():
        bt, n = _paged(S, L, 64)
        proj, cache, kn, dn = _bf(T, H * (D + R) + K + R, std=1.0), _bf(n, 64, K + R), torch.ones(K, device="cuda"), _bf(T, K + R)
        return lambda: lat.latent_append(proj, H * (D + R), None, kn, R, cs, pos, sot, bt, cache, 1e-5, dense=dn, dense_start=start), T * (K + R) * 6, 4 * T * K

    def append_like():
        bt, n = _paged(S, L, 16)
        qkv, kv = _bf(T, (Hq + 2 * Hkv) * 128, std=1.0), _bf(n, 2, Hkv, 16, 128)
        return lambda: ops.rope_kv_append(qkv, pos, sot, bt, cs_like, kv, Hq, Hkv, 128), T * (2 * Hq + 4 * Hkv) * 256, T * Hq * 512

    def rope():
        q = _bf(T, H * (D + R), std=1.0)
        return lambda: lat.rope_rows(q, H, D, R, cs, pos), T * H * R * 4, T * H * R * 3

    def conv():
        bt, n = _paged(S, L, 64)
        x, w, tail = f32(T, C), f32(4, C), _bf(n, 4, C)
        st = lat.ConvState(w, tail, 64)
        return lambda: lat.conv_input(x, st, pos, bt, sot, start), T * C * 6, 8 * T * C

    def norm(k):
        x, y = f32(T, C), _bf(T * max(1, k), C, std=1.0)
        idx = torch.randperm(T * k, device="cuda").to(torch.int32).view(T, k) if k else None
        w = torch.rand(T, k, device="cuda") if k else None
        return lambda: lat.post_norm(x, y, 3.0, one, 1e-5, idx, w), T * C * (10 + 2 * max(1, k)), 8 * T * C

    def norm_like(k):
        r, y, g = _bf(T, C, std=1.0), _bf(1, T * max(1, k), C, std=1.0), _bf(C)
        idx = torch.randperm(T * k, device="cuda").to(torch.int32).view(T, k) if k else None
        w = torch.rand(T, k, device="cuda") if k else None
        return lambda: ops.reduce_residual_rmsnorm(r, y, g, 1e-5, idx, w), T * C * (6 + 2 * max(1, k)), 8 * T * C

    out = [("attention", attn, attn_like), ("key / value expansion", lambda: dense(H * (D + V), K), lambda: dense((Hq + 2 * Hkv) * 128, C)),
           ("input projection", lambda: dense(H * (D + R) + K + R + H * V, C), lambda: dense((Hq + 2 * Hkv) * 128, C)),
           ("append", append, append_like), ("query rotation", rope, append_like), ("input convolution", conv, lambda: norm_like(0)),
           ("norm", lambda: norm(0), lambda: norm_like(0))]
    mlp = new.layers[0].mlp
    if isinstance(mlp, RoutedFFSpec):
        E, k = mlp.experts, mlp.top

        def route():
            x, wg = _bf(T, C, std=1.0), _bf(E, C)
            return lambda: lat.route_grouped(x, wg, k, mlp.groups, mlp.keep), T * C * 2 * (2 + 2 * k), 2 * T * E * C

        def route_like():
            x, wg = _bf(T, C, std=1.0), _bf(E, C)

            def fn():
                r = ops.route(x, wg, k)
                return ops.gather_rows(x, r[5])
            return fn, T * C * 2 * (2 + 2 * k), 2 * T * E * C
        out += [("router + gather", route, route_like), ("expert sum + norm", lambda: norm(k), lambda: norm_like(k))]
    else:
        def poly():
            z, act = _bf(T, mlp.ff, std=1.0), torch.ones(4, device="cuda")
            return lambda: lat.poly_norm(z, act, 1e-5), T * mlp.ff * 4, 12 * T * mlp.ff

        def poly_like():
            r, g = _bf(T, mlp.ff, std=1.0), _bf(mlp.ff)
            return lambda: ops.rmsnorm(r, g, 1e-5), T * mlp.ff * 6, 6 * T * mlp.ff
        out.append(("polynomial activation", poly, poly_like))
    return out


DESIGNS = {"zarorax": (("moe-2k", "moe-4k", "dense-4k"), size_config, decode_kernels, prefill_kernels),
           "sikalorn": (parallel.SIZES, parallel.size_config, parallel.decode_kernels, parallel.prefill_kernels),
           "barorax": (prenorm.SIZES, prenorm.size_config, prenorm.decode_kernels, prenorm.prefill_kernels),
           "derusun": (shifted.SIZES, shifted.size_config, shifted.decode_kernels, shifted.prefill_kernels)}
DESCRIBE = {"sikalorn": parallel.describe, "barorax": prenorm.describe, "derusun": shifted.describe}


def kernel_rows(design, new, near, iters=12, warmup=4):
    pk = peaks()

    def far(make, graph):
        fn, by, fl = make()
        us = timeit_graph(make, by, iters, warmup) if graph else timeit(fn, iters, warmup)
        best = max(by / (pk["hbm_gbs"] * 1e3), fl / (pk["bf16_tflops"] * 1e6))
        return us, us / best, by, fl
    rows = []
    for phase, table in (("decode", DESIGNS[design][2](new, near)), ("prefill", DESIGNS[design][3](new, near))):
        for name, a, b in table:
            ua, fa, by, fl = far(a, phase == "decode")
            torch.cuda.empty_cache()
            ub, fb, _, _ = far(b, phase == "decode")
            torch.cuda.empty_cache()
            rows.append({"phase": phase, "kernel": name, "us": round(ua, 2), "far": round(fa, 2), "GBps": round(by / ua * 1e-3), "TFLOPs": round(fl / ua * 1e-6, 1),
                         "like_us": round(ub, 2), "like_far": round(fb, 2), "ratio": round(fa / fb, 2)})
    ops.workspace().check_status()
    return rows


def run(design, sizes=None, only=("throughput", "kernels"), emit=print):
    for s in sizes or DESIGNS[design][0]:
        new, near = DESIGNS[design][1](s)
        about = DESCRIBE[design](new) if design in DESCRIBE else {"width": new.hidden_size, "heads": new.num_heads, "kv_rank": 512}
        res = {"size": s, "config": {"batch": 64, "prompt": 512, "decode_context": "512 + steps", "prefill_tokens": 8192, "weights": "random", **about},
               "peaks": peaks()}
        if "throughput" in only:
            res["design"] = throughput(new)
            torch.cuda.empty_cache()
            res["closest"] = throughput(near)
            torch.cuda.empty_cache()
        if "kernels" in only:
            res["kernels"] = kernel_rows(design, new, near)
        emit(json.dumps(res))


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--design", default="zarorax", choices=sorted(DESIGNS))
    ap.add_argument("--size", default="all", help="all, or a comma-separated list of: " + "; ".join(f"{d}: {', '.join(v[0])}" for d, v in DESIGNS.items()))
    ap.add_argument("--only", default="throughput,kernels")
    a = ap.parse_args(argv)
    with torch.no_grad():
        run(a.design, None if a.size == "all" else a.size.split(","), a.only.split(","))


if __name__ == "__main__":
    sys.exit(main())
