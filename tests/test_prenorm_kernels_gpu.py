"""CUDA kernels of pre-norm layers, of differential and chunked attention and of the selective scan against their plain PyTorch
references (ops/reference_parallel.py, ops/reference_prenorm.py, 32-bit math)."""
import dataclasses
import math
from types import SimpleNamespace

import pytest
import torch

from barorax_models import chunk, diff, moe
from skein_b200 import ops
from skein_b200.models.layered import RoutedFFSpec
from skein_b200.models.parallel_layers import SelectiveSpec, SelectiveWeights, WindowAttnSpec, up8
from skein_b200.ops import parallel as par, prenorm as pre, reference as ref, reference_parallel as rp, reference_prenorm as rn, selective as sel

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def rnd(*shape, dtype=BF, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def close(got, want, dtype, mul=1.0):
    got, want = got.float().cpu(), want.float()
    tol = (1e-2 if dtype == BF else 2e-5) * mul
    err = (got - want).abs().max().item()
    ref_ = max(want.abs().max().item(), 1e-3)
    assert math.isfinite(err) and err <= tol * ref_, (err, ref_)


def i32(x):
    return torch.tensor(x, dtype=torch.int32)


def dev(t):
    return t.to(DEV) if isinstance(t, torch.Tensor) else t


# ---- stream and router -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,C,top", [(1, 64, 1), (37, 77, 3), (600, 1024, 6), (9, 4096, 9), (700, 2500, 2), (3, 16384, 2), (5, 13001, 1)])
def test_add_norm(T, C, top, dtype):
    x, y, step, gain = rnd(T, C, dtype=F32, scale=3), rnd(T * top + 5, C, dtype=dtype, seed=1), rnd(C, dtype=F32), 1 + rnd(C, dtype=F32, scale=0.3, seed=2)
    x[0] *= 1e-3
    y[:] *= 1 if T > 1 else 1e-3           # eps inside the root matters
    idx = torch.randperm(T * top + 5, generator=torch.Generator().manual_seed(3))[:T * top].view(T, top).to(torch.int32)
    w = rnd(T, top, dtype=F32).abs()
    for yy, ss, gg in ((y, step, gain), (y, None, gain), (None, step, gain), (None, None, gain), (y, None, None)):
        routed = (yy, idx, w) if yy is not None else (None, None, None)
        wa, wact = rn.add_norm(x, *routed, ss, gg, 1e-5, dtype)
        a, act = pre.add_norm(dev(x), *map(dev, routed), dev(ss), dev(gg), 1e-5, dtype)
        close(a, wa, F32)
        assert (act is None) == (wact is None)
        if act is not None:
            close(act, wact, dtype, 0.6)


@pytest.mark.parametrize("T,F,K", [(1, 32, 512), (64, 160, 4096), (17, 161, 520), (64, 2048, 2048), (50, 33, 1000), (63, 288, 8192)])
def test_small_product(T, F, K):
    """Few rows and few weights: strided rows in and out, 16- and 32-bit sums, in place on the residual, the same result every time."""
    assert ops.functional.small_gemm_ok(T, F, K)
    x, w = rnd(T, K + 16)[:, 8:8 + K], rnd(F, K, scale=K ** -0.5)
    gx = rnd(T, K + 16).to(DEV)[:, 8:8 + K]
    wide = torch.full((T, F + 8), 7.0, dtype=BF, device=DEV)
    ops.linear(gx, w.to(DEV), out=wide[:, :F])
    close(wide[:, :F], ref.linear(x, w), BF)
    assert (wide[:, F:] == 7).all()
    r = rnd(T, F, dtype=F32, scale=4)
    a, b = r.to(DEV), r.to(DEV)
    for o in (a, b):
        ops.linear(gx, w.to(DEV), out=o, residual=o, out_f32=True)
    close(a, ref.linear(x, w, r, out_f32=True), F32)
    assert torch.equal(a, b)
    rb = rnd(T, F, seed=3)
    close(ops.linear(gx, w.to(DEV), residual=rb.to(DEV)), ref.linear(x, w, rb), BF)


RULES = [moe(experts=12, top=3, groups=4, keep=2), moe(experts=64, top=6, groups=8, keep=4), moe(experts=5, top=2, groups=1, keep=1, scale=1.0),
         moe(experts=8, top=4, groups=8, keep=5), moe(experts=128, top=12, groups=64, keep=9), moe(experts=200, top=7, groups=40, keep=3),
         RoutedFFSpec(8, 7.0, 16, 4, 4, 2), RoutedFFSpec(8, None, 16, 4, 4, 2, group_best=2, renorm=True)]


@pytest.mark.parametrize("f", RULES)
def test_router_rules(f):
    T, C = 300, 96
    x, wg = rnd(T, C), rnd(f.experts, C, scale=0.2)
    logits = x.float() @ wg.float().t()
    ids, w = rn.select(logits, f)
    got = pre.route(x.to(DEV), wg.to(DEV), f)
    # (a close call may fall either way: compare where the choice is clear)
    same = (got[0].cpu() == ids).all(-1)
    assert same.float().mean() > 0.97
    close(got[1].cpu()[same], w[same], F32, 5.0)
    counts, offsets, row_of, src = got[2:6]
    assert counts.sum() == T * f.top and torch.equal(got[6], x.to(DEV)[src.long()]) and (src.view(-1)[row_of.long()].view(T, f.top).cpu() == torch.arange(T)[:, None]).all()


@pytest.mark.parametrize("T,C,f", [(1, 128, RULES[0]), (64, 2048, RULES[1]), (33, 5000, RULES[3]), (148, 512, RULES[2]), (16, 1024, RULES[7])])
def test_fused_norm_and_router(T, C, f):
    x, gain, wg = rnd(T, C, dtype=F32, scale=2), 1 + rnd(C, dtype=F32, scale=0.3), rnd(f.experts, C, scale=2 * C ** -0.5)
    assert pre.can_fuse_route(x.to(DEV), f, BF)
    act, ids, w, counts, offsets, row_of, src, xs = pre.norm_route(x.to(DEV), gain.to(DEV), 1e-5, wg.to(DEV), f)
    _, want = rn.add_norm(x, None, None, None, None, gain, 1e-5, BF)
    close(act, want, BF)
    wid, ww = rn.select(act.cpu().float() @ wg.float().t(), f)
    same = (ids.cpu() == wid).all(-1)
    assert same.float().mean() > 0.97
    close(w.cpu()[same], ww[same], F32, 5.0)
    wc, wo, _, ws = ref.router_plan(ids.cpu(), f.experts)
    assert torch.equal(counts.cpu(), wc) and torch.equal(offsets.cpu(), wo) and torch.equal(src.cpu(), ws) and torch.equal(xs, act[src.long()])
    ops.workspace().check_status()


# ---- attention -----------------------------------------------------------------------------------------------------------
ATTN = {
    "diff": diff(), "diff_odd": diff(3, 1, 7, 5, 0.5, 2, 100.0, 0.2), "diff_tc": diff(4, 2, 64, 128, 0.125, 64, 1e5, 0.5),
    "diff_tc_wide": diff(8, 1, 64, 128, 0.2, 16, 1e4, 0.8), "diff_16_rows": diff(18, 2, 64, 128, 0.2, 16, 1e4, 0.8),
    "diff_window": dataclasses.replace(diff(4, 2, 64, 128, 0.125, 64, 1e5, 0.5), window=100),
    "chunk": chunk(), "chunk_odd": chunk(5, 5, 10, 7, 0.7, 4, 50.0, 5), "chunk_one": chunk(2, 1, 16, 16, 0.25, 16, 1e4, 1),
    "chunk_64": chunk(4, 2, 64, 64, 0.125, 64, 1e4, 100), "chunk_128": chunk(8, 1, 128, 128, 0.09, 32, 1e6, 130), "chunk_long": chunk(4, 4, 128, 128, 0.05, 128, 1e6, 1000),
    "half_pairs": WindowAttnSpec(6, 3, 24, 40, 0.2, 16, 1e4, window=33, row_norm=False, sink=True, gated=True),
    "sink_tc": WindowAttnSpec(8, 2, 128, 128, 0.1, 32, 1e6, window=130, row_norm=False, sink=True),
}


def _attn_case(a, lens, new, ps, dtype, seed=0):
    """Sequences of `lens` cached tokens and `new` tokens each in this step; a cache whose unused rows hold junk."""
    S, T = len(lens), sum(new)
    mb = max(-(-(l + n) // ps) for l, n in zip(lens, new))
    pages = torch.randperm(S * mb + 3, generator=torch.Generator().manual_seed(seed))[:S * mb].view(S, mb).to(torch.int32)
    cache = rnd(S * mb + 3, a.kv_heads * ps * (a.key_width + a.vdim), dtype=dtype, seed=seed)
    pos = i32([p for l, n in zip(lens, new) for p in range(l, l + n)])
    sot = i32([s for s, n in enumerate(new) for _ in range(n)])
    cols, at = {}, 0
    for n, rows in a.sections():
        cols[n], at = slice(at, at + rows), at + up8(rows)
    row = rnd(T, at + 8, dtype=dtype, seed=seed + 1)
    table = ref.rope_cos_sin_table(int(pos.max()) + 1, a.rot_dims, a.rope_base)
    inp = dict(positions=pos, seq_of_token=sot, block_table=pages, seq_lens=i32([l + n for l, n in zip(lens, new)]), q_start=i32([sum(new[:s]) for s in range(S)]),
               q_len=i32(new), max_q_len=max(new), ctx_hint=1024)
    return cache, row, cols, table, inp


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("ps", [16, 64])
@pytest.mark.parametrize("name", list(ATTN))
def test_head_append_and_attention(name, ps, dtype):
    a = ATTN[name]
    lam = torch.tensor([0.63])
    for decode, lens, new in ((False, [0, 30, 0, 250, 16], [150, 3, 1, 140, 2]), (False, [0, 126], [520, 130]),
                              (True, [0, 5, 127, 128, 129, 460, 15, 20, 21, 99, 100], [1] * 11), (True, [1500, 3], [1, 1])):
        cache, row, cols, table, inp = _attn_case(a, lens, new, ps, dtype)
        T = row.shape[0]
        qkv = lambda r: tuple(r[:, cols[n]] for n in "qkv")      # noqa: E731
        wc, wr = cache.clone(), row.clone()
        rp.head_append(*qkv(wr), a, table, inp["positions"], inp["seq_of_token"], inp["block_table"], wc, ps, 1e-5)
        gate = row[:, cols["g"]] if a.gated else None
        want = rp.window_attn_rows(qkv(wr)[0], a, inp["positions"], inp["seq_of_token"], inp["block_table"], wc, ps, 0.7, par.HeadMix(lam, gate, 1e-5))
        gi = SimpleNamespace(is_prefill=not decode, **{k: dev(v) for k, v in inp.items()})
        if decode:
            gi.seq_of_token = None
        gc, gr = cache.to(DEV), row.to(DEV)
        par.head_append(*qkv(gr), a, table.to(DEV), gi.positions, gi.seq_of_token, gi.block_table, gc, ps, 1e-5)
        close(gr, wr, dtype)
        close(gc, wc, dtype)
        gr, gc = wr.to(DEV), wc.to(DEV)        # the attention from identical inputs
        mix = par.HeadMix(lam.to(DEV), gr[:, cols["g"]] if a.gated else None, 1e-5)
        for fn in (par.window_attn, None):
            out = torch.zeros(T, up8(a.out_width) + 8, dtype=dtype, device=DEV)
            o = out[:, :a.out_width]
            if fn is None:
                par.window_attn_rows(qkv(gr)[0], a, gi.positions, gi.seq_of_token, gi.block_table, gc, ps, o, 0.7, mix)
            else:
                fn(qkv(gr)[0], a, gi, gc, ps, o, 0.7, mix)
            # a head norm divides by what the two maps leave: twice the rounding
            close(o, want, dtype, 2.0 if a.diff is not None else 1.0)
            assert (out[:, a.out_width:] == 0).all()
    ops.workspace().check_status()


@pytest.mark.parametrize("name", ["chunk_64", "chunk_128", "sink_tc", "chunk"])
def test_the_sink_counts(name):
    """Without the sink the first tokens of a chunk (few keys, low scores) differ: what the test above compares depends on it."""
    a = ATTN[name]
    cache, row, cols, table, inp = _attn_case(a, [0], [40], 16, F32)
    args = (inp["positions"], inp["seq_of_token"], inp["block_table"])
    q, k, v = (row[:, cols[n]] for n in "qkv")
    rp.head_append(q, k, v, a, table, *args, cache, 16, 1e-5)
    with_, without = (rp.window_attn_rows(q, s, *args, cache, 16, 1.0, par.HeadMix()) for s in (a, dataclasses.replace(a, sink=False)))
    assert (with_ - without).norm() > 0.05 * with_.norm()


# ---- selective scan --------------------------------------------------------------------------------------------------
SCANS = {"small": SelectiveSpec(120, 12, 9, 4), "odd": SelectiveSpec(37, 5, 3, 2), "ones": SelectiveSpec(64, 1, 1, 1), "taps": SelectiveSpec(88, 40, 16, 7),
         "tiles": SelectiveSpec(256, 16, 16, 4), "n8": SelectiveSpec(40, 7, 8, 3), "n64": SelectiveSpec(200, 64, 8, 4), "n128": SelectiveSpec(24, 100, 8, 4),
         "n256": SelectiveSpec(20, 200, 8, 4)}


def _scan_case(m, lens, new, dtype, seed=0):
    S, T = len(lens), sum(new)
    f = lambda *s, scale=1.0, k=0: rnd(*s, dtype=F32, scale=scale, seed=seed + k)      # noqa: E731
    x_cols = sum(up8(r) for _, r in m.x_sections())
    w = SelectiveWeights(None, None, conv=f(m.taps, m.inner), conv_b=f(m.inner, k=1), dt_bias=f(m.inner, k=2) - 1, neg_a=-f(m.state, m.inner, k=3).exp(),
                         skip=f(m.inner, k=4))
    state = sel.ScanState.make(m, S + 2, dtype, "cpu")
    state.mat.copy_(f(*state.mat.shape, k=5))
    if state.tail is not None:
        state.tail.copy_(rnd(*state.tail.shape, dtype=dtype, seed=seed + 6))
    slots = torch.randperm(S + 2, generator=torch.Generator().manual_seed(seed))[:S].to(torch.int32)
    row = rnd(T, 2 * up8(m.inner) + 8, dtype=dtype, seed=seed + 7)
    inp = dict(positions=i32([p for l, n in zip(lens, new) for p in range(l, l + n)]), seq_of_token=i32([s for s, n in enumerate(new) for _ in range(n)]),
               q_start=i32([sum(new[:s]) for s in range(S)]), q_len=i32(new), seq_lens=i32([l + n for l, n in zip(lens, new)]))
    return w, state, slots, row, rnd(T, x_cols, dtype=dtype, seed=seed + 8), f(T, m.inner, k=9), inp


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", list(SCANS))
def test_convolution_and_scan(name, dtype):
    m = SCANS[name]
    for decode, lens, new in ((False, [0, 30, 0, 250, 1], [150, 3, 1, 40, 2]), (False, [5], [65]), (True, [0, 5, 1, 2, 90, 6], [1] * 6)):
        w, state, slots, row, proj, dt, inp = _scan_case(m, lens, new, dtype)
        T, I = row.shape[0], m.inner
        xz = lambda r: (r[:, :I], r[:, up8(I):up8(I) + I])      # noqa: E731
        g = SimpleNamespace(**{k: dev(v) for k, v in inp.items()})
        gw, gs = SelectiveWeights(*(dev(v) for v in vars(w).values())), sel.ScanState(state.mat.to(DEV), dev(state.tail))
        want_x = rn.short_conv(xz(row)[0], m.taps, w, state, inp["positions"], slots, inp["q_start"], inp["q_len"])
        out = torch.zeros(T, I + 8, dtype=dtype)
        rn.scan(want_x, proj, dt, *xz(row), out[:, :I], m, w, state, inp["positions"], slots, inp["q_start"], inp["q_len"])
        grow = row.to(DEV)
        got_x = sel.short_conv(xz(grow)[0], m, gw, gs, g, slots.to(DEV), decode)
        close(got_x, want_x, dtype)
        got = torch.zeros(T, up8(I) + 8, dtype=dtype, device=DEV)
        sel.scan(want_x.to(DEV), proj.to(DEV), dt.to(DEV), *xz(grow), got[:, :I], m, gw, gs, g, slots.to(DEV), decode)
        close(got[:, :I], out[:, :I], dtype, 1.0 if dtype == BF else 2.0)
        close(gs.mat, state.mat, F32, 1.0 if dtype == F32 else 2.0)        # (slots of no sequence are left alone)
        if state.tail is not None:
            assert torch.equal(gs.tail.cpu(), state.tail)
        assert (got[:, I:] == 0).all()
    ops.workspace().check_status()


def test_padding_rows_leave_state_and_cache_alone():
    m = SCANS["tiles"]
    w, state, slots, row, proj, dt, inp = _scan_case(m, [3, 4, 5], [1] * 3, BF)
    inp["positions"][1] = -1
    gw, gs = SelectiveWeights(*(dev(v) for v in vars(w).values())), sel.ScanState(state.mat.to(DEV), dev(state.tail))
    g = SimpleNamespace(**{k: dev(v) for k, v in inp.items()})
    r, I = row.to(DEV), m.inner
    xc = sel.short_conv(r[:, :I], m, gw, gs, g, slots.to(DEV), True)
    sel.scan(xc, proj.to(DEV), dt.to(DEV), r[:, :I], r[:, I:2 * I], torch.zeros(3, I, dtype=BF, device=DEV), m, gw, gs, g, slots.to(DEV), True)
    keep = int(slots[1])
    assert torch.equal(gs.mat[keep].cpu(), state.mat[keep]) and torch.equal(gs.tail[keep].cpu(), state.tail[keep])
    assert not torch.equal(gs.mat[int(slots[0])].cpu(), state.mat[int(slots[0])])


def test_a_slow_decay_keeps_32_bit_accuracy():
    """Thousands of steps whose decays lie just below one, in portions and one by one, against the recurrence in 64-bit."""
    m, n = SelectiveSpec(32, 8, 8, 1), 3000
    w, state, slots, row, proj, dt, inp = _scan_case(m, [0], [n], F32)
    w.neg_a = -torch.full_like(w.neg_a, 2e-3)
    proj[:, :] = proj.abs()
    x = rnd(n, m.inner, dtype=F32, seed=5).abs()
    z = torch.ones(n, m.inner)
    S, want = torch.zeros(m.state, m.inner, dtype=torch.float64), torch.zeros(n, m.inner, dtype=torch.float64)
    step = torch.nn.functional.softplus(dt.double() + w.dt_bias.double())
    for t in range(n):
        S = torch.exp(step[t] * w.neg_a.double()) * S + step[t] * x[t].double() * proj[t, 8:16, None].double()
        want[t] = (proj[t, 16:24].double() @ S + w.skip.double() * x[t].double()) * torch.sigmoid(torch.tensor(1.0))
    gw = SelectiveWeights(*(dev(v) for v in vars(w).values()))
    for cuts in ([n], [1000, 1, 1999]):
        gs, at, got = sel.ScanState(torch.zeros_like(state.mat).to(DEV), None), 0, torch.zeros(n, m.inner, device=DEV)
        for k in cuts:
            rows = slice(at, at + k)
            g = SimpleNamespace(positions=i32(range(at, at + k)).to(DEV), seq_of_token=torch.zeros(k, dtype=torch.int32, device=DEV), q_start=i32([0]).to(DEV),
                                q_len=i32([k]).to(DEV), seq_lens=i32([at + k]).to(DEV))
            xz = torch.cat([x[rows], z[rows]], dim=1).to(DEV)
            sel.scan(x[rows].to(DEV).contiguous(), proj[rows].to(DEV).contiguous(), dt[rows].to(DEV).contiguous(), xz[:, :32], xz[:, 32:], got[rows], m, gw, gs, g,
                     slots.to(DEV), k == 1)
            at += k
        assert float(((got.cpu() - want).abs() / want.abs().clamp(min=1)).max()) < 1e-5
