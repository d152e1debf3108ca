"""CUDA kernels of parallel layers, sliding-window attention and recurrences against their plain PyTorch references
(ops/reference_parallel.py, 32-bit math)."""
import copy
import math
from types import SimpleNamespace

import pytest
import torch

from skein_b200 import ops
from skein_b200.models.parallel_layers import RecurrentSpec, RecurrentWeights, TanhNorm, WindowAttnSpec
from skein_b200.ops import parallel as par, recurrent as rec, reference as ref, reference_parallel as rp

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


def to_dev(obj):
    """A copy of a dataclass of tensors on the GPU."""
    out = copy.copy(obj)
    for k, v in vars(obj).items():
        if isinstance(v, torch.Tensor):
            setattr(out, k, v.to(DEV))
    return out


# ---- around the products -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,C", [(1, 64), (37, 77), (300, 1024)])
def test_residual_tanh(T, C, dtype):
    x, y, b = rnd(T, C, dtype=F32, scale=3), rnd(T, C, dtype=F32, seed=1), rnd(C, dtype=F32)
    norm = TanhNorm(torch.tensor([0.37]), 1 + rnd(C, dtype=F32, scale=0.3), rnd(C, dtype=F32, seed=2))
    small = TanhNorm(torch.tensor([1e-3]), norm.w, torch.zeros(C))            # tanh near zero keeps its relative accuracy
    for xx, yy, bb, nn in ((x, y, b, norm), (x, None, None, norm), (None, y, b, norm), (x, y.to(dtype), None, None), (x, None, None, small)):
        wa, wact = rp.residual_tanh(xx, yy, bb, nn, dtype)
        d = lambda t: None if t is None else t.to(DEV)      # noqa: E731
        a, act = par.residual_tanh(d(xx), d(yy), d(bb), to_dev(nn) if nn else None, dtype)
        close(a, wa, F32)
        close(act, wact, dtype, 0.5)
    wide = torch.full((T, 2 * C + 8), 7.0, dtype=dtype, device=DEV)
    par.residual_tanh(x.to(DEV), dtype=dtype, out=wide[:, C:2 * C])
    assert torch.equal(wide[:, C:2 * C].cpu(), x.to(dtype)) and (wide[:, :C] == 7).all() and (wide[:, 2 * C:] == 7).all()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("n,groups,period", [(96, 1, 96), (96, 4, 24), (2560, 2, 2560), (77 * 3, 3, 77), (1024, 8, 128), (5, 5, 1)])
@pytest.mark.parametrize("first,silu", [(True, True), (False, True), (False, False)])
def test_gated_norm(n, groups, period, first, silu, dtype):
    T = 19
    o, wide, w = rnd(T, n, dtype=dtype), rnd(T, n + 24, dtype=dtype, seed=1), 1 + rnd(period, dtype=F32, scale=0.4)
    o[3] *= 1e-3           # eps inside the root matters
    want = rp.gated_norm(o, wide[:, 8:8 + n], w, groups, 1e-5, first, silu, 0.6)
    out = torch.full((T, n + 16), 7.0, dtype=dtype, device=DEV)
    par.gated_norm(o.to(DEV), wide.to(DEV)[:, 8:8 + n], w.to(DEV), out[:, 8:8 + n], groups, 1e-5, first, silu, 0.6)
    close(out[:, 8:8 + n], want, dtype)
    assert (out[:, :8] == 7).all() and (out[:, 8 + n:] == 7).all()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,F,K,cols", [(3, 136, 64, 40), (65, 640, 256, 320), (300, 520, 96, 520), (9, 33, 21, 16), (64, 4096, 512, 2048)])
def test_product_with_squared_relu_and_fp32_sum(T, F, K, cols, dtype):
    x, w = rnd(T, K, dtype=dtype), rnd(F, K, dtype=dtype, scale=K ** -0.5)
    wide = torch.full((T, F + 16), 7.0, dtype=dtype, device=DEV)
    ops.linear(x.to(DEV), w.to(DEV), out=wide[:, 8:8 + F], relu2_cols=cols)
    close(wide[:, 8:8 + F], ref.linear(x, w, relu2_cols=cols), dtype)
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + F:] == 7).all()
    r = rnd(T, F, dtype=F32, scale=4)
    out = r.to(DEV)
    ops.linear(x.to(DEV), w.to(DEV), out=out, residual=out, out_f32=True)      # added in place
    close(out, ref.linear(x, w, r, out_f32=True), F32 if dtype == F32 else BF, 1.0 if dtype == F32 else 0.05)
    ops.workspace().check_status()


# ---- sliding-window attention -------------------------------------------------------------------------------------
WINDOWS = {
    "plain": WindowAttnSpec(heads=6, kv_heads=3, dim=24, vdim=40, scale=0.2, rot_dims=16, rope_base=1e4, rope_factor=2.0, window=21),
    "odd": WindowAttnSpec(heads=3, kv_heads=1, dim=7, vdim=5, scale=0.4, rot_dims=2, rope_base=100.0, window=1),
    "h64": WindowAttnSpec(heads=6, kv_heads=3, dim=64, vdim=64, scale=0.125, rot_dims=64, rope_base=1e5, rope_factor=4.0, window=100),
    "h128": WindowAttnSpec(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.1, rot_dims=32, rope_base=1e6, window=130),
    "wide": WindowAttnSpec(heads=16, kv_heads=1, dim=128, vdim=128, scale=0.09, rot_dims=128, rope_base=1e6, window=400),
    "none": WindowAttnSpec(heads=4, kv_heads=4, dim=64, vdim=64, scale=0.125, rot_dims=0, rope_base=1e4, window=0),
}


def _attn_case(a, lens, new, ps, dtype, seed=0):
    """Sequences of `lens` cached tokens and `new` tokens each in this step; a cache whose unused rows hold junk."""
    S, T = len(lens), sum(new)
    mb = max(-(-(l + n) // ps) for l, n in zip(lens, new))
    pages = torch.randperm(S * mb + 3, generator=torch.Generator().manual_seed(seed))[:S * mb].view(S, mb).to(torch.int32)
    cache = rnd(S * mb + 3, a.kv_heads * ps * (a.dim + a.vdim), dtype=dtype, seed=seed)
    pos = i32([p for l, n in zip(lens, new) for p in range(l, l + n)])
    sot = i32([s for s, n in enumerate(new) for _ in range(n)])
    W = sum(r for _, r in a.sections())
    row = rnd(T, W + 8, dtype=dtype, seed=seed + 1)
    table = ref.rope_cos_sin_table(int(pos.max()) + 1, a.rot_dims, a.rope_base, None, {"rope_type": "linear", "factor": a.rope_factor})
    starts = [sum(new[:s]) for s in range(S)]
    inp = dict(positions=pos, seq_of_token=sot, block_table=pages, seq_lens=i32([l + n for l, n in zip(lens, new)]), q_start=i32(starts),
               q_len=i32(new), max_q_len=max(new), ctx_hint=1024)
    return cache, row, table, inp, 1 + rnd(a.heads * a.dim, dtype=F32, scale=0.3), 1 + rnd(a.kv_heads * a.dim, dtype=F32, scale=0.3, seed=2)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("ps", [16, 64])
@pytest.mark.parametrize("name", list(WINDOWS))
def test_window_append_and_attention(name, ps, dtype):
    a = WINDOWS[name]
    nq, nk = a.heads * a.dim, a.kv_heads * a.dim
    for decode, lens, new in ((False, [0, 30, 0, 250, 16], [150, 3, 1, 140, 2]), (False, [0], [520]), (True, [0, 5, 127, 128, 129, 460, 15, 20, 21], [1] * 9)):
        cache, row, table, inp, qn, kn = _attn_case(a, lens, new, ps, dtype)
        T = row.shape[0]
        cut = lambda r: (r[:, :nq], r[:, nq:nq + nk], r[:, nq + nk:nq + nk + a.kv_heads * a.vdim])      # noqa: E731
        wc, wr = cache.clone(), row.clone()
        rp.window_append(*cut(wr), qn, kn, a, table, inp["positions"], inp["seq_of_token"], inp["block_table"], wc, ps, 1e-5)
        want = rp.window_attn_rows(cut(wr)[0], a, inp["positions"], inp["seq_of_token"], inp["block_table"], wc, ps, 0.7)
        d = {k: v.to(DEV) if isinstance(v, torch.Tensor) else v for k, v in inp.items()}
        if decode:
            d["seq_of_token"] = None
        gi = SimpleNamespace(is_prefill=not decode, **d)
        gc, gr = cache.to(DEV), row.to(DEV)
        par.window_append(*cut(gr), qn.to(DEV), kn.to(DEV), a, table.to(DEV), gi.positions, gi.seq_of_token, gi.block_table, gc, ps, 1e-5)
        close(gr, wr, dtype)
        close(gc, wc, dtype)
        gr, gc = wr.to(DEV), wc.to(DEV)        # the attention from identical inputs
        for fn in (par.window_attn, None):
            out = torch.zeros(T, a.out_width + 8, dtype=dtype, device=DEV)
            if fn is None:
                par.window_attn_rows(cut(gr)[0], a, gi.positions, gi.seq_of_token, gi.block_table, gc, ps, out[:, :a.out_width], 0.7)
            else:
                fn(cut(gr)[0], a, gi, gc, ps, out[:, :a.out_width], 0.7)
            close(out[:, :a.out_width], want, dtype)
            assert (out[:, a.out_width:] == 0).all()
    ops.workspace().check_status()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name,window", [("h128", 130), ("h128", 128), ("h64", 65), ("plain", 64), ("h128", 1)])
def test_window_edge_shows_one_key_in_and_one_out(name, window, dtype):
    """One key whose score stands out among all: seen window - 1 tokens later, gone one token after that; in a prompt and decoding,
    the key at page and tile borders."""
    a = WindowAttnSpec(**{**vars(WINDOWS[name]), "window": window})
    ps, n = 64, 400
    for p in (0, 63, 64, 127, 128, 200):
        cache, row, table, inp, _, _ = _attn_case(a, [0], [n], ps, dtype)
        keys, vals = rp._pages(cache, a.kv_heads, ps, a.dim, a.vdim)
        page, at = int(inp["block_table"][0, p // ps]), p % ps
        keys *= 0.05
        vals *= 0.05
        q = rnd(n, a.heads * a.dim, dtype=dtype, scale=0.05)
        direction = torch.nn.functional.normalize(rnd(a.dim, dtype=F32), dim=0) * (12 / a.scale) ** 0.5
        keys[page, :, at] = direction.to(dtype)
        vals[page, :, at] = 5.0
        inside, outside = p + window - 1, p + window
        for t in {inside, outside} & set(range(n)):
            q[t] = direction.repeat(a.heads).to(dtype)
        want = rp.window_attn_rows(q, a, inp["positions"], inp["seq_of_token"], inp["block_table"], cache, ps, 1.0)
        if inside < n:
            assert want[inside].float().mean() > 4.5
        if outside < n:
            assert want[outside].float().abs().max() < 1.0
        gc, gq = cache.to(DEV), q.to(DEV)
        d = {k: v.to(DEV) if isinstance(v, torch.Tensor) else v for k, v in inp.items()}
        out = torch.zeros(n, a.out_width, dtype=dtype, device=DEV)
        par.window_attn(gq, a, SimpleNamespace(is_prefill=True, **d), gc, ps, out)
        close(out, want, dtype)
        for t in {inside, outside} & set(range(n)):
            one = SimpleNamespace(is_prefill=False, positions=i32([t]).to(DEV), seq_of_token=None, block_table=d["block_table"], seq_lens=i32([t + 1]).to(DEV),
                                  ctx_hint=1024)
            out = torch.zeros(1, a.out_width, dtype=dtype, device=DEV)
            par.window_attn(gq[t:t + 1], a, one, gc, ps, out)
            close(out, want[t:t + 1], dtype)
    ops.workspace().check_status()


# ---- recurrences -----------------------------------------------------------------------------------------------------
RECS = {
    "delta": RecurrentSpec("delta", heads=4, groups=2, dim=24, vdim=40, taps=4),
    "delta_ones": RecurrentSpec("delta", heads=3, groups=3, dim=5, vdim=7, taps=1),
    "delta128": RecurrentSpec("delta", heads=4, groups=2, dim=128, vdim=128, taps=4),
    "delta64": RecurrentSpec("delta", heads=2, groups=1, dim=64, vdim=192, taps=2),
    "ssd": RecurrentSpec("ssd", heads=6, groups=3, dim=20, vdim=16, taps=4, norm_groups=2),
    "ssd128": RecurrentSpec("ssd", heads=4, groups=1, dim=128, vdim=64, taps=4),
    "ssd64": RecurrentSpec("ssd", heads=4, groups=2, dim=64, vdim=128, taps=3),
    "ssd64_pairs": RecurrentSpec("ssd", heads=12, groups=3, dim=64, vdim=64, taps=4),
    "ssd_odd_heads": RecurrentSpec("ssd", heads=3, groups=1, dim=128, vdim=64, taps=6),
    "delta_v256": RecurrentSpec("delta", heads=2, groups=2, dim=64, vdim=256, taps=3),
    "ssd_big": RecurrentSpec("ssd", heads=2, groups=1, dim=300, vdim=33, taps=2),
    "lightning": RecurrentSpec("lightning", heads=3, groups=3, dim=16, vdim=24, decay=(0.5, 0.9, 1.0)),
    "lightning128": RecurrentSpec("lightning", heads=3, groups=3, dim=128, vdim=128, decay=(0.0, 0.97, 0.9995)),
}


def rec_case(r, T, dtype, seed=0):
    H, ch = r.heads, r.conv_channels
    col, at = {}, 8
    for n, rows in r.sections():
        col[n] = at
        at += (rows + 7) // 8 * 8
    row = rnd(T, at, dtype=dtype, seed=seed)
    w = RecurrentWeights(norm=torch.ones(1))
    if r.kind == "lightning":
        w.decay = torch.tensor(r.decay)
        w.neg_decay = torch.tensor(r.decay, dtype=torch.float64).log().clamp(min=-1e30).float()
    else:
        w.neg_decay, w.dt_bias = -torch.exp(rnd(H, dtype=F32)), rnd(H, dtype=F32, seed=3) - 1.0
        w.conv = rnd(r.taps, ch, scale=r.taps ** -0.5).float()
        if r.kind == "ssd":
            w.conv_b, w.skip = rnd(ch, dtype=F32, scale=0.2), rnd(H, dtype=F32)
    return row, rec.RecColumns.of(r, col), w


def run_steps(r, row, cols, w, state, slots, plan, dev, impl=None):
    """plan: steps of [(sequence, tokens)]; every sequence reads its own rows of `row` in order. Returns outputs per sequence."""
    n_seq = len(row)
    at, outs = [0] * n_seq, [[] for _ in range(n_seq)]
    for step in plan:
        rows = torch.cat([row[s][at[s]:at[s] + k] for s, k in step]).to(dev)
        pos = i32([p for s, k in step for p in range(at[s], at[s] + k)]).to(dev)
        sl = i32([slots[s] for s, _ in step]).to(dev)
        if all(k == 1 for _, k in step) and impl is None:
            o = rec.rec_step(rows, cols, r, w, state, pos, sl)
        else:
            sot = i32([i for i, (_, k) in enumerate(step) for _ in range(k)]).to(dev)
            ks = [k for _, k in step]
            qs = i32([sum(ks[:i]) for i in range(len(ks))]).to(dev)
            o = rec.rec_chunk(rows, cols, r, w, state, pos, sl, sot, qs, i32(ks).to(dev), max(ks), impl=impl)
        i = 0
        for s, k in step:
            outs[s].append(o[i:i + k].float().cpu())
            i, at[s] = i + k, at[s] + k
    return [torch.cat(x) for x in outs]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", list(RECS))
def test_recurrence_in_portions_and_steps(name, dtype):
    """Unequal sequences in whole portions, in cut ones (down to a token), in decode steps and in both forms of the chunk kernel;
    slots that hold junk before position 0."""
    r = RECS[name]
    lens = [150, 66, 1, 64, 131]
    rows, cols, w = zip(*[rec_case(r, n, dtype, seed=10 * i) for i, n in enumerate(lens)])
    cols, w, slots = cols[0], w[0], [3, 0, 5, 1, 2]
    fresh = lambda dev: rec.RecState(*(t.normal_(generator=torch.Generator().manual_seed(1)).to(dev) if t is not None else None  # noqa: E731
                                       for t in vars(rec.RecState.make(r, 6, dtype, "cpu")).values()))
    whole = [[(s, n) for s, n in enumerate(lens)]]
    st = fresh("cpu")
    want = run_steps(r, rows, cols, w, st, slots, whole, "cpu")
    cut = [[(0, 2), (1, 3), (2, 1)], [(0, 64), (3, 1)], [(0, 17), (1, 2), (3, 40), (4, 70)], [(0, 1), (1, 1), (4, 1)], [(4, 2), (0, 60)],
           [(0, 1)], [(1, 60), (3, 23), (4, 58), (0, 5)]]
    left = [n - sum(k for step in cut for s2, k in step if s2 == s) for s, n in enumerate(lens)]
    assert left == [0, 0, 0, 0, 0], left
    steps = [[(s, 1) for s, n in enumerate(lens) if t < n] for t in range(max(lens))]
    gw = to_dev(w)
    for plan, impl in ((whole, "tc"), (whole, "scan"), (cut, "tc"), (cut, "scan"), (cut, None), (steps, None)):
        gs = fresh(DEV)
        got = run_steps(r, rows, cols, gw, gs, slots, plan, DEV, impl)
        for s in range(len(lens)):
            close(got[s], want[s], dtype, 1.0 if dtype == BF else 3.0)
            # the state is 32-bit in every form (a convolved input may round to the other neighbour in bf16)
            e = (gs.mat[slots[s]].cpu() - st.mat[slots[s]]).norm() / st.mat[slots[s]].norm()
            assert e < (3e-4 if dtype == BF else 1e-5), (plan is whole, impl, s, e)
            if gs.tail is not None:
                keep = [p % r.taps for p in range(max(0, lens[s] - r.taps + 1), lens[s])]
                assert torch.equal(gs.tail[slots[s]].cpu()[keep], st.tail[slots[s]][keep])
        unused = 4
        assert torch.equal(gs.mat[unused].cpu(), fresh("cpu").mat[unused])
    ops.workspace().check_status()


def test_step_with_padding_rows_touches_nothing():
    r = RECS["delta128"]
    row, cols, w = rec_case(r, 4, BF)
    gs = rec.RecState.make(r, 4, BF, DEV)
    gs.mat.normal_()
    before = gs.mat.clone(), gs.tail.clone()
    rec.rec_step(row.to(DEV), cols, r, to_dev(w), gs, i32([-1, 7, -1, -1]).to(DEV), i32([0, 2, 1, 3]).to(DEV))
    changed = (gs.mat != before[0]).flatten(1).any(1).cpu().tolist()
    assert changed == [False, False, True, False] and not (gs.tail[[0, 1, 3]] != before[1][[0, 1, 3]]).any()


@pytest.mark.parametrize("name", ["delta128", "ssd128", "lightning128"])
def test_long_recurrence_keeps_an_early_write(name):
    """Hundreds of tokens with little decay: what the first tokens wrote is still read at the end, by the chunk form and by steps."""
    r = RECS[name]
    n = 700
    row, cols, w = rec_case(r, n, BF, seed=5)
    w.neg_decay, w.decay = torch.full((r.heads,), -1e-4), None
    st = rec.RecState.make(r, 1, BF, "cpu")
    want = run_steps(r, [row], cols, w, st, [0], [[(0, n)]], "cpu")[0]
    lost = run_steps(r, [torch.cat([row[:60] * 0, row[60:]])], cols, w, rec.RecState.make(r, 1, BF, "cpu"), [0], [[(0, n)]], "cpu")[0]
    assert (lost[-20:] - want[-20:]).norm() > 0.02 * want[-20:].norm()
    for plan in ([[(0, n)]], [[(0, 333)], [(0, n - 333 - 30)]] + [[(0, 1)]] * 30):
        gs = rec.RecState.make(r, 1, BF, DEV)
        got = run_steps(r, [row], cols, to_dev(w), gs, [0], plan, DEV)[0]
        assert (got - want).norm() < 0.004 * want.norm()
        assert (gs.mat.cpu() - st.mat).norm() < 1e-4 * st.mat.norm()
    ops.workspace().check_status()
