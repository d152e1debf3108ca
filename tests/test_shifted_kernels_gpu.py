"""CUDA kernels of shifted pre-norm layers against their plain PyTorch references (ops/reference_parallel.py, ops/reference_prenorm.py,
ops/reference_latent.py, 32-bit math): depth average with grouped norm and token shift, append with biases, head norms and value mixing,
attention that keeps the first tokens, capped scores and sinks, the delta rule with a decay per key channel."""
import copy
import dataclasses
import math
from types import SimpleNamespace

import pytest
import torch

from derusun_models import attn, latent, rec as channel
from skein_b200 import ops
from skein_b200.models.parallel_layers import RecurrentWeights, WindowAttnWeights
from skein_b200.ops import latent as lat, parallel as par, prenorm as pre, recurrent as rec, reference as ref, reference_latent as rl
from skein_b200.ops import reference_parallel as rp, reference_prenorm as rn

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


def dev(obj):
    """A tensor, or a copy of an object of tensors, on the GPU."""
    if isinstance(obj, torch.Tensor):
        return obj.to(DEV)
    if obj is None or not hasattr(obj, "__dict__"):
        return obj
    out = copy.copy(obj)
    for k, v in vars(obj).items():
        if isinstance(v, torch.Tensor):
            setattr(out, k, v.to(DEV))
    return out


def step_inputs(lens, new, decode=False):
    """Sequences of `lens` cached tokens and `new` tokens each in this step."""
    pos = i32([p for l, n in zip(lens, new) for p in range(l, l + n)])
    sot = i32([s for s, n in enumerate(new) for _ in range(n)])
    return SimpleNamespace(positions=pos, seq_of_token=None if decode else sot, q_start=i32([sum(new[:s]) for s in range(len(new))]), q_len=i32(new),
                           max_q_len=max(new), seq_lens=i32([l + n for l, n in zip(lens, new)]), is_prefill=not decode, ctx_hint=1024)


# ---- stream ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("C,groups", [(64, 1), (320, 2), (77, 7), (512, 4), (2048, 2), (2560, 5), (4096, 1), (8192, 8), (8448, 3), (5, 5)])
def test_depth_norm(C, groups, dtype):
    """Portions of one to hundreds of tokens beside each other, decode rows with padding, several numbers of terms, slots that hold junk."""
    cases = [([0, 30, 0, 7], [5, 1, 2, 3], False), ([0, 9], [700 if C <= 2048 else 40, 333 if C <= 2048 else 3], False), ([0, 5, 127, 3], [1] * 4, True)]
    for n, (lens, new, decode) in zip((1, 6, 3), cases):
        T = sum(new)
        inp = step_inputs(lens, new, decode)
        if decode:
            inp.positions[3] = -1
        terms, w = rnd(n, T, C, dtype=F32, scale=2), rnd(n, dtype=F32)
        terms[:, 0] *= 1e-3                   # eps inside the root matters
        gain, mix, slots = 1 + rnd(C, dtype=F32, scale=0.3), rnd(C, dtype=F32, seed=1), i32([2, 0, 4, 1][:len(new)])
        state = rnd(5, C, dtype=F32, seed=2)
        for weights in (w, None) if n == 1 else (w,):
            ws, gs = state.clone(), state.to(DEV)
            wx, gx = torch.empty(T, C), torch.empty(T, C, device=DEV)
            want = rn.depth_norm(terms, weights, gain, groups, 1e-5, dtype, wx, pre.TokenShift(mix, ws), inp, slots, decode)
            got = pre.depth_norm(dev(terms), dev(weights), dev(gain), groups, 1e-5, dtype, gx, pre.TokenShift(dev(mix), gs), dev(inp), dev(slots), decode)
            live = inp.positions >= 0
            close(got.cpu()[live], want[live], dtype)
            close(gx, wx, F32)
            close(gs, ws, F32)
            unused = [s for s in range(5) if s not in slots.tolist()]
            assert torch.equal(gs.cpu()[unused], state[unused]) and (not decode or torch.equal(gs.cpu()[1], state[1]))
        close(pre.depth_norm(dev(terms), dev(w), dev(gain), groups, 1e-5, dtype), rn.depth_norm(terms, w, gain, groups, 1e-5, dtype, None, None, None, None, False), dtype)
    ops.workspace().check_status()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,F,K", [(3, 40, 64), (70, 640, 96), (300, 136, 520), (9, 33, 21), (64, 4096, 512)])
def test_clamped_pair_product(T, F, K, dtype):
    x, w = rnd(T, K, dtype=dtype), rnd(2 * F, K, dtype=dtype, scale=3 * K ** -0.5)
    for limit in (0.5, 7.0):
        close(ops.swiglu_linear(dev(x), dev(w), glu=(limit, 1.702)), ref.swiglu_linear(x, w, (limit, 1.702)), dtype, 1.0 if dtype == BF else 2.0)


@pytest.mark.parametrize("K", [8, 24, 40, 72, 104])
def test_product_over_columns_of_a_wider_matrix_reads_nothing_else(K):
    """The columns behind them, and those of the next row, hold NaN."""
    for T, F in ((5, 48), (70, 136), (200, 640)):
        wide = torch.full((T, 3 * 104), float("nan"), dtype=BF, device=DEV)
        x, w = rnd(T, K), rnd(F, K)
        wide[:, 104:104 + K] = dev(x)
        for f32 in (False, True):
            close(ops.linear(wide[:, 104:104 + K], dev(w), out_f32=f32), ref.linear(x, w, out_f32=f32), BF)


# ---- attention -----------------------------------------------------------------------------------------------------------
ATTN = {
    "plain": attn(), "odd": attn(3, 1, 7, 5, 0.5, 3, 9, 2.0), "one": attn(2, 2, 16, 16, 0.25, 1, 0, 5.0), "no_window": attn(4, 2, 24, 16, 0.3, 0, 0, 6.0),
    "h128": attn(8, 2, 128, 128, 0.09, 130, 20, 30.0), "h64": attn(6, 3, 64, 64, 0.125, 100, 17, 20.0), "wide": attn(16, 1, 128, 128, 0.2, 64, 300, 3.0),
    "keep_more": attn(4, 4, 64, 64, 0.2, 20, 200, 10.0), "uncapped": dataclasses.replace(attn(8, 2, 128, 128, 0.09, 64, 129, 30.0), softcap=0.0),
    "full_tc": attn(4, 1, 128, 128, 0.15, 0, 0, 9.0), "rotated": dataclasses.replace(attn(4, 2, 24, 16, 0.3, 33, 4, 6.0), rot_dims=8, interleaved=True),
    "halves": dataclasses.replace(attn(4, 2, 128, 128, 0.09, 70, 40, 6.0), rot_dims=64),
}


def attn_case(a, inp, ps, dtype, seed=0):
    S, T = inp.seq_lens.shape[0], inp.positions.shape[0]
    mb = -(-int(inp.seq_lens.max()) // ps)
    inp.block_table = torch.randperm(S * mb + 3, generator=torch.Generator().manual_seed(seed))[:S * mb].view(S, mb).to(torch.int32)
    cache = rnd(S * mb + 3, a.kv_heads * ps * (a.dim + a.vdim), dtype=dtype, seed=seed)
    row = rnd(T, sum(r for _, r in a.sections()) + 8, dtype=dtype, seed=seed + 1)
    w = WindowAttnWeights(q_norm=1 + rnd(a.dim, dtype=F32, scale=0.3), k_norm=1 + rnd(a.dim, dtype=F32, scale=0.3, seed=2), sinks=rnd(a.heads, dtype=F32, scale=2, seed=4),
                          q_bias=rnd(a.heads * a.dim, dtype=F32), k_bias=rnd(a.kv_heads * a.dim, dtype=F32), v_bias=rnd(a.kv_heads * a.vdim, dtype=F32),
                          vmix=torch.tensor([0.3]))
    table = ref.rope_cos_sin_table(mb * ps, a.rot_dims, 1e4, None) if a.rot_dims else None
    return cache, row, w, table


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("ps", [16, 64])
@pytest.mark.parametrize("name", list(ATTN))
def test_append_and_attention(name, ps, dtype):
    a = ATTN[name]
    nq, nk, nv = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim
    cut = lambda r: (r[:, :nq], r[:, nq:nq + nk], r[:, nq + nk:nq + nk + nv])      # noqa: E731
    for decode, lens, new in ((False, [0, 30, 0, 250, 16], [150, 3, 1, 140, 2]), (False, [0], [520]), (False, [500], [40]),
                              (True, [0, 5, 127, 128, 129, 460, 15, 20, 21], [1] * 9), (True, [1500, 3], [1, 1])):
        inp = step_inputs(lens, new, decode)
        cache, row, w, table = attn_case(a, inp, ps, dtype)
        T = row.shape[0]
        for mode in ("none", "keep", "mix"):
            first = rnd(T, nv, dtype=dtype, seed=9)
            wm, gm = (None, None) if mode == "none" else (par.ValueMix(first.clone(), mode == "keep"), par.ValueMix(first.to(DEV), mode == "keep"))
            wc, wr, gc, gr = cache.clone(), row.clone(), cache.to(DEV), row.to(DEV)
            args = lambda d, x: (inp.positions.to(d), None if decode else inp.seq_of_token.to(d), inp.block_table.to(d), x, ps, 1e-5)      # noqa: E731
            rp.head_append(*cut(wr), a, table, *args("cpu", wc), w, wm)
            par.head_append(*cut(gr), a, dev(table), *args(DEV, gc), dev(w), gm)
            close(gr, wr, dtype)
            close(gc, wc, dtype)
            if mode != "none":
                close(gm.v_first, wm.v_first, dtype)
        mix = par.HeadMix(eps=1e-5, sinks=w.sinks)
        want = rp.window_attn_rows(cut(wr)[0], a, inp.positions, inp.seq_of_token, inp.block_table, wc, ps, 0.7, mix)
        gr, gc, gi = wr.to(DEV), wc.to(DEV), dev(inp)        # the attention from identical inputs
        for rows in (False, True):
            out = torch.zeros(T, a.out_width + 8, dtype=dtype, device=DEV)
            if rows:
                par.window_attn_rows(cut(gr)[0], a, gi.positions, gi.seq_of_token, gi.block_table, gc, ps, out[:, :a.out_width], 0.7, dev(mix))
            else:
                par.window_attn(cut(gr)[0], a, gi, gc, ps, out[:, :a.out_width], 0.7, dev(mix))
            close(out[:, :a.out_width], want, dtype)
            assert (out[:, a.out_width:] == 0).all()
    ops.workspace().check_status()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,window,keep", [(128, 130, 20), (64, 65, 64), (28, 40, 17), (128, 20, 150), (64, 128, 129)])
def test_one_key_inside_and_outside_of_what_is_kept(dim, window, keep, dtype):
    """One key whose score stands out among all: a kept one is seen from everywhere, the next one only inside the window."""
    a = attn(4, 2, dim, dim, 0.1, window, keep, 40.0)
    ps, n = 64, 500
    for p in sorted({0, keep - 1, keep, keep + 1, 127, 128}):
        inp = step_inputs([0], [n])
        cache, _, w, _ = attn_case(a, inp, ps, dtype)
        keys, vals = rp._pages(cache, a.kv_heads, ps, dim, dim)
        keys *= 0.05
        vals *= 0.05
        q = rnd(n, a.heads * dim, dtype=dtype, scale=0.05)
        direction = torch.nn.functional.normalize(rnd(dim, dtype=F32), dim=0) * (30 / a.scale) ** 0.5
        page, at = int(inp.block_table[0, p // ps]), p % ps
        keys[page, :, at], vals[page, :, at] = direction.to(dtype), 5.0
        ask = [t for t in (p, p + window - 1, p + window, p + window + 1, 380, n - 1) if t < n]
        q[ask] = direction.repeat(a.heads).to(dtype)
        mix = par.HeadMix(sinks=w.sinks)
        want = rp.window_attn_rows(q, a, inp.positions, inp.seq_of_token, inp.block_table, cache, ps, 1.0, mix)
        for t in ask:
            assert (want[t].float().mean() > 4.5) == (p < keep or t - p < window), (p, t)
        gc, gq, gi = cache.to(DEV), q.to(DEV), dev(inp)
        out = torch.zeros(n, a.out_width, dtype=dtype, device=DEV)
        par.window_attn(gq, a, gi, gc, ps, out, mix=dev(mix))
        close(out, want, dtype)
        for t in ask:
            one = SimpleNamespace(is_prefill=False, positions=i32([t]).to(DEV), seq_of_token=None, block_table=gi.block_table, seq_lens=i32([t + 1]).to(DEV), ctx_hint=4096)
            out = torch.zeros(1, a.out_width, dtype=dtype, device=DEV)
            par.window_attn(gq[t:t + 1], a, one, gc, ps, out, mix=dev(mix))
            close(out, want[t:t + 1], dtype)
    ops.workspace().check_status()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m", [latent(), latent(16, 64, 64, 128, 512, 1e5, 0.1), latent(32, 128, 64, 128, 256, 1e5, 0.08), latent(5, 6, 2, 3, 11, 100.0, 0.6)])
def test_latent_rows_with_sinks(m, dtype):
    """Single rows over the cache (decode, splits of one long sequence) and, where it applies, expanded keys; sinks from negligible to dominant."""
    H, K, ps = m.heads, m.kv_rank, 64
    lens = [1, 64, 65, 700, 3000]
    mb = -(-max(lens) // ps)
    bt = torch.randperm(len(lens) * mb, generator=torch.Generator().manual_seed(0)).view(len(lens), mb).to(torch.int32)
    cache, table = rnd(len(lens) * mb, ps, m.cache_width, dtype=dtype), ref.rope_cos_sin_table(mb * ps, m.rot_dim, m.rope_base, None)
    sinks = torch.linspace(-20, 12, H)
    for pick in (list(range(len(lens))), [3], [4]):
        T, pos = len(pick), i32([lens[s] - 1 for s in pick])
        q_abs, q = rnd(T, H * K, dtype=dtype, scale=0.5), rnd(T, H * m.head_size, dtype=dtype, scale=0.5)
        want = rl.latent_attention_rows(q_abs.view(T, H, K), q.view(T, H, -1), m.dim, m.rot_dim, m.scale, table, pos, None, bt[pick], cache, sinks)
        got = lat.latent_attn_rows(dev(q_abs), dev(q), H, m.dim, m.rot_dim, m.scale, dev(table), dev(pos), None, dev(bt[pick]), dev(cache), max(lens), sinks=dev(sinks))
        close(got, want.reshape(T, -1), dtype)
    if not lat.expanded_ok(dtype, m.dim, m.rot_dim, m.vdim, K, torch.device(DEV)):
        return
    T, kv_len, q_len = 130, [300, 129], [100, 30]
    q, dense, kv = rnd(T, H * m.head_size, scale=0.5), rnd(sum(kv_len), m.cache_width), rnd(sum(kv_len), H * (m.dim + m.vdim))
    got = lat.latent_attn_prefill(dev(q), H, m.dim, m.rot_dim, m.vdim, m.scale, dev(dense), dev(kv), i32([0, 100]).to(DEV), i32(q_len).to(DEV), i32(kv_len).to(DEV),
                                  i32([0, 300]).to(DEV), 100, sinks=dev(sinks))
    for s, (r0, c0) in enumerate(((0, 0), (100, 300))):
        k = kv[c0:c0 + kv_len[s], :H * m.dim].float().view(-1, H, m.dim)
        v = kv[c0:c0 + kv_len[s], H * m.dim:].float().view(-1, H, m.vdim)
        qq = q[r0:r0 + q_len[s]].float().view(-1, H, m.head_size)
        sc = torch.einsum("qhd,khd->hqk", qq[..., :m.dim], k) + torch.einsum("qhd,kd->hqk", qq[..., m.dim:], dense[c0:c0 + kv_len[s], K:].float())
        i, j = torch.arange(q_len[s])[:, None] + kv_len[s] - q_len[s], torch.arange(kv_len[s])[None]
        sc = torch.cat([(sc * m.scale).masked_fill(j > i, -math.inf), sinks[:, None, None].expand(H, q_len[s], 1)], dim=-1)
        want = torch.einsum("hqk,khv->qhv", torch.softmax(sc, -1)[..., :-1], v).reshape(q_len[s], -1)
        close(got[r0:r0 + q_len[s]], want, BF)
    ops.workspace().check_status()


# ---- the recurrence ------------------------------------------------------------------------------------------------------
RECS = {
    "plain": channel(4, 2, 24, 40, 4), "ones": channel(3, 3, 5, 7, 1), "bulk": channel(4, 4, 32, 64, 3), "d128": channel(4, 2, 128, 128, 4),
    "d64": channel(2, 1, 64, 192, 2), "d64_v64": channel(6, 3, 64, 64, 6), "d128_v64": channel(4, 4, 128, 64, 4), "d64_v256": channel(2, 2, 64, 256, 3),
    "big": channel(2, 1, 300, 33, 2),
}


def rec_case(r, T, dtype, seed=0, strong=0.0):
    """strong: how far beyond what the factored form of a block takes some channels decay."""
    H, ch = r.heads, r.conv_channels
    col, at = {}, 8
    for n, rows in r.sections():
        col[n] = at
        at += (rows + 7) // 8 * 8
    row = rnd(T, at, dtype=dtype, seed=seed)
    w = RecurrentWeights(norm=torch.ones(1), neg_decay=-torch.exp(rnd(H, dtype=F32)), dt_bias=rnd(H * r.dim, dtype=F32, seed=3) - 2.0,
                         conv=rnd(r.taps, ch, scale=r.taps ** -0.5).float())
    step = rnd(T, H * r.dim, dtype=F32, seed=seed + 5)
    step[:, ::7] += strong
    return row, step, rec.RecColumns.of(r, col), w


def run_steps(r, row, step, cols, w, state, slots, plan, device, impl=None):
    """plan: steps of [(sequence, tokens)]; every sequence reads its own rows in order. Returns outputs per sequence."""
    at, outs = [0] * len(row), [[] for _ in row]
    for part in plan:
        rows, a = (torch.cat([x[s][at[s]:at[s] + k] for s, k in part]).to(device) for x in (row, step))
        pos = i32([p for s, k in part for p in range(at[s], at[s] + k)]).to(device)
        sl = i32([slots[s] for s, _ in part]).to(device)
        if all(k == 1 for _, k in part) and impl is None:
            o = rec.rec_step(rows, cols, r, w, state, pos, sl, step=a)
        else:
            ks = [k for _, k in part]
            sot, qs = i32([i for i, k in enumerate(ks) for _ in range(k)]).to(device), i32([sum(ks[:i]) for i in range(len(ks))]).to(device)
            o = rec.rec_chunk(rows, cols, r, w, state, pos, sl, sot, qs, i32(ks).to(device), max(ks), impl=impl, step=a)
        i = 0
        for s, k in part:
            outs[s].append(o[i:i + k].float().cpu())
            i, at[s] = i + k, at[s] + k
    return [torch.cat(x) for x in outs]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name,strong", [(n, 0.0) for n in RECS] + [("d128", 12.0), ("d64_v64", 60.0), ("plain", 60.0)])
def test_recurrence_in_portions_and_steps(name, strong, dtype):
    """Unequal sequences in whole portions, in cut ones (down to a token), in decode steps and in both forms of the chunk kernel; slots that
    hold junk before position 0; decays from slow ones to those that empty a row of the state at once."""
    r = RECS[name]
    lens = [150, 66, 1, 64, 131]
    rows, steps_in, cols, w = zip(*[rec_case(r, n, dtype, seed=10 * i, strong=strong) for i, n in enumerate(lens)])
    cols, w, slots = cols[0], w[0], [3, 0, 5, 1, 2]
    fresh = lambda d: rec.RecState(*(t.normal_(generator=torch.Generator().manual_seed(1)).to(d) if t is not None else None  # noqa: E731
                                     for t in vars(rec.RecState.make(r, 6, dtype, "cpu")).values()))
    whole = [[(s, n) for s, n in enumerate(lens)]]
    st = fresh("cpu")
    want = run_steps(r, rows, steps_in, cols, w, st, slots, whole, "cpu")
    cut = [[(0, 2), (1, 3), (2, 1)], [(0, 64), (3, 1)], [(0, 17), (1, 2), (3, 40), (4, 70)], [(0, 1), (1, 1), (4, 1)], [(4, 2), (0, 60)],
           [(0, 1)], [(1, 60), (3, 23), (4, 58), (0, 5)]]
    single = [[(s, 1) for s, n in enumerate(lens) if t < n] for t in range(max(lens))]
    gw = dev(w)
    for plan, impl in ((whole, "tc"), (whole, "scan"), (cut, "tc"), (cut, "scan"), (cut, None), (single, None)):
        gs = fresh(DEV)
        got = run_steps(r, rows, steps_in, cols, gw, gs, slots, plan, DEV, impl)
        for s in range(len(lens)):
            close(got[s], want[s], dtype, 1.0 if dtype == BF else 3.0)
            # the state is 32-bit in every form (a convolved input may round to the other neighbour in bf16)
            e = (gs.mat[slots[s]].cpu() - st.mat[slots[s]]).norm() / st.mat[slots[s]].norm()
            assert e < (3e-4 if dtype == BF else 1e-5), (plan is whole, impl, s, e)
            if gs.tail is not None:
                keep = [p % r.taps for p in range(max(0, lens[s] - r.taps + 1), lens[s])]
                assert torch.equal(gs.tail[slots[s]].cpu()[keep], st.tail[slots[s]][keep])
        assert torch.equal(gs.mat[4].cpu(), fresh("cpu").mat[4])          # nobody's slot
    ops.workspace().check_status()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", ["d128", "d64_v256", "bulk"])
def test_step_with_gate_and_padding_rows(name, dtype):
    """Many rows (several heads per CTA), head norm and gate inside the step; padding rows touch nothing."""
    r = RECS[name]
    B = 180
    row, step, cols, w = rec_case(r, B, dtype)
    w.norm = 1 + rnd(r.vdim, dtype=F32, scale=0.3)
    state, slots = rec.RecState.make(r, B, dtype, "cpu"), torch.randperm(B, generator=torch.Generator().manual_seed(2)).to(torch.int32)
    state.mat.normal_(generator=torch.Generator().manual_seed(3))
    pos = i32([-1 if i % 9 == 4 else i % 5 for i in range(B)])
    gs, z = dev(state), rnd(B, r.out_width + 8, dtype=dtype, seed=4)
    want = rec.rec_step(row, cols, r, w, state, pos, slots, step=step)
    want = rp.gated_norm(want, z[:, 8:], w.norm, r.heads, 1e-5, False, False, 0.9)
    out = torch.full((B, r.out_width + 8), 7.0, dtype=dtype, device=DEV)
    gate = rec.HeadGate(dev(w.norm), dev(z)[:, 8:], out[:, :r.out_width], 1e-5, 0.9, sigmoid=True)
    assert rec.rec_step(dev(row), cols, r, dev(w), gs, dev(pos), dev(slots), gate=gate, step=dev(step)) is None
    live = pos >= 0
    close(out.cpu()[live][:, :r.out_width], want[live], dtype)
    assert (out.cpu()[~live] == 7).all() and (out[:, r.out_width:] == 7).all()
    close(gs.mat, state.mat, F32, 1.0 if dtype == F32 else 30.0)
    assert torch.equal(gs.mat.cpu()[slots[~live].long()], state.mat[slots[~live].long()])


@pytest.mark.parametrize("name", ["d128", "d64_v64"])
def test_long_recurrence_keeps_an_early_write(name):
    """Hundreds of tokens with little decay: what the first tokens wrote is still read at the end, by the chunk form and by steps."""
    r = RECS[name]
    n = 700
    row, step, cols, w = rec_case(r, n, BF, seed=5)
    w.neg_decay = torch.full((r.heads,), -1e-3)
    st = rec.RecState.make(r, 1, BF, "cpu")
    want = run_steps(r, [row], [step], cols, w, st, [0], [[(0, n)]], "cpu")[0]
    lost = run_steps(r, [torch.cat([row[:60] * 0, row[60:]])], [step], cols, w, rec.RecState.make(r, 1, BF, "cpu"), [0], [[(0, n)]], "cpu")[0]
    assert (lost[-20:] - want[-20:]).norm() > 0.01 * want[-20:].norm()
    for plan in ([[(0, n)]], [[(0, 333)], [(0, n - 333 - 30)]] + [[(0, 1)]] * 30):
        gs = rec.RecState.make(r, 1, BF, DEV)
        got = run_steps(r, [row], [step], cols, dev(w), gs, [0], plan, DEV)[0]
        assert (got - want).norm() < 0.004 * want.norm()
        assert (gs.mat.cpu() - st.mat).norm() < 1e-4 * st.mat.norm()
    ops.workspace().check_status()
