"""CUDA kernels of post-norm latent-attention blocks against their plain PyTorch references (ops/reference_latent.py, fp32 math)."""
import math

import pytest
import torch

from skein_b200 import ops
from skein_b200.ops import latent as lat, reference as ref, reference_latent as rl

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def rnd(*shape, dtype=BF, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def close(got, want, dtype, mul=1.0):
    got, want = got.float().cpu(), want.float()
    tol = (2e-2 if dtype == BF else 2e-5) * mul
    err = (got - want).abs().max().item()
    ref_ = max(want.abs().max().item(), 1e-3)
    assert math.isfinite(err) and err <= tol * ref_, (err, ref_)


def i32(x):
    return torch.tensor(x, dtype=torch.int32)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,F,K", [(5, 40, 24), (70, 300, 200), (33, 130, 77), (257, 64, 520)])
def test_linear_any_row_length(T, F, K, dtype):
    x, w = rnd(T, K, dtype=dtype), rnd(F, K, dtype=dtype, scale=K ** -0.5)
    want = x.float() @ w.float().t()
    close(ops.linear(x.to(DEV), w.to(DEV)), want, dtype)
    wide = torch.cat([x, torch.full((T, 8), 3.0, dtype=dtype)], dim=1).to(DEV)      # the first K columns of wider rows
    close(ops.linear(wide[:, :K], w.to(DEV), out_f32=True), want, F32 if dtype == F32 else BF)
    ops.workspace().check_status()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,F,K,cols,gated", [(3, 80, 48, 64, False), (70, 16, 24, 40, True), (5, 40, 80, 80, True), (4, 33, 21, 30, True),
                                              (16, 512, 128, 192, False), (16, 128, 512, 512, True)])
@pytest.mark.parametrize("T", [1, 37])
def test_head_linear(H, F, K, cols, gated, T, dtype):
    x, w = rnd(T, H * cols, dtype=dtype), rnd(H, F, K, dtype=dtype, scale=K ** -0.5)
    gates = rnd(T, H * F + 16, dtype=dtype)
    g = gates[:, 8:8 + H * F] if gated else None
    got = lat.head_linear(x.to(DEV), cols, w.to(DEV), gates.to(DEV)[:, 8:8 + H * F] if gated else None)
    close(got, rl.head_linear(x, cols, w, g), dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("E,Fe,C", [(6, 72, 192), (70, 24, 64), (3, 128, 256), (4, 21, 35)])
def test_grouped_clamped_unit(E, Fe, C, dtype):
    counts = i32([(e * 7) % 5 for e in range(E)])
    offsets = torch.cat([torch.zeros(1, dtype=torch.int32), torch.cumsum(counts, 0).to(torch.int32)])
    n = int(offsets[-1])
    xs, w = rnd(n, C, dtype=dtype, scale=2.0), rnd(E, 2 * Fe, C, dtype=dtype, scale=C ** -0.5)
    want = ref.grouped_linear(xs, w, counts, offsets, True, (1.25, 1.702))
    got = ops.grouped_linear(xs.to(DEV), w.to(DEV), counts.to(DEV), offsets.to(DEV), swiglu=True, glu=(1.25, 1.702))
    close(got, want, dtype)
    assert want.float().max() > 1.5       # the limit is reached


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("F", [160, 77, 6000, 20000])
def test_poly_norm(F, dtype):
    z, act = rnd(9, F, dtype=dtype, scale=1.7), torch.tensor([0.4, -0.6, 0.9, 0.3])
    close(lat.poly_norm(z.to(DEV), act.to(DEV), 1e-5), rl.poly_norm(z, act, 1e-5), dtype)
    tiny = z * 1e-3                        # eps inside the root matters
    close(lat.poly_norm(tiny.to(DEV), act.to(DEV), 1e-5), rl.poly_norm(tiny, act, 1e-5), dtype)


@pytest.mark.parametrize("E,top,groups,keep", [(20, 4, 5, 3), (8, 2, 4, 1), (64, 6, 8, 3), (256, 8, 8, 4), (5, 5, 1, 1), (40, 1, 20, 1)])
def test_grouped_selection_and_layout(E, top, groups, keep):
    T, C = 301, 64
    x, w = rnd(T, C, dtype=F32), rnd(E, C, dtype=F32)
    ids, wt, *_ = lat.route_grouped(x, w, top, groups, keep)
    out = lat.route_grouped(x.to(DEV), w.to(DEV), top, groups, keep)
    assert torch.equal(out[0].cpu(), ids)
    close(out[1], wt, F32)
    counts, offsets, row_of, src = ref.router_plan(ids, E)
    for a, b in zip(out[2:6], (counts, offsets, row_of, src)):
        assert torch.equal(a.cpu(), b)
    assert torch.equal(out[6].cpu(), x[src.long()])


def paged(S, n_pages, ps, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randperm(S * n_pages, generator=g).view(S, n_pages).to(torch.int32)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("C,taps,ps", [(192, 4, 16), (77, 3, 2), (64, 1, 8), (128, 7, 4)])
def test_conv_state_lives_with_pages(C, taps, ps, dtype):
    """Chunks of all sizes, then decode rows (both kernels that run the convolution there), against one pass over the sequence."""
    S, n = 2, 21
    x, w = rnd(S, n, C, dtype=F32), rnd(taps, C, dtype=F32, scale=0.5)
    bt = paged(S, -(-n // ps), ps)
    full = torch.stack([rl.conv_input(x[s], w, None, torch.arange(n), torch.zeros(n).long(), torch.zeros(1).long(), bt[s:s + 1], ps, dtype, False)
                        for s in range(S)])
    R = min(taps, ps) if taps > 1 else 0
    tail = torch.zeros(bt.numel(), R, C, dtype=dtype, device=DEV) if R else None
    cs = lat.ConvState(w.to(DEV), tail, ps)
    btd = bt.to(DEV)
    at = 0
    for step in (5, 1, 2, 7):
        rows = torch.cat([x[s, at:at + step] for s in range(S)]).to(DEV)
        pos = i32(list(range(at, at + step)) * S).to(DEV)
        sot, qs = i32([s for s in range(S) for _ in range(step)]).to(DEV), i32([s * step for s in range(S)]).to(DEV)
        h = lat.conv_input(rows, cs, pos, btd, sot, qs, dtype)
        proj = torch.zeros(S * step, 24, dtype=dtype, device=DEV)
        lat.latent_append(proj, 0, None, torch.ones(16, device=DEV), 8, torch.zeros(64, 4, 2, device=DEV), pos, sot, btd,
                          torch.zeros(bt.numel(), ps, 24, dtype=dtype, device=DEV), 1e-5, rows, tail, i32([at + step] * S).to(DEV), taps)
        for s in range(S):
            close(h[s * step:(s + 1) * step], full[s, at:at + step], dtype)
        at += step
    one = torch.ones(1, device=DEV)
    while at < n:
        pos = i32([at] * S).to(DEV)
        rows = x[:, at].to(DEV).contiguous()
        if at % 2:
            h = lat.conv_input(rows, cs, pos, btd, dtype=dtype, write_tail=True)
            close(h, full[:, at], dtype)
        else:       # fused behind a norm: alpha 1, gain = the row's own root mean square keeps the row as it is
            for _ in range(2):      # a decode step may run twice
                rms = rows.pow(2).mean(-1).sqrt()
                xo, h = lat.post_norm(rows / rms[:, None], None, 1.0, one, 0.0, dtype=dtype, conv=cs, positions=pos, block_table=btd)
                want = torch.stack([rl.conv_input(x[s] / rms[s].cpu(), w, None, torch.arange(n), torch.zeros(n).long(), torch.zeros(1).long(),
                                                  bt[s:s + 1], ps, dtype, False)[at] for s in range(S)]) if taps == 1 else None
                if want is not None:
                    close(h, want, dtype)
            lat.conv_input(rows, cs, pos, btd, dtype=dtype, write_tail=True)      # the true input of this position
        at += 1
    ops.workspace().check_status()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("C", [192, 35, 4096, 13000])
def test_post_norm(C, dtype):
    B, k, n = 7, 3, 30
    x, y = rnd(B, C, dtype=F32), rnd(n, C, dtype=dtype)
    idx, w = torch.randint(0, n, (B, k), dtype=torch.int32), torch.rand(B, k)
    g, fg = torch.tensor([1.7]), torch.tensor([0.6])
    want = rl.post_norm(x, y, 3.0, g, 1e-3, idx, w)
    xo, act = lat.post_norm(x.to(DEV), y.to(DEV), 3.0, g.to(DEV), 1e-3, idx.to(DEV), w.to(DEV), dtype)
    close(xo, want, F32, 4)
    close(act, want, dtype, 4)
    want = rl.post_norm(x, y[:B], 0.5, g, 1e-3)
    xo, act = lat.post_norm(x.to(DEV), y[:B].contiguous().to(DEV), 0.5, g.to(DEV), 1e-3, dtype=dtype, final_gain=fg.to(DEV))
    close(xo, want, F32, 4)
    close(act, rl.post_norm(want, None, 1.0, fg, 1e-3), dtype, 4)


@pytest.mark.parametrize("T,C,E,top,groups,keep", [(5, 192, 18, 4, 6, 3), (64, 1024, 64, 6, 8, 3), (148, 256, 8, 2, 1, 1), (33, 4096, 40, 8, 10, 4)])
def test_post_norm_route_equals_separate_kernels(T, C, E, top, groups, keep):
    x, y, wg = rnd(T, C, dtype=F32).to(DEV), rnd(T, C).to(DEV), rnd(E, C, scale=C ** -0.5).to(DEV)
    g = torch.tensor([1.3], device=DEV)
    xo, act = lat.post_norm(x, y, 2.0, g, 1e-5)
    sep = lat.route_grouped(act, wg, top, groups, keep)
    for _ in range(2):       # the grid-wide arrival counter re-arms itself
        out = lat.post_norm_route(x, y, 2.0, g, 1e-5, wg, top, groups, keep)
        assert torch.allclose(out[0], xo, atol=1e-5)
        same = (out[1] == sep[0]).all(dim=1)
        assert same.float().mean() > 0.97      # a near tie may fall the other way (summation order of the logits)
        close(out[2][same], sep[1][same].cpu(), F32, 50)
        if bool(same.all()):
            for a, b in zip(out[3:7], sep[2:6]):
                assert torch.equal(a, b)
            close(out[7], sep[6].cpu(), BF)      # rows may differ in the last bit: the mean square is summed in another order
    ops.workspace().check_status()


# heads, dim, rot, kv_rank, page size: every head-tile and column-tile variant of the decode kernel, and sizes it does not take
SIZES = [(4, 48, 32, 96, 64), (7, 64, 32, 128, 64), (3, 48, 16, 80, 16), (16, 128, 64, 512, 64), (32, 128, 64, 512, 64), (40, 64, 32, 256, 32),
         (64, 128, 64, 512, 64), (70, 16, 16, 32, 128), (20, 24, 48, 320, 64), (5, 20, 6, 36, 8), (2, 33, 10, 24, 16)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,D,rot,K,ps", SIZES)
def test_rows_over_the_cache(H, D, rot, K, ps, dtype):
    """Lengths around tile and page borders, a padding row, several split counts. One row's query is aligned with one far key of
    its own so that losing that key shows."""
    lens = [1, 2, 63, 64, 65, 129, 0, 200, ps, ps + 1]
    T, n_pages = len(lens), -(-201 // ps)
    bt = paged(T, n_pages, ps)
    cache = rnd(bt.numel(), ps, K + rot, dtype=dtype, scale=0.3)
    cs = ref.rope_cos_sin_table(256, rot, 5000.0)
    q = rnd(T, H * (D + rot) + 8, dtype=dtype)
    q_abs = rnd(T, H * K, dtype=dtype, scale=0.5)
    for t, n in enumerate(lens):       # head 0 of every row asks for its oldest key
        if n:
            key = cache[bt[t, 0].long(), 0].float()
            q_abs[t, :K] = (key[:K] * 40).to(dtype)
    pos = i32([n - 1 for n in lens])
    want = rl.latent_attention_rows(q_abs.view(T, H, K), q[:, :H * (D + rot)].reshape(T, H, D + rot), D, rot, 0.2, cs, pos, None, bt, cache)
    args = (H, D, rot, 0.2, cs.to(DEV), pos.to(DEV), None, bt.to(DEV), cache.to(DEV))
    for splits in (None, 1, 3, 8):
        close(lat.latent_attn_rows(q_abs.to(DEV), q.to(DEV), *args, splits=splits), want.reshape(T, H * K), dtype)
    ops.workspace().check_status()


def test_rows_of_a_portion_share_their_sequence():
    H, D, rot, K, ps = 4, 48, 16, 96, 16
    bt = paged(2, 4, ps)
    cache = rnd(bt.numel(), ps, K + rot, scale=0.3)
    cs = ref.rope_cos_sin_table(64, rot, 1e4)
    sot, pos = i32([0, 0, 0, 1, 1]), i32([14, 15, 16, 40, 41])
    q, q_abs = rnd(5, H * (D + rot)), rnd(5, H * K)
    want = rl.latent_attention_rows(q_abs.view(5, H, K), q.view(5, H, D + rot), D, rot, 0.1, cs, pos, sot, bt, cache)
    got = lat.latent_attn_rows(q_abs.to(DEV), q.to(DEV), H, D, rot, 0.1, cs.to(DEV), pos.to(DEV), sot.to(DEV), bt.to(DEV), cache.to(DEV))
    close(got, want.reshape(5, -1), BF)


def plain_prefill(q, dense, kv, H, D, rot, V, scale, q_len, kv_len, gate):
    out, qa, ca = [], 0, 0
    for ql, kl in zip(q_len, kv_len):
        qs = q[qa:qa + ql, :H * (D + rot)].float().view(ql, H, D + rot)
        k = kv[ca:ca + kl, :H * D].float().view(kl, H, D)
        v = kv[ca:ca + kl, H * D:].float().view(kl, H, V)
        kr = dense[ca:ca + kl, -rot:].float()
        s = (torch.einsum("qhd,khd->hqk", qs[..., :D], k) + torch.einsum("qhr,kr->hqk", qs[..., D:], kr)) * scale
        vis = torch.arange(kl)[None, :] <= torch.arange(kl - ql, kl)[:, None]
        o = torch.einsum("hqk,khv->qhv", torch.softmax(s.masked_fill(~vis, -math.inf), -1), v).reshape(ql, H * V)
        out.append(o)
        qa, ca = qa + ql, ca + kl
    out = torch.cat(out)
    return out if gate is None else out * torch.sigmoid(gate.float())


@pytest.mark.parametrize("H,D,rot,V,K,gated", [(4, 32, 16, 48, 96, True), (2, 128, 64, 128, 512, False), (3, 48, 16, 40, 80, True),
                                               (5, 24, 32, 72, 96, False), (1, 72, 8, 8, 16, True)])
@pytest.mark.parametrize("q_len,kv_len", [([1], [1]), ([127, 40], [127, 300]), ([128, 129, 3], [128, 129, 260]), ([300, 257], [300, 700]), ([513], [641])])
def test_expanded_prefill(H, D, rot, V, K, gated, q_len, kv_len):
    T, ctx = sum(q_len), sum(kv_len)
    q, dense, kv = rnd(T, H * (D + rot) + 8), rnd(ctx, K + rot), rnd(ctx, H * (D + V))
    # the last query of every chunk asks for its sequence's first key, and the first query for the key just before its own
    qa = ca = 0
    for ql, kl in zip(q_len, kv_len):
        q[qa + ql - 1, :D] = (kv[ca, :D].float() * 6).to(BF)
        q[qa, :D] = (kv[ca + max(kl - ql - 1, 0), :D].float() * 6).to(BF)
        qa, ca = qa + ql, ca + kl
    gates = rnd(T, H * V + 8)
    gate = gates[:, :H * V] if gated else None
    starts = i32([sum(kv_len[:i]) for i in range(len(kv_len))]).to(DEV)
    qs = i32([sum(q_len[:i]) for i in range(len(q_len))]).to(DEV)
    got = lat.latent_attn_prefill(q.to(DEV), H, D, rot, V, 0.15, dense.to(DEV), kv.to(DEV), qs, i32(q_len).to(DEV), i32(kv_len).to(DEV), starts,
                                  max(q_len), gates.to(DEV)[:, :H * V] if gated else None)
    ops.workspace().check_status()
    close(got, plain_prefill(q, dense, kv, H, D, rot, V, 0.15, q_len, kv_len, gate), BF)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("q_rank,K,rot,ps", [(0, 72, 24, 64), (56, 80, 16, 16), (33, 21, 6, 3)])
def test_append_gather_rotate(q_rank, K, rot, ps, dtype):
    lens, cached = [5, 70, 1], [0, 9, 130]
    kv_len = [a + b for a, b in zip(lens, cached)]
    S, T = len(lens), sum(lens)
    bt = paged(S, -(-max(kv_len) // ps), ps)
    off = (q_rank + 7) // 8 * 8
    proj = rnd(T, off + K + rot + 8, dtype=dtype)
    cache = rnd(bt.numel(), ps, K + rot, dtype=dtype)
    cs = ref.rope_cos_sin_table(256, rot, 1e4)
    qn, kn = (torch.rand(q_rank) + 0.5 if q_rank else None), torch.rand(K) + 0.5
    pos = i32([c + i for c, n in zip(cached, lens) for i in range(n)])
    sot = i32([s for s, n in enumerate(lens) for _ in range(n)])
    d = lambda t: None if t is None else t.to(DEV)      # noqa: E731
    cg = cache.to(DEV)
    starts = i32([sum(kv_len[:i]) for i in range(S)]).to(DEV)
    dense = torch.full((sum(kv_len), K + rot), float("nan"), dtype=dtype, device=DEV)
    lat.latent_gather(cg, d(bt), i32(kv_len).to(DEV), i32(lens).to(DEV), starts, dense, max(cached))
    cq = lat.latent_append(d(proj), off, d(qn), d(kn), rot, d(cs), d(pos), d(sot), d(bt), cg, 1e-4, dense=dense, dense_start=starts)
    want = rl.latent_append(proj, off, qn, kn, rot, cs, pos, sot, bt, cache, 1e-4, None, None, None, 1)
    close(cg, cache, dtype)
    if q_rank:
        close(cq, want, dtype)
    rows = torch.cat([cache[bt[s, torch.arange(n) // ps].long(), torch.arange(n) % ps] for s, n in enumerate(kv_len)])
    close(dense, rows, dtype)
    q = rnd(T, 3 * (8 + rot) + 4, dtype=dtype)
    qg = q.to(DEV)
    lat.rope_rows(qg, 3, 8, rot, d(cs), d(pos))
    want = q.clone()
    for h in range(3):
        c = h * (8 + rot) + 8
        want[:, c:c + rot] = rl.rotate_pairs(q[:, c:c + rot], cs[pos.long()]).to(dtype)
    close(qg, want, dtype)
