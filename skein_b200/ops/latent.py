"""Operators of post-norm blocks of latent attention: fp32 residual stream, input convolution, latent cache, clamped gated
experts behind a group-limited router.

CUDA tensors run the kernels in csrc/kernels (postnorm.cu, latent.cu, attn_latent_decode.cu, attn_latent_prefill.cu,
router.cu and the GEMMs); CPU tensors run ops/reference_latent.py. Activations are bf16, or fp32 when the model's weights are
(a model run in 32-bit): every operator takes both.
"""
from __future__ import annotations

import os
from dataclasses import dataclass

import torch

from . import _lib, functional as F, reference as ref, reference_latent as rl

MAX_ROUTE_E = 256


def _fp32(t) -> int:
    return 1 if t.dtype == torch.float32 else 0


@dataclass
class ConvState:
    """What the input convolution of one layer reads and keeps: its taps [taps, C] (fp32, oldest first) and the tail rows of the
    cache pages [pages, R, C]."""
    taps: torch.Tensor
    tail: torch.Tensor | None
    page_size: int

    @property
    def n_taps(self) -> int:
        return self.taps.shape[0]

    @property
    def rows(self) -> int:
        return 0 if self.tail is None else self.tail.shape[1]


def embed_f32(ids, table, out=None):
    """Rows of the embedding table as an fp32 residual stream."""
    if not table.is_cuda:
        x = ref.embed(ids, table).float()
        return x if out is None else out.copy_(x)
    T, C = ids.shape[0], table.shape[1]
    if out is None:
        out = torch.empty(T, C, dtype=torch.float32, device=table.device)
    _lib.check(_lib.lib().skein_embed_f32(ids.data_ptr(), table.data_ptr(), out.data_ptr(), T, C, table.shape[0], _fp32(table),
                                          _lib.stream_ptr()), "embed_f32")
    _lib.count_launch()
    return out


def conv_input(x, cs: ConvState, positions, block_table, seq_of_token=None, q_start=None, dtype=torch.bfloat16, write_tail=False):
    """h = x + causal convolution of x over time. Rows of one chunk (q_start given) find their predecessors in x, others in the
    cache; write_tail appends each row's input to the cache (decode rows)."""
    if not x.is_cuda:
        return rl.conv_input(x, cs.taps, cs.tail, positions, seq_of_token, q_start, block_table, cs.page_size, dtype, write_tail)
    T, C = x.shape
    h = torch.empty(T, C, dtype=dtype, device=x.device)
    rc = _lib.lib().skein_conv_input(
        x.data_ptr(), h.data_ptr(), cs.taps.data_ptr(), _lib.ptr(cs.tail), positions.data_ptr(), _lib.ptr(seq_of_token), _lib.ptr(q_start),
        block_table.data_ptr(), F.workspace().status.data_ptr(), T, C, cs.n_taps, cs.rows, cs.page_size, block_table.stride(0),
        cs.tail.shape[0] if cs.tail is not None else 0, int(write_tail), _fp32(h), _lib.stream_ptr())
    _lib.check(rc, "conv_input")
    _lib.count_launch()
    return h


def post_norm(x, y, alpha, gain, eps, row_idx=None, row_w=None, dtype=torch.bfloat16, want_act=True, conv: ConvState | None = None,
              positions=None, block_table=None, final_gain=None):
    """x <- gain * v / rms(v) with v = alpha x + y (or the weighted sum of rows row_idx of y). Returns (new residual fp32, second):
    `second` is the residual in the activation type, or with `conv` (decode rows) the next mixer's input x + convolution, or with
    `final_gain` the norm of the new residual with that gain."""
    if not x.is_cuda:
        xn = rl.post_norm(x, y, alpha, gain, eps, row_idx, row_w)
        if conv is not None:
            return xn, rl.conv_input(xn, conv.taps, conv.tail, positions, None, None, block_table, conv.page_size, dtype, True)
        if final_gain is not None:
            return xn, rl.post_norm(xn, None, 1.0, final_gain, eps).to(dtype)
        return xn, (xn.to(dtype) if want_act else None)
    B, C = x.shape
    x_out = torch.empty_like(x)
    act = torch.empty(B, C, dtype=dtype, device=x.device) if (want_act or conv is not None or final_gain is not None) else None
    tail = conv.tail if conv is not None else None
    rc = _lib.lib().skein_post_norm(
        x.data_ptr(), _lib.ptr(y), _lib.ptr(row_idx), _lib.ptr(row_w), gain.data_ptr(), _lib.ptr(final_gain), x_out.data_ptr(), _lib.ptr(act),
        float(alpha), float(eps), B, C, row_idx.shape[1] if row_idx is not None else 0,
        conv.taps.data_ptr() if conv is not None else None, _lib.ptr(tail), _lib.ptr(positions), _lib.ptr(block_table),
        F.workspace().status.data_ptr(), conv.n_taps if conv is not None else 0, conv.rows if conv is not None else 0,
        conv.page_size if conv is not None else 1, block_table.stride(0) if block_table is not None else 0,
        tail.shape[0] if tail is not None else 0, 1 if dtype == torch.float32 else 0, _lib.stream_ptr())
    _lib.check(rc, "post_norm")
    _lib.count_launch()
    return x_out, act


def can_fuse_group_route(T, C, E, topk, dtype, device) -> bool:
    """Whether post_norm_route takes this step (every row's CTA resident at once, bf16, 16-byte rows)."""
    return (dtype == torch.bfloat16 and C % 8 == 0 and C <= 16384 and E <= 64 and topk <= 8 and F.can_fuse_route(T, topk, device))


def post_norm_route(x, y, alpha, gain, eps, wg, top, groups, keep):
    """post_norm + group-limited router + scatter into expert-sorted order, one launch (decode-sized batches).
    Returns (new residual, ids, weights, counts, offsets, row_of, src_token, xs)."""
    T, C = x.shape
    E = wg.shape[0]
    dev = x.device
    x_out = torch.empty_like(x)
    ids, w, counts, offsets, row_of, src_token = route_buffers(T, E, top, dev)
    xs = torch.empty(T * top, C, dtype=torch.bfloat16, device=dev)
    ws = F.workspace()
    rc = _lib.lib().skein_post_norm_route(
        x.data_ptr(), _lib.ptr(y), gain.data_ptr(), x_out.data_ptr(), float(alpha), float(eps), T, C, wg.data_ptr(), E, top, groups, keep,
        ids.data_ptr(), w.data_ptr(), counts.data_ptr(), offsets.data_ptr(), row_of.data_ptr(), src_token.data_ptr(), xs.data_ptr(),
        ws.route_barrier.data_ptr(), ws.sm_count, ws.status.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "post_norm_route")
    _lib.count_launch()
    return x_out, ids, w, counts, offsets, row_of, src_token, xs


def route_grouped(x, wg, top, groups, keep):
    """Group-limited router over the rows of x and the expert-sorted copy. Returns (ids, weights, counts, offsets, row_of,
    src_token, xs). The logits are fp32."""
    E = wg.shape[0]
    if not x.is_cuda:
        ids, w = rl.select_grouped(x.float() @ wg.float().t(), top, groups, keep)
        counts, offsets, row_of, src_token = ref.router_plan(ids, E)
        return ids, w, counts, offsets, row_of, src_token, x[src_token.long()]
    rule = _lib.RouteRule()
    rule.n_groups, rule.keep, rule.group_best, rule.scale = groups, keep, 1, 1.0
    return route_by_rule(x, wg, top, rule)


def route_buffers(T: int, E: int, top: int, dev):
    """(ids, weights, counts, offsets, row_of, src_token) of a routed step, uninitialised."""
    meta = torch.empty(2 * E + 1 + 2 * T * top, dtype=torch.int32, device=dev)
    return (torch.empty(T, top, dtype=torch.int32, device=dev), torch.empty(T, top, dtype=torch.float32, device=dev), meta[:E], meta[E:2 * E + 1],
            meta[2 * E + 1:2 * E + 1 + T * top], meta[2 * E + 1 + T * top:])


def route_by_rule(x, wg, top, rule: "_lib.RouteRule"):
    """Router over the rows of x by any rule (csrc/kernels/route.cuh) and the expert-sorted copy; see route_grouped."""
    T, E = x.shape[0], wg.shape[0]
    if E > MAX_ROUTE_E:
        raise ValueError(f"the router kernel takes at most {MAX_ROUTE_E} experts")
    logits = F.linear(x, wg, out_f32=True)
    ids, w, counts, offsets, row_of, src_token = route_buffers(T, E, top, x.device)
    rc = _lib.lib().skein_route_grouped(logits.data_ptr(), T, E, top, _lib.byref(rule), ids.data_ptr(), w.data_ptr(), counts.data_ptr(),
                                        offsets.data_ptr(), row_of.data_ptr(), src_token.data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "route_grouped")
    _lib.count_launch(3)
    return ids, w, counts, offsets, row_of, src_token, gather_rows(x, src_token)


def gather_rows(x, src_row):
    """out[r] = x[src_row[r]]; rows of 4-byte elements are moved as pairs of 2-byte ones."""
    if x.is_cuda and x.dtype == torch.float32:
        return F.gather_rows(x.view(torch.bfloat16), src_row).view(torch.float32)
    return F.gather_rows(x, src_row)


def poly_norm(z, act, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e with N dividing a row by its root mean square; act holds (a, b, c, e)."""
    if not z.is_cuda:
        return rl.poly_norm(z, act, eps).to(z.dtype)
    out = torch.empty_like(z)
    _lib.check(_lib.lib().skein_poly_norm(z.data_ptr(), act.data_ptr(), out.data_ptr(), z.shape[0], z.shape[1], float(eps), _fp32(z),
                                          _lib.stream_ptr()), "poly_norm")
    _lib.count_launch()
    return out


# ---- latent attention -------------------------------------------------------------------------------------------------
def latent_append(proj, off_kv, q_norm, kv_norm, rot, cos_sin, positions, seq_of_token, block_table, cache, eps, x=None, tail=None,
                  seq_lens=None, taps=1, dense=None, dense_start=None):
    """Norms the cache row (and the query latent) of every token, rotates its key part and writes it to the paged cache; with
    `dense` also to the dense copy of the step's context; with `x` the convolution's tail rows of a chunk. Returns the normed
    query latent or None."""
    if not proj.is_cuda:
        return rl.latent_append(proj, off_kv, q_norm, kv_norm, rot, cos_sin, positions, seq_of_token, block_table, cache, eps, x, tail,
                                seq_lens, taps)
    T = proj.shape[0]
    q_rank = q_norm.shape[0] if q_norm is not None else 0
    cq = torch.empty(T, q_rank, dtype=proj.dtype, device=proj.device) if q_rank else None
    rc = _lib.lib().skein_latent_append(
        proj.data_ptr(), proj.stride(0), off_kv, _lib.ptr(q_norm), q_rank, kv_norm.data_ptr(), kv_norm.shape[0], rot, cos_sin.data_ptr(),
        cos_sin.shape[0], positions.data_ptr(), _lib.ptr(seq_of_token), block_table.data_ptr(), block_table.stride(0), cache.data_ptr(),
        cache.shape[0], cache.shape[1], _lib.ptr(cq), _lib.ptr(dense), _lib.ptr(dense_start), _lib.ptr(x), _lib.ptr(tail), _lib.ptr(seq_lens),
        x.shape[1] if x is not None else 0, tail.shape[1] if tail is not None else 0, taps, float(eps), T, F.workspace().status.data_ptr(),
        _fp32(proj), _lib.stream_ptr())
    _lib.check(rc, "latent_append")
    _lib.count_launch()
    return cq


def head_linear(x, x_cols, w, gate=None, out=None):
    """Per-head product: head h multiplies columns h * x_cols .. + K of x by w[h] [F, K]; results side by side [T, H * F], possibly
    columns `out` of a wider matrix. `gate` ([T, H * F], rows may be strided): the result is multiplied by its sigmoid."""
    H, Fo, K = w.shape
    if not x.is_cuda:
        y = rl.head_linear(x, x_cols, w, gate)
        return y if out is None else out.copy_(y)
    T = x.shape[0]
    if out is None:
        out = torch.empty(T, H * Fo, dtype=x.dtype, device=x.device)
    if T == 0:
        return out
    tensor_core = F.tc_gemm_ok(x, K) and x.stride(0) % 8 == 0 and x_cols % 8 == 0 and x.data_ptr() % 16 == 0
    for h0 in range(0, H, _lib.MAX_GROUPS):
        hn = min(_lib.MAX_GROUPS, H - h0)
        p = F._base_params(x, w, out, Fo, K, F.pick_n_tile(T, False), 0)
        p.X, p.W = x[:, h0 * x_cols:].data_ptr(), w[h0:].data_ptr()
        p.G, p.w_rows_per_group = hn, Fo
        p.x_ld, p.x_group_cols, p.ldo, p.out_col0, p.out_group_cols = x.stride(0), x_cols, out.stride(0), h0 * Fo, Fo
        if gate is not None:
            p.gate, p.gate_ld = gate[:, h0 * Fo:].data_ptr(), gate.stride(0)
        if tensor_core:
            F._gemm_launch(p, "head_linear")
        else:
            F.simt_launch(p, x, T, "head_linear")
    return out


def _decode_tc_ok(q_abs, q, D, rot, K, cache) -> bool:
    ps = cache.shape[1]
    return (q_abs.dtype == torch.bfloat16 and K % 8 == 0 and rot % 8 == 0 and K <= 512
            and (ps in (16, 32) or ps % 64 == 0) and os.environ.get("SKEIN_LATENT_DECODE", "tc") == "tc"
            and hasattr(_lib.lib(), "skein_latent_attn_decode"))


def latent_attn_rows(q_abs, q, H, D, rot, scale, cos_sin, positions, seq_of_token, block_table, cache, ctx_hint=1024, splits=None, sinks=None):
    """Attention of single rows over the latent cache with the key expansion already applied to the queries.
    q_abs [T, H * K]; q [T, >= H * (D + rot)] whose rotated parts are not rotated yet; row t sees positions 0 .. positions[t] of
    its sequence. sinks [H] fp32: head h's denominator has one more term exp(sinks[h]). Returns the weighted latents [T, H * K]."""
    K = cache.shape[2] - rot
    T = q_abs.shape[0]
    if not q_abs.is_cuda:
        return rl.latent_attention_rows(q_abs.view(T, H, K), q[:, :H * (D + rot)].reshape(T, H, D + rot), D, rot, scale, cos_sin, positions,
                                        seq_of_token, block_table, cache, sinks).reshape(T, H * K)
    out = torch.empty(T, H * K, dtype=q_abs.dtype, device=q_abs.device)
    ws = F.workspace()
    L = _lib.lib()
    if _decode_tc_ok(q_abs, q, D, rot, K, cache):
        rc = L.skein_latent_attn_decode(
            q_abs.data_ptr(), q.data_ptr(), q.stride(0), cos_sin.data_ptr(), cos_sin.shape[0], positions.data_ptr(), _lib.ptr(seq_of_token),
            block_table.data_ptr(), block_table.stride(0), cache.data_ptr(), cache.shape[0], cache.shape[1], out.data_ptr(), T, H, D, rot, K,
            float(scale), _lib.ptr(sinks), int(splits or 0), int(ctx_hint), ws.status.data_ptr(), _lib.stream_ptr())
        if rc != -1:
            _lib.check(rc, "latent_attn_decode")
            _lib.count_launch()
            return out
    rc = L.skein_latent_attn_rows(
        q_abs.data_ptr(), q.data_ptr(), q.stride(0), cos_sin.data_ptr(), cos_sin.shape[0], positions.data_ptr(), _lib.ptr(seq_of_token),
        block_table.data_ptr(), block_table.stride(0), cache.data_ptr(), cache.shape[0], cache.shape[1], out.data_ptr(), T, H, D, rot, K,
        float(scale), _lib.ptr(sinks), ws.status.data_ptr(), _fp32(q_abs), _lib.stream_ptr())
    _lib.check(rc, "latent_attn_rows")
    _lib.count_launch()
    return out


def expanded_ok(dtype, D, rot, V, K, device) -> bool:
    """Whether the expanded prefill kernel (csrc/kernels/attn_latent_prefill.cu) takes this mixer."""
    return (device.type == "cuda" and dtype == torch.bfloat16 and D <= 128 and rot <= 64 and V <= 128 and D % 8 == 0 and rot % 8 == 0
            and V % 8 == 0 and K % 8 == 0 and os.environ.get("SKEIN_LATENT_PREFILL", "tc") == "tc"
            and hasattr(_lib.lib(), "skein_latent_attn_prefill"))


def latent_gather(cache, block_table, kv_len, q_len, dense_start, dense, max_ctx):
    """Cached rows before each chunk -> their places in the dense copy of the context."""
    rc = _lib.lib().skein_latent_gather(cache.data_ptr(), block_table.data_ptr(), block_table.stride(0), kv_len.data_ptr(), q_len.data_ptr(),
                                        dense_start.data_ptr(), dense.data_ptr(), kv_len.shape[0], int(max_ctx), cache.shape[2], cache.shape[1],
                                        cache.shape[0], F.workspace().status.data_ptr(), _fp32(cache), _lib.stream_ptr())
    _lib.check(rc, "latent_gather")
    _lib.count_launch()


def rope_rows(q, H, D, rot, cos_sin, positions):
    """Rotates the rotated part of every head of q [T, >= H * (D + rot)] in place."""
    rc = _lib.lib().skein_rope_rows(q.data_ptr(), q.stride(0), positions.data_ptr(), cos_sin.data_ptr(), q.shape[0], H, D, rot, cos_sin.shape[0],
                                    F.workspace().status.data_ptr(), _fp32(q), _lib.stream_ptr())
    _lib.check(rc, "rope_rows")
    _lib.count_launch()


def latent_attn_prefill(q, H, D, rot, V, scale, dense, kv, q_start, q_len, kv_len, dense_start, max_q_len, gate=None, sinks=None):
    """Causal attention of prefill chunks with keys and values expanded per head. q [T, >= H * (D + rot)] rotated; dense
    [ctx, K + rot] the step's context rows (rotated key part in the last columns); kv [ctx, H * (D + V)] keys then values.
    `gate` [T, H * V] (rows may be strided): the output is multiplied by its sigmoid. sinks [H] fp32: see latent_attn_rows. Returns
    [T, H * V]."""
    T = q.shape[0]
    out = torch.empty(T, H * V, dtype=q.dtype, device=q.device)
    rc = _lib.lib().skein_latent_attn_prefill(
        q.data_ptr(), q.stride(0), T, dense.data_ptr(), dense.shape[1], kv.data_ptr(), kv.shape[0], _lib.ptr(gate),
        gate.stride(0) if gate is not None else 0, q_start.data_ptr(), q_len.data_ptr(), kv_len.data_ptr(), dense_start.data_ptr(),
        out.data_ptr(), F.workspace().status.data_ptr(), q_len.shape[0], int(max_q_len), H, D, rot, V, float(scale), _lib.ptr(sinks),
        _lib.stream_ptr())
    _lib.check(rc, "latent_attn_prefill")
    _lib.count_launch()
    return out
