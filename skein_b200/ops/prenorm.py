"""Operators of pre-norm layers over an fp32 stream: stream sum + RMS norm, average over depth + RMS norm in groups + token shift, and the
router that scores every expert by itself.

CUDA tensors run csrc/kernels (prenorm.cu, router.cu); CPU tensors run ops/reference_prenorm.py. Activations are bf16, or fp32 when a
model runs in 32-bit; the stream is fp32.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import _lib, functional as F, latent, reference as ref, reference_prenorm as rn

SCORES = {"softmax": 0, "sigmoid": 1}


def _fp32(t) -> int:
    return 1 if t.dtype == torch.float32 else 0


def add_norm(x, y=None, row_idx=None, row_w=None, step=None, gain=None, eps=0.0, dtype=torch.bfloat16):
    """a = x + (sum over j of row_w[:, j] * y[row_idx[:, j]]) + step, fp32 (y, step: may be None). Returns (a, a / rms(a) * gain in
    `dtype`, or None without a gain)."""
    T, C = x.shape
    if not x.is_cuda:
        return rn.add_norm(x, y, row_idx, row_w, step, gain, eps, dtype)
    plain = y is None and step is None
    x_out = x if plain else torch.empty_like(x)
    act = torch.empty(T, C, dtype=dtype, device=x.device) if gain is not None else None
    if T and not (plain and act is None):
        _lib.check(_lib.lib().skein_add_norm(
            x.data_ptr(), _lib.ptr(y), _lib.ptr(row_idx), _lib.ptr(row_w), row_idx.shape[1] if row_idx is not None else 0, _lib.ptr(step),
            _lib.ptr(gain), None if plain else x_out.data_ptr(), _lib.ptr(act), T, C, float(eps), 1 if dtype == torch.float32 else 0,
            _lib.stream_ptr()), "add_norm")
        _lib.count_launch()
    return x_out, act


@dataclass
class TokenShift:
    """What the mixer of a shifted layer reads: h + (h' - h) mix with h the normed row and h' the previous token's. state [slots, C] fp32 keeps
    every sequence's last h; position 0 starts from zero whatever the slot holds."""
    mix: torch.Tensor            # [C] fp32
    state: torch.Tensor


def depth_norm(terms, weights, gain, groups, eps, dtype, x_out=None, shift: TokenShift | None = None, inp=None, slots=None, decode=False):
    """x = sum_j weights[j] terms[j] (weights None: the one term itself), fp32, into x_out where given; then its RMS norm over `groups` equal
    parts of a row times gain; then, with `shift`, the token shift over the step's sequences. terms [n, T, C]; returns [T, C] in `dtype`."""
    n, T, C = terms.shape
    if not terms.is_cuda:
        return rn.depth_norm(terms, weights, gain, groups, eps, dtype, x_out, shift, inp, slots, decode)
    act = torch.empty(T, C, dtype=dtype, device=terms.device)
    if T:
        p = _lib.DepthNormParams()
        p.terms, p.weights, p.x_out, p.gain, p.act_out = terms.data_ptr(), _lib.ptr(weights), _lib.ptr(x_out), gain.data_ptr(), act.data_ptr()
        p.term_stride, p.n_terms, p.T, p.C, p.groups, p.eps = terms.stride(0), n, T, C, groups, float(eps)
        p.status = F.workspace().status.data_ptr()
        if shift is not None:
            p.shift, p.state, p.num_slots = shift.mix.data_ptr(), shift.state.data_ptr(), shift.state.shape[0]
            p.positions, p.slots = inp.positions.data_ptr(), slots.data_ptr()
            if not decode:
                p.seq_of_token, p.q_start, p.q_len = inp.seq_of_token.data_ptr(), inp.q_start.data_ptr(), inp.q_len.data_ptr()
        _lib.check(_lib.lib().skein_depth_norm(_lib.byref(p), 1 if dtype == torch.float32 else 0, _lib.stream_ptr()), "depth_norm")
        _lib.count_launch()
    return act


def _rule(f) -> "_lib.RouteRule":
    r = _lib.RouteRule()
    r.n_groups, r.keep, r.score, r.group_best, r.renorm, r.scale = f.groups, f.keep, SCORES[f.score], f.group_best, int(f.renorm), float(f.scale)
    return r


def can_fuse_route(x, f, dtype) -> bool:
    """Whether norm_route takes this step (every row's CTA resident at once, bf16, 16-byte rows)."""
    T, C = x.shape
    return latent.can_fuse_group_route(T, C, f.experts, f.top, dtype, x.device)


def norm_route(x, gain, eps, wg, f):
    """RMS norm + router + scatter into expert-sorted order, one launch (decode-sized batches). Returns (normed rows, ids, weights,
    counts, offsets, row_of, src_token, xs)."""
    T, C = x.shape
    E, top, dev = wg.shape[0], f.top, x.device
    act = torch.empty(T, C, dtype=torch.bfloat16, device=dev)
    ids, w, counts, offsets, row_of, src_token = latent.route_buffers(T, E, top, dev)
    xs = torch.empty(T * top, C, dtype=torch.bfloat16, device=dev)
    ws, rule = F.workspace(), _rule(f)
    _lib.check(_lib.lib().skein_norm_route(
        x.data_ptr(), gain.data_ptr(), act.data_ptr(), float(eps), T, C, wg.data_ptr(), E, top, _lib.byref(rule), ids.data_ptr(), w.data_ptr(),
        counts.data_ptr(), offsets.data_ptr(), row_of.data_ptr(), src_token.data_ptr(), xs.data_ptr(), ws.route_barrier.data_ptr(), ws.sm_count,
        ws.status.data_ptr(), _lib.stream_ptr()), "norm_route")
    _lib.count_launch()
    return act, ids, w, counts, offsets, row_of, src_token, xs


def route(x, wg, f):
    """Router over the rows of x by the rule of `f` (models/layered.py: RoutedFFSpec) and the expert-sorted copy. Returns (ids, weights,
    counts, offsets, row_of, src_token, xs). The logits are fp32."""
    E = wg.shape[0]
    if not x.is_cuda:
        ids, w = rn.select(x.float() @ wg.float().t(), f)
        counts, offsets, row_of, src_token = ref.router_plan(ids, E)
        return ids, w, counts, offsets, row_of, src_token, x[src_token.long()]
    return latent.route_by_rule(x, wg, f.top, _rule(f))
