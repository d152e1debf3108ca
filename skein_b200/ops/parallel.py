"""Operators of parallel layers (x <- x + mixer(h) + ff(h), h = tanh(alpha x) w + b) and of grouped-query attention over a window or
chunks (models/parallel_layers.py: WindowAttnSpec).

CUDA tensors run csrc/kernels (parallel_layer.cu, attn_window.cu, attn_prefill_tc.cu, attn_decode_mma.cu); CPU tensors run
ops/reference_parallel.py. Activations are bf16, or fp32 when a model runs in 32-bit; the residual stream is fp32.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from . import _lib, functional as F, reference_parallel as rp


def _fp32(t) -> int:
    return 1 if t.dtype == torch.float32 else 0


def residual_tanh(x, y=None, bias=None, norm=None, dtype=torch.bfloat16, out=None, want_x=True):
    """a = x + y + bias (each may be None), fp32. Returns (a, or None unless want_x; tanh(alpha a) w + b in `dtype` with a norm
    (models/parallel_layers.py: TanhNorm), else a in `dtype`). `out`: where the latter goes, possibly columns of a wider matrix;
    False: nowhere."""
    like = x if x is not None else y
    T, C = like.shape
    if not like.is_cuda:
        a, act = rp.residual_tanh(x, y, bias, norm, dtype)
        if out is not None and out is not False:
            out.copy_(act)
            act = out
        return (a if want_x else None), (None if out is False else act)
    if out is None:
        out = torch.empty(T, C, dtype=dtype, device=like.device)
    act = None if out is False else out
    plain = y is None and bias is None      # a is x
    x_out = torch.empty(T, C, dtype=torch.float32, device=like.device) if want_x and not plain else None
    if T:
        _lib.check(_lib.lib().skein_residual_tanh(
            _lib.ptr(x), _lib.ptr(y), 1 if y is None else _fp32(y), _lib.ptr(bias), _lib.ptr(norm.alpha if norm else None),
            _lib.ptr(norm.w if norm else None), _lib.ptr(norm.b if norm else None), _lib.ptr(x_out), _lib.ptr(act),
            act.stride(0) if act is not None else 0, T, C, 1 if dtype == torch.float32 else 0, _lib.stream_ptr()), "residual_tanh")
        _lib.count_launch()
    return ((x if plain else x_out) if want_x else None), act


def gated_norm(o, gate, w, out, groups, eps, gate_first=False, silu=False, scale=1.0):
    """o [T, n] in `groups` equal parts, each divided by its root mean square, times w ([n], or one part's or less, repeated) and
    times the gate's activation (silu or sigmoid), which multiplies before the norm with gate_first; times scale, into `out`
    (columns of a wider matrix)."""
    T, n = o.shape
    if not o.is_cuda:
        out.copy_(rp.gated_norm(o, gate, w, groups, eps, gate_first, silu, scale))
        return out
    if T:
        _lib.check(_lib.lib().skein_gated_norm(
            o.data_ptr(), gate.data_ptr(), gate.stride(0), w.data_ptr(), w.shape[0], out.data_ptr(), out.stride(0), T, n, groups,
            int(gate_first), int(silu), float(eps), float(scale), _fp32(o), _lib.stream_ptr()), "gated_norm")
        _lib.count_launch()
    return out


# ---- attention over a window or chunks ----------------------------------------------------------------------------------
def window_cache(num_pages: int, page_size: int, kv_heads: int, dim: int, vdim: int, dtype, device) -> torch.Tensor:
    """[pages, kv_heads * page_size * (dim + vdim)]: keys [kv_heads, page_size, dim], then values [kv_heads, page_size, vdim]. `dim` is
    the width of a key head, its maps side by side."""
    return torch.zeros(num_pages, kv_heads * page_size * (dim + vdim), dtype=dtype, device=device)


def window_append(q, k, v, q_norm, k_norm, spec, cos_sin, positions, seq_of_token, block_table, cache, page_size, eps):
    """Norm and rotation of q (in place) and k, append of k and v to the cache. q, k, v: columns of one matrix."""
    T = q.shape[0]
    if not q.is_cuda:
        return rp.window_append(q, k, v, q_norm, k_norm, spec, cos_sin, positions, seq_of_token, block_table, cache, page_size, eps)
    if T:
        _lib.check(_lib.lib().skein_window_append(
            q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), q_norm.data_ptr(), k_norm.data_ptr(), cos_sin.data_ptr(), positions.data_ptr(),
            _lib.ptr(seq_of_token), block_table.data_ptr(), cache.data_ptr(), F.workspace().status.data_ptr(), T, spec.heads, spec.kv_heads,
            spec.dim, spec.vdim, spec.rot_dims, cos_sin.shape[0], block_table.stride(0), cache.shape[0], page_size, float(eps), _fp32(q),
            _lib.stream_ptr()), "window_append")
        _lib.count_launch()


@dataclass
class ValueMix:
    """The first mixing layer's values of the step's tokens, [T, kv_heads * vdim] in the activation type. `keep`: this layer is the first
    and writes them; otherwise its values become (1 - lam) v + lam v_first."""
    v_first: torch.Tensor
    keep: bool


def head_append(q, k, v, spec, cos_sin, positions, seq_of_token, block_table, cache, page_size, eps, w=None, mix: ValueMix | None = None):
    """Per head of q (in place) and k: bias, RMS norm with a weight, rotation, division by the root mean square, each where the
    specification asks for it; bias and mixing of v; append of k and v to the cache. q, k, v: columns of one matrix. A head with two maps is
    two heads here. w (models/parallel_layers.py: WindowAttnWeights): biases, norm weights, the mixing weight. cos_sin None: no rotation."""
    T = q.shape[0]
    if not q.is_cuda:
        return rp.head_append(q, k, v, spec, cos_sin, positions, seq_of_token, block_table, cache, page_size, eps, w, mix)
    if T:
        x = _lib.HeadExtras()
        if spec.bias:
            x.q_bias, x.k_bias, x.v_bias = w.q_bias.data_ptr(), w.k_bias.data_ptr(), w.v_bias.data_ptr()
        if spec.head_norm:
            x.q_norm, x.k_norm = w.q_norm.data_ptr(), w.k_norm.data_ptr()
        if mix is not None and mix.keep:
            x.v_keep = mix.v_first.data_ptr()
        elif mix is not None:
            x.mix, x.v_first = w.vmix.data_ptr(), mix.v_first.data_ptr()
        max_pos = cos_sin.shape[0] if cos_sin is not None else block_table.shape[1] * page_size
        _lib.check(_lib.lib().skein_head_append(
            q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), _lib.ptr(cos_sin), positions.data_ptr(), _lib.ptr(seq_of_token),
            block_table.data_ptr(), cache.data_ptr(), F.workspace().status.data_ptr(), C.byref(x), T, spec.heads, spec.kv_heads, spec.dim, spec.maps, spec.vdim,
            spec.rot_dims, int(spec.interleaved), int(spec.unit), max_pos, block_table.stride(0), cache.shape[0], page_size, float(eps),
            _fp32(q), _lib.stream_ptr()), "head_append")
        _lib.count_launch()


@dataclass
class HeadMix:
    """What belongs to a head's softmax and what follows it: the second map's weight (two maps), the gate, the head norm's eps, the learned
    sinks."""
    lam: torch.Tensor | None = None
    gate: torch.Tensor | None = None       # [T, heads * vdim], columns of a wider matrix
    eps: float = 0.0
    sinks: torch.Tensor | None = None      # [heads] fp32


def _attn_rule(spec, mix, out_scale) -> "_lib.AttnRule":
    """The mask, sink and what follows the softmax, as the kernels take it."""
    r = _lib.AttnRule()
    r.window, r.chunk, r.sink, r.maps = spec.window, spec.chunk, int(spec.sink), spec.maps
    r.scale, r.out_scale = float(spec.scale), float(out_scale)
    r.softcap, r.keep_first = float(spec.softcap), spec.keep_first if spec.window else 0
    if spec.head_sink:
        r.sinks = mix.sinks.data_ptr()
    if spec.diff is not None:
        r.lam, r.eps, r.out_scale = mix.lam.data_ptr(), float(mix.eps), float(out_scale) * (1.0 - spec.diff)
    if mix is not None and mix.gate is not None:
        r.gate, r.gate_ld = mix.gate.data_ptr(), mix.gate.stride(0)
    return r


def window_attn_rows(q, spec, positions, seq_of_token, block_table, cache, page_size, out, out_scale=1.0, mix: HeadMix | None = None):
    """Attention of single rows over the cache, any sizes (plain kernel)."""
    T = q.shape[0]
    if not q.is_cuda:
        out.copy_(rp.window_attn_rows(q, spec, positions, seq_of_token, block_table, cache, page_size, out_scale, mix))
        return out
    if T:
        r = _attn_rule(spec, mix, out_scale)
        _lib.check(_lib.lib().skein_window_attn_rows(
            q.data_ptr(), q.stride(0), cache.data_ptr(), positions.data_ptr(), _lib.ptr(seq_of_token), block_table.data_ptr(), out.data_ptr(),
            out.stride(0), F.workspace().status.data_ptr(), T, spec.heads, spec.kv_heads, spec.dim, spec.vdim, block_table.stride(0),
            cache.shape[0], page_size, C.byref(r), _fp32(q), _lib.stream_ptr()), "window_attn_rows")
        _lib.count_launch()
    return out


def window_attn(q, spec, inp, cache, page_size, out, out_scale=1.0, mix: HeadMix | None = None):
    """Attention of a step's rows (a decode step or a chunk) over the cache. bf16 heads of 128 or 64 (two maps of 64 over values of 128)
    run the tensor-core kernels (a decode step's with up to 16 query rows per key head), everything else the plain one."""
    KW = spec.key_width
    tc = (q.is_cuda and q.dtype == torch.bfloat16 and KW == spec.vdim and (KW == 128 or (KW == 64 and spec.maps == 1)) and page_size % 16 == 0
          and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0 and out.data_ptr() % 16 == 0 and out.stride(0) % 8 == 0 and spec.scale > 0)
    if tc and mix is not None and mix.gate is not None:
        tc = spec.maps == 2 and mix.gate.data_ptr() % 16 == 0 and mix.gate.stride(0) % 8 == 0
    if not tc or (not inp.is_prefill and (inp.seq_of_token is not None or spec.maps * (spec.heads // spec.kv_heads) > 16)):
        return window_attn_rows(q, spec, inp.positions, inp.seq_of_token, inp.block_table, cache, page_size, out, out_scale, mix)
    ws, bt, H, K, r = F.workspace(), inp.block_table, spec.heads, spec.kv_heads, _attn_rule(spec, mix, out_scale)
    if inp.is_prefill:
        rc = _lib.lib().skein_attn_prefill_window(
            q.data_ptr(), q.stride(0), q.shape[0], cache.data_ptr(), bt.data_ptr(), inp.q_start.data_ptr(), inp.q_len.data_ptr(),
            inp.seq_lens.data_ptr(), out.data_ptr(), out.stride(0), ws.status.data_ptr(), inp.q_len.shape[0], int(inp.max_q_len), H, K, KW,
            page_size, bt.stride(0), cache.shape[0], C.byref(r), _lib.stream_ptr())
    else:
        B, reach = q.shape[0], spec.window + spec.keep_first if spec.window else spec.chunk or inp.ctx_hint
        splits = F.pick_splits(B, K, min(inp.ctx_hint, reach), ws.sm_count)
        scratch = ws.attn_scratch(B, H * spec.maps, K, splits) if splits > 1 else None
        splits, (wsf, ctr) = (splits, scratch) if scratch is not None else (1, (None, None))
        rc = _lib.lib().skein_attn_decode_window(
            q.data_ptr(), q.stride(0), cache.data_ptr(), bt.data_ptr(), inp.seq_lens.data_ptr(), out.data_ptr(), out.stride(0), _lib.ptr(wsf),
            _lib.ptr(ctr), ws.status.data_ptr(), B, H, K, KW, page_size, bt.stride(0), cache.shape[0], splits, C.byref(r), _lib.stream_ptr())
    _lib.check(rc, "window_attn")
    _lib.count_launch()
    return out
