"""Selective scan (Mamba): short convolution over time, then a diagonal recurrence per channel with a 32-bit state per sequence.

CUDA tensors run csrc/kernels/selective.cu; CPU tensors run ops/reference_prenorm.py. The specification and weights are
models/parallel_layers.py: SelectiveSpec, SelectiveWeights. A sequence owns one slot of the state pools, as in ops/recurrent.py.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from . import _lib, functional as F, reference_prenorm as rn


@dataclass
class ScanState:
    """State pools of one layer: S [slots, state, inner] fp32 and the convolution's last inputs [slots, taps, inner] (None without a
    look-back), position p in row p mod taps. Position 0 starts from zero whatever the slot holds."""
    mat: torch.Tensor
    tail: torch.Tensor | None

    @staticmethod
    def make(spec, slots: int, dtype, device) -> "ScanState":
        mat = torch.zeros(slots, spec.state, spec.inner, dtype=torch.float32, device=device)
        tail = torch.zeros(slots, spec.conv_rows, spec.inner, dtype=dtype, device=device) if spec.conv_rows else None
        return ScanState(mat, tail)


def _portions(inp, decode: bool):
    """(first row, number of rows) of every sequence's portion, on the CPU path."""
    n = inp.seq_lens.shape[0]
    return (torch.arange(n), torch.ones(n, dtype=torch.int32)) if decode else (inp.q_start, inp.q_len)


def _params(spec, w, state, inp, slots, decode: bool) -> "_lib.ScanParams":
    p = _lib.ScanParams()
    p.state, p.tail = state.mat.data_ptr(), _lib.ptr(state.tail)
    p.conv_w, p.conv_b, p.dt_bias, p.neg_a, p.skip = (t.data_ptr() for t in (w.conv, w.conv_b, w.dt_bias, w.neg_a, w.skip))
    p.positions, p.slots, p.status = inp.positions.data_ptr(), slots.data_ptr(), F.workspace().status.data_ptr()
    if not decode:
        p.seq_of_token, p.q_start, p.q_len = inp.seq_of_token.data_ptr(), inp.q_start.data_ptr(), inp.q_len.data_ptr()
    p.I, p.N, p.taps, p.num_slots = spec.inner, spec.state, spec.taps, state.mat.shape[0]
    return p


def short_conv(x, spec, w, state: ScanState, inp, slots, decode: bool):
    """silu(convolution of x over time + bias), x columns of a wider matrix [T, inner]. A decode step also keeps its input for the next
    ones; a portion's last inputs are kept by `scan`, which runs behind every reader of the old ones."""
    T = x.shape[0]
    if not x.is_cuda:
        return rn.short_conv(x, spec.taps, w, state, inp.positions, slots, *_portions(inp, decode))
    out = torch.empty(T, spec.inner, dtype=x.dtype, device=x.device)
    if T:
        p = _params(spec, w, state, inp, slots, decode)
        p.x, p.x_ld, p.xc = x.data_ptr(), x.stride(0), out.data_ptr()
        _lib.check(_lib.lib().skein_short_conv(C.byref(p), T, int(decode), 1 if x.dtype == torch.float32 else 0, _lib.stream_ptr()), "short_conv")
        _lib.count_launch()
    return out


def scan(xc, proj, dt, x, z, out, spec, w, state: ScanState, inp, slots, decode: bool):
    """The recurrence over the step's rows, into `out` (columns of a wider matrix): y silu(z). xc [T, inner] from short_conv; proj its
    projections (sections of SelectiveSpec.x_sections, each from a multiple of 8 columns); dt [T, inner] fp32 step sizes before bias and
    softplus; x the convolution's inputs, of which a portion's last ones are kept."""
    T = xc.shape[0]
    if not xc.is_cuda:
        return rn.scan(xc, proj, dt, x, z, out, spec, w, state, inp.positions, slots, *_portions(inp, decode))
    if T:
        p = _params(spec, w, state, inp, slots, decode)
        p.x, p.x_ld, p.xc = x.data_ptr(), x.stride(0), xc.data_ptr()
        p.proj, p.proj_ld, p.dt, p.z, p.out, p.out_ld = proj.data_ptr(), proj.stride(0), dt.data_ptr(), z.data_ptr(), out.data_ptr(), out.stride(0)
        if z.stride(0) != x.stride(0):
            raise ValueError("scan: x and z must be columns of one matrix")
        p.b_col = (spec.dt_rank + 7) // 8 * 8
        p.c_col = p.b_col + (spec.state + 7) // 8 * 8
        fn = _lib.lib().skein_scan_step if decode else _lib.lib().skein_scan_rows
        _lib.check(fn(C.byref(p), T if decode else inp.q_len.shape[0], 1 if xc.dtype == torch.float32 else 0, _lib.stream_ptr()), "selective_scan")
        _lib.count_launch()
    return out
