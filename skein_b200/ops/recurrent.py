"""Recurrences with a 32-bit matrix state per head (gated delta rule with a decay per head or per key channel, state-space duality, fixed decay).

CUDA tensors run csrc/kernels/recurrent.cu, recurrent_tc.cu and recurrent_channel_tc.cu; CPU tensors run ops/reference_parallel.py. The specification
(models/parallel_layers.py: RecurrentSpec) says which recurrence; the weights are its RecurrentWeights.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from . import _lib, functional as F, reference_parallel as rp

KINDS = {"delta": 0, "ssd": 1, "lightning": 2, "channel_delta": 3}
TC_MIN_ROWS = 17         # portions of at least this many rows take the tensor-core form


def tc_ok(spec, row) -> bool:
    return row.is_cuda and row.dtype == torch.bfloat16 and spec.dim in (64, 128) and spec.vdim % 64 == 0


@dataclass
class RecState:
    """State pools of one recurrent layer: matrices [slots, heads, dim, vdim] fp32 and the convolution's last inputs
    [slots, taps, channels] (None without a convolution), position p in row p mod taps."""
    mat: torch.Tensor
    tail: torch.Tensor | None

    @staticmethod
    def make(spec, slots: int, dtype, device) -> "RecState":
        mat = torch.zeros(slots, spec.heads, spec.dim, spec.vdim, dtype=torch.float32, device=device)
        tail = torch.zeros(slots, spec.conv_rows, spec.conv_channels, dtype=dtype, device=device) if spec.conv_rows else None
        return RecState(mat, tail)


@dataclass
class RecColumns:
    """First columns of the recurrence's projections in a row."""
    q: int
    k: int
    v: int
    a: int = 0               # input of the decay (delta: a; ssd: dt)
    b: int = 0               # input of the write strength (delta)

    @staticmethod
    def of(spec, col: dict) -> "RecColumns":
        if spec.kind == "ssd":      # values | keys | queries, the order of the checkpoint's matrix
            v = col["conv"]
            k = v + spec.heads * spec.vdim
            return RecColumns(k + spec.groups * spec.dim, k, v, a=col["dt"])
        return RecColumns(col["q"], col["k"], col["v"], col.get("a", 0), col.get("b", 0))


def _params(row, cols, spec, w, state, positions, slots, out, step=None) -> "_lib.RecParams":
    p = _lib.RecParams()
    p.row, p.out, p.ld = row.data_ptr(), out.data_ptr(), row.stride(0)
    p.state, p.tail = state.mat.data_ptr(), _lib.ptr(state.tail)
    p.conv_w, p.conv_b, p.neg_decay, p.decay, p.dt_bias, p.skip = (
        _lib.ptr(t) for t in (w.conv, w.conv_b, w.neg_decay, w.decay, w.dt_bias, w.skip))
    p.step = _lib.ptr(step)
    p.positions, p.slots, p.status = positions.data_ptr(), slots.data_ptr(), F.workspace().status.data_ptr()
    p.kind, p.H, p.G, p.D, p.V, p.taps, p.C = KINDS[spec.kind], spec.heads, spec.groups, spec.dim, spec.vdim, spec.taps, spec.conv_channels
    p.q_col, p.k_col, p.v_col, p.a_col, p.b_col, p.num_slots = cols.q, cols.k, cols.v, cols.a, cols.b, state.mat.shape[0]
    return p


@dataclass
class HeadGate:
    """Norm and gate of a head's own read-out (delta rules): o / rms(o) * norm * silu(gate) * scale, into `out`. gate and out
    [rows, heads * vdim]: columns of a wider matrix; `sigmoid`: the gate's activation is a sigmoid."""
    norm: torch.Tensor
    gate: torch.Tensor
    out: torch.Tensor
    eps: float
    scale: float = 1.0
    sigmoid: bool = False


def rec_step(row, cols: RecColumns, spec, w, state: RecState, positions, slots, gate: HeadGate | None = None, step=None):
    """One token per sequence: row [B, ld] holds the projections, step [B, heads * dim] fp32 ("channel_delta") the inputs of the decays
    before bias and softplus. Returns the read-outs [B, heads * vdim], or None when the step applied `gate` to them (it does where a
    kernel holds whole heads); the state moves on."""
    B = row.shape[0]
    if not row.is_cuda:
        return rp.rec_chunk(row, cols, spec, w, state, positions, slots, torch.arange(B), torch.ones(B, dtype=torch.int32), step)
    out = torch.empty(B, spec.out_width, dtype=row.dtype, device=row.device)
    p, g = _params(row, cols, spec, w, state, positions, slots, out, step), _lib.RecGate()
    L = _lib.lib()
    if gate is not None and L.skein_rec_step_gates(C.byref(p)):
        g.norm, g.out, g.out_ld, g.eps, g.scale = gate.norm.data_ptr(), gate.out.data_ptr(), gate.out.stride(0), gate.eps, gate.scale
        g.gate, g.gate_ld, g.sigmoid = gate.gate.data_ptr(), gate.gate.stride(0), int(gate.sigmoid)
    _lib.check(L.skein_rec_step(C.byref(p), C.byref(g), B, 1 if row.dtype == torch.float32 else 0, _lib.stream_ptr()), "rec_step")
    _lib.count_launch()
    return None if g.out else out


class ChunkRun:
    """Portions of several sequences on the GPU: the launches of rec_chunk and what they share."""

    def __init__(self, row, cols, spec, w, state, positions, slots, seq_of_token, q_start, q_len, max_q_len, impl=None, step=None):
        dev, self.T, self.S = row.device, row.shape[0], q_len.shape[0]
        self.out = torch.empty(self.T, spec.out_width, dtype=row.dtype, device=dev)
        self.p, self.c = _params(row, cols, spec, w, state, positions, slots, self.out, step), _lib.RecChunk()
        self.fp32, self.tail_rows = 1 if row.dtype == torch.float32 else 0, state.tail is not None
        self.tc = (impl or ("tc" if max_q_len >= TC_MIN_ROWS else "scan")) == "tc" and tc_ok(spec, row)
        c = self.c
        c.v_off = (2 * spec.groups * spec.dim + 7) // 8 * 8
        c.qkv_ld = c.v_off + (spec.out_width + 7) // 8 * 8
        qkv = torch.empty(self.T, c.qkv_ld, dtype=row.dtype, device=dev)
        gates = torch.empty(self.T, spec.heads, 2, dtype=torch.float32, device=dev)
        unit = torch.empty(self.T, 2, spec.groups, dtype=torch.float32, device=dev) if spec.corrects else None
        scratch = None
        if self.tc:
            size = _lib.lib().skein_rec_channel_scratch_bytes if spec.kind == "channel_delta" else _lib.lib().skein_rec_tc_scratch_bytes
            scratch = torch.empty(int(size(C.byref(self.p), self.T, self.S)), dtype=torch.uint8, device=dev)
        c.seq_of_token, c.q_start, c.q_len, c.max_q_len = seq_of_token.data_ptr(), q_start.data_ptr(), q_len.data_ptr(), int(max_q_len)
        c.qkv, c.gates, c.unit, c.chunk_mat = qkv.data_ptr(), gates.data_ptr(), _lib.ptr(unit), _lib.ptr(scratch)
        self._keep = (row, step, w, state, positions, slots, seq_of_token, q_start, q_len, qkv, gates, unit, scratch)

    def prep(self):
        """Convolution, silu, gates, unit norms."""
        _lib.check(_lib.lib().skein_rec_prep(C.byref(self.p), C.byref(self.c), self.T, self.fp32, _lib.stream_ptr()), "rec_prep")
        _lib.count_launch()

    def walk(self):
        """The recurrence; the state moves on."""
        if self.tc:
            form = _lib.lib().skein_rec_channel if self.p.kind == KINDS["channel_delta"] else _lib.lib().skein_rec_tc
            _lib.check(form(C.byref(self.p), C.byref(self.c), self.T, self.S, _lib.stream_ptr()), "rec_tc")
            _lib.count_launch(2)
        else:
            _lib.check(_lib.lib().skein_rec_scan(C.byref(self.p), C.byref(self.c), self.S, self.fp32, _lib.stream_ptr()), "rec_scan")
            _lib.count_launch()

    def tail(self):
        """The convolution's last inputs, once nothing reads the old ones any more."""
        if self.tail_rows:
            _lib.check(_lib.lib().skein_rec_tail(C.byref(self.p), C.byref(self.c), self.S, self.fp32, _lib.stream_ptr()), "rec_tail")
            _lib.count_launch()


def rec_chunk(row, cols: RecColumns, spec, w, state: RecState, positions, slots, seq_of_token, q_start, q_len, max_q_len, impl=None, step=None):
    """Portions of several sequences, one after another: rows q_start[s] .. + q_len[s] are consecutive tokens of the sequence in
    slots[s]. impl "tc" (chunks of 64 tokens on the tensor cores; the default for longer portions where it takes the sizes) or
    "scan" (one token after the other). step: see rec_step."""
    if not row.is_cuda:
        return rp.rec_chunk(row, cols, spec, w, state, positions, slots, q_start, q_len, step)
    run = ChunkRun(row, cols, spec, w, state, positions, slots, seq_of_token, q_start, q_len, max_q_len, impl, step)
    run.prep()
    run.walk()
    run.tail()
    return run.out
