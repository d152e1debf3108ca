"""Parallel layers, x <- x + (mixer(h) + ff(h)) with h = tanh(alpha x) w + b: specification, parameter names, weights; and the mixers
that other layers (models/prenorm_layers.py) share with them.

Mixers (specifications are data; a design picks some and fixes nothing else):

  WindowAttnSpec   grouped-query attention over a sliding window, over chunks or over everything before; RMS norm of the whole q and k
                   projections (or none), then rotation of the first rot_dims dimensions of every head (pairs i, i + rot_dims / 2, or
                   neighbours; frequencies divided by rot_factor), then unit heads (or not); a sink; two maps per head of which the
                   second is subtracted; an output gate; biases on the projections; RMS norm with a weight per head; a cap on the scores;
                   a window's first tokens kept in sight; a learned sink per head; values mixed with those of the first such layer
  RecurrentSpec    a matrix state S [dim, vdim] per head, 32-bit, carried from token to token:
                       S <- g S + k u^T,   o = S^T q (+ D v)
                     "delta"      g per head and token, u = beta (v - (g S)^T k), q and k unit vectors
                     "ssd"        g = exp(-exp(A) dt), u = dt v (Mamba-2; q, k, v are C, B, x)
                     "lightning"  g fixed per head, u = v
                     "channel_delta"  "delta" with one g per head, token and row of S; g and the output's gate come from a bottleneck each
  SelectiveSpec    a diagonal recurrence per channel (Mamba), 32-bit, behind a short convolution:
                       S[n, c] <- exp(dt[c] A[n, c]) S[n, c] + dt[c] x[c] B[n],   y[c] = sum_n S[n, c] C[n] + D[c] x[c],   y silu(z)
  MixerPairSpec    an attention and a recurrence beside each other, summed with a weight each

A parallel layer runs as one product from h (w_in: the feed-forward's up projection and every projection of the mixer, stacked), the
mixer's own kernels, and one product back (w_out: the mixers' output projections and the feed-forward's down projection side
by side, so that their sum is the product's). LayerLayout says where everything sits in the row between the two products:

    [ mixer outputs | feed-forward (activated in place) | projections of the mixers ]
      <------------ read by w_out ------------------->
                      <--------------- written by w_in ------------------------------>

Every section starts at a multiple of 8 elements.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch


class SpecError(ValueError):
    pass


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class WindowAttnSpec:
    heads: int
    kv_heads: int
    dim: int                 # of a query / key head
    vdim: int
    scale: float
    rot_dims: int
    rope_base: float
    rope_factor: float = 1.0
    window: int = 0          # position i sees j with 0 <= i - j < window (0: every earlier position)
    kind: str = ""           # mixer type of the configuration, where the attention is a mixer of its own
    chunk: int = 0           # position i sees the j of its own chunk of this many positions, counted from 0 (0: no chunks)
    row_norm: bool = True    # RMS norm over all of q and all of k, with a weight, before the rotation
    interleaved: bool = False    # rotated pairs are neighbours
    unit: bool = False       # heads of q and k are divided by their root mean square after the rotation
    sink: bool = False       # one more term exp(0) in the softmax's denominator
    diff: float | None = None    # two maps per head over the same values: (1 - diff) N(map 1 - lambda map 2) with lambda learned around diff
    gated: bool = False      # the output is multiplied by the sigmoid of a projection
    bias: bool = False       # q, k and v have biases
    head_norm: bool = False  # RMS norm of every head of q and k, with a weight that the heads share, before the rotation
    softcap: float = 0.0     # scores are softcap * tanh(score / softcap) (0: as they are)
    keep_first: int = 0      # with a window: the sequence's first tokens that every position sees
    head_sink: bool = False  # one more term exp(a learned number per head) in the softmax's denominator
    v_mix: bool = False      # values are mixed with those that the first such layer has for the token

    @property
    def maps(self) -> int:
        return 1 if self.diff is None else 2

    @property
    def head_size(self) -> int:
        return self.dim

    @property
    def key_width(self) -> int:
        """Elements of a key head in the cache: its maps side by side."""
        return self.maps * self.dim

    @property
    def cache_elems_per_token(self) -> int:
        return self.kv_heads * (self.key_width + self.vdim)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def sections(self) -> list:
        """(tensor, rows) of the projections of h, in stacking order."""
        s = [("q", self.heads * self.key_width), ("k", self.kv_heads * self.key_width), ("v", self.kv_heads * self.vdim)]
        return s + [("g", self.out_width)] if self.gated else s

    def param_shapes(self, C: int) -> dict:
        s = {n: (rows, C) for n, rows in self.sections()}
        if self.row_norm:
            s["q.norm"], s["k.norm"] = (self.heads * self.dim,), (self.kv_heads * self.dim,)
        if self.bias:
            s.update({n + ".b": (rows,) for n, rows in self.sections()[:3]})
        if self.head_norm:
            s["q.norm"], s["k.norm"] = (self.dim,), (self.dim,)
        if self.diff is not None:
            s.update({n: (self.dim,) for n in LAMBDA_VECTORS})
        if self.v_mix:
            s["vmix"] = ()
        if self.head_sink:
            s["sink"] = (self.heads,)
        s["o"] = (C, self.out_width)
        return s

    def to_dict(self) -> dict:
        rot = {"base": self.rope_base, "dims": self.rot_dims}
        if self.rope_factor != 1.0:
            rot["scaling"] = {"factor": self.rope_factor}
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot_dims or not self.head_norm:
            d["rot"] = rot
        if self.window or self.chunk:
            d["mask"] = {"size": self.window or self.chunk}
            if self.keep_first:
                d["mask"]["keep_first"] = self.keep_first
        if self.softcap:
            d["softcap"] = self.softcap
        if self.v_mix:
            d["v_mix"] = True
        if self.diff is not None:
            d["diff"] = self.diff
        return d


LAMBDA_VECTORS = ("lq1", "lk1", "lq2", "lk2")      # lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff


@dataclass(frozen=True)
class RecurrentSpec:
    kind: str                # "delta", "channel_delta", "ssd" or "lightning"
    heads: int               # value heads (one state each)
    groups: int              # query / key heads; head h uses h // (heads / groups)
    dim: int                 # of a query / key head: rows of the state
    vdim: int                # columns of the state
    taps: int = 1            # of the short convolutions over time (1 for "lightning": none)
    norm_groups: int = 1     # equal parts of the normed output that have a root mean square each ("ssd")
    decay: tuple = ()        # "lightning"
    decay_rank: int = 0      # "channel_delta": widths of the bottlenecks in front of the decays ...
    gate_rank: int = 0       # ... and of the output's gate

    @property
    def corrects(self) -> bool:
        """The delta rules: what the state holds for k is replaced, and q and k are unit vectors."""
        return self.kind in ("delta", "channel_delta")

    @property
    def cache_elems_per_token(self) -> int:
        return 0

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def head_size(self) -> int:
        return self.dim

    @property
    def conv_channels(self) -> int:
        """Channels that pass a convolution: queries, keys and values together."""
        return 2 * self.groups * self.dim + self.heads * self.vdim if self.kind != "lightning" else 0

    @property
    def conv_rows(self) -> int:
        """Cached inputs of the convolution. One more than it looks back, so that a step writes no row that it reads."""
        return self.taps if self.conv_channels and self.taps > 1 else 0

    @property
    def state_elems(self) -> int:
        return self.heads * self.dim * self.vdim

    def state_bytes(self, elem: int = 2) -> int:
        """Bytes of one sequence's state: the 32-bit matrices and the convolution's last inputs."""
        return 4 * self.state_elems + elem * self.conv_rows * self.conv_channels

    def sections(self) -> list:
        GD, HV = self.groups * self.dim, self.heads * self.vdim
        if self.kind == "ssd":      # rows of the one input matrix: z | x | B | C | dt
            return [("z", HV), ("conv", HV + 2 * GD), ("dt", self.heads)]
        if self.kind == "channel_delta":
            return [("q", GD), ("k", GD), ("v", HV), ("b", self.heads), ("a1", self.decay_rank), ("g1", self.gate_rank)]
        qkv = [("q", GD), ("k", GD), ("v", HV), ("g", HV)]
        return qkv + [("b", self.heads), ("a", self.heads)] if self.kind == "delta" else qkv

    def param_shapes(self, C: int) -> dict:
        H, GD, HV = self.heads, self.groups * self.dim, self.heads * self.vdim
        if self.kind == "ssd":
            ch = self.conv_channels
            return {"in": (2 * HV + 2 * GD + H, C), "conv": (ch, self.taps), "conv.b": (ch,), "dt_bias": (H,), "A_log": (H,), "D": (H,),
                    "norm": (HV,), "o": (C, HV)}
        s = {n: (rows, C) for n, rows in self.sections()}
        if self.kind == "delta":
            s.update({n + ".conv": (rows, self.taps) for n, rows in self.sections()[:3]})
            s.update({"A_log": (H,), "dt_bias": (H,), "norm": (self.vdim,)})
        elif self.kind == "channel_delta":
            s.update({n + ".conv": (rows, self.taps) for n, rows in self.sections()[:3]})
            s.update({"A_log": (H,), "norm": (self.vdim,), "a2": (H * self.dim, self.decay_rank), "dt_bias": (H * self.dim,),
                      "g2": (HV, self.gate_rank)})
        else:
            s["norm"] = (HV,)
        s["o"] = (C, HV)
        return s

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}
        if self.kind == "ssd":
            return {"conv": self.taps, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups, "state": self.dim,
                    "vdim": self.vdim}
        if self.kind == "delta":
            return {**d, "conv": self.taps, "kv_heads": self.groups}
        if self.kind == "channel_delta":
            return {**d, "conv": self.taps, "kv_heads": self.groups, "decay_rank": self.decay_rank, "gate_rank": self.gate_rank}
        return {**d, "decay": list(self.decay)}


@dataclass(frozen=True)
class SelectiveSpec:
    inner: int               # channels
    state: int               # state dimensions of a channel
    dt_rank: int             # width of the step sizes' bottleneck
    taps: int = 1            # of the short convolution over time
    kind: str = "mamba1"
    heads: int = 1

    @property
    def cache_elems_per_token(self) -> int:
        return 0

    @property
    def out_width(self) -> int:
        return self.inner

    @property
    def head_size(self) -> int:
        return self.state

    @property
    def conv_channels(self) -> int:
        return self.inner

    @property
    def conv_rows(self) -> int:
        """Cached inputs of the convolution. One more than it looks back, so that a step writes no row that it reads."""
        return self.taps if self.taps > 1 else 0

    @property
    def state_elems(self) -> int:
        return self.inner * self.state

    def state_bytes(self, elem: int = 2) -> int:
        return 4 * self.state_elems + elem * self.conv_rows * self.inner

    def sections(self) -> list:
        return [("x", self.inner), ("z", self.inner)]

    def x_sections(self) -> list:
        """(name, rows) of the projections of the convolved x: step sizes' bottleneck, B, C."""
        return [("dt", self.dt_rank), ("B", self.state), ("C", self.state)]

    def param_shapes(self, C: int) -> dict:
        I, N, R = self.inner, self.state, self.dt_rank
        return {"in": (2 * I, C), "conv": (I, self.taps), "conv.b": (I,), "x": (R + 2 * N, I), "dt": (I, R), "dt.b": (I,), "A_log": (I, N),
                "D": (I,), "o": (C, I)}

    def to_dict(self) -> dict:
        return {"conv": self.taps, "dt_rank": self.dt_rank, "inner": self.inner, "state": self.state}


@dataclass(frozen=True)
class MixerPairSpec:
    left: WindowAttnSpec
    right: RecurrentSpec
    left_scale: float = 1.0
    right_scale: float = 1.0
    kind: str = "parallel"

    @property
    def heads(self) -> int:
        return self.left.heads

    @property
    def head_size(self) -> int:
        return self.left.dim

    @property
    def cache_elems_per_token(self) -> int:
        return self.left.cache_elems_per_token

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(), "right_scale": self.right_scale}


def attention_of(mixer) -> WindowAttnSpec | None:
    return mixer.left if isinstance(mixer, MixerPairSpec) else mixer if isinstance(mixer, WindowAttnSpec) else None


def recurrence_of(mixer) -> RecurrentSpec | SelectiveSpec | None:
    return mixer.right if isinstance(mixer, MixerPairSpec) else mixer if isinstance(mixer, (RecurrentSpec, SelectiveSpec)) else None


# ---- configuration -------------------------------------------------------------------------------------------------
def _need(ok: bool, what: str) -> None:
    if not ok:
        raise SpecError(what)


def parse_window(m: dict, mask: str = "window", **fixed) -> WindowAttnSpec:
    """An attention mixer; `mask` is what mask.size counts ("window" or "chunk"), `fixed` the properties that the design fixes."""
    rot, size = m["rot"], int((m.get("mask") or {}).get("size") or 0)
    a = WindowAttnSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                       rot_dims=int(rot["dims"]), rope_base=float(rot["base"]), rope_factor=float((rot.get("scaling") or {}).get("factor", 1.0)),
                       **{mask: size}, **fixed)
    _need(a.heads % a.kv_heads == 0, "heads must be a multiple of kv_heads")
    _need(a.rot_dims % 2 == 0 and 0 <= a.rot_dims <= a.dim, "rot.dims must be even and at most dim (rotation turns pairs)")
    _need(size >= 0 and a.rope_factor > 0, "mask.size and rot.scaling.factor must be positive")
    return a


def parse_differential(m: dict) -> WindowAttnSpec:
    return parse_window(m, kind="attention", row_norm=False, interleaved=True, diff=float(m["diff"]), gated=True)


def parse_chunked(m: dict) -> WindowAttnSpec:
    a = parse_window(m, mask="chunk", kind="attention_2", row_norm=False, interleaved=True, unit=True, sink=True)
    _need(a.chunk > 0, "mask.size must be positive")
    return a


def parse_selective(m: dict) -> SelectiveSpec:
    r = SelectiveSpec(inner=int(m["inner"]), state=int(m["state"]), dt_rank=int(m["dt_rank"]), taps=int(m["conv"]))
    _need(min(r.inner, r.state, r.dt_rank) >= 1, "inner, state and dt_rank must be positive")
    _need(r.taps >= 1, "conv must be at least 1")
    return r


def parse_ssd(m: dict) -> RecurrentSpec:
    r = RecurrentSpec("ssd", heads=int(m["heads"]), groups=int(m["groups"]), dim=int(m["state"]), vdim=int(m["vdim"]), taps=int(m["conv"]),
                      norm_groups=int(m["norm_groups"]))
    _need(r.heads % r.groups == 0, "heads must be a multiple of groups")
    _need(r.norm_groups >= 1 and r.out_width % r.norm_groups == 0, "norm_groups must divide heads * vdim")
    _need(r.taps >= 1, "conv must be at least 1")
    return r


def parse_delta(m: dict) -> RecurrentSpec:
    r = RecurrentSpec("delta", heads=int(m["heads"]), groups=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), taps=int(m["conv"]))
    _need(r.heads % r.groups == 0, "heads must be a multiple of kv_heads")
    _need(r.taps >= 1, "conv must be at least 1")
    return r


def parse_channel_delta(m: dict) -> RecurrentSpec:
    """A configuration that does not name the bottlenecks' widths leaves them to the checkpoint (models/prenorm_layers.py: fill_ranks); where
    there is none they are a key head's size."""
    r = RecurrentSpec("channel_delta", heads=int(m["heads"]), groups=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), taps=int(m["conv"]),
                      decay_rank=int(m.get("decay_rank") or m["dim"]), gate_rank=int(m.get("gate_rank") or m["dim"]))
    _need(r.heads % r.groups == 0, "heads must be a multiple of kv_heads")
    _need(r.taps >= 1, "conv must be at least 1")
    return r


def parse_kept_window(m: dict) -> WindowAttnSpec:
    """Attention without rotation over a window that keeps the first tokens in sight."""
    mask = m.get("mask") or {}
    a = WindowAttnSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), rot_dims=0,
                       rope_base=1e4, window=int(mask.get("size") or 0), kind="attention", row_norm=False, bias=True, head_norm=True,
                       softcap=float(m.get("softcap") or 0.0), keep_first=int(mask.get("keep_first") or 0), head_sink=True,
                       v_mix=bool(m.get("v_mix")))
    _need(a.heads % a.kv_heads == 0, "heads must be a multiple of kv_heads")
    _need(a.window >= 0 and a.keep_first >= 0 and a.softcap >= 0, "mask.size, mask.keep_first and softcap must not be negative")
    return a


def parse_lightning(m: dict) -> RecurrentSpec:
    r = RecurrentSpec("lightning", heads=int(m["heads"]), groups=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                      decay=tuple(float(x) for x in m["decay"]))
    _need(len(r.decay) == r.heads, "decay must list one number per head")
    _need(all(0.0 <= d <= 1.0 for d in r.decay), "decay must lie in [0, 1]")
    return r


def parse_pair(m: dict) -> MixerPairSpec:
    return MixerPairSpec(parse_window(m["left"]), parse_ssd(m["right"]), float(m["left_scale"]), float(m["right_scale"]))


def parse_loop(loop: dict | None, n: int):
    """(start, stop, times) or None."""
    if not loop:
        return None
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start < stop <= n or times < 1:
        raise SpecError(f"loop {start}..{stop} x {times} is not a range of the {n} layers")
    return start, stop, times


def layer_runs(n: int, loop) -> list:
    """(layer, pass) in the order they run; pass is None outside the loop."""
    if loop is None:
        return [(i, None) for i in range(n)]
    a, b, times = loop
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(times) for i in range(a, b)] + [(i, None) for i in range(b, n)])


# ---- parameters --------------------------------------------------------------------------------------------------
def _mixer_parts(mixer):
    """(name prefix under the layer, specification, weight of its output)."""
    if isinstance(mixer, MixerPairSpec):
        return [("mix.left.", mixer.left, mixer.left_scale), ("mix.right.", mixer.right, mixer.right_scale)]
    return [("mix.", mixer, 1.0)]


def _norm_shapes(name: str, C: int) -> dict:
    return {name: (C,), name + ".b": (C,), name + ".alpha": ()}


def param_shapes(cfg) -> dict:
    C, s = cfg.hidden_size, {}
    if cfg.loop is not None:
        s["loop.in"], s["loop.step"] = (C, 2 * C), (cfg.loop[2], C)
    for sp in sorted((sp for sp in cfg.layers if sp.weights_of is None), key=lambda sp: sp.tensors):
        p = f"l{sp.tensors}."
        s.update(_norm_shapes(p + "norm1", C))
        for pre, m, _ in _mixer_parts(sp.mixer):
            s.update({p + pre + n: shape for n, shape in m.param_shapes(C).items()})
        if sp.mlp is not None:
            s[p + "mlp.up"], s[p + "mlp.down"] = (sp.mlp.ff, C), (C, sp.mlp.ff)
    s.update(_norm_shapes("final.norm", C))
    return s


def active_params(cfg) -> int:
    C = cfg.hidden_size
    n = 2 * C * C * cfg.loop[2] if cfg.loop is not None else 0
    for sp in cfg.layers:
        lay = LayerLayout(sp)
        n += C * (lay.in_rows + lay.out_cols)
    return n


@dataclass
class Section:
    """Columns of a layer's row (LayerLayout) that belong to one mixer."""
    spec: object
    scale: float             # weight of the mixer's output in the layer's sum
    out: int                 # first column of its output
    col: dict                # projection -> first column


class LayerLayout:
    """`ff` False: the feed-forward is not part of the row (layers that run it behind the mixer)."""

    def __init__(self, sp, ff: bool = True):
        self.parts, at = [], 0
        parts = _mixer_parts(sp.mixer)
        for _, m, scale in parts:
            self.parts.append(Section(m, scale, at, {}))
            at += up8(m.out_width)
        self.ff, self.ff_cols = at, up8(sp.mlp.ff) if ff and sp.mlp is not None else 0
        self.in_first = at               # w_in writes from here
        at += self.ff_cols
        self.out_cols = at               # w_out reads up to here
        for sec in self.parts:
            for name, rows in sec.spec.sections():
                sec.col[name] = at
                at += up8(rows)
        self.width, self.in_rows = at, at - self.in_first
        self.zero_fill = any(m.out_width % 8 for _, m, _ in parts)      # columns that w_out reads and nothing writes

    def part(self, cls):
        return next((s for s in self.parts if isinstance(s.spec, cls)), None)


# ---- weights ------------------------------------------------------------------------------------------------------
@dataclass
class TanhNorm:
    """tanh(alpha x) w + b."""
    alpha: torch.Tensor      # [1] fp32
    w: torch.Tensor          # [C] fp32
    b: torch.Tensor          # [C] fp32


@dataclass
class WindowAttnWeights:
    q_norm: torch.Tensor | None = None     # [heads * dim] fp32, or [dim] with a norm per head
    k_norm: torch.Tensor | None = None     # [kv_heads * dim] fp32, or [dim]
    lam: torch.Tensor | None = None        # [1] fp32: weight of the second map
    q_bias: torch.Tensor | None = None     # fp32
    k_bias: torch.Tensor | None = None
    v_bias: torch.Tensor | None = None
    sinks: torch.Tensor | None = None      # [heads] fp32
    vmix: torch.Tensor | None = None       # [1] fp32: weight of the first such layer's values


@dataclass
class SelectiveWeights:
    w_x: torch.Tensor                      # [x_rows, inner]: the sections of x_sections, each from a multiple of 8 rows
    w_dt: torch.Tensor                     # [inner, dt_rank], columns padded with zeros to a multiple of 8
    conv: torch.Tensor                     # [taps, inner] fp32
    conv_b: torch.Tensor                   # [inner] fp32
    dt_bias: torch.Tensor                  # [inner] fp32
    neg_a: torch.Tensor                    # [state, inner] fp32: -exp(A_log)
    skip: torch.Tensor                     # [inner] fp32: D


@dataclass
class RecurrentWeights:
    norm: torch.Tensor                     # output norm, fp32: [vdim] (delta rules) or [heads * vdim]
    conv: torch.Tensor | None = None       # [taps, channels] fp32, channels q | k | v (zero taps of "lightning": none)
    conv_b: torch.Tensor | None = None     # [channels] fp32
    neg_decay: torch.Tensor | None = None  # [heads] fp32: -exp(A_log), or log(decay) of "lightning"
    decay: torch.Tensor | None = None      # [heads] fp32, "lightning"
    dt_bias: torch.Tensor | None = None    # [heads] fp32, or [heads * dim] ("channel_delta")
    skip: torch.Tensor | None = None       # [heads] fp32: D
    w_decay: torch.Tensor | None = None    # [heads * dim, decay_rank], columns padded with zeros to a multiple of 8 ("channel_delta")
    w_gate: torch.Tensor | None = None     # [heads * vdim, gate_rank], likewise


@dataclass
class ParallelLayerWeights:
    norm: TanhNorm
    w_in: torch.Tensor                     # [in_rows, C]
    w_out: torch.Tensor                    # [C, out_cols]
    attn: WindowAttnWeights | None = None
    rec: RecurrentWeights | None = None
    fp8: dict = field(default_factory=dict)


@dataclass
class LoopWeights:
    w_in: torch.Tensor                     # [C, 2 C]: the stream, then the embedding output
    step: torch.Tensor                     # [times, C] fp32


def load_tanh_norm(get, name: str) -> TanhNorm:
    return TanhNorm(get(name + ".alpha").float().reshape(1), get(name).float(), get(name + ".b").float())


def load_loop(cfg, get) -> LoopWeights | None:
    return None if cfg.loop is None else LoopWeights(get("loop.in").contiguous(), get("loop.step").float())


def _pad(t: torch.Tensor, dim: int) -> torch.Tensor:
    n = up8(t.shape[dim]) - t.shape[dim]
    if n == 0:
        return t
    shape = list(t.shape)
    shape[dim] = n
    return torch.cat([t, torch.zeros(shape, dtype=t.dtype, device=t.device)], dim=dim)


def load_attention(m: WindowAttnSpec, get, p: str) -> WindowAttnWeights:
    w = WindowAttnWeights()
    if m.row_norm or m.head_norm:
        w.q_norm, w.k_norm = get(p + "q.norm").float(), get(p + "k.norm").float()
    if m.diff is not None:
        lq1, lk1, lq2, lk2 = (get(p + n).double() for n in LAMBDA_VECTORS)
        w.lam = ((lq1 * lk1).sum().exp() - (lq2 * lk2).sum().exp() + m.diff).float().reshape(1)
    if m.bias:
        w.q_bias, w.k_bias, w.v_bias = (get(p + n + ".b").float() for n in ("q", "k", "v"))
    if m.head_sink:
        w.sinks = get(p + "sink").float()
    if m.v_mix:
        w.vmix = get(p + "vmix").float().reshape(1)
    return w


def load_selective(m: SelectiveSpec, get, p: str) -> SelectiveWeights:
    x = get(p + "x").split([rows for _, rows in m.x_sections()])
    return SelectiveWeights(w_x=torch.cat([_pad(t, 0) for t in x]).contiguous(), w_dt=_pad(get(p + "dt"), 1).contiguous(),
                            conv=get(p + "conv").float().t().contiguous(), conv_b=get(p + "conv.b").float(), dt_bias=get(p + "dt.b").float(),
                            neg_a=-get(p + "A_log").float().t().exp().contiguous(), skip=get(p + "D").float())


def load_recurrence(m: RecurrentSpec, get, p: str) -> RecurrentWeights:
    w = RecurrentWeights(norm=get(p + "norm").float())
    GD, HV = m.groups * m.dim, m.heads * m.vdim
    if m.kind == "lightning":
        d = torch.tensor(m.decay, dtype=torch.float64)
        w.decay, w.neg_decay = (t.to(w.norm.device) for t in (d.float(), d.log().clamp(min=-1e30).float()))
        return w
    w.neg_decay, w.dt_bias = -get(p + "A_log").float().exp(), get(p + "dt_bias").float()
    if m.kind == "channel_delta":
        w.w_decay, w.w_gate = _pad(get(p + "a2"), 1).contiguous(), _pad(get(p + "g2"), 1).contiguous()
    if m.corrects:
        w.conv = torch.cat([get(p + n + ".conv").float() for n in ("q", "k", "v")]).t().contiguous()
    else:      # the checkpoint's order is x (values) | B (keys) | C (queries)
        c, b = get(p + "conv").float(), get(p + "conv.b").float()
        order = torch.cat([torch.arange(HV + GD, HV + 2 * GD), torch.arange(HV, HV + GD), torch.arange(HV)]).to(c.device)
        w.conv, w.conv_b, w.skip = c[order].t().contiguous(), b[order].contiguous(), get(p + "D").float()
    return w


def assemble_layer(sp, get) -> ParallelLayerWeights:
    p = f"l{sp.tensors}."
    ins, outs = [], []
    attn = rec = None
    if sp.mlp is not None:
        ins.append(get(p + "mlp.up"))
    for pre, m, _ in _mixer_parts(sp.mixer):
        q = p + pre
        if isinstance(m, WindowAttnSpec):
            attn = load_attention(m, get, q)
        else:
            rec = load_recurrence(m, get, q)
        if isinstance(m, RecurrentSpec) and m.kind == "ssd":
            rows, whole = m.sections(), get(q + "in")
            ins.extend(whole.split([n for _, n in rows]))
        else:
            ins.extend(get(q + n) for n, _ in m.sections())
        outs.append(_pad(get(q + "o"), 1))
    if sp.mlp is not None:
        outs.append(_pad(get(p + "mlp.down"), 1))
    return ParallelLayerWeights(norm=load_tanh_norm(get, p + "norm1"), w_in=torch.cat([_pad(t, 0) for t in ins]).contiguous(),
                                w_out=torch.cat(outs, dim=1).contiguous(), attn=attn, rec=rec)


def random_param(name: str, shape, gen, device):
    """Seeded random values of the parameters that are neither projections nor gains: decays between slow and fast, small steps,
    convolution taps and biases of order one; None for the others."""
    def normal(std, mean=0.0):
        return torch.empty(shape, dtype=torch.float32, device=device).normal_(mean, std, generator=gen)
    if name.endswith(".alpha"):
        return torch.ones(shape, device=device)
    if name.endswith((".norm1.b", "norm.b", ".conv.b", "loop.step", ".q.b", ".k.b", ".v.b", ".sink")):
        return normal(0.02)
    if name.endswith(".conv"):
        return normal(shape[-1] ** -0.5)
    if name.endswith(".A_log"):
        return normal(1.0)
    if name.endswith((".dt_bias", ".dt.b")):
        return normal(1.0, -3.0)
    if name.endswith(tuple("." + n for n in LAMBDA_VECTORS)):
        return normal(0.1)
    if name.endswith(".D"):
        return torch.ones(shape, device=device)
    if name.endswith((".shift", ".vmix")):
        return normal(0.1, 0.5)
    if name.endswith(".dwa"):      # near the layer's own result
        t = normal(0.02)
        t[-1] += 1.0
        return t
    return None
