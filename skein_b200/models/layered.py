"""Designs whose configuration lists the layers one by one, each with its own mixer and feed-forward: specification,
parameter names and shapes, weights.

Three kinds of layers exist. A post-norm layer is x <- norm1(alpha x + mixer(h)), x <- norm2(alpha x + ff(x)), with RMS norms
whose gain is one number, and h = x + (short causal convolution of x over time). A parallel layer is
x <- x + (mixer(h) + ff(h)) with h = tanh(a x) w + b (models/parallel_layers.py). A pre-norm layer is x <- x + mixer(norm1(x)),
x <- x + ff(norm2(x)) with RMS norms (models/prenorm_layers.py). Several layers may use one layer's tensors
(`weights_of`); each keeps a cache of its own. A range of layers may run several times (`loop`): ModelConfig.layers then lists
every run, the later ones with `weights_of` the first. The registry below names, per architecture, the kind of its layers and
which mixers exist:

  Zarorax   latent_attention     latent attention, queries through a latent of their own
            latent_attention_2   latent attention, queries straight from the input, output gated by a sigmoid
  Sikalorn  parallel             sliding-window attention beside a state-space recurrence, both on the same input
            delta                gated delta rule
            lightning            linear attention with a fixed decay per head
  Barorax   attention            differential attention (two maps per head over the same values), gated
            attention_2          attention inside chunks, unit queries and keys, a sink
            mamba1               selective scan
  Derusun   latent_attention     latent attention, queries straight from the input, a learned sink per head
            attention            grouped-query attention over a window that keeps the first tokens; biases, head norms, capped scores, a
                                 learned sink per head, values mixed with the first such layer's
            channel_delta        gated delta rule with a decay per head and key channel
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from . import parallel_layers as pl
from .parallel_layers import MixerPairSpec, RecurrentSpec, SelectiveSpec, SpecError, WindowAttnSpec  # noqa: F401

# architecture -> mixer type -> (queries through a latent, output gate), or the parser of the mixer
LAYERED_ARCHS = {"Zarorax": {"latent_attention": (True, False), "latent_attention_2": (False, True)},
                 "Sikalorn": {"parallel": pl.parse_pair, "delta": pl.parse_delta, "lightning": pl.parse_lightning},
                 "Barorax": {"attention": pl.parse_differential, "attention_2": pl.parse_chunked, "mamba1": pl.parse_selective},
                 "Derusun": {"latent_attention": lambda m: parse_latent(m, "latent_attention", False, False, sink=True),
                             "attention": pl.parse_kept_window, "channel_delta": pl.parse_channel_delta}}
PARALLEL_ARCHS = {"Sikalorn"}              # the architectures of parallel layers
PRENORM_ARCHS = {"Barorax", "Derusun"}     # ... and of pre-norm layers
SHIFTED_ARCHS = {"Derusun"}                # pre-norm layers behind a token shift and an average over depth (models/prenorm_layers.py)

GLU_SLOPE = 1.702          # g * sigmoid(GLU_SLOPE * g) of the clamped gated unit


@dataclass(frozen=True)
class LatentMixerSpec:
    kind: str                # mixer type of the configuration
    heads: int
    dim: int                 # unrotated query / key dimensions per head
    rot_dim: int             # rotated query / key dimensions per head (the key part is shared by all heads)
    vdim: int
    kv_rank: int
    rope_base: float
    scale: float
    q_rank: int = 0          # 0: queries straight from the input
    gated: bool = False
    sink: bool = False       # one more term exp(a learned number per head) in the softmax's denominator

    @property
    def cache_width(self) -> int:
        """Elements cached per token: the normed latent and the rotated key part."""
        return self.kv_rank + self.rot_dim

    @property
    def q_width(self) -> int:
        return self.heads * (self.dim + self.rot_dim)

    @property
    def head_size(self) -> int:
        return self.dim + self.rot_dim

    @property
    def cache_elems_per_token(self) -> int:
        return self.cache_width

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def sections(self) -> list:
        """(tensor, rows) of the projections of a pre-norm layer's input, in stacking order."""
        return [("q", self.q_width), ("dkv", self.cache_width)]

    def param_shapes(self, C: int) -> dict:
        s = {n: (rows, C) for n, rows in self.sections()}
        s["dkv.norm"], s["uk"], s["uv"] = (self.kv_rank,), (self.heads * self.dim, self.kv_rank), (self.heads * self.vdim, self.kv_rank)
        if self.sink:
            s["sink"] = (self.heads,)
        s["o"] = (C, self.out_width)
        return s

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank, "scale": self.scale,
             "rot": {"base": self.rope_base, "dims": self.rot_dim}}
        return {**d, "q_rank": self.q_rank} if self.q_rank else d


def parse_latent(m: dict, kind: str, q_latent: bool, gated: bool, sink: bool = False) -> LatentMixerSpec:
    rot = m["rot"]
    if int(rot["dims"]) != int(m["rot_dim"]):
        raise SpecError("rot.dims must equal rot_dim")
    mixer = LatentMixerSpec(kind=kind, heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                            kv_rank=int(m["kv_rank"]), rope_base=float(rot["base"]), scale=float(m["scale"]),
                            q_rank=int(m["q_rank"]) if q_latent else 0, gated=gated, sink=sink)
    if mixer.rot_dim % 2:
        raise SpecError("rot_dim must be even (rotation turns pairs)")
    return mixer


@dataclass(frozen=True)
class DenseFFSpec:
    ff: int
    limit: float | None = None   # of a clamped gated unit (gate and up projections); None: the design's ungated unit


@dataclass(frozen=True)
class RoutedFFSpec:
    ff: int                  # of one expert
    limit: float | None      # of the clamped gated unit; None: silu(g) u
    experts: int
    top: int
    groups: int = 1          # neighbouring experts form equal groups ...
    keep: int = 1            # ... of which the best `keep` are eligible
    score: str = "softmax"   # of the router's logits: softmax over all experts, or a sigmoid each
    group_best: int = 1      # a group's score is the sum of its 1 or 2 largest scores
    renorm: bool = False     # the chosen scores are divided by their sum
    scale: float = 1.0       # ... and multiplied by this
    shared_ff: int = 0       # size of an expert that runs for every token (0: none)

    def check(self) -> None:
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep <= self.groups or not 1 <= self.top <= self.keep * (self.experts // self.groups):
            raise SpecError(f"{self.top} of {self.experts} experts cannot be chosen from {self.keep} of {self.groups} groups")


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentMixerSpec | MixerPairSpec | RecurrentSpec | WindowAttnSpec | SelectiveSpec
    mlp: DenseFFSpec | RoutedFFSpec | None
    weights_of: int | None = None
    tensors: int | None = None     # number of this layer in the checkpoint's names, where that is not its place in the list
    loop_pass: int | None = None   # this layer opens the loop's pass of that number


def parse_layers(arch: str, layers: list, loop: dict | None = None) -> tuple:
    """The configuration's `layers` list (and `loop`) -> LayerSpec tuple (`weights_of` chains resolved to the layer that owns
    tensors, loops to one entry per run)."""
    if arch in PARALLEL_ARCHS | PRENORM_ARCHS:
        return _parse_runs(arch, layers, loop)
    kinds = LAYERED_ARCHS[arch]
    out = []
    for i, d in enumerate(layers):
        if d.get("type") not in kinds:
            raise SpecError(f"layer {i}: mixer type {d.get('type')!r} is not part of {arch}")
        try:
            mixer = parse_latent(d["mixer"], d["type"], *kinds[d["type"]])
        except SpecError as e:
            raise SpecError(f"layer {i}: {e}") from e
        mlp = d.get("mlp")
        if mlp is None:
            ff = None
        elif mlp["kind"] == "dense":
            ff = DenseFFSpec(int(mlp["ff"]))
        elif mlp["kind"] == "moe":
            r = mlp["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            ff = RoutedFFSpec(int(mlp["expert"]["ff"]), float(mlp["expert"]["limit"]), int(r["experts"]), int(r["top"]),
                              int(g["count"]), int(g["keep"]))
            try:
                ff.check()
            except SpecError as e:
                raise SpecError(f"layer {i}: {e}") from e
        else:
            raise SpecError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not supported")
        src = d.get("weights_of")
        if src is not None:
            src = int(src)
            if not 0 <= src < i:
                raise SpecError(f"layer {i}: weights_of {src} does not name an earlier layer")
            owner = out[src]
            if (owner.mixer, owner.mlp) != (mixer, ff):
                raise SpecError(f"layer {i} differs from layer {src}, whose tensors it uses")
            src = owner.weights_of if owner.weights_of is not None else src
        out.append(LayerSpec(mixer, ff, src))
    return tuple(out)


def _parse_dense(mlp: dict) -> DenseFFSpec:
    if mlp["kind"] != "dense":
        raise SpecError(f"feed-forward kind {mlp['kind']!r} is not supported")
    return DenseFFSpec(int(mlp["ff"]))


def _parse_runs(arch: str, layers: list, loop: dict | None) -> tuple:
    """Layers whose mixers have a parser each, one entry per run of a loop."""
    specs, parse_ff = [], pn.PARSE_FF.get(arch, _parse_dense)
    for i, d in enumerate(layers):
        parse = LAYERED_ARCHS[arch].get(d.get("type"))
        if parse is None:
            raise SpecError(f"layer {i}: mixer type {d.get('type')!r} is not part of {arch}")
        mlp = d.get("mlp")
        try:
            specs.append((parse(d["mixer"]), parse_ff(mlp) if mlp is not None else None))
        except SpecError as e:
            raise SpecError(f"layer {i}: {e}") from e
    if arch in SHIFTED_ARCHS:
        if loop:
            raise SpecError(f"{arch} has no loop")
        pn.check_value_mixing([m for m, _ in specs])
    return unroll_loop(specs, pl.parse_loop(loop, len(specs)))


def unroll_loop(specs, loop) -> tuple:
    """(mixer, mlp) pairs in checkpoint order and a loop (start, stop, times) or None -> one LayerSpec per run."""
    first, out = {}, []
    for i, t in pl.layer_runs(len(specs), loop):
        opens = t if (loop is not None and i == loop[0]) else None
        out.append(LayerSpec(*specs[i], weights_of=first.get(i), tensors=i, loop_pass=opens))
        first.setdefault(i, len(out) - 1)
    return tuple(out)


def layers_to_list(layers) -> list:
    """Inverse of parse_layers."""
    if layers and layers[0].tensors is not None:
        own = [sp for sp in layers if sp.weights_of is None]
        return [{"type": sp.mixer.kind, "mixer": sp.mixer.to_dict(), "mlp": _ff_to_dict(sp.mlp)} for sp in sorted(own, key=lambda sp: sp.tensors)]
    out = []
    for sp in layers:
        d = {"type": sp.mixer.kind, "mixer": sp.mixer.to_dict(), "mlp": _ff_to_dict(sp.mlp)}
        if sp.weights_of is not None:
            d["weights_of"] = sp.weights_of
        out.append(d)
    return out


def _ff_to_dict(f) -> dict | None:
    if f is None:
        return None
    if isinstance(f, DenseFFSpec):
        return {"kind": "dense", "ff": f.ff} if f.limit is None else {"kind": "dense", "ff": f.ff, "limit": f.limit}
    r, expert = {"experts": f.experts, "top": f.top}, {"ff": f.ff}
    if (f.groups, f.keep) != (1, 1):
        r["groups"] = {"count": f.groups, "keep": f.keep}
    if f.limit is not None:
        expert["limit"] = f.limit
    if f.renorm:
        r["scale"] = f.scale
    d = {"kind": "moe", "expert": expert, "router": r}
    if f.shared_ff:
        d["shared"] = {"ff": f.shared_ff}
    return d


def param_shapes(cfg) -> dict:
    """Checkpoint tensor name -> shape, in file order (layers with `weights_of` own none)."""
    C = cfg.hidden_size
    s = {"embed": (cfg.vocab_size, C)}
    if cfg.is_parallel or cfg.is_prenorm:
        s.update((pl if cfg.is_parallel else pn).param_shapes(cfg))
        s["head"] = (cfg.vocab_size, C)
        return s
    for i, sp in enumerate(cfg.layers):
        if sp.weights_of is not None:
            continue
        p, m = f"l{i}.", sp.mixer
        s[p + "norm1"] = ()
        if sp.mlp is not None:
            s[p + "norm2"] = ()
        if m.q_rank:
            s[p + "mix.dq"], s[p + "mix.dq.norm"], s[p + "mix.uq"] = (m.q_rank, C), (m.q_rank,), (m.q_width, m.q_rank)
        else:
            s[p + "mix.q"] = (m.q_width, C)
        s[p + "mix.dkv"], s[p + "mix.dkv.norm"] = (m.cache_width, C), (m.kv_rank,)
        s[p + "mix.uk"], s[p + "mix.uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
        if m.gated:
            s[p + "mix.g"] = (m.heads * m.vdim, C)
        s[p + "mix.o"] = (C, m.heads * m.vdim)
        if isinstance(sp.mlp, DenseFFSpec):
            s[p + "mlp.up"], s[p + "mlp.down"], s[p + "mlp.act"] = (sp.mlp.ff, C), (C, sp.mlp.ff), (4,)
        elif isinstance(sp.mlp, RoutedFFSpec):
            for e in range(sp.mlp.experts):
                q = f"{p}mlp.e{e}."
                s[q + "gate"], s[q + "up"], s[q + "down"] = (sp.mlp.ff, C), (sp.mlp.ff, C), (C, sp.mlp.ff)
            s[p + "mlp.router"] = (sp.mlp.experts, C)
        s[p + "canon1"] = (C, cfg.conv_taps)
    s["final.norm"] = ()
    s["head"] = (cfg.vocab_size, C)
    return s


def active_params(cfg) -> int:
    """Weights one token multiplies with (its chosen experts only), output projection included."""
    C, n = cfg.hidden_size, cfg.vocab_size * cfg.hidden_size
    if cfg.is_parallel or cfg.is_prenorm:
        return n + (pl if cfg.is_parallel else pn).active_params(cfg)
    for sp in cfg.layers:
        m = sp.mixer
        n += C * (m.cache_width + m.heads * m.vdim * (2 if m.gated else 1)) + m.heads * (m.dim + m.vdim) * m.kv_rank
        n += m.q_rank * (C + m.q_width) if m.q_rank else C * m.q_width
        if isinstance(sp.mlp, DenseFFSpec):
            n += 2 * C * sp.mlp.ff
        elif isinstance(sp.mlp, RoutedFFSpec):
            n += 3 * C * sp.mlp.ff * sp.mlp.top + C * sp.mlp.experts
    return n


def decode_gemm_shapes(cfg) -> list:
    """(name, features, K, experts or 0, gate/up pair) of the distinct projections of a decode step that the tensor-core GEMM
    runs."""
    C, seen, out = cfg.hidden_size, set(), []

    def add(name, F, K, E=0, swiglu=False):
        if (F, K, E, swiglu) not in seen and K % 8 == 0 and E <= 64:
            seen.add((F, K, E, swiglu))
            out.append((name, F, K, E, swiglu))
    for i, sp in enumerate(cfg.layers):
        m = sp.mixer
        if cfg.is_prenorm:
            for name, F, K, E, swiglu in pn.gemm_shapes(sp, C):
                add(f"l{i}.{name}", F, K, E, swiglu)
            continue
        if cfg.is_parallel:
            lay = pl.LayerLayout(sp)
            add(f"l{i}.in", lay.in_rows, C)
            add(f"l{i}.out", C, lay.out_cols)
            continue
        add(f"l{i}.in", _up8(m.q_rank or m.q_width) + _up8(m.cache_width) + (_up8(m.heads * m.vdim) if m.gated else 0), C)
        if m.q_rank:
            add(f"l{i}.uq", m.q_width, m.q_rank)
        add(f"l{i}.o", C, m.heads * m.vdim)
        if isinstance(sp.mlp, DenseFFSpec):
            add(f"l{i}.up", sp.mlp.ff, C)
            add(f"l{i}.down", C, sp.mlp.ff)
        elif isinstance(sp.mlp, RoutedFFSpec):
            add(f"l{i}.experts_gate_up", 2 * sp.mlp.ff, C, sp.mlp.experts, True)
            add(f"l{i}.experts_down", C, sp.mlp.ff, sp.mlp.experts)
    add("head", cfg.vocab_size, C)
    return out


# ---- weights ------------------------------------------------------------------------------------------------------
_up8 = pl.up8


@dataclass
class LatentMixerWeights:
    """Tensors of a latent-attention mixer in the layouts the kernels read.

    w_in stacks every projection of the mixer's input (queries or their latent, cache row, gate); each section starts at a
    multiple of 8 rows (zero rows in between), so that a row of its output can be read with 16-byte accesses."""
    w_in: torch.Tensor                 # [in_rows, C]
    q_norm: torch.Tensor | None        # [q_rank] fp32
    w_uq: torch.Tensor | None          # [H (dim + rot), q_rank]
    kv_norm: torch.Tensor              # [kv_rank] fp32
    w_ukv: torch.Tensor                # [H dim + H vdim, kv_rank]: keys then values of every head from the latent
    w_uk_t: torch.Tensor               # [H, kv_rank, dim]: the key expansion transposed, applied to the queries
    wo: torch.Tensor | None            # [C, H vdim]
    off_kv: int = 0                    # first column of the cache row / the gate in the input projection's output
    off_gate: int = -1
    sinks: torch.Tensor | None = None  # [H] fp32


@dataclass
class LayeredWeights:
    mixer: LatentMixerWeights
    conv: torch.Tensor                 # [taps, C] fp32
    norm1: torch.Tensor                # [1] fp32
    norm2: torch.Tensor | None
    w_up: torch.Tensor | None = None   # dense feed-forward
    act: torch.Tensor | None = None    # [4] fp32
    router: torch.Tensor | None = None
    w13: torch.Tensor | None = None    # experts: [E, 2 ff, C], gate rows first
    w2: torch.Tensor | None = None     # experts [E, C, ff], or the dense down projection [C, ff]
    fp8: dict = field(default_factory=dict)


def stack_rows(parts):
    """Row-stacks matrices, each section padded to a multiple of 8 rows. Returns (stacked, first row of each section)."""
    rows, offs, at = [], [], 0
    for p in parts:
        offs.append(at)
        rows.append(p)
        pad = _up8(p.shape[0]) - p.shape[0]
        if pad:
            rows.append(torch.zeros(pad, p.shape[1], dtype=p.dtype, device=p.device))
        at += _up8(p.shape[0])
    return torch.cat(rows, dim=0).contiguous(), offs


def expansions(m: LatentMixerSpec, get, prefix: str):
    """(keys then values of every head from the latent [H dim + H vdim, kv_rank], the key expansion transposed [H, kv_rank, dim])."""
    uk, uv = get(prefix + "uk"), get(prefix + "uv")
    return torch.cat([uk, uv], dim=0).contiguous(), uk.view(m.heads, m.dim, m.kv_rank).transpose(1, 2).contiguous()


def assemble_mixer(m: LatentMixerSpec, get, prefix: str) -> LatentMixerWeights:
    parts = [get(prefix + ("dq" if m.q_rank else "q")), get(prefix + "dkv")] + ([get(prefix + "g")] if m.gated else [])
    w_in, offs = stack_rows(parts)
    w_ukv, w_uk_t = expansions(m, get, prefix)
    return LatentMixerWeights(
        w_in=w_in, q_norm=get(prefix + "dq.norm").float() if m.q_rank else None, w_uq=get(prefix + "uq").contiguous() if m.q_rank else None,
        kv_norm=get(prefix + "dkv.norm").float(), w_ukv=w_ukv, w_uk_t=w_uk_t, wo=get(prefix + "o").contiguous(),
        off_kv=offs[1], off_gate=offs[2] if m.gated else -1)


def stack_experts(f: RoutedFFSpec, get, p: str):
    """(router, gate and up rows of every expert [E, 2 ff, C], down [E, C, ff]) of the layer with prefix p."""
    E = range(f.experts)
    return (get(p + "mlp.router").contiguous(),
            torch.stack([torch.cat([get(f"{p}mlp.e{e}.gate"), get(f"{p}mlp.e{e}.up")], dim=0) for e in E]).contiguous(),
            torch.stack([get(f"{p}mlp.e{e}.down") for e in E]).contiguous())


def assemble_layers(cfg, get) -> list:
    """One LayeredWeights per layer; layers that share tensors share the object."""
    out = []
    for i, sp in enumerate(cfg.layers):
        if sp.weights_of is not None:
            out.append(out[sp.weights_of])
            continue
        if cfg.is_parallel or cfg.is_prenorm:
            out.append(pl.assemble_layer(sp, get) if cfg.is_parallel else pn.assemble_layer(sp, get, cfg.is_shifted))
            continue
        p = f"l{i}."
        lw = LayeredWeights(mixer=assemble_mixer(sp.mixer, get, p + "mix."), conv=get(p + "canon1").float().t().contiguous(),
                            norm1=get(p + "norm1").float().reshape(1),
                            norm2=get(p + "norm2").float().reshape(1) if sp.mlp is not None else None)
        if isinstance(sp.mlp, DenseFFSpec):
            lw.w_up, lw.w2, lw.act = get(p + "mlp.up").contiguous(), get(p + "mlp.down").contiguous(), get(p + "mlp.act").float()
        elif isinstance(sp.mlp, RoutedFFSpec):
            lw.router, lw.w13, lw.w2 = stack_experts(sp.mlp, get, p)
        out.append(lw)
    return out


def random_param(name: str, shape, gen, std: float, dtype, device):
    """Seeded random parameter: N(0, std), gains 1, the polynomial activation near its linear term, convolution taps small."""
    special = pl.random_param(name, shape, gen, device)
    if special is not None:
        return special.to(dtype)
    if name.endswith("norm") or name.endswith(("norm1", "norm2")):
        return torch.ones(shape, dtype=dtype, device=device)
    t = torch.empty(shape, dtype=torch.float32, device=device)
    t.normal_(0.0, 0.25 if name.endswith((".act", ".canon1")) else std, generator=gen)
    if name.endswith(".act"):
        t += 0.5
    return t.to(dtype)


from . import prenorm_layers as pn  # noqa: E402  (uses the specifications above)
