"""Pre-norm layers over an fp32 stream, x <- x + mixer(norm1(x)), x <- x + ff(norm2(x)) with RMS norms: parameter names, weights.

Mixers are those of models/parallel_layers.py (attention, selective scan). A mixer runs as one product from the normed stream (every
projection stacked), its own kernels, and one product back that adds to the stream; both products and the kernels between them work on
one row per token (parallel_layers.LayerLayout without a feed-forward). The feed-forward is routed: scores of a sigmoid each, the best
groups of experts, the chosen scores divided by their sum; an expert that runs for every token beside them (layered.RoutedFFSpec); or it is
one clamped gated unit (layered.DenseFFSpec). A range of layers may run several times, each pass after the addition of a vector of its
own ("loop.step").

Designs of shifted layers (layered.SHIFTED_ARCHS) have three things more. Norms divide every one of `norm_groups` equal parts of a row by
its own root mean square. The mixer reads h + (h' - h) * shift with h' the previous token's normed row, which a sequence carries from step
to step like a recurrent state. And what a layer hands on is sum_j dwa[j] X_j over the embedding output X_0 and the results X_1 .. of all
layers so far.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from . import parallel_layers as pl
from .layered import DenseFFSpec, LatentMixerSpec, LatentMixerWeights, RoutedFFSpec, SpecError, expansions, stack_experts


def parse_ff(m: dict) -> RoutedFFSpec:
    if m["kind"] != "moe":
        raise SpecError(f"feed-forward kind {m['kind']!r} is not supported")
    r, shared = m["router"], m.get("shared")
    g = r.get("groups") or {"count": 1, "keep": 1}
    f = RoutedFFSpec(ff=int(m["expert"]["ff"]), limit=None, experts=int(r["experts"]), top=int(r["top"]), groups=int(g["count"]), keep=int(g["keep"]),
                     score="sigmoid", group_best=2, renorm=True, scale=float(r.get("scale", 1.0)), shared_ff=int(shared["ff"]) if shared else 0)
    f.check()
    return f


def parse_clamped(m: dict) -> DenseFFSpec:
    if m["kind"] != "dense":
        raise SpecError(f"feed-forward kind {m['kind']!r} is not supported")
    return DenseFFSpec(int(m["ff"]), float(m["limit"]))


PARSE_FF = {"Barorax": parse_ff, "Derusun": parse_clamped}


def check_value_mixing(mixers) -> None:
    """Layers whose values are mixed with the first such layer's must have values of its shape."""
    first = None
    for m in mixers:
        if getattr(m, "v_mix", False):
            first = first or m
            if (m.kv_heads, m.vdim) != (first.kv_heads, first.vdim):
                raise SpecError("layers that mix values must have the same kv_heads and vdim")


def fill_ranks(d: dict, shape_of) -> dict:
    """The configuration with the bottlenecks' widths of its channel_delta mixers filled in from a checkpoint: shape_of(tensor name) is a
    tensor's shape, or None where there is no such tensor."""
    layers = []
    for i, layer in enumerate(d["layers"]):
        if layer.get("type") == "channel_delta":
            ranks = {key: shape_of(f"l{i}.mix.{n}") for key, n in (("decay_rank", "a1"), ("gate_rank", "g1"))}
            layer = {**layer, "mixer": {**layer["mixer"], **{k: int(sh[0]) for k, sh in ranks.items() if sh is not None}}}
        layers.append(layer)
    return {**d, "layers": layers}


def _shift_shapes(cfg, i: int) -> dict:
    return {f"l{i}.shift": (cfg.hidden_size,), f"l{i}.dwa": (i + 2,)} if cfg.is_shifted else {}


def param_shapes(cfg) -> dict:
    C, s = cfg.hidden_size, {}
    if cfg.loop is not None:
        s["loop.step"] = (cfg.loop[2], C)
    for sp in sorted((sp for sp in cfg.layers if sp.weights_of is None), key=lambda sp: sp.tensors):
        p, f = f"l{sp.tensors}.", sp.mlp
        s[p + "norm1"] = (C,)
        if f is not None:
            s[p + "norm2"] = (C,)
        s.update({p + "mix." + n: shape for n, shape in sp.mixer.param_shapes(C).items()})
        s.update(_shift_shapes(cfg, sp.tensors))
        if f is None:
            continue
        if isinstance(f, DenseFFSpec):
            s[p + "mlp.gate"], s[p + "mlp.up"], s[p + "mlp.down"] = (f.ff, C), (f.ff, C), (C, f.ff)
            continue
        for e in range(f.experts):
            q = f"{p}mlp.e{e}."
            s[q + "gate"], s[q + "up"], s[q + "down"] = (f.ff, C), (f.ff, C), (C, f.ff)
        s[p + "mlp.router"] = (f.experts, C)
        if f.shared_ff:
            q = p + "mlp.shared."
            s[q + "gate"], s[q + "up"], s[q + "down"] = (f.shared_ff, C), (f.shared_ff, C), (C, f.shared_ff)
    s["final.norm"] = (C,)
    return s


def gemm_shapes(sp, C: int) -> list:
    """(name, features, K, experts or 0, gate/up pair) of a layer's products."""
    m, f, lay = sp.mixer, sp.mlp, pl.LayerLayout(sp, ff=False)
    out = [("in", lay.in_rows, C, 0, False), ("out", C, lay.out_cols, 0, False)]
    if isinstance(m, pl.SelectiveSpec):
        out += [("x", sum(pl.up8(rows) for _, rows in m.x_sections()), m.inner, 0, False), ("dt", m.inner, pl.up8(m.dt_rank), 0, False)]
    if isinstance(m, pl.RecurrentSpec):
        out += [("decay", m.heads * m.dim, pl.up8(m.decay_rank), 0, False), ("gate", m.out_width, pl.up8(m.gate_rank), 0, False)]
    if isinstance(f, DenseFFSpec):
        out += [("down", C, f.ff, 0, False)]
    elif f is not None:
        out += [("experts_gate_up", 2 * f.ff, C, f.experts, True), ("experts_down", C, f.ff, f.experts, False)]
        if f.shared_ff:
            out += [("shared_down", C, f.shared_ff, 0, False)]
    return out


def active_params(cfg) -> int:
    C, n = cfg.hidden_size, 0
    for sp in cfg.layers:
        f = sp.mlp
        n += sum(F * K for _, F, K, E, _ in gemm_shapes(sp, C) if E == 0)
        if isinstance(sp.mixer, LatentMixerSpec):
            n += sp.mixer.heads * (sp.mixer.dim + sp.mixer.vdim) * sp.mixer.kv_rank
        if isinstance(f, DenseFFSpec):
            n += 2 * C * f.ff
        elif f is not None:
            n += 3 * C * f.ff * f.top + C * f.experts + 2 * C * f.shared_ff
    return n


@dataclass
class PrenormLayerWeights:
    norm1: torch.Tensor                    # [C] fp32
    w_in: torch.Tensor                     # [in_rows, C]
    w_out: torch.Tensor                    # [C, out_cols]
    norm2: torch.Tensor | None = None
    attn: pl.WindowAttnWeights | None = None
    scan: pl.SelectiveWeights | None = None
    latent: LatentMixerWeights | None = None
    rec: pl.RecurrentWeights | None = None
    shift: torch.Tensor | None = None      # [C] fp32: share of the previous token's row in the mixer's input
    depth: torch.Tensor | None = None      # [layers so far + 1] fp32: weights of the embedding output and of every layer's result
    router: torch.Tensor | None = None     # [E, C]
    w13: torch.Tensor | None = None        # [E, 2 ff, C], gate rows first
    w2: torch.Tensor | None = None         # [E, C, ff]
    shared13: torch.Tensor | None = None   # [2 shared_ff, C], gate rows first
    shared2: torch.Tensor | None = None    # [C, shared_ff]
    dense13: torch.Tensor | None = None    # [2 ff, C], gate rows first
    dense2: torch.Tensor | None = None     # [C, ff]
    fp8: dict = field(default_factory=dict)


@dataclass
class StepWeights:
    """Loop of pre-norm layers: what is added to the stream before each pass."""
    step: torch.Tensor                     # [times, C] fp32


def load_loop(cfg, get) -> StepWeights | None:
    return None if cfg.loop is None else StepWeights(get("loop.step").float())


def assemble_layer(sp, get, shifted: bool = False) -> PrenormLayerWeights:
    p, m, f = f"l{sp.tensors}.", sp.mixer, sp.mlp
    q = p + "mix."
    sections = m.sections()
    parts = get(q + "in").split([rows for _, rows in sections]) if isinstance(m, pl.SelectiveSpec) else [get(q + n) for n, _ in sections]
    lw = PrenormLayerWeights(norm1=get(p + "norm1").float(), w_in=torch.cat([pl._pad(t, 0) for t in parts]).contiguous(),
                             w_out=pl._pad(get(q + "o"), 1).contiguous())
    if isinstance(m, pl.SelectiveSpec):
        lw.scan = pl.load_selective(m, get, q)
    elif isinstance(m, pl.RecurrentSpec):
        lw.rec = pl.load_recurrence(m, get, q)
    elif isinstance(m, LatentMixerSpec):
        w_ukv, w_uk_t = expansions(m, get, q)
        lw.latent = LatentMixerWeights(w_in=lw.w_in, q_norm=None, w_uq=None, kv_norm=get(q + "dkv.norm").float(), w_ukv=w_ukv, w_uk_t=w_uk_t, wo=None,
                                       sinks=get(q + "sink").float() if m.sink else None)
    else:
        lw.attn = pl.load_attention(m, get, q)
    if shifted:
        lw.shift, lw.depth = get(p + "shift").float(), get(p + "dwa").float()
    if f is not None:
        lw.norm2 = get(p + "norm2").float()
    if isinstance(f, DenseFFSpec):
        lw.dense13, lw.dense2 = torch.cat([get(p + "mlp.gate"), get(p + "mlp.up")]).contiguous(), get(p + "mlp.down").contiguous()
    elif f is not None:
        lw.router, lw.w13, lw.w2 = stack_experts(f, get, p)
        if f.shared_ff:
            s = p + "mlp.shared."
            lw.shared13, lw.shared2 = torch.cat([get(s + "gate"), get(s + "up")]).contiguous(), get(s + "down").contiguous()
    return lw
