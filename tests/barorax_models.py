"""Small random models of the Barorax design for the tests: configuration, raw dict for the plain implementation, tensors."""
import dataclasses

import torch

from skein_b200.models import config as mc
from skein_b200.models.layered import RoutedFFSpec, unroll_loop
from skein_b200.models.parallel_layers import SelectiveSpec, WindowAttnSpec


def diff(heads=4, kv_heads=2, dim=20, vdim=32, scale=0.3, rot=12, base=5e4, diff=0.6):
    return WindowAttnSpec(heads, kv_heads, dim, vdim, scale, rot, base, kind="attention", row_norm=False, interleaved=True, diff=diff, gated=True)


def chunk(heads=6, kv_heads=2, dim=24, vdim=16, scale=0.4, rot=24, base=1e4, size=21):
    return WindowAttnSpec(heads, kv_heads, dim, vdim, scale, rot, base, kind="attention_2", chunk=size, row_norm=False, interleaved=True, unit=True,
                          sink=True)


def scan(inner=120, state=12, dt_rank=9, taps=4):
    return SelectiveSpec(inner, state, dt_rank, taps)


def moe(ff=40, shared=56, experts=12, top=3, groups=4, keep=2, scale=1.7):
    return RoutedFFSpec(ff, None, experts, top, groups, keep, score="sigmoid", group_best=2, renorm=True, scale=scale, shared_ff=shared)


# "base": every mixer, a layer without feed-forward, two passes over three layers
VARIANTS = {
    "base": dict(width=96, vocab=100, specs=[(scan(), moe()), (diff(), moe(32, 24)), (chunk(), None), (scan(100, 20, 8, 3), moe(24, 48, 8, 2, 1, 1))],
                 loop=(1, 4, 2)),
    # nothing a multiple of 8, a group more than the eligible ones, no expert for every token in one layer, tiny pages
    "ragged": dict(width=77, vocab=61, eps=1e-3, page_size=2,
                   specs=[(diff(3, 1, 7, 5, 0.5, 2, 100.0, 0.2), moe(11, 13, 6, 2, 3, 2, 0.9)), (scan(37, 5, 3, 2), moe(9, 0, 5, 2, 1, 1)),
                          (chunk(5, 5, 10, 7, 0.7, 4, 50.0, 5), moe(7, 3, 6, 1, 2, 1, 2.0))], loop=(0, 2, 3)),
    # one head, chunks of one token, one state dimension, no look-back, one expert chosen, no loop
    "ones": dict(width=64, vocab=50, specs=[(chunk(1, 1, 16, 16, 0.25, 16, 1e4, 1), moe(16, 16, 2, 1, 1, 1, 1.0)), (diff(1, 1, 8, 16, 0.35, 0, 1e4, 0.0), None),
                                            (scan(64, 1, 1, 1), moe(16, 16, 4, 4, 1, 1, 1.0))], loop=None),
    # the loop holds the last layer and runs once; more taps than tokens of a page; groups of one expert; many query heads per key head
    "late": dict(width=80, vocab=90, page_size=4, specs=[(scan(88, 40, 16, 7), moe(24, 8, 4, 2, 4, 2)), (chunk(20, 1, 8, 24, 0.8, 4, 1e5, 70), None),
                                                         (diff(18, 2, 12, 16, 0.4, 12, 1e5, 0.8), moe(20, 28, 16, 5, 2, 2))], loop=(2, 3, 1)),
    # the sizes that the tensor-core kernels take: two maps of 64 over values of 128, heads of 64 and 128
    "tiles": dict(width=128, vocab=120, specs=[(scan(128, 16, 8, 4), moe(64, 64, 8, 2, 4, 2)), (diff(4, 2, 64, 128, 0.125, 64, 1e5, 0.5), moe(64, 128, 8, 2, 2, 1)),
                                               (chunk(8, 1, 128, 128, 0.09, 32, 1e6, 130), moe(64, 64, 8, 3, 4, 2)), (chunk(4, 2, 64, 64, 0.125, 64, 1e4, 100), None),
                                               (diff(8, 1, 64, 128, 0.1, 16, 1e4, 0.7), None)], loop=(1, 3, 2)),
}


def make(name, seed=0, clear=False, **over):
    """clear: every expert is chosen, so that no close call falls the other way in 16 bits."""
    v = {**VARIANTS[name], **over}
    if clear:
        v["specs"] = [(m, f and dataclasses.replace(f, keep=f.groups, top=f.experts)) for m, f in v["specs"]]
    cfg = mc.ModelConfig.layered("Barorax", unroll_loop(v["specs"], v["loop"]), width=v["width"], vocab=v["vocab"], eps=v.get("eps", 1e-5),
                                 max_pos=4096, name=name, loop=v["loop"])
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for n, shape in cfg.param_shapes().items():
        t = torch.randn(shape, generator=g)
        if n.endswith((".norm1", ".norm2", ".norm")):
            t = 1.0 + 0.3 * t
        elif n.endswith(".conv"):
            t = t / shape[-1] ** 0.5
        elif n.endswith((".dt.b", ".A_log")):
            t = t - 1.0
        elif n.endswith((".q", ".k")):
            t = t * (1.5 / shape[-1] ** 0.5)          # sharp attention: a wrong or missing key shows
        elif n.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = t * 0.3
        elif n == "loop.step":
            t = 0.5 * t
        elif n.endswith(".router"):
            t = t * (2.0 / shape[-1] ** 0.5)
        elif len(shape) == 2 and n != "embed":
            t = t / shape[-1] ** 0.5
        tensors[n] = t.to(torch.bfloat16)
    return cfg, cfg.to_hf_dict(), tensors


def rel_err(got, want):
    """Root mean square of the difference over that of the wanted values, worst row."""
    got, want = got.double().reshape(-1, got.shape[-1]).cpu(), want.double().reshape(-1, want.shape[-1])
    return float(((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()).max())
