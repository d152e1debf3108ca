"""Small random models of the Derusun design for the tests: configuration, raw dict for the plain implementation, tensors."""
import torch

from skein_b200.models import config as mc
from skein_b200.models.layered import DenseFFSpec, LatentMixerSpec, unroll_loop
from skein_b200.models.parallel_layers import RecurrentSpec, WindowAttnSpec


def latent(heads=3, dim=24, rot=16, vdim=40, rank=56, base=2e4, scale=0.3):
    return LatentMixerSpec("latent_attention", heads, dim, rot, vdim, rank, base, scale, sink=True)


def attn(heads=6, kv_heads=2, dim=28, vdim=20, scale=0.3, window=19, keep=5, cap=9.0, mix=True):
    return WindowAttnSpec(heads, kv_heads, dim, vdim, scale, rot_dims=0, rope_base=1e4, window=window, kind="attention", row_norm=False, bias=True,
                          head_norm=True, softcap=cap, keep_first=keep, head_sink=True, v_mix=mix)


def rec(heads=4, groups=2, dim=24, vdim=32, taps=3, decay_rank=16, gate_rank=8):
    return RecurrentSpec("channel_delta", heads, groups, dim, vdim, taps, decay_rank=decay_rank, gate_rank=gate_rank)


def ff(n=144, limit=1.5):
    return DenseFFSpec(n, limit)


# "base": every mixer, layers without feed-forward, values mixed in two of three layers of different windows
VARIANTS = {
    "base": dict(width=96, vocab=100, groups=3, specs=[(rec(), ff()), (attn(), None), (latent(), ff(80, 3.0)), (attn(window=33, keep=0, cap=30.0, mix=False), ff(64, 2.5)),
                                                       (attn(keep=11, cap=4.0), ff(120, 1.0)), (rec(6, 1, 20, 24, 4, 24, 40), None)]),
    # nothing a multiple of 8, one group per norm, tiny pages, a window shorter than what it keeps
    "ragged": dict(width=77, vocab=61, groups=1, eps=1e-3, page_size=2,
                   specs=[(attn(3, 1, 7, 5, 0.5, 3, 9, 2.0), ff(11, 0.7)), (rec(3, 3, 5, 7, 2, 3, 5), ff(9, 4.0)), (latent(5, 6, 2, 3, 11, 100.0, 0.6), None),
                          (attn(5, 1, 10, 5, 0.7, 6, 1, 50.0), ff(13, 1.1))]),
    # one head, one token in the window, no look-back, norms over groups of four, one layer that mixes values
    "ones": dict(width=64, vocab=50, groups=16, specs=[(attn(1, 1, 16, 16, 0.25, 1, 0, 5.0, False), ff(16, 1.0)), (rec(1, 1, 8, 16, 1, 1, 1), ff(16, 2.0)),
                                                       (latent(1, 8, 2, 16, 8, 1e4, 0.4), None), (attn(1, 1, 8, 16, 0.3, 1, 1, 5.0, True), None)]),
    # many query heads per key head, more taps than tokens of a page, the first mixing layer late, rotated parts larger than the others
    "late": dict(width=80, vocab=90, groups=2, page_size=4, specs=[(latent(4, 16, 40, 24, 64, 1e5, 0.2), ff(40, 1.3)), (rec(8, 4, 40, 40, 7, 40, 16), None),
                                                                   (attn(20, 1, 8, 24, 0.8, 70, 30, 12.0), None), (attn(18, 1, 12, 24, 0.4, 11, 2, 25.0), ff(72, 0.5))]),
    # the sizes that the tensor-core kernels take: heads of 64 and 128, bottlenecks of whole blocks
    "tiles": dict(width=256, vocab=120, groups=2, specs=[(rec(4, 2, 128, 128, 4, 64, 64), ff(256, 2.0)), (attn(8, 2, 128, 128, 0.09, 130, 20, 30.0), ff(128, 7.0)),
                                                         (latent(16, 64, 64, 128, 128, 1e5, 0.09), ff(256, 2.0)), (rec(4, 4, 64, 64, 4, 24, 128), None),
                                                         (attn(4, 2, 128, 128, 0.1, 70, 150, 8.0), None), (attn(6, 3, 64, 64, 0.125, 100, 17, 20.0, False), ff(192, 1.0))]),
}


def make(name, seed=0, **over):
    v = {**VARIANTS[name], **over}
    cfg = mc.ModelConfig.layered("Derusun", unroll_loop(v["specs"], None), width=v["width"], vocab=v["vocab"], eps=v.get("eps", 1e-5), max_pos=4096,
                                 name=name, groups=v["groups"])
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for n, shape in cfg.param_shapes().items():
        t = torch.randn(shape, generator=g)
        if n.endswith((".norm1", ".norm2", ".norm")):
            t = 1.0 + 0.3 * t
        elif n.endswith(".conv"):
            t = t / shape[-1] ** 0.5
        elif n.endswith((".dt_bias", ".A_log")):
            t = t - 1.0
        elif n.endswith((".shift", ".vmix")):
            t = 0.5 + 0.3 * t
        elif n.endswith(".dwa"):
            t = 0.3 * t + (torch.arange(shape[0]) == shape[0] - 1)
        elif n.endswith((".q.b", ".k.b", ".v.b")):
            t = 0.3 * t
        elif n.endswith((".mix.q", ".mix.k", ".mix.uk", ".mix.dkv")):
            t = t * (1.5 / shape[-1] ** 0.5)          # sharp attention: a wrong or missing key shows
        elif len(shape) == 2 and n != "embed":
            t = t / shape[-1] ** 0.5
        tensors[n] = t.to(torch.bfloat16)
    return cfg, cfg.to_hf_dict(), tensors


def rel_err(got, want):
    """Root mean square of the difference over that of the wanted values, worst row."""
    got, want = got.double().reshape(-1, got.shape[-1]).cpu(), want.double().reshape(-1, want.shape[-1])
    return float(((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()).max())
