"""Small random models of the Sikalorn design for the tests: configuration, raw dict for the plain implementation, tensors."""
import torch

from skein_b200.models import config as mc
from skein_b200.models.layered import DenseFFSpec, unroll_loop
from skein_b200.models.parallel_layers import MixerPairSpec, RecurrentSpec, WindowAttnSpec


def window(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.17, rot=16, base=5e4, factor=2.0, size=21):
    return WindowAttnSpec(heads, kv_heads, dim, vdim, scale, rot, base, factor, size)


def ssd(heads=6, groups=3, dim=20, vdim=16, taps=4, norm_groups=2):
    return RecurrentSpec("ssd", heads, groups, dim, vdim, taps, norm_groups)


def delta(heads=4, groups=2, dim=24, vdim=32, taps=4):
    return RecurrentSpec("delta", heads, groups, dim, vdim, taps)


def lightning(dim=16, vdim=24, decay=(0.5, 0.9, 0.995)):
    return RecurrentSpec("lightning", len(decay), len(decay), dim, vdim, decay=decay)


def pair(left=None, right=None, a=0.8, b=0.7):
    return MixerPairSpec(left or window(), right or ssd(), a, b)


FF = DenseFFSpec
# "base": every mixer, a layer without feed-forward, three passes over two layers
VARIANTS = {
    "base": dict(width=96, vocab=100, specs=[(delta(), FF(144)), (pair(), FF(120)), (lightning(), None), (pair(), FF(64))], loop=(1, 3, 3)),
    # nothing a multiple of 8, several norm groups, two convolution lengths, no scaling of the frequencies, tiny pages
    "ragged": dict(width=77, vocab=61, eps=1e-3, page_size=2,
                   specs=[(pair(window(3, 1, 7, 5, 0.4, 2, 100.0, 1.0, 5), ssd(6, 2, 9, 7, 2, 3), 1.3, -0.4), FF(33)), (lightning(5, 3, (0.7, 1.0)), FF(21)),
                          (delta(3, 1, 5, 7, 3), FF(19))], loop=(0, 2, 2)),
    # one head, one group, no look-back, no loop; the window is one token
    "ones": dict(width=64, vocab=50, specs=[(pair(window(1, 1, 16, 16, 0.25, 16, 1e4, 1.0, 1), ssd(1, 1, 16, 16, 1, 1), 1.0, 1.0), FF(64)),
                                            (delta(1, 1, 16, 16, 1), FF(64)), (lightning(16, 16, (0.0,)), FF(64))], loop=None),
    # the loop holds the last layer and runs once; more taps than tokens of a page; heads that share keys four ways
    "late": dict(width=80, vocab=90, page_size=4, specs=[(lightning(8, 16, (0.3, 0.8, 0.97, 0.999)), FF(56)), (delta(8, 2, 16, 8, 7), None),
                                                         (pair(window(8, 2, 32, 16, 0.2, 8, 1e5, 8.0, 70), ssd(4, 4, 12, 24, 6, 1)), FF(72))], loop=(2, 3, 1)),
    # the sizes that the tensor-core kernels take: heads of 64 and 128
    "tiles": dict(width=128, vocab=120, specs=[(delta(2, 1, 64, 64, 4), FF(128)), (pair(window(4, 2, 64, 64, 0.125, 64, 1e5, 4.0, 100), ssd(4, 1, 64, 64, 3, 2)), FF(96)),
                                               (lightning(128, 128, (0.9, 0.99)), FF(64)),
                                               (pair(window(8, 1, 128, 128, 0.09, 32, 1e6, 1.0, 130), ssd(2, 1, 128, 128, 4, 1)), None)], loop=(1, 3, 2)),
}


def make(name, seed=0, **over):
    v = {**VARIANTS[name], **over}
    cfg = mc.ModelConfig.layered("Sikalorn", unroll_loop(v["specs"], v["loop"]), width=v["width"], vocab=v["vocab"], eps=v.get("eps", 1e-5),
                                 max_pos=4096, name=name, loop=v["loop"])
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for n, shape in cfg.param_shapes().items():
        t = torch.randn(shape, generator=g)
        if n.endswith((".norm1", ".norm")):
            t = 1.0 + 0.3 * t
        elif n.endswith(".alpha"):
            t = 0.6 + 0.1 * t
        elif n.endswith((".norm1.b", "norm.b")):
            t = 0.2 * t
        elif n.endswith(".conv"):
            t = t / shape[-1] ** 0.5
        elif n.endswith((".dt_bias", ".A_log")):
            t = t - 1.0
        elif n.endswith((".q", ".k")):
            t = t * (2.0 / shape[-1] ** 0.5)          # sharp attention: a wrong or missing key shows
        elif n == "loop.step":
            t = 0.5 * t
        elif len(shape) == 2 and n != "embed":
            t = t / shape[-1] ** 0.5
        tensors[n] = t.to(torch.bfloat16)
    return cfg, cfg.to_hf_dict(), tensors


def rel_err(got, want):
    """Root mean square of the difference over that of the wanted values, worst row."""
    got, want = got.double().reshape(-1, got.shape[-1]).cpu(), want.double().reshape(-1, want.shape[-1])
    return float(((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()).max())
