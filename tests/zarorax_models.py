"""Small random models of the Zarorax design for the tests: configuration, raw dict for the plain implementation, tensors."""
import torch

from skein_b200.models import config as mc
from skein_b200.models.layered import DenseFFSpec, LatentMixerSpec, LayerSpec, RoutedFFSpec


def _gated(heads=3, dim=48, rot=16, vdim=40, rank=80, base=1e4, scale=0.11):
    return LatentMixerSpec("latent_attention_2", heads, dim, rot, vdim, rank, base, scale, gated=True)


def _latent_q(heads=5, dim=24, rot=32, vdim=32, rank=96, base=5e3, scale=0.13, q_rank=56):
    return LatentMixerSpec("latent_attention", heads, dim, rot, vdim, rank, base, scale, q_rank=q_rank)


def _moe(ff=72, limit=1.5, experts=8, top=2, groups=4, keep=2):
    return RoutedFFSpec(ff, limit, experts, top, groups, keep)


# "base": both mixers, both feed-forwards, a layer that uses another's tensors, a layer without feed-forward, two rotation bases
VARIANTS = {
    "base": dict(width=192, vocab=100, taps=4, alpha=2.5,
                 layers=(LayerSpec(_gated(), DenseFFSpec(160)), LayerSpec(_latent_q(), _moe()), LayerSpec(_latent_q(), _moe(), weights_of=1),
                         LayerSpec(_gated(), None))),
    # nothing a multiple of 8, experts in one group, a single tap pair, tiny pages
    "ragged": dict(width=77, vocab=61, taps=2, alpha=0.7, eps=1e-3, page_size=2,
                   layers=(LayerSpec(_latent_q(heads=3, dim=5, rot=6, vdim=9, rank=21, q_rank=11), DenseFFSpec(33)),
                           LayerSpec(_gated(heads=2, dim=7, rot=2, vdim=3, rank=13), RoutedFFSpec(19, 0.5, 5, 4)))),
    # one head, one expert of one group chosen, no look-back, alpha 1
    "ones": dict(width=64, vocab=50, taps=1, alpha=1.0,
                 layers=(LayerSpec(_gated(heads=1, dim=16, rot=16, vdim=16, rank=16), RoutedFFSpec(16, 7.0, 6, 1, 3, 1)),
                         LayerSpec(_gated(heads=1, dim=16, rot=16, vdim=16, rank=16), RoutedFFSpec(16, 7.0, 6, 1, 3, 1), weights_of=0))),
    # more taps than a page has tokens, all experts chosen, many heads
    "wide": dict(width=96, vocab=80, taps=7, alpha=4.0, page_size=4,
                 layers=(LayerSpec(_latent_q(heads=18, dim=8, rot=16, vdim=8, rank=32, q_rank=24), RoutedFFSpec(24, 1.0, 4, 4)),
                         LayerSpec(_gated(heads=18, dim=8, rot=16, vdim=24, rank=48), DenseFFSpec(56)))),
}


def make(name, seed=0, **over):
    v = {**VARIANTS[name], **over}
    cfg = mc.ModelConfig.layered("Zarorax", v["layers"], width=v["width"], vocab=v["vocab"], taps=v["taps"], alpha=v["alpha"],
                                 eps=v.get("eps", 1e-5), max_pos=4096, name=name)
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for n, shape in cfg.param_shapes().items():
        t = torch.randn(shape, generator=g)
        if n.endswith(("norm", "norm1", "norm2")):
            t = 1.0 + 0.3 * t
        elif n.endswith(".canon1"):
            t = 0.4 * t
        elif n.endswith((".uk", ".q", ".uq", ".dkv", ".dq")):
            t = t * (2.0 / shape[-1] ** 0.5)          # sharp attention: a wrong or missing key shows
        elif len(shape) == 2 and n != "embed":
            t = t / shape[-1] ** 0.5
        tensors[n] = t.to(torch.bfloat16)
    return cfg, cfg.to_hf_dict(), tensors


def rel_err(got, want):
    """Root mean square of the difference over that of the wanted values, worst row."""
    got, want = got.double().reshape(-1, got.shape[-1]).cpu(), want.double().reshape(-1, want.shape[-1])
    return float(((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()).max())
