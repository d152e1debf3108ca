"""The Zarorax design on the GPU, end to end against the plain implementation in tests/oracles: in 32-bit (tight) and in bf16
(within rounding), prompts, decoding, portions, mixed batches, reused pages, generation through the engine."""
import pytest
import torch
from safetensors.torch import save_file

from oracles import plain_zarorax as plain
from skein_b200 import ops
from skein_b200.compile.artifact import load_checkpoint
from skein_b200.models import config as mc
from skein_b200.models.decoder import Decoder, random_weights
from skein_b200.models.layered import DenseFFSpec, LayerSpec
from skein_b200.ops import _lib
from skein_b200.runtime.engine import Engine, EngineConfig, SamplingParams
from skein_b200.runtime.trace import TraceSession
from zarorax_models import VARIANTS, _gated, _latent_q, _moe, make, rel_err

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0)
BF, F32 = torch.bfloat16, torch.float32


def session(cfg, tensors, tmp, dtype, page_size=None, max_tokens=512):
    save_file(tensors, str(tmp / "model.safetensors"))
    w = load_checkpoint(cfg, tmp, DEV, dtype)
    ps = page_size or cfg.default_page_size
    return TraceSession(Decoder(cfg, w, num_pages=-(-max_tokens // ps), page_size=ps, max_pos=max_tokens), max_tokens)


def agree(got, want, dtype, what=""):
    """fp32: every row. bf16: rounding, judged by the rows' errors; a router decision may flip at a near tie, so a few rows may be
    further off."""
    if dtype == F32:
        assert rel_err(got, want) < 2e-4, what
        return
    e = torch.tensor([rel_err(g[None], w[None]) for g, w in zip(got, want)])
    assert torch.isfinite(e).all() and e.median() < 0.05 and (e > 0.15).float().mean() <= 0.1, (what, e.median(), e.max())


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(VARIANTS))
def test_prompt_decode_and_portions(name, dtype, tmp_path):
    cfg, raw, tensors = make(name)
    n = 150
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(3)).tolist()
    want = plain.forward(raw, tensors, toks)
    for ps in {VARIANTS[name].get("page_size", 16), 64}:
        s = session(cfg, tensors, tmp_path, dtype, ps)
        whole = s.step([("a", toks, range(n))], ["a"])
        agree(whole, want, dtype, "whole")
        for sizes in ([1] * n, [2, 3, 16, 2, 2, 17, 64, 1, 2, 40, 1], [100, 50]):
            out, at = [], 0
            for k in sizes:
                out.append(s.step([("b", toks[at:at + k], range(k))], ["b"] if at + k == n else []))
                at += k
            agree(torch.cat(out), want, dtype, sizes[:3])
        assert s.kv.in_use_pages == 0


@pytest.mark.parametrize("dtype", [F32, BF])
def test_layers(dtype, tmp_path):
    from skein_b200.compile.parity import DecoderForward
    cfg, raw, tensors = make("base")
    toks, layers = list(range(7, 7 + 40)), []
    plain.forward(raw, tensors, toks, layers_out=layers)
    s = session(cfg, tensors, tmp_path, dtype)
    hid, _ = DecoderForward(s.dec).run(toks)
    for i, (a, b) in enumerate(zip(hid, layers)):
        agree(a, b, dtype, i)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_unequal_requests_and_pages_used_again(dtype, tmp_path):
    cfg, raw, tensors = make("base", seed=2)
    g = torch.Generator().manual_seed(5)
    seqs = {n: torch.randint(0, cfg.vocab_size, (k,), generator=g).tolist() for n, k in (("a", 140), ("b", 70), ("c", 9), ("d", 130), ("e", 64))}
    want = {n: plain.forward(raw, tensors, t) for n, t in seqs.items()}
    s = session(cfg, tensors, tmp_path, dtype, page_size=64, max_tokens=384)      # 6 pages: a (3), b (2) and c (1)
    s.dec.kv[0].uniform_(-3, 3)       # what is left in a page must not matter
    for t in s.dec.conv_tail:
        t.uniform_(-3, 3)
    at = {n: 0 for n in seqs}

    def run(parts, end=()):
        ents = [(n, seqs[n][at[n]:at[n] + k], range(k)) for n, k in parts]
        lg, i = s.step(ents, end), 0
        for n, k in parts:
            agree(lg[i:i + k], want[n][at[n]:at[n] + k], dtype, (n, at[n]))
            i, at[n] = i + k, at[n] + k
    run([("a", 63), ("b", 1), ("c", 2)])
    run([("a", 1), ("b", 1), ("c", 1)])
    run([("a", 1), ("c", 1)])
    run([("b", 60), ("a", 1)])
    run([("c", 5), ("a", 50), ("b", 1)], end=["c"])
    run([("b", 7), ("a", 1)], end=["b"])
    run([("d", 126), ("a", 1)])
    run([("d", 1), ("a", 1), ("e", 1)])
    run([("a", 21), ("d", 1), ("e", 62)], end=["a"])
    run([("d", 2), ("e", 1)], end=["d", "e"])
    assert s.kv.in_use_pages == 0 and all(at[n] == len(seqs[n]) for n in seqs)


def _spiked():
    """A one-layer model in which token 2 looks up token 1 wherever it stands: token 2's query (head 0) points along token 1's key,
    so that one score stands out among hundreds; token 2's own key does not."""
    cfg, raw, t = make("base", layers=(LayerSpec(_gated(heads=2, dim=32, rot=16, vdim=32, rank=64, scale=0.3), DenseFFSpec(64)),), taps=3, alpha=0.3)
    t["l0.canon1"] *= 0
    g = torch.Generator().manual_seed(1)
    u, v = torch.randn(cfg.hidden_size, generator=g), torch.randn(cfg.hidden_size, generator=g)
    v -= u * (u @ v) / (u @ u)
    t["embed"][1], t["embed"][2] = (2 * u).to(BF), (2 * v).to(BF)
    c = plain.vector_norm(t["l0.mix.dkv"].float()[:64] @ (2 * u), t["l0.mix.dkv.norm"].float(), 1e-5)
    k0 = t["l0.mix.uk"].float()[:32] @ c
    q = t["l0.mix.q"].float()
    q[:48] = 0
    q[:32] = torch.outer(k0 / k0.norm(), v / v.norm()) * 3
    t["l0.mix.q"] = q.to(BF)
    return cfg, raw, t


@pytest.mark.parametrize("dtype", [F32, BF])
def test_one_far_key_among_hundreds(dtype, tmp_path):
    """The key at position p is asked for from far away, at page and tile borders, by a prompt and by decoding; moving it by one
    place, or losing it, changes the logits far beyond rounding (checked on the plain model)."""
    n = 420
    cfg, raw, t = _spiked()
    base = torch.randint(3, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(4)).tolist()
    s = session(cfg, t, tmp_path, dtype, page_size=64)
    for p in (0, 1, 63, 64, 127, 128, 255, 256):
        toks = list(base)
        toks[p] = 1
        for q in (n - 1, n - 2, p + 1):
            toks[q] = 2
        want = plain.forward(raw, t, toks)
        lost = list(toks)
        lost[p] = base[p]
        assert rel_err(plain.forward(raw, t, lost)[-1:], want[-1:]) > 0.3
        whole = s.step([("w", toks, range(n))], ["w"])
        agree(whole[[p + 1, n - 2, n - 1]], want[[p + 1, n - 2, n - 1]], dtype, p)
        s.step([("d", toks[:n - 2], [])])
        a = s.step([("d", toks[n - 2:n - 1], [0])])
        b = s.step([("d", toks[n - 1:], [0])], ["d"])
        agree(torch.cat([a, b]), want[n - 2:], dtype, p)


def test_long_decoding_stays_with_the_plain_model(tmp_path):
    cfg, raw, tensors = make("wide")
    n = 400
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(6)).tolist()
    want = plain.forward(raw, tensors, toks)
    s = session(cfg, tensors, tmp_path, F32, page_size=16)
    out = [s.step([("a", toks[:3], range(3))])] + [s.step([("a", [t], [0])]) for t in toks[3:]]
    agree(torch.cat(out), want, F32)
    assert s.runner.graph_replays >= n - 4        # decoding replays captured steps


@pytest.mark.parametrize("dtype", [F32, BF])
def test_greedy_generation_through_the_engine(dtype, tmp_path):
    cfg, raw, tensors = make("base", seed=7)
    save_file(tensors, str(tmp_path / "model.safetensors"))
    w = load_checkpoint(cfg, tmp_path, DEV, dtype)
    g = torch.Generator().manual_seed(8)
    common = torch.randint(0, cfg.vocab_size, (70,), generator=g).tolist()
    prompts = [common + [5, 6], common + [9], common[:11], common + [5, 6, 7], common[:40]]
    for chunk in (0, 24):
        eng = Engine(Decoder(cfg, w, num_pages=64, page_size=16, max_pos=256),
                     EngineConfig(max_batch=4, chunk_tokens=chunk, tpot_ms=1e9, ttft_ms=1e9, prefix_cache=True))
        n0 = _lib.launches()
        out = eng.generate(prompts, 12)
        assert _lib.launches() > n0 and eng.kv.prefix_hit_tokens_total > 0 and eng.kv.in_use_pages == 0
        for p, o in zip(prompts, out):
            assert len(o) == 12
            lg = plain.forward(raw, tensors, p + o[:-1])[len(p) - 1:]
            # every chosen token is the plain model's best, or within rounding of it (the sampler reads bf16 logits)
            gap = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
            assert gap.median() <= 1e-6 and (gap > 0.1 * lg.std(-1)).float().mean() <= (0.0 if dtype == F32 else 0.2), gap
    sampled = eng.generate([prompts[2]], 6, SamplingParams(temperature=1.0, seed=3))
    assert sampled == eng.generate([prompts[2]], 6, SamplingParams(temperature=1.0, seed=3))


def test_real_sizes_agree_between_forms():
    """Head sizes of a large model: the expanded prefill, row-wise attention and decoding of one prompt agree."""
    m = dict(heads=16, dim=128, rot=64, vdim=128, rank=512, scale=192 ** -0.5)
    cfg = mc.ModelConfig.layered("Zarorax", (LayerSpec(_gated(**m), _moe(ff=256, experts=16, top=4, groups=4, keep=2)),
                                             LayerSpec(_latent_q(q_rank=384, **m), DenseFFSpec(1024))), width=1024, vocab=2048, taps=4, alpha=2.0)
    w = random_weights(cfg, mc.ParallelLayout(), DEV, seed=1, std=0.04)
    toks = torch.randint(0, 2048, (300,), generator=torch.Generator().manual_seed(1)).tolist()
    s = TraceSession(Decoder(cfg, w, num_pages=10, max_pos=640), 640)
    a = s.step([("a", toks, range(300))], ["a"])
    out, at = [], 0
    for k in (32, 32, 200, 30) + (1,) * 6:
        out.append(s.step([("b", toks[at:at + k], range(k))]))
        at += k
    e = torch.tensor([rel_err(x[None], y[None]) for x, y in zip(torch.cat(out), a)])
    assert e.median() < 0.03 and (e > 0.15).float().mean() < 0.05, (e.median(), e.max())
    ops.workspace().check_status()
