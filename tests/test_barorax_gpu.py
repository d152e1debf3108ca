"""The Barorax design on the GPU, end to end against the plain implementation in tests/oracles: in 32-bit (tight) and in bf16
(within rounding), prompts, decoding, portions, mixed batches, reused pages and slots, far keys, generation through the engine."""
import pytest
import torch
from safetensors.torch import save_file

from oracles import plain_barorax as plain
from barorax_models import VARIANTS, chunk, diff, make, moe, rel_err, scan
from skein_b200 import ops
from skein_b200.compile.artifact import load_checkpoint
from skein_b200.models import config as mc
from skein_b200.models.decoder import Decoder, random_weights
from skein_b200.models.layered import unroll_loop
from skein_b200.ops import _lib
from skein_b200.runtime.engine import Engine, EngineConfig, SamplingParams
from skein_b200.runtime.trace import TraceSession

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0)
BF, F32 = torch.bfloat16, torch.float32


def session(cfg, tensors, tmp, dtype, page_size=None, max_tokens=512, slots=4):
    save_file(tensors, str(tmp / "model.safetensors"))
    w = load_checkpoint(cfg, tmp, DEV, dtype)
    ps = page_size or cfg.default_page_size
    return TraceSession(Decoder(cfg, w, num_pages=-(-max_tokens // ps), page_size=ps, max_pos=max_tokens, state_slots=slots), max_tokens)


def agree(got, want, dtype, what=""):
    """fp32: every row. bf16: rounding, judged by the rows' errors."""
    if dtype == F32:
        assert rel_err(got, want) < 3e-4, what
        return
    e = torch.tensor([rel_err(g[None], w[None]) for g, w in zip(got, want)])
    assert torch.isfinite(e).all() and e.median() < 0.05 and (e > 0.15).float().mean() <= 0.05, (what, e.median(), e.max())


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(VARIANTS))
def test_prompt_decode_and_portions(name, dtype, tmp_path):
    cfg, raw, tensors = make(name, clear=dtype == BF)
    n = 150
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(3)).tolist()
    want = plain.forward(raw, tensors, toks)
    for ps in {VARIANTS[name].get("page_size", 16), 64}:
        s = session(cfg, tensors, tmp_path, dtype, ps)
        agree(s.step([("a", toks, range(n))], ["a"]), want, dtype, "whole")
        for sizes in ([1] * n, [2, 3, 16, 2, 2, 17, 64, 1, 2, 40, 1], [100, 50], [63, 1, 65, 21]):
            out, at = [], 0
            for k in sizes:
                out.append(s.step([("b", toks[at:at + k], range(k))], ["b"] if at + k == n else []))
                at += k
            agree(torch.cat(out), want, dtype, sizes[:3])
        assert s.kv.in_use_pages == 0 and s.kv.free_state_slots == 4


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["base", "tiles"])
def test_layers(name, dtype, tmp_path):
    from skein_b200.compile.parity import DecoderForward
    cfg, raw, tensors = make(name, clear=dtype == BF)
    toks, layers = list(range(7, 7 + 40)), []
    plain.forward(raw, tensors, toks, layers_out=layers)
    s = session(cfg, tensors, tmp_path, dtype)
    hid, _ = DecoderForward(s.dec).run(toks)
    assert len(hid) == len(layers)
    for i, (a, b) in enumerate(zip(hid, layers)):
        agree(a, b, dtype, i)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["base", "tiles"])
def test_unequal_requests_pages_and_slots_used_again(name, dtype, tmp_path):
    cfg, raw, tensors = make(name, seed=2, clear=dtype == BF)
    g = torch.Generator().manual_seed(5)
    seqs = {n: torch.randint(0, cfg.vocab_size, (k,), generator=g).tolist() for n, k in (("a", 140), ("b", 70), ("c", 9), ("d", 130), ("e", 64))}
    want = {n: plain.forward(raw, tensors, t) for n, t in seqs.items()}
    s = session(cfg, tensors, tmp_path, dtype, page_size=64, max_tokens=384, slots=3)      # 6 pages: a (3), b (2) and c (1); 3 slots
    for t in s.dec.kv:                # what is left in a page or a slot must not matter
        if t is not None:
            t.uniform_(-3, 3)
    for r in s.dec.rec_state:
        if r is not None:
            r.mat.uniform_(-3, 3)
            if r.tail is not None:
                r.tail.uniform_(-3, 3)
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
    assert s.kv.in_use_pages == 0 and s.kv.free_state_slots == 3 and all(at[n] == len(seqs[n]) for n in seqs)


def _spiked(mixer, width=96):
    """A one-layer model in which token 2 looks up token 1: its query points along token 1's key, so that one score stands out among
    hundreds. (Two maps: the first one does.)"""
    cfg, raw, t = make("base", width=width, specs=[(mixer, moe(16, 16, 4, 1, 1, 1))], loop=None)
    g = torch.Generator().manual_seed(1)
    u, v = torch.randn(width, generator=g), torch.randn(width, generator=g)
    v -= u * (u @ v) / (u @ u)
    t["l0.norm1"] = torch.ones(width).to(BF)
    t["embed"][1], t["embed"][2] = (u * width ** 0.5 / u.norm()).to(BF), (v * width ** 0.5 / v.norm()).to(BF)
    for n in ("v", "o"):
        t["l0.mix." + n] = (t["l0.mix." + n].float() * 3).to(BF)
    D, K = mixer.dim, mixer.kv_heads
    k = torch.randn(D, generator=g)
    k *= D ** 0.5 / k.norm()
    unit = lambda z: z / z.norm() / width ** 0.5      # noqa: E731
    wq, wk = t["l0.mix.q"].float().view(-1, mixer.maps, D, width), t["l0.mix.k"].float().view(-1, mixer.maps, D, width)
    # scores of other pairs stay small; token 1's key and token 2's query lie along k
    wq[:, 0], wk[:, 0] = 0.1 * wq[:, 0] + 0.9 * torch.outer(k, unit(v)), 0.1 * wk[:, 0] + 0.9 * torch.outer(k, unit(u))
    t["l0.mix.q"], t["l0.mix.k"] = wq.reshape(-1, width).to(BF), wk.reshape(-1, width).to(BF)
    return cfg, raw, t


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("dim,size", [(64, 100), (24, 65), (128, 256), (16, 33)])
def test_chunk_edges_in_prompts_and_decoding(dim, size, dtype, tmp_path):
    """The key at position p is asked for by the last position of its chunk and by the first of the next one, p at the chunk's first and
    last places and at page borders, by a prompt, by portions that end at the edge and by decoding; leaving it out changes the logits
    inside and does not outside (plain model)."""
    n = 3 * size + 2
    cfg, raw, t = _spiked(chunk(2, 1, dim, dim, 16.0 / dim, 0, 1e4, size))
    base = torch.randint(3, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(4)).tolist()
    s = session(cfg, t, tmp_path, dtype, page_size=64, max_tokens=1024)
    for p in (0, 1, size - 2, size, size + 1, 2 * size - 2, min(64, size - 2)):
        inside, outside = p // size * size + size - 1, p // size * size + size
        toks = list(base)
        toks[p] = 1
        toks[inside] = toks[outside] = 2
        toks = toks[:outside + 1]
        want, lost = plain.forward(raw, t, toks), plain.forward(raw, t, toks[:p] + [base[p]] + toks[p + 1:])
        assert rel_err(lost[inside:inside + 1], want[inside:inside + 1]) > 0.2
        assert rel_err(lost[outside:], want[outside:]) < 1e-9
        agree(s.step([("w", toks, [inside, outside])], ["w"]), want[[inside, outside]], dtype, p)
        for first in (inside, max(1, inside - 1)):
            s.step([("d", toks[:first], [])])
            out = [s.step([("d", [tok], [0])]) for tok in toks[first:]]
            agree(torch.cat(out)[-2:], want[inside:], dtype, (p, first))
            s.step([], ["d"])
        a = s.step([("c", toks[:outside], [inside])])            # a portion that ends with the chunk
        agree(torch.cat([a, s.step([("c", toks[outside:], [0])], ["c"])]), want[inside:], dtype, p)
    assert s.kv.in_use_pages == 0


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("dim,vdim", [(64, 128), (20, 32)])
def test_far_keys_of_differential_attention(dim, vdim, dtype, tmp_path):
    """One key among a thousand, at the first places and at page borders, is asked for from far away by a prompt, a short portion and a
    decoded token."""
    n = 1000
    cfg, raw, t = _spiked(diff(4, 2, dim, vdim, 18.0 / dim, 0, 1e4, 0.4))
    base = torch.randint(3, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(4)).tolist()
    s = session(cfg, t, tmp_path, dtype, page_size=64, max_tokens=1024)
    for p in (0, 1, 63, 64, 511, 700):
        toks = list(base)
        toks[p], toks[-1] = 1, 2
        want, lost = plain.forward(raw, t, toks, F32)[-1:], plain.forward(raw, t, toks[:p] + [base[p]] + toks[p + 1:], F32)[-1:]
        assert rel_err(lost, want) > 0.2
        agree(s.step([("w", toks, [n - 1])], ["w"]), want, dtype, p)
        for k in (1, 2, 37):
            s.step([("d", toks[:-k], [])])
            agree(s.step([("d", toks[-k:], [k - 1])], ["d"]), want, dtype, (p, k))


def test_an_early_token_is_remembered_by_the_state(tmp_path):
    """Slow decays: the first token still shows in the logits hundreds of tokens later, in every way of cutting the sequence."""
    cfg, raw, t = make("base", specs=[(scan(96, 16, 8, 3), None), (scan(64, 4, 8, 1), moe())], loop=(0, 1, 2))
    for n in t:
        if n.endswith("A_log"):
            t[n] = torch.full_like(t[n], -7.0)
    n = 420
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(4)).tolist()
    want = plain.forward(raw, t, toks)
    lost = plain.forward(raw, t, [(toks[0] + 1) % cfg.vocab_size] + toks[1:])
    assert rel_err(lost[-1:], want[-1:]) > 3e-3
    s = session(cfg, t, tmp_path, F32)
    for sizes in ([n], [1, n - 1], [1] * 20 + [380] + [1] * 20):
        at, out = 0, []
        for k in sizes:
            out.append(s.step([("a", toks[at:at + k], range(k))], ["a"] if at + k == n else []))
            at += k
        agree(torch.cat(out), want, F32, sizes[:2])


@pytest.mark.parametrize("name", ["late", "tiles"])
def test_long_decoding_stays_with_the_plain_model(name, tmp_path):
    cfg, raw, tensors = make(name)
    n = 400
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(6)).tolist()
    want = plain.forward(raw, tensors, toks)
    s = session(cfg, tensors, tmp_path, F32, page_size=16)
    out = [s.step([("a", toks[:3], range(3))])] + [s.step([("a", [t], [0])]) for t in toks[3:]]
    agree(torch.cat(out), want, F32)
    assert s.runner.graph_replays >= n - 4        # decoding replays captured steps


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["base", "tiles"])
def test_greedy_generation_through_the_engine(name, dtype, tmp_path):
    cfg, raw, tensors = make(name, seed=7)
    save_file(tensors, str(tmp_path / "model.safetensors"))
    w = load_checkpoint(cfg, tmp_path, DEV, dtype)
    g = torch.Generator().manual_seed(8)
    common = torch.randint(0, cfg.vocab_size, (70,), generator=g).tolist()
    prompts = [common + [5, 6], common + [9], common[:11], common + [5, 6, 7], common[:40]]
    for chunk in (0, 24):
        eng = Engine(Decoder(cfg, w, num_pages=64, page_size=16, max_pos=256, state_slots=3),
                     EngineConfig(max_batch=4, chunk_tokens=chunk, tpot_ms=1e9, ttft_ms=1e9, prefix_cache=True, warm_graphs=chunk > 0))
        n0 = _lib.launches()
        out = eng.generate(prompts, 12)
        assert _lib.launches() > n0 and eng.kv.in_use_pages == 0 and eng.kv.free_state_slots == 3
        for p, o in zip(prompts, out):
            assert len(o) == 12
            lg = plain.forward(raw, tensors, p + o[:-1])[len(p) - 1:]
            # every chosen token is the plain model's best, or within rounding of it (the sampler reads bf16 logits)
            gap = lg.max(-1).values - lg.gather(1, torch.tensor(o)[:, None])[:, 0]
            assert gap.median() <= 1e-6 and (gap > 0.1 * lg.std(-1)).float().mean() <= (0.0 if dtype == F32 else 0.2), gap
    sampled = eng.generate([prompts[2]], 6, SamplingParams(temperature=1.0, seed=3))
    assert sampled == eng.generate([prompts[2]], 6, SamplingParams(temperature=1.0, seed=3))


def test_real_sizes_agree_between_forms():
    """Sizes of a large model's layers: one prompt whole, in portions and decoded."""
    ff = moe(512, 1024, 32, 4, 8, 4)
    specs = [(scan(2048, 16, 64, 4), ff), (diff(8, 2, 64, 128, 0.125, 64, 5e5, 0.8), ff), (chunk(8, 2, 128, 128, 128 ** -0.5, 128, 1e4, 200), ff)]
    cfg = mc.ModelConfig.layered("Barorax", unroll_loop(specs, (1, 3, 2)), width=1024, vocab=2048, loop=(1, 3, 2))
    w = random_weights(cfg, mc.ParallelLayout(), DEV, seed=1, std=0.04)
    toks = torch.randint(0, 2048, (300,), generator=torch.Generator().manual_seed(1)).tolist()
    s = TraceSession(Decoder(cfg, w, num_pages=10, max_pos=640, state_slots=4), 640)
    a = s.step([("a", toks, range(300))], ["a"])
    out, at = [], 0
    for k in (32, 16, 216, 30) + (1,) * 6:
        out.append(s.step([("b", toks[at:at + k], range(k))]))
        at += k
    e = torch.tensor([rel_err(x[None], y[None]) for x, y in zip(torch.cat(out), a)])
    assert e.median() < 0.03 and (e > 0.15).float().mean() < 0.05, (e.median(), e.max())
    ops.workspace().check_status()
