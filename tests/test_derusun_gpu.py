"""The Derusun design on the GPU, end to end against the plain implementation in tests/oracles: in 32-bit (tight) and in bf16
(within rounding), prompts, decoding, portions, mixed batches, reused pages and slots, window edges, far keys, generation through the engine."""
import pytest
import torch
from safetensors.torch import save_file

from derusun_models import VARIANTS, attn, ff, latent, make, rec, rel_err
from oracles import plain_derusun as plain
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
        assert rel_err(got, want) < 3e-4, (what, rel_err(got, want))
        return
    e = torch.tensor([rel_err(g[None], w[None]) for g, w in zip(got, want)])
    assert torch.isfinite(e).all() and e.median() < 0.05 and (e > 0.15).float().mean() <= 0.05, (what, e.median(), e.max())


def poison(dec):
    """What is left in a page or a slot must not matter."""
    for t in dec.kv:
        if t is not None:
            t.uniform_(-3, 3)
    for r in dec.rec_state:
        if r is not None:
            r.mat.uniform_(-3, 3)
            if r.tail is not None:
                r.tail.uniform_(-3, 3)
    dec.shift_state.uniform_(-3, 3)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(VARIANTS))
def test_prompt_decode_and_portions(name, dtype, tmp_path):
    cfg, raw, tensors = make(name)
    n = 150
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(3)).tolist()
    want = plain.forward(raw, tensors, toks)
    for ps in {VARIANTS[name].get("page_size", 16), 64}:
        s = session(cfg, tensors, tmp_path, dtype, ps)
        poison(s.dec)
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
    cfg, raw, tensors = make(name)
    toks, layers = list(range(7, 7 + 40)), []
    plain.forward(raw, tensors, toks, layers_out=layers)
    s = session(cfg, tensors, tmp_path, dtype)
    hid, _ = DecoderForward(s.dec).run(toks)
    assert len(hid) == len(layers)
    for i, (a, b) in enumerate(zip(hid, layers)):
        agree(a, b, dtype, i)


@pytest.mark.parametrize("name,dtype", [("base", F32), ("base", BF), ("tiles", F32), ("tiles", BF), ("ragged", F32)])
def test_unequal_requests_pages_and_slots_used_again(name, dtype, tmp_path):
    cfg, raw, tensors = make(name, seed=2)
    g = torch.Generator().manual_seed(5)
    seqs = {n: torch.randint(0, cfg.vocab_size, (k,), generator=g).tolist() for n, k in (("a", 140), ("b", 70), ("c", 9), ("d", 130), ("e", 64))}
    want = {n: plain.forward(raw, tensors, t) for n, t in seqs.items()}
    s = session(cfg, tensors, tmp_path, dtype, page_size=64, max_tokens=384, slots=3)      # 6 pages: a (3), b (2) and c (1); 3 slots
    poison(s.dec)
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


def test_junk_between_the_rows_of_a_product_does_not_reach_it(tmp_path, monkeypatch):
    """Strided products whose inner size is no whole block: fresh buffers are filled with NaN."""
    cfg, raw, tensors = make("tiles")
    toks = torch.randint(0, cfg.vocab_size, (90,), generator=torch.Generator().manual_seed(3)).tolist()
    want = plain.forward(raw, tensors, toks)
    s = session(cfg, tensors, tmp_path, BF)
    empty = torch.empty

    def poisoned(*a, **k):
        t = empty(*a, **k)
        return t.fill_(float("nan")) if t.is_cuda and t.is_floating_point() else t
    monkeypatch.setattr(torch, "empty", poisoned)
    for cut in ([90], [1, 40, 2, 47]):
        at, out = 0, []
        for k in cut:
            out.append(s.step([("a", toks[at:at + k], range(k)), ("b", toks[at:at + k], [])], ["a", "b"] if at + k == 90 else []))
            at += k
        agree(torch.cat(out), want, BF, cut)


def _lookup(mixer, width=96):
    """A one-layer model in which token 2 looks up token 1: its query points along token 1's key, every other key is at right angles to it,
    so that one score stands out among hundreds."""
    cfg, raw, t = make("base", width=width, groups=1, specs=[(mixer, ff(16, 1.0))])
    g = torch.Generator().manual_seed(1)
    u, v = (torch.nn.functional.normalize(torch.randn(width, generator=g), dim=0) for _ in range(2))
    v = torch.nn.functional.normalize(v - u * (u @ v), dim=0)
    emb = t["embed"].float()
    emb -= (emb @ u)[:, None] * u + (emb @ v)[:, None] * v
    emb[1], emb[2] = u * width ** 0.5, v * width ** 0.5
    t["embed"], t["l0.norm1"], t["l0.shift"], t["l0.dwa"] = emb.to(BF), torch.ones(width).to(BF), torch.zeros(width).to(BF), torch.tensor([0.0, 1.0]).to(BF)
    t["l0.mix.o"] = (t["l0.mix.o"].float() * 3).to(BF)
    D = mixer.dim
    k = torch.nn.functional.normalize(torch.randn(D, generator=g), dim=0)
    flat = lambda w: w - torch.einsum("d,e,hec->hdc", k, k, w)      # noqa: E731
    if hasattr(mixer, "kv_rank"):
        a = torch.nn.functional.normalize(torch.randn(mixer.kv_rank, generator=g), dim=0)
        w = t["l0.mix.dkv"].float()
        w[:mixer.kv_rank] += 8 * torch.outer(a, u) - torch.outer(a, a @ w[:mixer.kv_rank])
        w[mixer.kv_rank:] *= 0.02
        t["l0.mix.dkv"], t["l0.mix.dkv.norm"] = w.to(BF), torch.ones(mixer.kv_rank).to(BF)
        uk = 0.02 * t["l0.mix.uk"].float().view(mixer.heads, D, -1) + torch.outer(k, a)
        t["l0.mix.uk"], t["l0.mix.uv"] = uk.reshape(mixer.heads * D, -1).to(BF), (t["l0.mix.uv"].float() * 3).to(BF)
        q = 0.02 * t["l0.mix.q"].float().view(mixer.heads, mixer.head_size, width)
        q[:, :D] += torch.outer(k, v)
        t["l0.mix.q"] = q.reshape(-1, width).to(BF)
        return cfg, raw, t
    for n in ("q", "k"):
        t[f"l0.mix.{n}.b"], t[f"l0.mix.{n}.norm"] = torch.zeros_like(t[f"l0.mix.{n}.b"]), torch.ones(D).to(BF)
        w = flat(t["l0.mix." + n].float().view(-1, D, width))
        t["l0.mix." + n] = (0.1 * w + torch.outer(k, u if n == "k" else v)).reshape(-1, width).to(BF)
    t["l0.mix.v"] = (t["l0.mix.v"].float() * 3).to(BF)
    return cfg, raw, t


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("dim,size,keep", [(64, 100, 5), (24, 65, 3), (128, 130, 40), (16, 33, 17), (128, 20, 150), (64, 1, 0)])
def test_window_edges_and_kept_tokens_in_prompts_and_decoding(dim, size, keep, dtype, tmp_path):
    """The key at position p is asked for by the last position whose window holds it and by the next one, p inside and just behind the kept
    first tokens, at page borders and elsewhere, by a prompt, by portions that end at the edge and by decoding; leaving it out changes the
    logits where it is seen and nowhere else (plain model)."""
    cfg, raw, t = _lookup(attn(2, 1, dim, dim, 20.0 / dim, size, keep, 30.0, False))
    n = max(2 * size, keep) + 190
    base = torch.randint(3, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(4)).tolist()
    s = session(cfg, t, tmp_path, dtype, page_size=64, max_tokens=1024)
    for p in sorted({0, max(keep - 1, 0), keep, keep + 1, 63, 64, 127, 128}):
        inside, outside = p + size - 1, p + size
        toks = list(base)
        toks[p] = 1
        toks[inside] = 2 if inside != p else 1
        toks[outside] = 2
        toks = toks[:outside + 1]
        want, lost = plain.forward(raw, t, toks), plain.forward(raw, t, toks[:p] + [base[p]] + toks[p + 1:])
        if inside != p:
            assert rel_err(lost[inside:inside + 1], want[inside:inside + 1]) > 0.2
        seen = rel_err(lost[outside:], want[outside:])
        assert seen > 0.2 if p < keep else seen < 1e-9
        agree(s.step([("w", toks, [inside, outside])], ["w"]), want[[inside, outside]], dtype, p)
        for first in {inside, max(1, inside - 1)} - {0}:
            s.step([("d", toks[:first], [])])
            out = [s.step([("d", [tok], [0])]) for tok in toks[first:]]
            agree(torch.cat(out), want[first:], dtype, (p, first))
            s.step([], ["d"])
        a = s.step([("c", toks[:outside], [inside])])
        agree(torch.cat([a, s.step([("c", toks[outside:], [0])], ["c"])]), want[inside:], dtype, p)
    assert s.kv.in_use_pages == 0


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("mixer", [latent(16, 64, 64, 128, 128, 1e5, 1.2), latent(3, 24, 16, 40, 56, 2e4, 2.0), attn(4, 2, 128, 128, 0.15, 60, 400, 30.0, False),
                                   attn(4, 2, 28, 20, 0.7, 60, 400, 30.0, False)])
def test_far_keys(mixer, dtype, tmp_path):
    """One key among a thousand, at the first places and at page borders, is asked for from far away by a prompt, a short portion and a
    decoded token."""
    n = 1000
    cfg, raw, t = _lookup(mixer)
    base = torch.randint(3, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(4)).tolist()
    s = session(cfg, t, tmp_path, dtype, page_size=64, max_tokens=1024)
    for p in (0, 1, 63, 64, 127, 128, 399):
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
    cfg, raw, t = make("base", specs=[(rec(4, 2, 64, 64, 3, 16, 8), None), (rec(2, 2, 16, 24, 1, 8, 8), ff())])
    for n in t:
        if n.endswith("A_log"):
            t[n] = torch.full_like(t[n], -7.0)
        if n.endswith(".mix.b"):
            t[n] = t[n] * 0.1
    n = 420
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(4)).tolist()
    want = plain.forward(raw, t, toks)
    lost = plain.forward(raw, t, [(toks[0] + 1) % cfg.vocab_size] + toks[1:])
    assert rel_err(lost[-1:], want[-1:]) > 1e-4
    s = session(cfg, t, tmp_path, F32)
    for sizes in ([n], [1, n - 1], [1] * 20 + [380] + [1] * 20):
        at, out = 0, []
        for k in sizes:
            out.append(s.step([("a", toks[at:at + k], range(k))], ["a"] if at + k == n else []))
            at += k
        assert rel_err(torch.cat(out), want) < 3e-5, sizes[:2]


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
    specs = [(rec(8, 8, 128, 128, 4, 128, 128), ff(2048, 7.0)), (attn(8, 2, 128, 128, 128 ** -0.5, 200, 20, 50.0), ff(2048, 7.0)),
             (latent(16, 128, 64, 128, 512, 5e5, 192 ** -0.5), ff(2048, 7.0)), (attn(8, 2, 128, 128, 128 ** -0.5, 130, 4, 30.0), None)]
    cfg = mc.ModelConfig.layered("Derusun", unroll_loop(specs, None), width=1024, vocab=2048, groups=2)
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
