"""The Barorax design through the framework (configuration, loops, lowering, weights, cache, state slots, scheduler, command line)
against the plain implementation in tests/oracles. CPU: the reference operators; the GPU tests are in test_barorax_gpu.py."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch
from safetensors.torch import save_file

from barorax_models import VARIANTS, make, rel_err
from oracles import plain_barorax as plain
from skein_b200 import core
from skein_b200.compile import parity
from skein_b200.compile.artifact import Artifact, ArtifactError, load_checkpoint
from skein_b200.compile.pipeline import compile_model
from skein_b200.models import config as mc
from skein_b200.models.decoder import Decoder, random_weights
from skein_b200.ops import reference_prenorm as rn
from skein_b200.runtime.engine import Engine, EngineConfig
from skein_b200.runtime.trace import TraceSession

ROOT = Path(__file__).resolve().parent.parent
CPU, F32 = torch.device("cpu"), torch.float32


def session(cfg, tensors, tmp, page_size=None, max_tokens=512, slots=4):
    save_file(tensors, str(tmp / "model.safetensors"))
    w = load_checkpoint(cfg, tmp, CPU, F32)
    ps = page_size or cfg.default_page_size
    return TraceSession(Decoder(cfg, w, num_pages=-(-max_tokens // ps), page_size=ps, max_pos=max_tokens, state_slots=slots), max_tokens)


# ---- the plain implementation's mechanisms, each against a direct statement of it ---------------------------------------
def _turned(v, p, dims, base):
    """Rotation of neighbouring pairs as multiplication by complex numbers of modulus one."""
    z = torch.view_as_complex(v[:dims].reshape(-1, 2).contiguous())
    a = p * torch.tensor([base ** (-2 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    return torch.cat([torch.view_as_real(z * torch.polar(torch.ones_like(a), a)).reshape(-1), v[dims:]])


def test_plain_differential_attention_subtracts_two_maps():
    m = dict(heads=2, kv_heads=1, dim=6, vdim=4, scale=0.5, rot=dict(base=100.0, dims=4), diff=0.3)
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)      # noqa: E731
    W = {"q": r(24, 8), "k": r(12, 8), "v": r(4, 8), "g": r(8, 8), "o": torch.eye(8, dtype=torch.float64)} | {n: r(6) * 0.3 for n in ("lq1", "lk1", "lq2", "lk2")}
    h = r(9, 8)
    out = plain.differential_attention(h, m, W.__getitem__, 1e-5)
    lam = math.exp(float(W["lq1"] @ W["lk1"])) - math.exp(float(W["lq2"] @ W["lk2"])) + 0.3
    for t in (0, 1, 5, 8):
        for n in range(2):
            maps = []
            for j in range(2):
                q = _turned((W["q"] @ h[t])[12 * n + 6 * j:12 * n + 6 * j + 6], t, 4, 100.0)
                s = torch.stack([q @ _turned((W["k"] @ h[i])[6 * j:6 * j + 6], i, 4, 100.0) * 0.5 for i in range(t + 1)])
                maps.append(torch.softmax(s, 0) @ torch.stack([W["v"] @ h[i] for i in range(t + 1)]))
            o = maps[0] - lam * maps[1]
            o = o / (o.pow(2).mean() + 1e-5).sqrt() * 0.7 * torch.sigmoid(W["g"] @ h[t])[4 * n:4 * n + 4]
            assert torch.allclose(out[t, 4 * n:4 * n + 4], o)


def test_plain_chunks_unit_heads_and_sink():
    m = dict(heads=2, kv_heads=2, dim=6, vdim=4, scale=0.5, rot=dict(base=100.0, dims=6), mask=dict(size=4))
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)      # noqa: E731
    W = {"q": r(12, 8), "k": r(12, 8), "v": r(8, 8), "o": torch.eye(8, dtype=torch.float64)}
    h = r(11, 8)
    out = plain.chunked_attention(h, m, W.__getitem__, 1e-5)
    unit = lambda z: z / (z.pow(2).mean() + 1e-5).sqrt()            # noqa: E731
    for t in (0, 3, 4, 6, 10):
        for n in range(2):
            q = unit(_turned((W["q"] @ h[t])[6 * n:6 * n + 6], t, 6, 100.0))
            js = range(t - t % 4, t + 1)
            e = torch.stack([(q @ unit(_turned((W["k"] @ h[j])[6 * n:6 * n + 6], j, 6, 100.0)) * 0.5).exp() for j in js])
            want = (e / (1.0 + e.sum())) @ torch.stack([(W["v"] @ h[j])[4 * n:4 * n + 4] for j in js])
            assert torch.allclose(out[t, 4 * n:4 * n + 4], want)


def test_plain_scan_has_a_closed_form():
    g = torch.Generator().manual_seed(2)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)      # noqa: E731
    T, I, N = 9, 3, 2
    x, dt, A, B, C, D = r(T, I), r(T, I).abs(), -r(I, N).abs(), r(T, N), r(T, N), r(I)
    y = plain.selective_scan(x, dt, A, B, C, D)
    for t in (0, 4, 8):
        for c in range(I):
            want = D[c] * x[t, c] + sum(C[t, n] * sum(dt[j, c] * x[j, c] * B[j, n] * torch.exp(dt[j + 1:t + 1, c].sum() * A[c, n]) for j in range(t + 1))
                                        for n in range(N))
            assert torch.allclose(y[t, c], want)


def test_expert_choice_counts_the_two_best_of_a_group():
    # group 1 holds the single best expert, group 0 the best pair
    s = torch.tensor([0.7, 0.65, 0.1, 0.9, 0.2, 0.1, 0.5, 0.5, 0.1])
    assert plain.choose_experts(s, 2, 3, 1) == [0, 1] and plain.choose_experts(s, 3, 3, 2) == [3, 0, 1]
    f = VARIANTS["base"]["specs"][0][1]
    z = torch.randn(40, f.experts, generator=torch.Generator().manual_seed(3))
    ids, w = rn.select(z, f)
    for t in range(40):
        sc = torch.sigmoid(z[t])
        want = plain.choose_experts(sc, f.top, f.groups, f.keep)
        assert ids[t].tolist() == want and torch.allclose(w[t], f.scale * sc[want] / sc[want].sum())


# ---- the framework -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(VARIANTS))
def test_prompt_decode_and_portions_agree_with_the_plain_model(name, tmp_path):
    cfg, raw, tensors = make(name)
    n = 45
    toks = torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(3)).tolist()
    want = plain.forward(raw, tensors, toks)
    s = session(cfg, tensors, tmp_path, page_size=VARIANTS[name].get("page_size", 16))
    assert rel_err(s.step([("a", toks, range(n))], ["a"]), want) < 5e-5
    for sizes in ([1] * n, [2, 3, 16, 2, 2, 17, 3], [33, 12]):
        out, at = [], 0
        for k in sizes:
            out.append(s.step([("b", toks[at:at + k], range(k))], ["b"] if at + k == n else []))
            at += k
        assert rel_err(torch.cat(out), want) < 5e-5, sizes
    assert s.kv.in_use_pages == 0 and (s.kv.free_state_slots == 4 or not cfg.has_state)


def test_layers_agree_with_the_plain_model_and_the_dense_oracle(tmp_path):
    for name in ("base", "ragged"):
        cfg, raw, tensors = make(name)
        toks, layers = list(range(7, 7 + 19)), []
        want = plain.forward(raw, tensors, toks, layers_out=layers)
        s = session(cfg, tensors, tmp_path)
        hid, lg = parity.DecoderForward(s.dec).run(toks)
        assert len(hid) == len(layers) == cfg.num_layers == len(plain.layer_runs(raw))
        hid2, lg2 = parity.DenseForward(cfg, s.dec.w).run(toks)
        for a, b, c in zip(hid, hid2, layers):
            assert rel_err(a, c) < 5e-5 and rel_err(b, c) < 5e-5
        assert rel_err(lg, want[-1]) < 5e-5 and rel_err(lg2, want[-1]) < 5e-5


def test_unequal_requests_in_one_batch_pages_and_slots_used_again(tmp_path):
    """Requests of unequal length, portions beside single tokens, one paused; pages and slots given back and handed to later ones."""
    cfg, raw, tensors = make("base")
    g = torch.Generator().manual_seed(5)
    seqs = {n: torch.randint(0, cfg.vocab_size, (k,), generator=g).tolist() for n, k in (("a", 40), ("b", 23), ("c", 9), ("d", 37))}
    want = {n: plain.forward(raw, tensors, t) for n, t in seqs.items()}
    s = session(cfg, tensors, tmp_path, page_size=8, max_tokens=88, slots=3)       # 11 pages and 3 slots: a, b and c just fit
    at = {n: 0 for n in seqs}

    def run(parts, end=()):
        ents = [(n, seqs[n][at[n]:at[n] + k], range(k)) for n, k in parts]
        lg, i = s.step(ents, end), 0
        for n, k in parts:
            assert rel_err(lg[i:i + k], want[n][at[n]:at[n] + k]) < 5e-5, (n, at[n])
            i, at[n] = i + k, at[n] + k
    run([("a", 13), ("b", 1), ("c", 2)])
    run([("a", 1), ("b", 1), ("c", 1)])
    run([("b", 7), ("a", 1)])
    run([("c", 6), ("a", 9), ("b", 1)], end=["c"])
    run([("b", 13), ("a", 1)], end=["b"])
    run([("d", 30), ("a", 1)])
    run([("a", 14), ("d", 1)], end=["a"])
    run([("d", 6)], end=["d"])
    assert s.kv.in_use_pages == 0 and s.kv.free_state_slots == 3


def test_generation_through_the_engine_with_fewer_slots_than_requests(tmp_path):
    cfg, raw, tensors = make("base")
    save_file(tensors, str(tmp_path / "model.safetensors"))
    w = load_checkpoint(cfg, tmp_path, CPU, F32)
    g = torch.Generator().manual_seed(8)
    common = torch.randint(0, cfg.vocab_size, (21,), generator=g).tolist()
    prompts = [common + [5, 6], common + [9], common[:11], common + [5, 6, 7, 8, 9]]
    for chunk in (0, 7):
        eng = Engine(Decoder(cfg, w, num_pages=64, page_size=8, max_pos=128, state_slots=2),
                     EngineConfig(max_batch=4, chunk_tokens=chunk, tpot_ms=1e9, ttft_ms=1e9, prefix_cache=True))
        out = eng.generate(prompts, 6)
        assert eng.kv.prefix_hit_tokens_total == 0 and not eng.kv.prefix_enabled      # pages alone do not bring a state back
        assert eng.kv.in_use_pages == 0 and eng.kv.free_state_slots == 2
        for p, o in zip(prompts, out):
            lg = plain.forward(raw, tensors, p + o[:-1])[len(p) - 1:]
            assert len(o) == 6 and all(lg[i, tok] >= lg[i].max() - 1e-4 for i, tok in enumerate(o))


def test_a_model_without_a_state_keeps_the_prefix_cache(tmp_path):
    """Attention layers alone: cached pages bring a prefix back, also where a chunk ends inside it."""
    v = VARIANTS["base"]["specs"]
    cfg, raw, tensors = make("base", specs=[v[1], v[2]], loop=(0, 2, 2))
    assert not cfg.has_state and cfg.state_bytes_per_slot() == 0
    save_file(tensors, str(tmp_path / "model.safetensors"))
    w = load_checkpoint(cfg, tmp_path, CPU, F32)
    common = torch.randint(0, cfg.vocab_size, (30,), generator=torch.Generator().manual_seed(8)).tolist()
    eng = Engine(Decoder(cfg, w, num_pages=64, page_size=8, max_pos=128), EngineConfig(max_batch=4, tpot_ms=1e9, ttft_ms=1e9, prefix_cache=True))
    first, second = eng.generate([common + [5]], 4)[0], eng.generate([common + [9, 7]], 4)[0]
    assert eng.kv.prefix_hit_tokens_total >= 24
    for p, o in ((common + [5], first), (common + [9, 7], second)):
        lg = plain.forward(raw, tensors, p + o[:-1])[len(p) - 1:]
        assert all(lg[i, tok] >= lg[i].max() - 1e-4 for i, tok in enumerate(o))


def test_configuration_round_trip_and_refusals():
    for name in VARIANTS:
        cfg, raw, _ = make(name)
        again = mc.ModelConfig.from_hf_dict(json.loads(json.dumps(raw)))
        assert again.layers == cfg.layers and again.loop == cfg.loop
        j = json.dumps(raw)
        assert core.model_param_count(j) == cfg.param_count() == sum(math.prod(s) for s in cfg.param_shapes().values())
        ir = json.loads(core.import_model(j))
        assert {p["name"]: [d["fixed"] for d in p["shape"]] for l in ir["layers"] for p in l["params"]} == {n: list(s) for n, s in cfg.param_shapes().items()}
    cfg, raw, _ = make("base")
    assert [(l.tensors, l.weights_of, l.loop_pass) for l in cfg.layers] == [
        (0, None, None), (1, None, 0), (2, None, None), (3, None, None), (1, 1, 1), (2, 2, None), (3, 3, None)]
    assert cfg.state_bytes_per_slot() == 4 * 120 * 12 + 2 * 4 * 120 + 2 * (4 * 100 * 20 + 2 * 3 * 100)
    assert cfg.cache_bytes_per_page(64) == 2 * 64 * 2 * (2 * (40 + 32) + 2 * (24 + 16))
    for change in (lambda d: d["layers"][0].update(type="delta"), lambda d: d["loop"].update(stop=9), lambda d: d["loop"].update(times=0),
                   lambda d: d["layers"][1]["mixer"]["rot"].update(dims=22), lambda d: d["layers"][1]["mixer"].update(kv_heads=3),
                   lambda d: d["layers"][1]["mixer"].pop("diff"), lambda d: d["layers"][2]["mixer"].pop("mask"), lambda d: d["layers"][0]["mixer"].update(conv=0),
                   lambda d: d["layers"][0]["mlp"].update(kind="dense"), lambda d: d["layers"][0]["mlp"]["router"].update(top=9), lambda d: d.pop("norm")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(mc.ImportError_):
            mc.ModelConfig.from_hf_dict(bad)
    with pytest.raises(core.PlanError):
        core.lower_device_for(json.dumps(raw), 2, 1, 1, 0)


def test_missing_or_misshapen_tensor_is_named(tmp_path):
    cfg, _, tensors = make("base")
    t = dict(tensors)
    del t["l1.mix.lk2"]
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="l1.mix.lk2"):
        load_checkpoint(cfg, tmp_path, CPU)
    t["l1.mix.lk2"] = torch.zeros(3, dtype=torch.bfloat16)
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="shape"):
        load_checkpoint(cfg, tmp_path, CPU)


def test_compile_verify_and_serve_on_cpu(tmp_path):
    """plan -> artifact -> parity -> engine, as the command line does it."""
    cfg, raw, tensors = make("base")
    save_file(tensors, str(tmp_path / "model.safetensors"))
    read = lambda p: (ROOT / p).read_text()      # noqa: E731
    r = compile_model(json.dumps(raw), read("cluster/b200_4x.toml"), read("cluster/sample_trace.jsonl"), read("models/barorax_9b_drift.toml"),
                      read("cluster/cost_constants.toml"), tmp_path / "art", weights=str(tmp_path), n_parity_prompts=1)
    assert r.plan["parallelism"] == {"tp": 1, "pp": 1, "ep": 1} and r.report.passed
    assert not r.plan["execution"]["prefix_cache"]["enable"]
    art = Artifact(r.artifact_dir)
    art.check_lowering(0)
    w = art.load_weights(0, "cpu")
    assert w.layers[4] is w.layers[1] and torch.equal(w.loop.step, tensors["loop.step"].float())
    out = subprocess.run([sys.executable, "-m", "skein_b200.parallel.worker", "--artifact", str(r.artifact_dir), "--cpu", "--prompt", "abc",
                          "--max-new-tokens", "4", "--max-seq-len", "64", "--max-batch", "2"], capture_output=True, text=True, cwd=ROOT)
    assert out.returncode == 0, out.stderr[-2000:]
    assert len(json.loads(out.stdout.strip().splitlines()[-1])["generated"][0]) == 4


def test_hot_swap_copies_every_slot(tmp_path):
    from types import SimpleNamespace
    from skein_b200.runtime import hotswap
    cfg = mc.tiny_barorax()
    a, b = (random_weights(cfg, mc.ParallelLayout(), "cpu", seed=s) for s in (0, 1))
    art = SimpleNamespace(load_weights=lambda rank, dev: b)
    eng = SimpleNamespace(dec=Decoder(cfg, a, num_pages=2), kv=SimpleNamespace(clear_prefix_cache=lambda: None))
    real, hotswap.Artifact = hotswap.Artifact, lambda path: art
    try:
        hotswap.mount_weights(eng, "x", 0)
    finally:
        hotswap.Artifact = real
    flat = lambda w: [t for v in [*w.layers, w.loop] for t in hotswap._slots(v) if t is not None] + [w.final_norm, w.embed, w.lm_head]      # noqa: E731
    assert len(flat(a)) > 60 and all(torch.equal(x, y) for x, y in zip(flat(a), flat(b)))


def test_trace_runner_program_on_cpu(tmp_path):
    cfg, raw, tensors = make("base")
    (tmp_path / "m").mkdir()
    (tmp_path / "m" / "config.json").write_text(json.dumps(raw))
    save_file(tensors, str(tmp_path / "m" / "model.safetensors"))
    toks = list(range(30, 50))
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:12], "want": [3, 11]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[12:13], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[13:14], "want": [0]}, {"id": "y", "tokens": toks[:1], "want": [0]}], "end": ["x", "y"]}]
    r = subprocess.run([str(ROOT / "bin/trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens",
                        "128", "--device", "cpu"], input="\n".join(map(json.dumps, steps)), capture_output=True, text=True)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = plain.forward(raw, tensors, toks[:14])
    rows = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg.vocab_size)      # noqa: E731
    assert rel_err(rows(0), want[[3, 11]]) < 5e-5 and not (tmp_path / "1.f32").exists()
    assert rel_err(rows(2)[:1], want[13:]) < 5e-5 and rel_err(rows(2)[1:], plain.forward(raw, tensors, toks[:1])) < 5e-5
