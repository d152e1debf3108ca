"""The Sikalorn design through the framework (configuration, loops, lowering, weights, cache, state slots, scheduler, command line)
against the plain implementation in tests/oracles. CPU: the reference operators; the GPU tests are in test_sikalorn_gpu.py."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch
from safetensors.torch import save_file

from oracles import plain_sikalorn as plain
from sikalorn_models import VARIANTS, make, rel_err
from skein_b200 import core
from skein_b200.compile import parity
from skein_b200.compile.artifact import Artifact, ArtifactError, load_checkpoint
from skein_b200.compile.pipeline import compile_model
from skein_b200.models import config as mc
from skein_b200.models.decoder import Decoder, random_weights
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
def test_plain_window_is_attention_over_the_last_keys():
    m = dict(heads=2, kv_heads=1, dim=6, vdim=4, scale=0.5, rot=dict(base=100.0, dims=4, scaling=dict(factor=3.0)), mask=dict(size=3))
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)      # noqa: E731
    W = {"q": r(12, 8), "k": r(6, 8), "v": r(4, 8), "q.norm": r(12), "k.norm": r(6), "o": torch.eye(8, dtype=torch.float64)}
    h = r(9, 8)
    out = plain.windowed_attention(h, m, W.__getitem__, 1e-5)
    unit = lambda z, w: z / (z.pow(2).mean() + 1e-5).sqrt() * w            # noqa: E731

    def turned(v, p):
        v = v.clone()
        for i in range(2):
            a = torch.tensor(p * 100.0 ** (-2 * i / 4) / 3.0, dtype=torch.float64)
            u, w = v[i].clone(), v[i + 2].clone()
            v[i], v[i + 2] = u * a.cos() - w * a.sin(), w * a.cos() + u * a.sin()
        return v
    for t in (0, 1, 2, 5, 8):
        for n in range(2):
            q = turned(unit(W["q"] @ h[t], W["q.norm"])[6 * n:6 * n + 6], t)
            js = range(max(0, t - 2), t + 1)
            s = torch.stack([q @ turned(unit(W["k"] @ h[j], W["k.norm"]), j) * 0.5 for j in js])
            want = torch.softmax(s, 0) @ torch.stack([W["v"] @ h[j] for j in js])
            assert torch.allclose(out[t, 4 * n:4 * n + 4], want)


def test_plain_recurrences_have_a_closed_form():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)      # noqa: E731
    T, H, D, V = 11, 2, 3, 2
    W = {n: r(H * D, 5) for n in "qk"} | {"v": r(H * V, 5), "g": r(H * V, 5), "norm": torch.ones(H * V, dtype=torch.float64), "o": torch.eye(H * V, dtype=torch.float64)}
    h = r(T, 5)
    out = plain.lightning(h, dict(heads=H, dim=D, vdim=V, decay=[0.5, 0.9]), W.__getitem__, 0.0)
    q, k, v = (torch.nn.functional.silu(h @ W[n].T) for n in "qkv")
    o = torch.stack([sum(d ** (T - 1 - j) * (q[-1, D * n:D * n + D] @ k[j, D * n:D * n + D]) * v[j, V * n:V * n + V] for j in range(T))
                     for n, d in ((0, 0.5), (1, 0.9))]).reshape(-1)
    assert torch.allclose(out[-1], o / o.pow(2).mean().sqrt() * torch.sigmoid(h[-1] @ W["g"].T))
    # the delta rule with full write strength and no decay recalls what a key was last written with
    q1 = plain.unit(r(D))
    S = torch.zeros(D, V, dtype=torch.float64)
    for val in (r(V), r(V)):
        S = S + q1[:, None] * (val - S.T @ q1)[None]
    assert torch.allclose(S.T @ q1, val, atol=1e-5)


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
    assert s.kv.in_use_pages == 0 and s.kv.free_state_slots == 4


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
    with pytest.raises(Exception, match="slot"):
        s.kv.admit(999, [1])                     # no slot is left
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
        out = eng.generate(prompts, 8)
        assert eng.kv.prefix_hit_tokens_total == 0 and not eng.kv.prefix_enabled      # pages alone do not bring a state back
        assert eng.kv.in_use_pages == 0 and eng.kv.free_state_slots == 2
        for p, o in zip(prompts, out):
            seq = list(p)
            for tok in o:
                lg = plain.forward(raw, tensors, seq)[-1]
                assert lg[tok] >= lg.max() - 1e-4
                seq.append(tok)


def test_state_slots_of_the_block_manager():
    kv = core.KvBlockManager(8, 16, False, state_slots=2)
    a, b = kv.admit(1, [1] * 20), kv.admit(2, [1])
    assert {a.slot, b.slot} == {0, 1} and kv.slot_of(1) == a.slot and kv.free_state_slots == 0 and not kv.can_admit([1])
    kv.release(1)
    assert kv.can_admit([1]) and kv.admit(3, [2]).slot == a.slot and kv.slot_of(7) == -1
    with pytest.raises(Exception, match="prefix"):
        core.KvBlockManager(8, 16, True, state_slots=2)
    assert core.KvBlockManager(8, 16, False).admit(1, [1]).slot == -1


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
        (0, None, None), (1, None, 0), (2, None, None), (1, 1, 1), (2, 2, None), (1, 1, 2), (2, 2, None), (3, None, None)]
    assert cfg.state_bytes_per_slot() == sum(
        4 * r.heads * r.dim * r.vdim + 2 * (r.taps if r.kind != "lightning" else 0) * r.conv_channels
        for r in (getattr(l.mixer, "right", l.mixer) for l in cfg.layers))
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["loop"].update(stop=9), lambda d: d["loop"].update(times=0),
                   lambda d: d["layers"][1]["mixer"]["left"]["rot"].update(dims=26), lambda d: d["layers"][1]["mixer"]["left"].update(kv_heads=3),
                   lambda d: d["layers"][1]["mixer"]["right"].update(norm_groups=7), lambda d: d["layers"][2]["mixer"].update(decay=[0.5]),
                   lambda d: d["layers"][0]["mlp"].update(kind="moe"), lambda d: d.pop("norm")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(mc.ImportError_):
            mc.ModelConfig.from_hf_dict(bad)
    with pytest.raises(core.PlanError):
        core.lower_device_for(json.dumps(raw), 2, 1, 1, 0)
    from skein_b200.runtime.speculative import SpeculativeDecoder
    dec = Decoder(cfg, random_weights(cfg, mc.ParallelLayout(), "cpu"), num_pages=2)
    with pytest.raises(ValueError, match="rolled back"):
        SpeculativeDecoder(dec, dec)


def test_missing_or_misshapen_tensor_is_named(tmp_path):
    cfg, _, tensors = make("base")
    t = dict(tensors)
    del t["l1.mix.right.A_log"]
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="l1.mix.right.A_log"):
        load_checkpoint(cfg, tmp_path, CPU)
    t["l1.mix.right.A_log"] = torch.zeros(3, dtype=torch.bfloat16)
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="shape"):
        load_checkpoint(cfg, tmp_path, CPU)


def test_compile_verify_and_serve_on_cpu(tmp_path):
    """plan -> artifact -> parity -> engine, as the command line does it."""
    cfg, raw, tensors = make("base")
    save_file(tensors, str(tmp_path / "model.safetensors"))
    read = lambda p: (ROOT / p).read_text()      # noqa: E731
    r = compile_model(json.dumps(raw), read("cluster/b200_4x.toml"), read("cluster/sample_trace.jsonl"), read("models/sikalorn_7b_drift.toml"),
                      read("cluster/cost_constants.toml"), tmp_path / "art", weights=str(tmp_path), n_parity_prompts=1)
    assert r.plan["parallelism"] == {"tp": 1, "pp": 1, "ep": 1} and r.report.passed
    assert not r.plan["execution"]["prefix_cache"]["enable"]
    art = Artifact(r.artifact_dir)
    art.check_lowering(0)
    w = art.load_weights(0, "cpu")
    assert w.layers[3] is w.layers[1] and w.layers[5] is w.layers[1] and torch.equal(w.loop.step, tensors["loop.step"].float())
    out = subprocess.run([sys.executable, "-m", "skein_b200.parallel.worker", "--artifact", str(r.artifact_dir), "--cpu", "--prompt", "abc",
                          "--max-new-tokens", "4", "--max-seq-len", "64", "--max-batch", "2"], capture_output=True, text=True, cwd=ROOT)
    assert out.returncode == 0, out.stderr[-2000:]
    assert len(json.loads(out.stdout.strip().splitlines()[-1])["generated"][0]) == 4


def test_hot_swap_copies_every_slot(tmp_path):
    from types import SimpleNamespace
    from skein_b200.runtime import hotswap
    cfg = mc.tiny_sikalorn()
    a, b = (random_weights(cfg, mc.ParallelLayout(), "cpu", seed=s) for s in (0, 1))
    art = SimpleNamespace(load_weights=lambda rank, dev: b)
    eng = SimpleNamespace(dec=Decoder(cfg, a, num_pages=2), kv=SimpleNamespace(clear_prefix_cache=lambda: None))
    real, hotswap.Artifact = hotswap.Artifact, lambda path: art
    try:
        hotswap.mount_weights(eng, "x", 0)
    finally:
        hotswap.Artifact = real
    flat = lambda w: [t for v in [*w.layers, w.final_norm, w.loop] for t in hotswap._slots(v) if t is not None] + [w.embed, w.lm_head]      # noqa: E731
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
