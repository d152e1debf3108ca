"""The Derusun design through the framework (configuration, lowering, weights, cache, state slots, scheduler, command line) against the
plain implementation in tests/oracles. CPU: the reference operators; the GPU tests are in test_derusun_gpu.py."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch
from safetensors.torch import save_file

from derusun_models import VARIANTS, attn, latent, make, rec, rel_err
from oracles import plain_derusun as plain
from skein_b200 import core
from skein_b200.compile import parity
from skein_b200.compile.artifact import Artifact, ArtifactError, load_checkpoint
from skein_b200.compile.pipeline import compile_model
from skein_b200.models import config as mc
from skein_b200.models.decoder import Decoder, random_weights
from skein_b200.runtime.engine import Engine, EngineConfig
from skein_b200.runtime.trace import TraceSession

ROOT = Path(__file__).resolve().parent.parent
CPU, F32, F64 = torch.device("cpu"), torch.float32, torch.float64


def session(cfg, tensors, tmp, page_size=None, max_tokens=512, slots=4):
    save_file(tensors, str(tmp / "model.safetensors"))
    w = load_checkpoint(cfg, tmp, CPU, F32)
    ps = page_size or cfg.default_page_size
    return TraceSession(Decoder(cfg, w, num_pages=-(-max_tokens // ps), page_size=ps, max_pos=max_tokens, state_slots=slots), max_tokens)


def rand(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=F64)


# ---- the plain implementation's mechanisms, each against a direct statement of it ---------------------------------------
def test_plain_norm_shift_and_depth_average():
    r = rand(0)
    x, w, mix = r(5, 12), r(12), r(12)
    h = plain.grouped_norm(x, w, 3, 1e-5)
    for t in range(5):
        for g in range(3):
            part = x[t, 4 * g:4 * g + 4]
            assert torch.allclose(h[t, 4 * g:4 * g + 4], part / math.sqrt(float(part @ part) / 4 + 1e-5) * w[4 * g:4 * g + 4])
    s = plain.token_shift(h, mix)
    assert torch.allclose(s[0], h[0] * (1 - mix)) and all(torch.allclose(s[t], (1 - mix) * h[t] + mix * h[t - 1]) for t in range(1, 5))
    xs, a = [r(5, 12) for _ in range(4)], r(4)
    assert torch.allclose(plain.depth_average(xs, a), torch.einsum("j,jtc->tc", a, torch.stack(xs)))


def test_plain_window_cap_sink_and_mixing():
    m = dict(heads=2, kv_heads=1, dim=6, vdim=4, scale=0.5, softcap=1.5, mask=dict(size=3, keep_first=2))
    r = rand(1)
    W = {"q": r(12, 8), "k": r(6, 8), "v": r(4, 8), "q.b": r(12), "k.b": r(6), "v.b": r(4), "q.norm": r(6), "k.norm": r(6), "sink": r(2), "vmix": r(()),
         "o": torch.eye(8, dtype=F64)}
    h, first = r(9, 8), r(9, 4)
    out = plain.attention(h, m, W.__getitem__, 1e-5, first)
    norm = lambda z, w: z / (z.pow(2).mean() + 1e-5).sqrt() * w            # noqa: E731
    for t in (0, 1, 2, 4, 8):
        js = [j for j in range(t + 1) if t - j < 3 or j < 2]
        assert js == {0: [0], 1: [0, 1], 2: [0, 1, 2], 4: [0, 1, 2, 3, 4], 8: [0, 1, 6, 7, 8]}[t]
        for n in range(2):
            q = norm((W["q"] @ h[t] + W["q.b"])[6 * n:6 * n + 6], W["q.norm"])
            s = torch.stack([q @ norm(W["k"] @ h[j] + W["k.b"], W["k.norm"]) * 0.5 for j in js])
            p = torch.softmax(torch.cat([1.5 * torch.tanh(s / 1.5), W["sink"][n:n + 1]]), 0)[:-1]
            v = torch.stack([W["v"] @ h[j] + W["v.b"] for j in js])
            v = v + W["vmix"] * (first[js] - v)
            assert torch.allclose(out[t, 4 * n:4 * n + 4], p @ v)


def test_plain_latent_attention_equals_attention_over_expanded_keys():
    m = dict(heads=2, dim=4, rot_dim=4, vdim=3, kv_rank=5, scale=0.7, rot=dict(base=100.0, dims=4))
    r = rand(2)
    W = {"q": r(16, 8), "dkv": r(9, 8), "dkv.norm": r(5), "uk": r(8, 5), "uv": r(6, 5), "sink": r(2), "o": torch.eye(6, dtype=F64)}
    h = r(7, 8)
    out = plain.latent_attention(h, m, W.__getitem__, 1e-5)

    def turned(v, p):
        z = torch.complex(v[0::2], v[1::2])
        a = p * torch.tensor([100.0 ** (-2 * i / 4) for i in range(2)], dtype=F64)
        return torch.view_as_real(z * torch.polar(torch.ones_like(a), a)).reshape(-1)
    for t in (0, 3, 6):
        for n in range(2):
            q = (W["q"] @ h[t])[8 * n:8 * n + 8]
            s, v = [], []
            for j in range(t + 1):
                ckr = W["dkv"] @ h[j]
                c = ckr[:5] / (ckr[:5].pow(2).mean() + 1e-5).sqrt() * W["dkv.norm"]
                s.append((q[:4] @ (W["uk"] @ c)[4 * n:4 * n + 4] + turned(q[4:], t) @ turned(ckr[5:], j)) * 0.7)
                v.append((W["uv"] @ c)[3 * n:3 * n + 3])
            e = torch.stack(s).exp()
            assert torch.allclose(out[t, 3 * n:3 * n + 3], (e / (W["sink"][n].exp() + e.sum())) @ torch.stack(v))


def test_plain_delta_rule_per_channel():
    """Without correction the state is a decayed sum; with it and no decay, a written key reads back its value."""
    r = rand(3)
    T, H, D, V = 6, 2, 4, 3
    q, k, v, g = r(T, H, D), plain.unit(r(T, H, D)), r(T, H, V), torch.sigmoid(r(T, H, D))
    tiny = plain.delta_rule(q, k, v, torch.full((T, H), 1e-6, dtype=F64), g) * 1e6      # the correction is of second order
    for t in (0, 3, 5):
        for h in range(H):
            want = sum((q[t, h] * k[j, h] * g[j + 1:t + 1, h].prod(0)).sum() * v[j, h] for j in range(t + 1))
            assert torch.allclose(tiny[t, h], want, atol=1e-4)
    full = plain.delta_rule(k, k, v, torch.ones(T, H, dtype=F64), torch.ones(T, H, D, dtype=F64))
    assert torch.allclose(full, v, atol=1e-5)
    W = {"a1": r(3, 8), "a2": r(8, 3), "dt_bias": r(8), "A_log": r(2)}
    x = r(5, 8)
    d = plain.channel_decay(x, W.__getitem__, 2)
    assert torch.allclose(d[4, 1, 2], torch.exp(-W["A_log"][1].exp() * torch.log1p((W["a2"][6] @ (W["a1"] @ x[4]) + W["dt_bias"][6]).exp())))


def test_plain_clamped_unit():
    r = rand(4)
    W = {"gate": r(6, 4) * 3, "up": r(6, 4) * 3, "down": torch.eye(6, dtype=F64)}
    h = r(3, 4)
    y = plain.clamped_unit(h, 1.2, W.__getitem__)
    for t in range(3):
        for f in range(6):
            g, u = min(float(W["gate"][f] @ h[t]), 1.2), max(-1.2, min(1.2, float(W["up"][f] @ h[t])))
            assert math.isclose(float(y[t, f]), g / (1 + math.exp(-1.702 * g)) * (u + 1), rel_tol=1e-9)


# ---- the framework -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", [n for n in VARIANTS if n != "tiles"])
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
        assert len(hid) == len(layers) == cfg.num_layers
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


@pytest.mark.parametrize("name", ["base", "attention"])
def test_generation_through_the_engine_with_fewer_slots_than_requests(name, tmp_path):
    """Also without a recurrence: the last normed rows are a state all the same."""
    cfg, raw, tensors = make("base", **({} if name == "base" else {"specs": [(attn(), None), (latent(), None), (attn(keep=2), None)]}))
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


def test_configuration_round_trip_and_refusals():
    for name in VARIANTS:
        cfg, raw, _ = make(name)
        again = mc.ModelConfig.from_hf_dict(json.loads(json.dumps(raw)))
        assert again.layers == cfg.layers and again.norm_groups == cfg.norm_groups
        j = json.dumps(raw)
        assert core.model_param_count(j) == cfg.param_count() == sum(math.prod(s) for s in cfg.param_shapes().values())
        ir = json.loads(core.import_model(j))
        assert {p["name"]: [d["fixed"] for d in p["shape"]] for l in ir["layers"] for p in l["params"]} == {n: list(s) for n, s in cfg.param_shapes().items()}
    cfg, raw, _ = make("base")
    assert cfg.has_state and cfg.cache_bytes_per_page(64) == 2 * 64 * (3 * 2 * (28 + 20) + 56 + 16)
    assert cfg.state_bytes_per_slot() == 6 * 4 * 96 + 4 * 4 * 24 * 32 + 2 * 3 * (2 * 2 * 24 + 4 * 32) + 4 * 6 * 20 * 24 + 2 * 4 * (2 * 20 + 6 * 24)
    low = json.loads(core.lower_device_for(json.dumps(raw), 1, 1, 1, 0))["segments"][0]["ops"]
    assert low[1:9] == ["block_0_" + o for o in ("depth_shift_norm", "mixer_in", "recurrence_inputs", "recurrence", "gated_norm", "mixer_out", "group_norm2",
                                                 "clamped_gate_up")] and low[-3] == "final_depth_norm"
    for change in (lambda d: d["layers"][0].update(type="delta"), lambda d: d["norm"].update(groups=5), lambda d: d["layers"][1]["mixer"].update(kv_heads=4),
                   lambda d: d["layers"][4]["mixer"].update(vdim=24), lambda d: d["layers"][2]["mixer"]["rot"].update(dims=8), lambda d: d.update(loop={"start": 0, "stop": 1, "times": 2}),
                   lambda d: d["layers"][0]["mixer"].update(conv=0), lambda d: d["layers"][0]["mlp"].update(kind="moe"), lambda d: d["layers"][0]["mlp"].pop("limit"),
                   lambda d: d["layers"][0]["mixer"].update(kv_heads=3), lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=-1), lambda d: d.pop("norm")):
        bad = copy.deepcopy(raw)
        change(bad)
        with pytest.raises(mc.ImportError_):
            mc.ModelConfig.from_hf_dict(bad)
    with pytest.raises(core.PlanError):
        core.lower_device_for(json.dumps(raw), 2, 1, 1, 0)


def test_bottleneck_widths_come_from_the_checkpoint(tmp_path):
    """A configuration need not name them; the tensors do."""
    cfg, raw, tensors = make("base")
    bare = copy.deepcopy(raw)
    for layer in bare["layers"]:
        if layer["type"] == "channel_delta":
            del layer["mixer"]["decay_rank"], layer["mixer"]["gate_rank"]
    (tmp_path / "config.json").write_text(json.dumps(bare))
    alone = mc.ModelConfig.from_file(tmp_path / "config.json")
    assert alone.layers[0].mixer.decay_rank == alone.layers[0].mixer.dim            # nothing to look at
    save_file(tensors, str(tmp_path / "model.safetensors"))
    assert mc.ModelConfig.from_file(tmp_path / "config.json").layers == cfg.layers
    assert mc.ModelConfig.from_hf_dict(json.loads(mc.sized_config(json.dumps(bare), tmp_path / "model.safetensors"))).layers == cfg.layers


def test_missing_or_misshapen_tensor_is_named(tmp_path):
    cfg, _, tensors = make("base")
    t = dict(tensors)
    del t["l2.mix.sink"]
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="l2.mix.sink"):
        load_checkpoint(cfg, tmp_path, CPU)
    t["l2.mix.sink"] = torch.zeros(7, dtype=torch.bfloat16)
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="shape"):
        load_checkpoint(cfg, tmp_path, CPU)


def test_compile_verify_and_serve_on_cpu(tmp_path):
    """plan -> artifact -> parity -> engine, as the command line does it."""
    cfg, raw, tensors = make("base")
    save_file(tensors, str(tmp_path / "model.safetensors"))
    read = lambda p: (ROOT / p).read_text()      # noqa: E731
    r = compile_model(json.dumps(raw), read("cluster/b200_4x.toml"), read("cluster/sample_trace.jsonl"), read("models/derusun_4b_drift.toml"),
                      read("cluster/cost_constants.toml"), tmp_path / "art", weights=str(tmp_path), n_parity_prompts=1)
    assert r.plan["parallelism"] == {"tp": 1, "pp": 1, "ep": 1} and r.report.passed
    assert not r.plan["execution"]["prefix_cache"]["enable"]
    art = Artifact(r.artifact_dir)
    art.check_lowering(0)
    w = art.load_weights(0, "cpu")
    assert torch.equal(w.layers[4].depth, tensors["l4.dwa"].float()) and torch.equal(w.layers[2].latent.sinks, tensors["l2.mix.sink"].float())
    out = subprocess.run([sys.executable, "-m", "skein_b200.parallel.worker", "--artifact", str(r.artifact_dir), "--cpu", "--prompt", "abc",
                          "--max-new-tokens", "4", "--max-seq-len", "64", "--max-batch", "2"], capture_output=True, text=True, cwd=ROOT)
    assert out.returncode == 0, out.stderr[-2000:]
    assert len(json.loads(out.stdout.strip().splitlines()[-1])["generated"][0]) == 4


def test_hot_swap_copies_every_slot():
    from types import SimpleNamespace
    from skein_b200.runtime import hotswap
    cfg = mc.tiny_derusun()
    a, b = (random_weights(cfg, mc.ParallelLayout(), "cpu", seed=s) for s in (0, 1))
    art = SimpleNamespace(load_weights=lambda rank, dev: b)
    eng = SimpleNamespace(dec=Decoder(cfg, a, num_pages=2), kv=SimpleNamespace(clear_prefix_cache=lambda: None))
    real, hotswap.Artifact = hotswap.Artifact, lambda path: art
    try:
        hotswap.mount_weights(eng, "x", 0)
    finally:
        hotswap.Artifact = real
    flat = lambda w: [t for v in w.layers for t in hotswap._slots(v) if t is not None] + [w.final_norm, w.embed, w.lm_head]      # noqa: E731
    assert len(flat(a)) > 80 and all(torch.equal(x, y) for x, y in zip(flat(a), flat(b)))


def test_other_families_know_nothing_of_the_new_properties():
    assert not any(c.is_shifted for c in (mc.tiny_barorax(), mc.tiny_sikalorn(), mc.tiny_zarorax(), mc.tiny_llama())) and mc.tiny_derusun().is_prenorm
    assert "groups" not in mc.tiny_barorax().to_hf_dict()["norm"] and rec().corrects


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
