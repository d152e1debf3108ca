"""The Zarorax design through the framework (configuration, lowering, weights, cache, scheduler, sampling, command line) against
the plain implementation in tests/oracles. CPU: the reference operators; the GPU tests are in test_zarorax_gpu.py."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch
from safetensors.torch import save_file

from oracles import plain_zarorax as plain
from skein_b200 import core
from skein_b200.compile import parity
from skein_b200.compile.artifact import Artifact, ArtifactError, WeightSource, load_checkpoint
from skein_b200.compile.pipeline import compile_model
from skein_b200.models import config as mc
from skein_b200.models.decoder import Decoder
from skein_b200.runtime.engine import Engine, EngineConfig
from skein_b200.runtime.trace import TraceSession
from zarorax_models import VARIANTS, make, rel_err

ROOT = Path(__file__).resolve().parent.parent


def session(cfg, tensors, tmp, dtype=torch.float32, page_size=None, max_tokens=512, device="cpu"):
    save_file(tensors, str(tmp / "model.safetensors"))
    w = load_checkpoint(cfg, tmp, torch.device(device), dtype)
    ps = page_size or cfg.default_page_size
    return TraceSession(Decoder(cfg, w, num_pages=-(-max_tokens // ps), page_size=ps, max_pos=max_tokens), max_tokens)


@pytest.mark.parametrize("name", list(VARIANTS))
def test_prompt_decode_and_portions_agree_with_the_plain_model(name, tmp_path):
    cfg, raw, tensors = make(name)
    toks = torch.randint(0, cfg.vocab_size, (45,), generator=torch.Generator().manual_seed(3)).tolist()
    want = plain.forward(raw, tensors, toks)
    ps = VARIANTS[name].get("page_size", 16)
    s = session(cfg, tensors, tmp_path, page_size=ps)
    got = s.step([("a", toks, range(45))], ["a"])
    assert rel_err(got, want) < 2e-5
    for sizes in ([1] * 45, [2, 3, 16, 2, 2, 17, 3], [33, 12]):
        out, at = [], 0
        for n in sizes:
            out.append(s.step([("b", toks[at:at + n], range(n))], ["b"] if at + n == 45 else []))
            at += n
        assert rel_err(torch.cat(out), want) < 2e-5, sizes
    assert s.kv.in_use_pages == 0


def test_layers_agree_with_the_plain_model_and_the_dense_oracle(tmp_path):
    cfg, raw, tensors = make("base")
    toks = list(range(7, 7 + 19))
    layers = []
    want = plain.forward(raw, tensors, toks, layers_out=layers)
    s = session(cfg, tensors, tmp_path)
    hid, lg = parity.DecoderForward(s.dec).run(toks)
    assert len(hid) == len(layers) == cfg.num_layers
    for a, b in zip(hid, layers):
        assert rel_err(a, b) < 2e-5
    assert rel_err(lg, want[-1]) < 2e-5
    hid2, lg2 = parity.DenseForward(cfg, s.dec.w).run(toks)
    for a, b in zip(hid2, layers):
        assert rel_err(a, b) < 2e-5
    assert rel_err(lg2, want[-1]) < 2e-5


def test_unequal_requests_in_one_batch_and_pages_used_again(tmp_path):
    """Requests of unequal length, portions beside single tokens, one paused, pages given back and handed to a later request."""
    cfg, raw, tensors = make("base")
    g = torch.Generator().manual_seed(5)
    seqs = {n: torch.randint(0, cfg.vocab_size, (k,), generator=g).tolist() for n, k in (("a", 40), ("b", 23), ("c", 9), ("d", 37))}
    want = {n: plain.forward(raw, tensors, t) for n, t in seqs.items()}
    s = session(cfg, tensors, tmp_path, page_size=8, max_tokens=88)       # 11 pages: a, b and c just fit
    at = {n: 0 for n in seqs}

    def run(parts, end=()):
        ents = [(n, seqs[n][at[n]:at[n] + k], range(k)) for n, k in parts]
        lg, i = s.step(ents, end), 0
        for n, k in parts:
            assert rel_err(lg[i:i + k], want[n][at[n]:at[n] + k]) < 2e-5, (n, at[n])
            i, at[n] = i + k, at[n] + k
    run([("a", 13), ("b", 1), ("c", 2)])
    run([("a", 1), ("b", 1), ("c", 1)])
    run([("b", 7), ("a", 1)])
    run([("c", 6), ("a", 9), ("b", 1)], end=["c"])
    run([("b", 13), ("a", 1)], end=["b"])
    run([("d", 30), ("a", 1)])
    run([("a", 14), ("d", 1)], end=["a"])
    run([("d", 6)], end=["d"])
    assert s.kv.in_use_pages == 0


def test_generation_through_the_engine_with_shared_prefixes(tmp_path):
    """Greedy generation of a batch through the scheduler: chunked prompts, prefix cache (whose pages bring the convolution's state
    along), requests that start later."""
    cfg, raw, tensors = make("base")
    save_file(tensors, str(tmp_path / "model.safetensors"))
    w = load_checkpoint(cfg, tmp_path, torch.device("cpu"), torch.float32)
    g = torch.Generator().manual_seed(8)
    common = torch.randint(0, cfg.vocab_size, (21,), generator=g).tolist()
    prompts = [common + [5, 6], common + [9], common[:11], common + [5, 6, 7, 8, 9]]
    for chunk in (0, 7):
        eng = Engine(Decoder(cfg, w, num_pages=64, page_size=8, max_pos=128),
                     EngineConfig(max_batch=4, chunk_tokens=chunk, tpot_ms=1e9, ttft_ms=1e9, prefix_cache=True))
        out = eng.generate(prompts[:2], 8) + eng.generate(prompts[2:], 8)
        assert eng.kv.prefix_hit_tokens_total > 0 and eng.kv.in_use_pages == 0
        for p, o in zip(prompts, out):
            seq = list(p)
            for tok in o:
                lg = plain.forward(raw, tensors, seq)[-1]
                assert lg[tok] >= lg.max() - 1e-4
                seq.append(tok)


def test_configuration_round_trip_and_refusals():
    cfg, raw, _ = make("base")
    assert mc.ModelConfig.from_hf_dict(cfg.to_hf_dict()).layers == cfg.layers
    assert cfg.layers[2].weights_of == 1 and cfg.layers[3].mlp is None
    j = json.dumps(cfg.to_hf_dict())
    assert core.model_param_count(j) == cfg.param_count() == sum(math.prod(s) for s in cfg.param_shapes().values())
    names = {p["name"] for l in json.loads(core.import_model(j))["layers"] for p in l["params"]}
    assert names == set(cfg.param_shapes())
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][2].update(weights_of=2), lambda d: d.pop("canon"),
                   lambda d: d["layers"][0]["mixer"]["rot"].update(dims=8), lambda d: d["layers"][2]["mixer"].update(heads=2),
                   lambda d: d["layers"][1]["mlp"]["router"].update(top=7)):
        bad = copy.deepcopy(cfg.to_hf_dict())
        change(bad)
        with pytest.raises(mc.ImportError_):
            mc.ModelConfig.from_hf_dict(bad)
    with pytest.raises(core.PlanError):
        core.lower_device_for(j, 2, 1, 1, 0)
    with pytest.raises(ValueError):
        from skein_b200.runtime.speculative import SpeculativeDecoder
        w = mc.ParallelLayout()
        from skein_b200.models.decoder import random_weights
        dec = Decoder(cfg, random_weights(cfg, w, "cpu"), num_pages=2)
        SpeculativeDecoder(dec, dec)


def test_missing_or_misshapen_tensor_is_named(tmp_path):
    cfg, _, tensors = make("base")
    t = dict(tensors)
    del t["l0.mix.uk"]
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="l0.mix.uk"):
        load_checkpoint(cfg, tmp_path, torch.device("cpu"))
    t["l0.mix.uk"] = torch.zeros(3, 3, dtype=torch.bfloat16)
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(ArtifactError, match="shape"):
        load_checkpoint(cfg, tmp_path, torch.device("cpu"))


def test_compile_verify_and_serve_on_cpu(tmp_path):
    """plan -> artifact -> parity -> engine, as the command line does it."""
    cfg, raw, tensors = make("base")
    save_file(tensors, str(tmp_path / "model.safetensors"))
    read = lambda p: (ROOT / p).read_text()      # noqa: E731
    r = compile_model(json.dumps(cfg.to_hf_dict()), read("cluster/b200_4x.toml"), read("cluster/sample_trace.jsonl"),
                      read("models/zarorax_13b_drift.toml"), read("cluster/cost_constants.toml"), tmp_path / "art",
                      weights=str(tmp_path), n_parity_prompts=1)
    assert r.plan["parallelism"] == {"tp": 1, "pp": 1, "ep": 1} and r.report.passed
    assert {tuple(d.values()) for d in r.plan["dtype_map"]["per_layer"]} == {("bf16", "bf16", "bf16")}
    art = Artifact(r.artifact_dir)
    art.check_lowering(0)
    w, src = art.load_weights(0, "cpu"), WeightSource(cfg, str(tmp_path))
    assert torch.equal(w.layers[1].w2[3], src.get("l1.mlp.e3.down", cfg.param_shapes()["l1.mlp.e3.down"])) and w.layers[2] is w.layers[1]
    out = subprocess.run([sys.executable, "-m", "skein_b200.parallel.worker", "--artifact", str(r.artifact_dir), "--cpu", "--prompt", "abc",
                          "--max-new-tokens", "4", "--max-seq-len", "64", "--max-batch", "2"], capture_output=True, text=True, cwd=ROOT)
    assert out.returncode == 0, out.stderr[-2000:]
    assert len(json.loads(out.stdout.strip().splitlines()[-1])["generated"][0]) == 4


def test_hot_swap_copies_every_slot(tmp_path):
    from skein_b200.models.decoder import random_weights
    from skein_b200.runtime.hotswap import _copy_into, _slots
    cfg = mc.tiny_zarorax()
    a, b = (random_weights(cfg, mc.ParallelLayout(), "cpu", seed=s) for s in (0, 1))
    for x, y in zip(a.layers, b.layers):
        for o, n in zip(_slots(x), _slots(y)):
            _copy_into(o, n)
    for x, y in zip(a.layers, b.layers):
        assert torch.equal(x.mixer.w_in, y.mixer.w_in) and torch.equal(x.conv, y.conv)
        assert x.w13 is None or torch.equal(x.w13, y.w13)


def test_trace_runner_program_on_cpu(tmp_path):
    cfg, raw, tensors = make("base")
    (tmp_path / "m").mkdir()
    (tmp_path / "m" / "config.json").write_text(json.dumps(cfg.to_hf_dict()))
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
    assert rel_err(rows(0), want[[3, 11]]) < 2e-5 and not (tmp_path / "1.f32").exists()
    assert rel_err(rows(2)[:1], want[13:]) < 2e-5 and rel_err(rows(2)[1:], want[:1] * 0 + plain.forward(raw, tensors, toks[:1])) < 2e-5
