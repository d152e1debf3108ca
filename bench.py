#!/usr/bin/env python
"""Headline benchmark: Mixtral-8x7B-shaped decode throughput (tokens/s) at 1/2/4/8 B200.

    python bench.py --gpus 1 --steps 128 --warmup 8
    python -m torch.distributed.run --nnodes=1 --nproc-per-node 8 --master-addr 127.0.0.1 \
        --master-port 29511 bench.py --gpus 8 --steps 128 --warmup 8

Workload (the serving config of the headline): random-init bf16 weights N(0, 0.02), 64 concurrent
sequences, prompts of 512 random token ids, 256 generated tokens, paged KV with block size 16,
tensor parallel over all N GPUs. A "step" is one decode step of the whole batch (64 tokens).

Two measurements, both with every kernel of the step (sampling included) inside the timed region, each
repeated (state reset in between) with the median reported:
  value  device-timed (CUDA events, max over ranks): K replays of the captured decode step with the
         sampled tokens fed back on the device.
  e2e    the serving path a client of `skein serve` gets: the 64 requests are submitted to the engine
         (C++ batcher, paged-KV manager), prefilled, and K iterations of Engine.step() are timed by wall
         clock. Every step copies its inputs (token ids, positions, lengths, sampling parameters, block
         tables) from pinned host memory to the device and reads the sampled tokens back; at N > 1 every
         rank runs its engine in lock step through the control page of runtime/driver.py, exactly as the
         rank processes of `skein serve --gpus` do.
The weights (93 GB at N=1) are far larger than L2, so no explicit L2 flush is needed between steps.

At N > 1 the run first proves that these N ranks compute the right tokens (a tiny Mixtral sharded over them,
teacher-forced against the unsharded CPU graph: "selfcheck"), and reports the same step with the fusion taken
out (GEMM -> copy/publish kernel -> pull, also captured in a CUDA graph: "unfused_ms_per_step").
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

BASELINE_TOK_S = 168.0  # the reference's only published number (2x RTX PRO 6000, PP=2)


def parse():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--model", default="mixtral-8x7b")
    ap.add_argument("--batch", type=int, default=64)
    ap.add_argument("--prompt", type=int, default=512)
    ap.add_argument("--gen", type=int, default=256)
    ap.add_argument("--layers", type=int, default=0, help="debug only: override the layer count (marks the run invalid)")
    ap.add_argument("--ep", type=int, default=1, help="expert-parallel degree (tensor parallel = gpus / ep / pp)")
    ap.add_argument("--pp", type=int, default=1, help="pipeline stages (tensor parallel = gpus / pp inside every stage)")
    ap.add_argument("--fp8-blocks", default="", help="'a:b' = blocks a..b-1 (of the whole model) in block-scaled fp8, all four projections")
    ap.add_argument("--fp8-experts", action="store_true", help="block-scaled e4m3 expert / FFN weights (marks dtype)")
    ap.add_argument("--prefill-chunk", type=int, default=4096, help="tokens per prefill chunk (device-timed prefill and the engine)")
    ap.add_argument("--no-e2e", action="store_true")
    ap.add_argument("--burst", type=int, default=0,
                    help="also replay a synthetic burst trace of this many requests through the serving engine (on/off Poisson "
                         "arrivals 50 / 2 per second every 10 s, log-normal prompts of median 600 capped at --prompt, outputs "
                         "uniform 32 .. --gen): adds the key 'burst' (TTFT / TPOT under load)")
    ap.add_argument("--burst-time-scale", type=float, default=1.0, help="trace seconds per wall second")
    ap.add_argument("--burst-only", action="store_true",
                    help="run only the burst replay (after the multi-rank self-check): --batch is the number of sequences "
                         "served at a time, --prompt / --gen cap the trace's prompt and output lengths and size the KV pool")
    ap.add_argument("--pp-continuous", action="store_true",
                    help="with --pp: the end-to-end engine keeps one group of sequences per stage in flight across steps "
                         "instead of draining the pipeline at the end of every step")
    ap.add_argument("--replicated-attention", action="store_true",
                    help="expert parallelism: every rank runs attention for all sequences (the comparison arm) instead of "
                         "each rank attending over its own slice with token dispatch between the ranks")
    ap.add_argument("--repeats", type=int, default=5, help="how often each timed K-step loop is repeated (median reported)")
    ap.add_argument("--no-selfcheck", action="store_true")
    ap.add_argument("--no-unfused", action="store_true", help="skip the un-fused comparison arm at N > 1")
    ap.add_argument("--design", default="", choices=["", "zarorax", "sikalorn", "barorax", "derusun"],
                    help="instead of the headline workload: throughput of this design at a few layer sizes beside the closest uniform model, "
                         "and its kernels' rooflines beside the like kernels (one JSON line per size; skein_b200/utils/design_bench.py)")
    ap.add_argument("--design-sizes", default="all", help="with --design: comma-separated sizes (zarorax: moe-2k, moe-4k, dense-4k; sikalorn: width-2k, width-4k; barorax: scan-2k, scan-4k; derusun: shift-2k, shift-4k)")
    ap.add_argument("--eager", action="store_true",
                    help="launch the step's kernels one by one instead of replaying the captured graph "
                         "(for a per-kernel launch list; the timed loop sits in an NVTX range named 'timed')")
    return ap.parse_args()


def reference_arm(args):
    # The reference is a Rust workspace (cargo, luminal, cudarc). It has no Python package to install
    # (`pip install` of its source tree: "Neither 'setup.py' nor 'pyproject.toml' found") and this image
    # has no Rust toolchain, so it cannot be built or run here.
    if int(os.environ.get("RANK", "0")) == 0:      # one line per job, not one per rank
        print(json.dumps({"impl": "reference",
                          "unavailable": "reference is a Rust/cargo workspace: pip reports no setup.py/pyproject.toml "
                                         "and the image has no cargo/rustc, so it cannot be built offline"}), flush=True)
    return 0


def measured_peaks():
    """The pool's measured copy bandwidth and cuBLAS bf16 rate (written next to this file by the harness), else the
    earlier measurement on the same pool."""
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    except (OSError, KeyError, ValueError):
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def step_roofline(cfg, tp, ep, B, ctx, fp8_experts, ms_per_step, n_gpus, dp=1):
    """Bytes one decode step must move per GPU (weights that the batch touches, KV read, logits) and over NVLink,
    and the step time those imply at the measured peaks. The step's target time is the slower of the two.
    dp: ranks that share the batch's sequences among them for attention (data-parallel attention under expert
    parallelism): a GPU then reads the KV of B / dp sequences only."""
    H, D, I, L, V = cfg.hidden_size, cfg.head_dim, cfg.intermediate_size, cfg.num_layers, cfg.vocab_size
    hq, hkv = cfg.num_heads // tp, max(1, cfg.num_kv_heads // tp)
    attn_w = ((hq + 2 * hkv) * D * H + H * hq * D) * 2
    wb = 1 if fp8_experts else 2
    if cfg.is_moe:
        e_local = cfg.num_experts // ep
        # experts that receive at least one of the B * top_k pairs (uniform routing): all of them at these batches
        pairs = B * cfg.top_k
        hit = cfg.num_experts * (1.0 - (1.0 - 1.0 / cfg.num_experts) ** pairs)
        ffn_w = min(e_local, hit / ep) * 3 * H * (I // tp) * wb + cfg.num_experts * H * 2
    else:
        ffn_w = 3 * H * (I // tp) * wb
    kv = (B // dp) * ctx * 2 * hkv * D * 2
    per_layer = attn_w + ffn_w + kv
    hbm = L * per_layer + (V // tp) * H * 2 + B * H * 2 * 8 * L        # + lm_head + activations (small)
    # NVLink: per all-reduce every GPU must receive the other ranks' partials of its batch ([B, H] bf16 each) unless the
    # switch adds them; the lower bound with in-switch reduction is one [B, H] per all-reduce
    n_ar = 2 * L if tp > 1 else 0
    nvl = n_ar * B * H * 2
    if ep > 1 and cfg.is_moe:
        # token dispatch: a GPU receives the rows routed to its experts from the other ranks ((ep-1)/ep of B top_k / ep rows
        # under uniform routing); combine: it fetches the expert outputs of its own rows' pairs from their owners
        own_rows = B // dp
        nvl += L * (B * cfg.top_k // ep + own_rows * cfg.top_k) * H * 2 * (ep - 1) // ep
    peaks = measured_peaks()
    t_hbm = hbm / (peaks["hbm_gbs"] * 1e9) * 1e3
    t_nvl = nvl / 770e9 * 1e3
    target = max(t_hbm, t_nvl)
    return {"hbm_bytes_per_step_per_gpu": int(hbm), "nvlink_bytes_in_per_step_per_gpu": int(nvl),
            "hbm_gbs_peak": peaks["hbm_gbs"], "nvlink_gbs_peak": 770.0, "peaks": peaks["source"],
            "target_ms_per_step": round(target, 4), "achieved_fraction": round(target / ms_per_step, 4),
            "achieved_hbm_gbs_per_gpu": round(hbm / (ms_per_step * 1e-3) / 1e9, 1)}



def cost_model_prediction(cfg, tp, ep, B, ctx, fp8_experts, n_gpus):
    """What the placement cost model (csrc/core/cost.hpp with cluster/cost_constants.toml, the numbers the planner ranks plans
    by) says this decode step takes, so that every run shows the model beside the measurement. None when the inputs of
    the model are not at hand (a GPU count without a cluster file)."""
    try:
        import re

        from skein_b200 import core
        root = os.path.dirname(os.path.abspath(__file__))
        cluster = open(os.path.join(root, "cluster", f"b200_{n_gpus}x.toml")).read()
        const = re.sub(r"decode_kv_tokens\s*=\s*\d+", f"decode_kv_tokens = {int(ctx)}", open(os.path.join(root, "cluster", "cost_constants.toml")).read())
        cfg_json = json.dumps(cfg.to_hf_dict())
        meta = json.loads(core.model_meta(cfg_json))
        # the model's dtype map is per block: expert weights in e4m3 are the bulk of a block's bytes
        wd = "fp8_e4m3" if fp8_experts else "bf16"
        plan = {"parallelism": {"tp": tp, "pp": 1, "ep": ep}, "kv": {"layout": {"kind": "paged", "page_size": 16}, "kv_sharded": True},
                "batching": {"kind": "continuous", "max_batch": B},
                "dtype_map": {"per_layer": [{"weight": wd, "activation": "bf16", "kv_cache": "bf16"}] * meta["num_layers"]},
                "execution": {"cuda_graphs": {"enable": True, "capture_classes": [{"batch_size": 1 << i, "kv_class": 0} for i in range(4)]},
                              "spec_decode": {"enable": False, "draft": None}, "prefix_cache": {"enable": True, "reuse_policy": "lru_by_last_access"}},
                "disaggregation": None, "model_meta": meta}
        b = core.cost_breakdown(json.dumps(plan), cfg_json, cluster, const, 0)
        return {"predicted_ms_per_step": round(b["total"] / 1e3, 3), "streaming_us": round(b["compute"]), "collectives_us": round(b["comm"]),
                "per_kernel_us": round(b["launch"]), "kernels": int(b["kernels"])}
    except Exception as e:      # noqa: BLE001  (the prediction is a side note of the benchmark line, never its failure)
        return {"unavailable": f"{type(e).__name__}: {e}"[:200]}


class ClockSampler:
    """SM clock and throttle reasons of one GPU, sampled DURING the timed region: NVML reads from a thread every
    10 ms (read-only queries), or `nvidia-smi -lms 100` when NVML cannot be loaded."""
    QUERY = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
             "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")
    REASON_BITS = {0x4: "sw_power_cap", 0x8: "hw_slowdown", 0x20: "sw_thermal_slowdown", 0x40: "hw_thermal_slowdown",
                   0x80: "hw_power_brake_slowdown"}

    def __init__(self, gpu_index: int):
        self.idx = gpu_index
        self.proc = None
        self.thread = None
        self.samples, self.reasons, self.max_mhz = [], set(), None
        self._stop = False

    def _physical_index(self):
        vis = os.environ.get("CUDA_VISIBLE_DEVICES")
        if vis:
            ids = [v.strip() for v in vis.split(",") if v.strip()]
            if self.idx < len(ids) and ids[self.idx].isdigit():
                return int(ids[self.idx])
        return self.idx

    def start(self):
        try:
            import threading

            import pynvml
            pynvml.nvmlInit()
            h = pynvml.nvmlDeviceGetHandleByIndex(self._physical_index())
            self.max_mhz = float(pynvml.nvmlDeviceGetMaxClockInfo(h, pynvml.NVML_CLOCK_SM))

            def loop():
                while not self._stop:
                    try:
                        self.samples.append(float(pynvml.nvmlDeviceGetClockInfo(h, pynvml.NVML_CLOCK_SM)))
                        bits = int(pynvml.nvmlDeviceGetCurrentClocksThrottleReasons(h))
                        for bit, name in self.REASON_BITS.items():
                            if bits & bit:
                                self.reasons.add(name)
                    except Exception:
                        pass
                    time.sleep(0.01)

            self.thread = threading.Thread(target=loop, daemon=True)
            self.thread.start()
            return
        except Exception:
            self.thread = None
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self._physical_index())], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.proc = None

    def stop(self):
        if self.thread is not None:
            self._stop = True
            self.thread.join(timeout=2)
            sm = self.samples
            return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": self.max_mhz,
                    "reasons": sorted(self.reasons), "samples": len(sm), "source": "nvml"}
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            out, _ = self.proc.communicate(timeout=5)
        except subprocess.TimeoutExpired:
            self.proc.kill()
            out, _ = self.proc.communicate()
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for line in out.strip().splitlines():
            f = [x.strip() for x in line.split(",")]
            if len(f) < 9:
                continue
            try:
                sm.append(float(f[1])); mx.append(float(f[2]))
            except ValueError:
                continue
            for n, v in zip(names, f[5:9]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(mx) if mx else None,
                "reasons": sorted(reasons), "samples": len(sm), "source": "nvidia-smi"}


def replay_burst(args, cfg, dec, runner, make_control, world, rank, B, P, Gn, use_graphs, max_over_ranks, barrier):
    """Replays a synthetic burst trace (the arrival process of the Mixtral-8x22B serving configuration this build is measured on) through the serving engine on all ranks in
    lock step: rank 0's clock is announced through the control page every step, every rank submits the requests that
    have arrived by then (the trace is generated from a seed, identically everywhere) and steps its engine. Chunked
    prefill interleaves with decode (at most 2048 prompt tokens per step while sequences decode), at most B sequences
    run at a time, the rest queue. Times are wall clock on rank 0, from a request's arrival to its tokens."""
    import torch

    from skein_b200 import core
    from skein_b200.runtime.engine import Engine, EngineConfig

    lines = core.synth_burst_trace(args.burst, 0, 50.0, 2.0, 10.0, 600.0, P, 32, Gn).splitlines()
    reqs = [json.loads(l) for l in lines[1:] if l.strip()]
    g = torch.Generator().manual_seed(4321)
    for kv in dec.kv:
        kv.zero_()
    ecfg = EngineConfig(max_batch=B, tpot_ms=1e9, ttft_ms=1e9, use_graphs=use_graphs, prefix_cache=False,
                        max_prefill_tokens=8192, interleave_prefill_tokens=2048)
    eng = Engine(dec, ecfg)
    eng.runner = runner
    ctl = make_control()
    prompts = [torch.randint(0, cfg.vocab_size, (max(1, min(int(r["prompt_tokens"]), P)),), generator=g).tolist() for r in reqs]
    arrival = [float(r["arrival_ms"]) / args.burst_time_scale for r in reqs]       # wall milliseconds after the start
    nxt, n_tok = 0, 0
    t_first, t_last, n_out, step_ms, batch_sizes = {}, {}, {}, [], []
    barrier()
    t0 = time.perf_counter()
    while nxt < len(reqs) or not eng.idle:
        t_s = time.perf_counter()
        if world > 1:
            if rank == 0:
                now = int((time.perf_counter() - t0) * 1e3)
                ctl.lead(None, now)
            else:
                _, now = ctl.follow()
        else:
            now = int((time.perf_counter() - t0) * 1e3)
        while nxt < len(reqs) and arrival[nxt] <= now:
            eng.submit(prompts[nxt], int(reqs[nxt]["output_tokens"]), now_ms=now, request_id=nxt + 1)
            nxt += 1
        evs = eng.step(now)
        if ctl.agree_failed(eng.last_step_failed):
            raise RuntimeError("an engine step failed during the burst replay: " + str([e.error for e in evs if e.error][:1]))
        t_e = time.perf_counter()
        if evs:
            step_ms.append((t_e - t_s) * 1e3)
            batch_sizes.append(len(evs))
        else:
            time.sleep(0.0002)
        for e in evs:
            if e.error is None:
                n_tok += 1
                t_first.setdefault(e.request_id, t_e)
                t_last[e.request_id] = t_e
                n_out[e.request_id] = n_out.get(e.request_id, 0) + 1
    torch.cuda.synchronize()
    wall = max_over_ranks(time.perf_counter() - t0)
    ctl.close()
    q = lambda xs, f: (sorted(xs)[min(len(xs) - 1, int(f * len(xs)))] if xs else None)
    ttft = [(t_first[i + 1] - t0) * 1e3 - arrival[i] for i in range(len(reqs)) if i + 1 in t_first]
    tpot = [(t_last[i] - t_first[i]) * 1e3 / (n_out[i] - 1) for i in t_first if n_out[i] > 1]
    rnd = lambda v: None if v is None else round(v, 2)
    return {"requests": len(reqs), "completed": len(t_first), "output_tokens": n_tok, "wall_s": round(wall, 2),
            "tokens_per_s": round(n_tok / wall, 1), "ttft_p50_ms": rnd(q(ttft, 0.5)), "ttft_p95_ms": rnd(q(ttft, 0.95)),
            "tpot_p50_ms": rnd(q(tpot, 0.5)), "tpot_p99_ms": rnd(q(tpot, 0.99)), "step_p50_ms": rnd(q(step_ms, 0.5)),
            "step_p99_ms": rnd(q(step_ms, 0.99)), "mean_batch": rnd(sum(batch_sizes) / max(1, len(batch_sizes))),
            "max_concurrent": B, "time_scale": args.burst_time_scale,
            "trace": "on/off Poisson 50 / 2 req/s every 10 s, log-normal prompts (median 600, max %d), outputs uniform 32..%d, seed 0" % (P, Gn)}


def run_pipeline(args, emit_json):
    """--pp > 1: tensor parallel inside each of `pp` stages (the Llama-3-70B configuration: TP=4 x PP=2). The device-
    timed loop is the steady-state pipelined decode (pp micro-batches in flight across steps, per-stage CUDA graphs,
    asynchronous point-to-point between stages); the end-to-end number runs the serving engine over the pipeline."""
    import datetime

    import torch
    import torch.distributed as dist

    from skein_b200 import ops
    from skein_b200.models import config as mc
    from skein_b200.models.decoder import BatchInputs, Decoder, quantize_blocks, random_weights
    from skein_b200.parallel import pp as pp_mod
    from skein_b200.parallel.tp import TPComm
    from skein_b200.runtime.driver import SharedControl
    from skein_b200.runtime.engine import Engine, EngineConfig
    from skein_b200.runtime.runner import ModelRunner

    world, rank, local_rank = int(os.environ["WORLD_SIZE"]), int(os.environ["RANK"]), int(os.environ["LOCAL_RANK"])
    torch.cuda.set_device(local_rank)
    dev = torch.device("cuda", local_rank)
    os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
    dist.init_process_group("nccl", device_id=dev, timeout=datetime.timedelta(seconds=300))
    control_group = dist.new_group(backend="gloo")
    cfg = {"mixtral-8x7b": mc.mixtral_8x7b, "mixtral-8x22b": mc.mixtral_8x22b, "llama3-70b": mc.llama3_70b}[args.model]()
    if args.layers:
        cfg.num_layers = args.layers
    npp = args.pp
    tp = world // npp
    lay = mc.ParallelLayout(tp=tp, pp=npp, rank=rank)
    tp_group, pp_ranks, pp_group = pp_mod.make_groups((tp, npp, 1), rank)
    fb_group = dist.new_group(list(range(world)))        # token feedback travels on its own communicator
    comm = TPComm(tp_group, dev, hidden=cfg.hidden_size, fused_rows=8192) if tp > 1 else None
    B, P, Gn, ps = args.batch, args.prompt, args.gen, 16
    Gn = max(Gn, args.steps + max(args.warmup, 3) + 8)       # room for a timed loop longer than the generation length
    blocks_per_seq = (P + Gn + ps - 1) // ps + 1
    num_pages = B * blocks_per_seq + 8
    weights = random_weights(cfg, lay, dev, seed=0, std=0.02, shard_embed=True)
    fp8_note = "bf16"
    if args.fp8_blocks:
        a, b = (int(x) for x in args.fp8_blocks.split(":"))
        mine = list(lay.stage_layers(cfg.num_layers))
        quantize_blocks(weights, [i for i, g in enumerate(mine) if a <= g < b])
        fp8_note = f"blocks {a}..{b - 1} block-scaled fp8 (e4m3, 1x128), the rest bf16"
    dec = Decoder(cfg, weights, lay, num_pages=num_pages, page_size=ps, max_pos=P + Gn + 64, comm=comm)
    stage = pp_mod.PipelineStage(dec, lay, pp_ranks, pp_group)
    runner = ModelRunner(stage, max_blocks_per_seq=blocks_per_seq, use_graphs=False, ctx_hint=P + Gn // 2)
    g = torch.Generator().manual_seed(1234)
    prompts = torch.randint(0, cfg.vocab_size, (B, P), generator=g).tolist()
    tables = [list(range(1 + s * blocks_per_seq, 1 + (s + 1) * blocks_per_seq)) for s in range(B)]

    def barrier():
        dist.barrier()
        torch.cuda.synchronize()

    def max_over_ranks(x):
        t = torch.tensor([x], device=dev, dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t[0])

    def check_all(where):
        code = ops.workspace().status[:1].clone()
        dist.all_reduce(code, op=dist.ReduceOp.MAX)
        if int(code[0]) != 0:
            if rank == 0:
                emit_json({"error": f"device status {int(code[0])} after {where}", "n_gpus": world})
            os._exit(3)

    # ---- prefill: chunks of up to 8192 tokens through the pipeline ----
    per_chunk = max(1, 8192 // P)
    barrier()
    t_pf = time.perf_counter()
    first_tokens = []
    for c0 in range(0, B, per_chunk):
        first_tokens.extend(runner.prefill([(prompts[s], tables[s], 0) for s in range(c0, min(B, c0 + per_chunk))]))
    torch.cuda.synchronize()
    prefill_cold_ms = max_over_ranks((time.perf_counter() - t_pf) * 1e3)
    check_all("prefill")
    # the same prefill once more: the first pass also pays for one-time set-up (communicator connections between the
    # stages, kernel attributes, allocator growth)
    barrier()
    t_pf = time.perf_counter()
    again = []
    for c0 in range(0, B, per_chunk):
        again.extend(runner.prefill([(prompts[s], tables[s], 0) for s in range(c0, min(B, c0 + per_chunk))]))
    torch.cuda.synchronize()
    prefill_ms = max_over_ranks((time.perf_counter() - t_pf) * 1e3)
    prefill_repeatable = again == first_tokens

    # ---- steady-state pipelined decode: pp micro-batches in flight ----
    M = npp
    per = B // M
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    K, W, R = args.steps, max(args.warmup, 3), max(1, args.repeats)

    def make_micro():
        micro = []
        for m in range(M):
            rows = list(range(m * per, (m + 1) * per))
            bt = torch.zeros(per, blocks_per_seq, dtype=torch.int32, device=dev)
            for i, r_ in enumerate(rows):
                bt[i] = i32(tables[r_])
            micro.append(BatchInputs(token_ids=i32([first_tokens[r_] for r_ in rows]), positions=i32([P] * per), block_table=bt,
                                     seq_lens=i32([P + 1] * per), ctx_hint=P + Gn // 2))
        return micro

    micro = make_micro()

    def advance(inp, toks):
        ops.advance_decode_state(toks if toks is not None else inp.token_ids, inp.token_ids, inp.positions, inp.seq_lens)

    def reset(micro):
        for m, inp in enumerate(micro):
            rows = list(range(m * per, (m + 1) * per))
            inp.token_ids.copy_(i32([first_tokens[r_] for r_ in rows]))
            inp.positions.fill_(P)
            inp.seq_lens.fill_(P + 1)

    from skein_b200.ops import _lib
    times, idle, launches_per_step = [], None, None
    for r in range(R):
        reset(micro)
        torch.cuda.synchronize()
        l0 = _lib.launches()
        pp_mod.pipelined_decode(stage, micro, W, advance, fb_group, resume=False, more=True)
        if r == 0:
            # the first step ran eagerly and the second was captured: each counted this rank's launches of one step once
            # (minus the position updates, which are counted on every step)
            launches_per_step = (_lib.launches() - l0 - M * (W - 1)) // 2
        barrier()
        stage.stage_busy_events, stage.time_stages = [], (r == R - 1)
        ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        ev0.record()
        pp_mod.pipelined_decode(stage, micro, K, advance, fb_group, resume=True, more=False)
        ev1.record()
        barrier()
        ms_r = ev0.elapsed_time(ev1)
        if r == R - 1:
            idle = stage.idle_fraction(ms_r)
            stage.time_stages = False
        times.append(max_over_ranks(ms_r))
        check_all("the pipelined decode")
    times.sort()
    ms = times[len(times) // 2]
    value = B * K / (ms / 1e3)
    idles = [None] * world
    dist.all_gather_object(idles, idle)

    # ---- end to end: the serving engine over the pipeline (micro-batched steps, lock-step control page) ----
    e2e = None
    if not args.no_e2e:
        for kv in dec.kv:
            kv.zero_()
        ecfg = EngineConfig(max_batch=B, tpot_ms=1e9, ttft_ms=1e9, use_graphs=False, prefix_cache=False, max_prefill_tokens=8192,
                            interleave_prefill_tokens=0, pp_continuous=args.pp_continuous)
        stage.feedback_group = fb_group
        ctl = SharedControl(f"/dev/shm/skein_bench_ctl_{os.environ.get('MASTER_PORT', '0')}", rank, world, control_group, wait_s=300)
        eng = Engine(stage, ecfg)
        for s_ in range(B):
            eng.submit(prompts[s_], Gn, now_ms=0, request_id=s_ + 1)

        def one_step():
            if rank == 0:
                now = eng.clock()
                ctl.lead(None, now)
            else:
                _, now = ctl.follow()
            evs = eng.step(now)
            if ctl.agree_failed(eng.last_step_failed):
                raise RuntimeError("an engine step failed: " + str([e.error for e in evs if e.error][:1]))
            return evs

        # continuous mode: a step accepts the tokens of one of the pp groups of sequences, so pp steps make one token per sequence
        per_tok = npp if args.pp_continuous else 1
        n_dec = 0
        while n_dec < W * per_tok:
            evs = one_step()
            if len(evs) == B // per_tok and all(not e.is_final for e in evs):
                n_dec += 1
        barrier()
        t_a = time.perf_counter()
        n_tok = 0
        for _ in range(K * per_tok):
            n_tok += sum(1 for e in one_step() if e.error is None)
        torch.cuda.synchronize()
        wall = max_over_ranks(time.perf_counter() - t_a)
        bk = eng.runner.bucket(B // per_tok, slot=0 if args.pp_continuous else None)
        e2e = {"value": round(n_tok / wall, 2), "unit": "tokens/s", "h2d_bytes_per_step": bk.h2d_bytes * per_tok,
               "d2h_bytes_per_step": bk.d2h_bytes * per_tok,
               "path": ("Engine.step over PipelineStage, one group of sequences per stage kept in flight across steps" if args.pp_continuous
                        else "Engine.step over PipelineStage (pp micro-batches per step, per-stage CUDA graphs)") + "; lock-step control page"}
        ctl.close()
    if rank == 0:
        emit_json({
            "metric": args.model.replace("-", "_") + "_decode_tokens_per_s", "value": round(value, 2), "unit": "tokens/s",
            "n_gpus": world, "steps": K, "warmup": W, "ms_per_step": round(ms / K, 4), "higher_is_better": True, "scaling": "strong",
            "vs_baseline": None, "dtype": "bf16" if not args.fp8_blocks else "bf16 activations; " + fp8_note,
            "data": "synthetic (random-init weights N(0,0.02), random prompt token ids)",
            "config": {"model": cfg.name + ("" if not args.layers else f"-{args.layers}layers-INVALID"), "global_batch": B, "seq_len": P,
                       "gen_len": args.gen, "parallelism": f"tp{tp}xpp{npp}", "kv": "paged, block 16", "micro_batches": M,
                       "l2": "inputs (weights) larger than L2, no flush", "cuda_graph": "per stage and micro-batch",
                       "weights": fp8_note, "repeats": R},
            "prefill_ms": round(prefill_ms, 1), "prefill_first_pass_ms": round(prefill_cold_ms, 1), "prefill_repeatable": prefill_repeatable, "stage_idle_fraction_per_rank": [None if x is None else round(x, 3) for x in idles],
            "e2e": e2e, "gpu_launches": (launches_per_step or 0) * K, "kernels_per_step_on_rank0": launches_per_step, "impl": "ours"})
    dist.barrier()
    dist.destroy_process_group()
    return 0


def main():
    args = parse()
    if args.impl == "reference":
        return reference_arm(args)
    if args.design:
        import torch

        from skein_b200.utils import design_bench
        sizes = design_bench.DESIGNS[args.design][0] if args.design_sizes == "all" else args.design_sizes.split(",")
        for size in sizes:
            sampler = ClockSampler(0)
            sampler.start()
            lines = []
            with torch.no_grad():
                design_bench.run(args.design, [size], emit=lines.append)
            out = json.loads(lines[0])
            out["clocks"] = sampler.stop()
            print(json.dumps(out), flush=True)
        return 0
    if args.pp > 1:
        sys.stdout.flush()
        fd = os.dup(1)
        os.dup2(2, 1)
        return run_pipeline(args, lambda obj: os.write(fd, (json.dumps(obj) + "\n").encode()))

    # Libraries (NCCL's version banner, for one) write to file descriptor 1. Keep the real stdout for the one JSON
    # line and send everything else that lands on descriptor 1 to stderr.
    sys.stdout.flush()
    json_fd = os.dup(1)
    os.dup2(2, 1)

    def emit_json(obj):
        os.write(json_fd, (json.dumps(obj) + "\n").encode())

    import torch
    import torch.distributed as dist

    from skein_b200 import ops
    from skein_b200.models import config as mc
    from skein_b200.models.decoder import Decoder, random_weights
    from skein_b200.ops import _lib
    from skein_b200.runtime.driver import LocalControl, SharedControl
    from skein_b200.runtime.engine import Engine, EngineConfig
    from skein_b200.runtime.runner import ModelRunner

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus:
        if world == 1 and args.gpus > 1:
            raise SystemExit("launch multi-GPU runs with torch.distributed.run (WORLD_SIZE must equal --gpus)")
    torch.cuda.set_device(local_rank)
    dev = torch.device("cuda", local_rank)
    cfg = {"mixtral-8x7b": mc.mixtral_8x7b, "mixtral-8x22b": mc.mixtral_8x22b, "llama3-70b": mc.llama3_70b}[args.model]()
    if args.layers:
        cfg.num_layers = args.layers
    ep = max(1, args.ep)
    if world % ep != 0 or (ep > 1 and not cfg.is_moe):
        raise SystemExit("--ep must divide the number of GPUs and needs a mixture-of-experts model")
    tp = world // ep
    if tp >= 8:
        # in-switch reduction of the tensor-parallel partials: measured 4.46 against 4.74 ms per step at 8 ranks (no gain
        # at 2 and 4, where it stays off); SKEIN_MULTIMEM=0 keeps the peer-load path
        os.environ.setdefault("SKEIN_MULTIMEM", "1")
    comm, comm_moe, control_group = None, None, None
    selfcheck = None
    if world > 1:
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        import datetime
        dist.init_process_group("nccl", device_id=dev, timeout=datetime.timedelta(seconds=180))
        control_group = dist.new_group(backend="gloo")
        from skein_b200.parallel.tp import TPComm
        groups = [dist.new_group(list(range(b0, b0 + tp))) for b0 in range(0, world, tp)] if (ep > 1 and tp > 1) else None
        tp_group = (groups[rank // tp] if groups else dist.group.WORLD) if tp > 1 else None
        if not args.no_selfcheck:
            # the same ranks, groups, collectives and graph runner on a tiny model with a CPU oracle
            from skein_b200.parallel.selfcheck import teacher_forced_check
            c1 = TPComm(tp_group, dev, hidden=1024, fused_rows=256, max_batch=64) if tp > 1 else None
            c2 = TPComm(dist.group.WORLD, dev, hidden=1024, fused_rows=256, max_batch=64) if ep > 1 else None
            # Two independently drawn tiny models: a wrong collective or kernel fails on both, while a rounding coincidence
            # that the near-tie rules do not cover is tied to one draw. Every rank sees the same tokens, so all ranks take
            # the same branch here.
            failures = []
            for seed in (11, 12):
                try:
                    info = teacher_forced_check(world, rank, dev, comm=c1, comm_moe=c2, tp=tp, ep=ep, hidden=1024,
                                                fp8_experts=args.fp8_experts, seed=seed,
                                                dp_attention=ep > 1 and tp == 1 and not args.replicated_attention)
                    selfcheck = dict(info, result="ok", seed=seed, failed_seeds=[f[0] for f in failures])
                    break
                except AssertionError as e:
                    failures.append((seed, str(e)[:1500]))
            if selfcheck is None:
                if rank == 0:
                    emit_json({"error": "selfcheck failed", "detail": failures, "n_gpus": world})
                os._exit(4)       # the other ranks may be waiting in a collective: leave without one
            dist.barrier()
            for c in (c1, c2):
                if c is not None:
                    c.close()
        if tp > 1:
            # room for the partials of one 8192-token prefill chunk (its expert-sorted rows for a MoE model)
            comm = TPComm(tp_group, dev, hidden=cfg.hidden_size, fused_rows=max(512, 8192 * max(1, cfg.top_k if cfg.is_moe else 1)))
        if ep > 1:   # communicator over all tp x ep ranks for the expert-parallel combine
            comm_moe = TPComm(dist.group.WORLD, dev, hidden=cfg.hidden_size, fused_rows=max(512, 8192 * cfg.top_k),
                              max_batch=max(256, args.batch))
    lay = mc.ParallelLayout(tp=tp, ep=ep, rank=rank)
    B, P, Gn, ps = args.batch, args.prompt, args.gen, 16
    # a timed loop longer than the workload's generation length keeps decoding the same sequences: room for those tokens
    Gn = max(Gn, args.steps + max(args.warmup, 3) + 8)
    blocks_per_seq = (P + Gn + ps - 1) // ps + 1
    num_pages = B * blocks_per_seq + 8
    t0 = time.time()
    weights = random_weights(cfg, lay, dev, seed=0, std=0.02, shard_embed=True)    # vocabulary-parallel embedding under TP
    if args.fp8_experts:
        from skein_b200.models.decoder import quantize_blocks
        quantize_blocks(weights, range(len(weights.layers)), names=("w13", "w2"))
    dec = Decoder(cfg, weights, lay, num_pages=num_pages, page_size=ps, max_pos=P + Gn + 64, comm=comm, comm_moe=comm_moe)
    if ep > 1 and tp == 1 and not args.replicated_attention:
        dec.dp_attention = True      # rows are static in this benchmark: a sequence stays on its rank
    fused = all(c is None or c.mode != "nccl" for c in (comm, comm_moe))
    use_graphs = fused and not args.eager   # the NCCL baseline mode launches eagerly
    runner = ModelRunner(dec, max_blocks_per_seq=blocks_per_seq, use_graphs=use_graphs, ctx_hint=P + Gn // 2)
    torch.cuda.synchronize()
    t_init = time.time() - t0

    # ---- requests: identical on every rank ---------------------------------------------------------
    g = torch.Generator().manual_seed(1234)
    prompts = torch.randint(0, cfg.vocab_size, (B, P), generator=g).tolist()
    tables = [list(range(1 + s * blocks_per_seq, 1 + (s + 1) * blocks_per_seq)) for s in range(B)]

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    def check_all(where):
        # every rank learns of a device-side error (a peer wait that ran out, a bad index) on any rank
        code = ops.workspace().status[:1].clone()
        if world > 1:
            dist.all_reduce(code, op=dist.ReduceOp.MAX)
        if int(code[0]) != 0:
            if rank == 0:
                emit_json({"error": f"device status {int(code[0])} after {where}", "n_gpus": world})
            if world > 1:
                dist.destroy_process_group()
            sys.exit(3)

    def max_over_ranks(x: float) -> float:
        if world == 1:
            return x
        t = torch.tensor([x], device=dev, dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t[0])

    if args.burst_only:
        if args.burst <= 0:
            raise SystemExit("--burst-only needs --burst N")

        def make_control_():
            if world > 1:
                return SharedControl(f"/dev/shm/skein_bench_ctl_{os.environ.get('MASTER_PORT', '0')}", rank, world, control_group, wait_s=120)
            return LocalControl()
        if use_graphs:
            runner.capture_buckets(B)
        burst = replay_burst(args, cfg, dec, runner, make_control_, world, rank, B, P, Gn, use_graphs, max_over_ranks, barrier)
        check_all("the burst replay")
        if rank == 0:
            emit_json({"metric": args.model.replace("-", "_") + "_burst_trace_tokens_per_s", "value": burst["tokens_per_s"],
                       "unit": "tokens/s", "n_gpus": world, "higher_is_better": True, "dtype": "bf16" if not args.fp8_experts else
                       "bf16 activations, fp8 expert weights", "data": "synthetic (random-init weights N(0,0.02), synthetic burst trace)",
                       "config": {"model": cfg.name, "parallelism": f"tp{tp}" + (f"xep{ep}" if ep > 1 else ""), "max_concurrent": B,
                                  "cuda_graph": use_graphs, "expert_weights": "fp8 e4m3 1x128" if args.fp8_experts else "bf16"},
                       "burst": burst, "selfcheck": "single rank" if world == 1 else (selfcheck or {}).get("result", "skipped"),
                       "impl": "ours"})
        if world > 1:
            dist.barrier()
            dist.destroy_process_group()
        return

    # ---- prefill (chunks of up to --prefill-chunk tokens) ----------------------------------------------
    per_chunk = max(1, args.prefill_chunk // P)
    barrier()
    first_tokens = []
    t_pf = time.perf_counter()
    for c0 in range(0, B, per_chunk):
        first_tokens.extend(runner.prefill([(prompts[s], tables[s], 0) for s in range(c0, min(B, c0 + per_chunk))]))
    torch.cuda.synchronize()
    prefill_cold_ms = max_over_ranks((time.perf_counter() - t_pf) * 1e3)   # first pass: also pays for one-time set-up
    check_all("prefill")
    barrier()
    t_pf = time.perf_counter()
    again = []
    for c0 in range(0, B, per_chunk):
        again.extend(runner.prefill([(prompts[s], tables[s], 0) for s in range(c0, min(B, c0 + per_chunk))]))
    torch.cuda.synchronize()
    prefill_ms = max_over_ranks((time.perf_counter() - t_pf) * 1e3)        # whole batch, tokens read back per chunk
    prefill_repeatable = again == first_tokens

    K, W, R = args.steps, max(args.warmup, 3), max(1, args.repeats)
    if K + W > Gn - 1:
        raise SystemExit(f"--steps + --warmup must stay below the {Gn} generated tokens of the workload")

    def device_timed(run: ModelRunner, label: str):
        """R repeats of: reset the decode state, W warm-up steps, K timed steps (CUDA events, max over ranks)."""
        bk = run.bucket(B)
        if run.use_graphs:
            run._ensure_graph(bk, True)
        times, clocks = [], None
        for r in range(R):
            run.load_decode_inputs(bk, first_tokens, [P] * B, [P + 1] * B, tables)
            bk.dev_in.copy_(bk.host_in)
            torch.cuda.synchronize()
            for i in range(W):
                run.decode_loop_step(bk)
                if r == 0 and i == 0:
                    check_all(f"the first decode step ({label})")
            sampler = ClockSampler(local_rank) if r == R // 2 else None
            barrier()
            if sampler:
                sampler.start()
            ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            ev0.record()
            torch.cuda.nvtx.range_push("timed")
            for _ in range(K):
                run.decode_loop_step(bk)
            torch.cuda.nvtx.range_pop()
            ev1.record()
            barrier()
            if sampler:
                clocks = sampler.stop()
            times.append(max_over_ranks(ev0.elapsed_time(ev1)))
            check_all(f"the timed loop ({label})")
        times.sort()
        return times[len(times) // 2], times, clocks, bk

    ms, all_ms, clocks, bk = device_timed(runner, "fused")
    value = B * K / (ms / 1e3)
    # kernels per step: count one eager step's launches on a scratch copy of the state
    saved = bk.dev_in.clone()
    torch.cuda.synchronize()
    l1 = _lib.launches()
    runner._decode_body(bk, True)
    torch.cuda.synchronize()
    launches_per_step = _lib.launches() - l1
    bk.dev_in.copy_(saved)

    # ---- the same step with the fusion taken out (graph against graph) ---------------------------------------
    unfused_ms = None
    if world > 1 and not args.no_unfused and use_graphs and all(c is None or c.mode == "fused" for c in (comm, comm_moe)):
        from skein_b200.parallel.tp import TPComm
        u1 = TPComm(comm.group, dev, hidden=cfg.hidden_size, mode="unfused", multimem=comm.multimem, max_batch=comm.max_batch) if comm is not None else None
        u2 = TPComm(comm_moe.group, dev, hidden=cfg.hidden_size, mode="unfused", multimem=comm_moe.multimem) if comm_moe is not None else None
        dec_u = Decoder(cfg, weights, lay, num_pages=0, page_size=ps, max_pos=P + Gn + 64, comm=u1, comm_moe=u2)
        dec_u.kv, dec_u.num_pages = dec.kv, dec.num_pages          # same weights, same cache
        run_u = ModelRunner(dec_u, max_blocks_per_seq=blocks_per_seq, use_graphs=True, ctx_hint=P + Gn // 2)
        unfused_ms, _, _, _ = device_timed(run_u, "unfused")

    def make_control():
        if world > 1:
            return SharedControl(f"/dev/shm/skein_bench_ctl_{os.environ.get('MASTER_PORT', '0')}", rank, world, control_group, wait_s=120)
        return LocalControl()

    # ---- end to end through the serving engine ----------------------------------------------------------------
    e2e, ttft_p50, tpot_p99 = None, None, None
    if not args.no_e2e:
        ecfg = EngineConfig(max_batch=B, tpot_ms=1e9, ttft_ms=1e9, use_graphs=use_graphs, prefix_cache=False,
                            max_prefill_tokens=args.prefill_chunk, interleave_prefill_tokens=0)
        for kv in dec.kv:
            kv.zero_()
        ctl = make_control()
        if use_graphs:
            runner.capture_buckets(B)      # as the server does while it starts: no request pays for a graph capture
        e2e_vals, step_ms = [], []
        parts = {"announce": 0.0, "engine_step": 0.0, "agree": 0.0, "n": 0}
        for r in range(min(R, 3)):
            eng = Engine(dec, ecfg)
            eng.runner = runner                                   # reuse the captured graphs
            t_sub = eng.clock()
            for s in range(B):
                eng.submit(prompts[s], Gn, now_ms=t_sub, request_id=s + 1)
            n_decode_steps, t_a = 0, None
            first_seen = {}
            t_wall0 = time.perf_counter()

            def one_step():
                t0_ = time.perf_counter()
                if world > 1:
                    if rank == 0:
                        now = eng.clock()
                        ctl.lead(None, now)
                    else:
                        _, now = ctl.follow()
                else:
                    now = eng.clock()
                t1_ = time.perf_counter()
                evs = eng.step(now)
                t2_ = time.perf_counter()
                if ctl.agree_failed(eng.last_step_failed):
                    raise RuntimeError("an engine step failed: " + str([e.error for e in evs if e.error][:1]))
                t3_ = time.perf_counter()
                parts["announce"] += t1_ - t0_; parts["engine_step"] += t2_ - t1_; parts["agree"] += t3_ - t2_; parts["n"] += 1
                return evs

            # prefill iterations, then warm-up decode iterations
            while True:
                evs = one_step()
                for e in evs:
                    first_seen.setdefault(e.request_id, (time.perf_counter() - t_wall0) * 1e3)
                if len(evs) == B and eng.batcher.inflight_len == B and all(not e.is_final for e in evs):
                    n_decode_steps += 1
                    if n_decode_steps >= W:
                        break
            barrier()
            for k_ in parts:
                parts[k_] = 0 if k_ == "n" else 0.0
            t_a = time.perf_counter()
            for _ in range(K):
                t_s = time.perf_counter()
                evs = one_step()                 # batcher + H2D inputs + graph replay + D2H tokens + control page
                step_ms.append((time.perf_counter() - t_s) * 1e3)
                assert len(evs) == B
            torch.cuda.synchronize()
            wall = max_over_ranks(time.perf_counter() - t_a)
            e2e_vals.append(B * K / wall)
            if r == 0:      # time from submission of all B requests to each request's first token, wall clock
                ttfts = sorted(first_seen.values())
                ttft_p50 = ttfts[len(ttfts) // 2]
            eng.abort_all("benchmark repeat finished")
            barrier()
        ctl.close()
        e2e_vals.sort()
        step_ms.sort()
        tpot_p99 = round(step_ms[min(len(step_ms) - 1, int(0.99 * len(step_ms)))], 3)
        e2e = {"value": round(e2e_vals[len(e2e_vals) // 2], 2), "unit": "tokens/s", "h2d_bytes_per_step": bk.h2d_bytes,
               "d2h_bytes_per_step": bk.d2h_bytes, "tpot_p50_ms": round(step_ms[len(step_ms) // 2], 3), "tpot_p99_ms": tpot_p99,
               "path": "Engine.step (C++ batcher + paged-KV manager) -> ModelRunner.decode_step; lock-step control page at N > 1",
               "repeats": [round(v, 1) for v in e2e_vals],
               "host_us_per_step_rank0": {k: round(v / max(1, parts["n"]) * 1e6, 1) for k, v in parts.items() if k != "n"}}

    burst = None
    if args.burst > 0:
        burst = replay_burst(args, cfg, dec, runner, make_control, world, rank, B, P, Gn, use_graphs, max_over_ranks, barrier)

    if rank == 0:
        out = {
            "metric": args.model.replace("-", "_") + "_decode_tokens_per_s", "value": round(value, 2), "unit": "tokens/s",
            "n_gpus": world, "steps": K, "warmup": W, "ms_per_step": round(ms / K, 4), "higher_is_better": True,
            "scaling": "strong",
            "vs_baseline": round(value / BASELINE_TOK_S, 2) if args.model == "mixtral-8x7b" and not args.layers else None,
            "dtype": "bf16" if not args.fp8_experts else "bf16 activations, fp8 expert weights",
            "data": "synthetic (random-init weights N(0,0.02), random prompt token ids)",
            "config": {"model": cfg.name + ("" if not args.layers else f"-{args.layers}layers-INVALID"),
                       "global_batch": B, "seq_len": P, "gen_len": args.gen, "parallelism": f"tp{tp}" + (f"xep{ep}" if ep > 1 else ""),
                       "kv": "paged, block 16", "l2": "inputs (weights) larger than L2, no flush",
                       "cuda_graph": use_graphs, "comm": ((comm or comm_moe).mode if (comm or comm_moe) else "none"),
                       "in_switch_reduction": bool((comm or comm_moe).heap.mc_ptr) if (comm or comm_moe) else False,
                       "attention": ("data-parallel (each expert-parallel rank attends over its own sequences, token dispatch "
                                     "over peer memory)" if dec.dp_attention else "replicated across expert-parallel ranks") if ep > 1 else "tensor-parallel",
                       "expert_weights": "fp8 e4m3 1x128" if args.fp8_experts else "bf16",
                       "repeats": R, "ms_per_k_steps_all_repeats": [round(x, 3) for x in all_ms]},
            "roofline": step_roofline(cfg, tp, ep, B, P + (W + K // 2), args.fp8_experts, ms / K, world,
                                      dp=ep if dec.dp_attention else 1),
            "cost_model": cost_model_prediction(cfg, tp, ep, B, P + (W + K // 2), args.fp8_experts, world),
            "prefill_ms": round(prefill_ms, 1), "prefill_first_pass_ms": round(prefill_cold_ms, 1), "prefill_repeatable": prefill_repeatable,
            "prefill_tokens_per_s": round(B * P / prefill_ms * 1e3, 1),
            "ttft_p50_ms": None if ttft_p50 is None else round(ttft_p50, 2),
            "tpot_p99_ms": tpot_p99,
            "e2e": e2e, "burst": burst, "gpu_launches": launches_per_step * K, "kernels_per_step": launches_per_step,
            "selfcheck": selfcheck["result"] if selfcheck else ("skipped" if world > 1 else "single rank"),
            "selfcheck_detail": selfcheck,
            "unfused_ms_per_step": None if unfused_ms is None else round(unfused_ms / K, 4),
            "clocks": clocks, "init_s": round(t_init, 1), "impl": "ours",
        }
        emit_json(out)
    if world > 1:
        dist.barrier()
        dist.destroy_process_group()
    return 0


if __name__ == "__main__":
    sys.exit(main())
