"""Replay of a token trace: given token ids are fed through a model step by step and the logits of chosen places are written.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

A step is one JSON object a line: {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [ids]}. Every
entry brings a request's next tokens (a portion of a prompt, or one decoded token); all entries run as one batch from the cache
that earlier steps left; "end" lists requests whose pages are given back afterwards. Logits of the wanted places go to
OUT/<step>.f32 (little-endian fp32, in order) and "done <step>" is printed after every step. The model, its cache manager, the
step function and the captured decode steps are the ones that serve generations; nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


MAX_LIVE = 4          # state slots: most requests that may be live at a time (models with a recurrent state)


class TraceSession:
    """Requests by name over one decoder, a page pool of `max_tokens` tokens and (with a recurrent state) MAX_LIVE state slots."""

    def __init__(self, decoder, max_tokens: int, use_graphs: bool = True):
        from .. import core
        from .runner import ModelRunner
        self.dec = decoder
        self.kv = core.KvBlockManager(decoder.num_pages, decoder.page_size, False, state_slots=decoder.num_state_slots)
        self.runner = ModelRunner(decoder, max(1, -(-max_tokens // decoder.page_size)), use_graphs=use_graphs, ctx_hint=max_tokens)
        self._rid, self._cached, self._next = {}, {}, 1

    def step(self, entries, end=()):
        """entries: (id, tokens, want) triples. Returns the wanted logits [n, vocab] fp32 on the host, or None."""
        seqs, wants = [], []
        for name, tokens, want in entries:
            tokens = [int(t) for t in tokens]
            if name not in self._rid:
                self._rid[name], self._cached[name] = self._next, 0
                self._next += 1
                self.kv.admit(self._rid[name], tokens)
            else:
                self.kv.advance(self._rid[name], len(tokens))
            seqs.append((tokens, self.kv.pages_for(self._rid[name]), self._cached[name], self.kv.slot_of(self._rid[name])))
            wants.append([int(w) for w in want])
        logits = None
        if seqs:
            logits = self.runner.extend(seqs, wants)
            for (name, _, _), s in zip(entries, seqs):
                self._cached[name] += len(s[0])
            logits = logits.float().cpu() if any(wants) else None
            if self.dec.device.type == "cuda":
                from .. import ops
                ops.workspace().check_status()
        for name in end:
            self.kv.release(self._rid.pop(name))
            self._cached.pop(name)
        return logits


def open_session(model_dir, dtype: str, max_tokens: int, device) -> TraceSession:
    import torch

    from ..compile.artifact import load_checkpoint
    from ..models.config import ModelConfig
    from ..models.decoder import Decoder
    cfg = ModelConfig.from_file(os.path.join(model_dir, "config.json"))
    weights = load_checkpoint(cfg, model_dir, device, getattr(torch, dtype))
    ps = cfg.default_page_size
    dec = Decoder(cfg, weights, num_pages=max(1, -(-max_tokens // ps)), page_size=ps, max_pos=max_tokens, state_slots=MAX_LIVE)
    return TraceSession(dec, max_tokens)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at a time (the page pool's size)")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu: the reference operators (for debugging)")
    args = ap.parse_args(argv)
    from .. import _build
    from ..models.config import ModelConfig
    cfg = ModelConfig.from_file(os.path.join(args.model, "config.json"))
    _build.ensure_built(cfg.architecture, kernels=args.device == "cuda")
    import torch
    if args.device == "cuda" and not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 2
    torch.backends.cuda.matmul.allow_tf32 = False
    session = open_session(args.model, args.dtype, args.max_tokens, torch.device(args.device, 0) if args.device == "cuda" else torch.device("cpu"))
    with torch.no_grad():
        for line in sys.stdin:
            if not line.strip():
                continue
            st = json.loads(line)
            lg = session.step([(e["id"], e["tokens"], e.get("want", [])) for e in st["entries"]], st.get("end", []))
            if lg is not None:
                path = os.path.join(args.out, f"{st['step']}.f32")
                lg.contiguous().numpy().astype("<f4").tofile(path)
            print(f"done {st['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
