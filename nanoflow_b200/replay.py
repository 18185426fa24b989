"""Replay of a token trace through the engine: given tokens in, logits out, step by step.

    bin/trace_run --model DIR --dtype bfloat16 --out OUT --max-tokens 4096 < steps.jsonl

Each line of standard input is one step, a JSON object: ``entries`` lists, per request, its ``id``, its next
``tokens`` and ``want``, the places among them whose logits are asked for; ``end`` lists the requests that are
finished after the step. All entries of a step run as one batch of the engine (single tokens on the decode
path, longer portions on the prefill path), from the pages and state that earlier steps left. A step in which
something is wanted writes ``OUT/<step>.f32`` (little-endian fp32, [wanted, vocab]), and every step prints
``done <step>``. Nothing is sampled.

Useful to compare the engine with another implementation token by token, and to time recorded batches.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Iterable, List, Optional

import numpy as np

REQUEST_TOKENS = 64           # a request's share of --max-tokens is rounded up to this many


class TraceReplay:
    """Requests of a trace on one engine: page lists and state slots from the pools of the serving loop, batches
    in the scheduler's layout."""

    def __init__(self, engine, num_pages: int, state_slots: int):
        from .serving import DistKVPool, StateSlotPool

        m = engine.model
        self.engine, self.model = engine, m
        self.pool = DistKVPool(m.run_layers, m.num_kv_heads, m.head_dim, num_pages, engine.eng.page_size, 1)
        self.slots = StateSlotPool(state_slots) if getattr(m, "has_state", False) else None
        self.first_seen = getattr(m, "first_seen", None)
        self.live: Dict[str, object] = {}
        self.steps = 0

    def step(self, entries: Iterable[dict], end: Iterable[str] = ()) -> Optional[np.ndarray]:
        """Run one batch; returns the wanted logits, fp32 [wanted, vocab], or None if nothing is wanted."""
        from .serving import DistKVCache, Portion, plan_portions

        portions: List[Portion] = []
        for e in entries:
            tokens = np.asarray(e["tokens"], dtype=np.int32)
            if tokens.size == 0:
                continue
            kv = self.live.get(e["id"])
            if kv is None:
                kv = self.live[e["id"]] = DistKVCache(self.pool, self.slots)
            if self.first_seen is not None:
                kv.trim(self.first_seen(kv.seqlen))
            kv.allocate_tokens(tokens.size)
            portions.append(Portion(kv, tokens, e.get("want") or ()))
        out = None
        if portions:
            plan = plan_portions(portions, self.steps, tile_tokens=max(1, 128 // self.model.group_size))
            self.engine.run(plan)
            n = int(plan.sample_rows.size)
            if n:
                out = self.engine.last_logits(n).float().cpu().numpy()
        for rid in end:
            kv = self.live.pop(rid, None)
            if kv is not None:
                kv.release()
        self.steps += 1
        return out


def build_replay(model_dir: str, dtype: str, max_tokens: int, max_requests: int = 4, device=None) -> TraceReplay:
    import torch

    from .config import folder_config
    from .models.registry import family_of

    tokens = max(REQUEST_TOKENS, -(-max_tokens // REQUEST_TOKENS) * REQUEST_TOKENS)
    cfg = folder_config(model_dir, dtype=dtype, global_batch_size=tokens,
                        model_configs={"max_batch_size": max_requests, "max_sample_rows": tokens,
                                       "state_slots": max_requests, "num_pages": tokens // 16},
                        pipeline_configs={"autotune_gemm": False})
    fam = family_of(cfg.raw["model"])
    if dtype == "float32" and not fam.runs_float32:
        raise NotImplementedError(f"the {fam.name} family does not run in 32-bit")
    device = device or torch.device("cuda", torch.cuda.current_device())
    engine = fam.engine(cfg, fam.load_folder(cfg, model_dir, device), device=device)
    return TraceReplay(engine, engine.num_pages, max_requests)


def build_parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=4, help="most requests that are live at any time")
    return ap


def main(argv=None, steps=None, out=None) -> int:
    args = build_parser().parse_args(argv)
    steps, out = steps or sys.stdin, out or sys.stdout
    from .ops.build import build_runtime

    build_runtime()
    try:
        replay = build_replay(args.model, args.dtype, args.max_tokens, args.max_requests)
    except NotImplementedError as e:
        print(e, file=sys.stderr)
        return 3
    os.makedirs(args.out, exist_ok=True)
    for line in iter(steps.readline, ""):
        if not line.strip():
            continue
        st = json.loads(line)
        logits = replay.step(st.get("entries", ()), st.get("end", ()))
        if logits is not None:
            logits.astype("<f4").tofile(os.path.join(args.out, f"{st['step']}.f32"))
        print(f"done {st['step']}", file=out, flush=True)
    replay.engine.finalize()
    return 0


if __name__ == "__main__":
    sys.exit(main())
