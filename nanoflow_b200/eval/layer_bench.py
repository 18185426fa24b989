"""Prefill and decode throughput of a layer-list model beside the Llama model of equal size, layer by layer.

    python bench.py --layer-list 8B            (or 2B, or both: 2B,8B)
    python bench.py --layer-list 8B --layer-model zubedra

Both models get the same width, feed-forward (of a mixture of experts: what a token uses), head count and number of
layers, random weights, and the same batches: whole prompts in one iteration, and single-token decoding over a given context. Engines, kernels
and step function are those of serving; each workload has an engine of its own batch size, so that both models'
GEMM shapes are the tuned ones. Time: CUDA events around repeated iterations (CUDA graphs, weights far larger than
L2), then one iteration with an event pair around every op for the per-kernel table. Each kernel is set against
its roofline, the larger of FLOPs over the measured GEMM rate and bytes over the measured copy bandwidth.
"""
from __future__ import annotations

import json
from pathlib import Path
from typing import Any, Dict, List, Tuple

import numpy as np
import torch

SIZES = {
    # name: (width, ff, heads, kv heads of the Llama, vocab, latent rank, window, mLSTM heads, dim, vdim,
    #        WKV decay rank, ff of an expert and of the shared one: 6 experts per token and the shared one make up ff,
    #        blocks of the linear recurrent unit, ff of an expert without a gate: 6 of them have as many weights as ff,
    #        tokens per chunk of chunked attention)
    "8B": dict(width=4096, ff=14336, heads=32, kv=8, vocab=128256, rank=512, window=1024, mh=8, md=256, mv=512, decay=128,
               eff=2048, sff=2048, blocks=16, uff=3584, chunk=8192),
    "2B": dict(width=2048, ff=8192, heads=16, kv=4, vocab=32000, rank=256, window=512, mh=4, md=256, mv=512, decay=64,
               eff=1024, sff=2048, blocks=16, uff=2048, chunk=1536),
}
EXPERTS, TOP, GROUPS, KEEP, IDENTITY = 64, 6, 8, 4, 4
WORKLOADS = [("prefill 4 x 1024", [(0, 1024)] * 4), ("prefill 1 x 4096", [(0, 4096)]),
             ("decode 256 at 1280", [(1280, 1)] * 256), ("decode 32 at 4096", [(4096, 1)] * 32)]
LAYERS = 4


def peaks() -> Tuple[float, float]:
    """(FLOP/s, bytes/s) measured on this machine's GPUs, or the earlier measurement if the file is missing."""
    f = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if f.exists():
        d = json.loads(f.read_text())
        return d["bf16_tflops"] * 1e12, d["hbm_gbs"] * 1e9
    return 1.59e15, 6.65e12


def model_dict(kind: str, s: Dict[str, int]) -> Dict[str, Any]:
    from ..config import _hf
    from ..models import gimudra, gupizen, volarax, zubedra
    if kind == "llama":
        return _hf(s["width"], s["ff"], LAYERS, s["heads"], s["kv"], s["vocab"], 500000.0)
    if kind == "zubedra":
        return zubedra.builtin(s["width"], s["vocab"], "aw" * (LAYERS // 2), heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128,
                               softcap=50.0, w_heads=s["width"] // 64, w_dim=64, rank=s["decay"], experts=EXPERTS, top=TOP,
                               ff=s["eff"], groups=GROUPS, keep=KEEP, shared_ff=s["sff"])
    if kind == "gupizen":
        return gupizen.builtin(s["width"], s["vocab"], "pd" * (LAYERS // 2), heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128,
                               window=s["window"], rec_width=s["width"], rec_blocks=s["blocks"], d_heads=s["heads"],
                               d_kv_heads=s["heads"], d_dim=128, d_vdim=128, rank=128, experts=EXPERTS, top=TOP, ff=s["uff"])
    if kind == "gimudra":
        return gimudra.builtin(s["width"], s["vocab"], "dmms"[:LAYERS], heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128,
                               chunks=(s["chunk"],), ff=s["ff"], experts=EXPERTS - IDENTITY, top=TOP, e_ff=s["uff"], groups=GROUPS,
                               keep=KEEP, identity=IDENTITY)
    return volarax.builtin(s["width"], s["vocab"], "am" * (LAYERS // 2), heads=s["heads"], dim=128, vdim=128, kv_rank=s["rank"],
                   window=s["window"], m_heads=s["mh"], m_dim=s["md"], m_vdim=s["mv"], ff=s["ff"], m_ff=s["ff"])


def make_engine(kind: str, size: Dict[str, int], spans, device, pages: int, **pipeline):
    from ..config import parse_config
    from ..models.registry import family_of
    T, B = sum(n for _, n in spans), len(spans)
    hf = model_dict(kind, size)
    cfg = parse_config({"model": hf, "model_configs": {"gpu_num": 1, "max_batch_size": B, "num_pages": pages},
                        "pipeline_configs": {"global_batch_size": T, **pipeline},
                        "serve_configs": {"model": kind, "actual_gpu_num": 1, "pipeline_type": "NON_OVERLAP_LOCAL"}})
    fam = family_of(hf)
    return fam.engine(cfg, fam.random_weights(cfg, 0, 1, device), device=device, executor="graph")


def make_plan(engine, spans, pages: int):
    from ..serving import DistKVCache, DistKVPool, Portion, StateSlotPool, plan_portions
    m = engine.model
    pool = DistKVPool(m.run_layers, m.num_kv_heads, m.head_dim, pages, 16, 1)
    slots = StateSlotPool(len(spans)) if getattr(m, "has_state", False) else None
    first_seen = getattr(m, "first_seen", None)
    parts = []
    for ctx, n in spans:
        kv = DistKVCache(pool, slots)
        if ctx:
            kv.allocate_tokens(ctx)
        if first_seen is not None:
            kv.trim(first_seen(ctx))
        kv.allocate_tokens(n)
        parts.append(Portion(kv, np.random.default_rng(len(parts)).integers(0, m.vocab_size, n), [n - 1]))
    return plan_portions(parts, tile_tokens=max(1, 128 // m.group_size))


def op_work(engine, op, spans) -> Tuple[float, float]:
    """(FLOPs, bytes) an op has to do; (0, 0) for ops that are not set against a roofline."""
    from ..runtime import graph as G
    m, p = engine.model, op.params
    T = sum(n for _, n in spans)
    es = 2
    def sees(w, chunk=0):
        """(query, key) pairs, with a window or chunks."""
        return sum(sum(min(c + t + 1, w or c + t + 1) - ((c + t) // chunk * chunk if chunk else 0) for t in range(n)) for c, n in spans)
    if isinstance(p, G.GemmParams):
        dyn = dict(op.dyn)["M"]
        M = engine._last_sym.get(dyn, 0)
        if M == 0:
            return 0.0, 0.0
        gated = 2 if p.epilogue == 1 else 1
        groups = max(1, p.groups)
        wide = p.N - p.f32_col0 if p.D32 else 0          # columns that leave as fp32
        return 2.0 * M * p.N * p.K * gated, es * (gated * p.N * p.K + M * (p.K * groups + p.N)) + (4 - es) * M * wide
    if isinstance(p, G.AttnParams):
        pre = "prefill" in op.kernel
        if (spans[0][1] == 1) == pre:
            return 0.0, 0.0
        w = p.window
        pairs = sees(w, p.chunk)
        keys = sum(min(c + n, (w + n - 1) if w else c + n) - (c // p.chunk * p.chunk if p.chunk else 0) for c, n in spans)
        return 4.0 * pairs * p.q_heads * p.head_dim, es * (2 * keys * p.kv_heads * p.head_dim + 2 * T * p.q_heads * p.head_dim)
    if isinstance(p, G.LatentAttnParams):
        if spans[0][1] != 1:
            return 0.0, 0.0
        pairs = sees(p.window)
        return 4.0 * pairs * p.heads * p.ld, es * (pairs * p.ld + 2 * T * p.heads * p.ld)
    if isinstance(p, G.MlstmParams):
        dec = "decode" in op.kernel
        if (spans[0][1] == 1) != dec:
            return 0.0, 0.0
        state = len(spans) * p.heads * (p.dim * p.vdim + 2 * p.dim) * 4
        io = T * p.heads * ((2 * p.dim + p.vdim) * es + p.vdim * 4)
        chunk = 0 if dec else 64
        return T * p.heads * (chunk * (p.dim + p.vdim) + 4.0 * p.dim * p.vdim), (2 if dec else 1) * state + io
    if isinstance(p, G.ResidualNormParams):
        rows = T if not p.rows_idx else len(spans)
        more = (1 if p.y2 else 0) + (p.e_top if p.e_out else 0)
        earlier = (p.hist_n if p.hist_w else 0) + (1 if p.hist_out else 0)
        return 0.0, rows * p.cols * (8 + 4 * earlier + (2 + more) * es)
    if isinstance(p, G.GqaAppendParams):
        return 0.0, T * 2 * ((p.heads if p.q_out else 0) + 2 * p.kv_heads) * p.hd * es
    if isinstance(p, G.TalkAttnParams):
        if (spans[0][1] == 1) != (dict(op.dyn).get("n_tokens") == "n_dec"):
            return 0.0, 0.0
        pairs = sees(p.window)
        keys = sum(min(c + n, (p.window + n - 1) if p.window else c + n) for c, n in spans)
        return pairs * p.heads * (4.0 * p.hd + 2.0 * p.heads), es * (2 * keys * p.kv_heads * p.hd + 2 * T * p.heads * p.hd)
    if isinstance(p, G.ShortConvParams):
        if spans[0][1] == 1 and ("row_begin", "n_dec") in op.dyn:
            return 0.0, 0.0                             # single tokens go through it in the residual step
        return 0.0, T * 2 * p.cols * es
    if isinstance(p, G.RgLruParams):
        if (spans[0][1] == 1) != ("decode" in op.kernel):
            return 0.0, 0.0
        return 0.0, T * p.cols * (3 * es + 8) + 2 * len(spans) * p.cols * 4
    if isinstance(p, G.DeltaParams):
        dec = "decode" in op.kernel
        if (spans[0][1] == 1) != dec:
            return 0.0, 0.0
        state = len(spans) * p.heads * p.dim * p.vdim * 4
        io = T * ((2 * p.kv_heads * p.dim + 3 * p.heads * p.vdim) * es + p.heads * p.dim * 4)
        chunk = 0 if dec else 64
        return T * p.heads * (2.0 * chunk * (p.dim + p.vdim) + 6.0 * p.dim * p.vdim), 2 * state + io
    if isinstance(p, G.TokenShiftParams):
        return 0.0, T * (1 + p.n_mix) * p.ld_h * es
    if isinstance(p, G.WkvParams):
        dec = "decode" in op.kernel
        if (spans[0][1] == 1) != dec:
            return 0.0, 0.0
        state = len(spans) * p.heads * p.dim * p.dim * 4
        io = T * p.heads * p.dim * (5 * es + 4)
        chunk = 0 if dec else 64
        return T * p.heads * (2.0 * chunk * p.dim + 4.0 * p.dim * p.dim), 2 * state + io
    if isinstance(p, G.MoeRouteParams):
        return 0.0, T * 4 * (p.experts + 3 * p.top)
    if isinstance(p, G.MoePermuteParams):
        return 0.0, (T + engine._expert_rows) * p.cols * es
    if isinstance(p, G.MoeGemmParams):
        rows, mats = engine._expert_rows, 2 if p.B2 else 1
        used = min(p.experts, engine._experts_used)
        return 2.0 * rows * p.N * p.K * mats, es * (mats * used * p.N * p.K + rows * (p.K + p.N))
    if isinstance(p, G.HeadNormGateParams):
        return 0.0, T * p.heads * p.vdim * (4 + 2 * es)
    if isinstance(p, G.LatentAppendParams):
        return 0.0, T * p.rank * 2 * es
    if isinstance(p, G.RopeAppendParams):
        return 0.0, T * (2 * p.q_heads + 4 * p.kv_heads) * p.head_dim * es
    if isinstance(p, G.LatentGatherParams):
        return 0.0, 2.0 * engine._last_sym.get(dict(op.dyn)["n_pages"], 0) * p.page_size * p.ld * es
    if isinstance(p, G.NormParams):
        return 0.0, 2 * T * p.cols * es
    return 0.0, 0.0


def measure(engine, plan, spans, steps: int, warmup: int) -> Dict[str, Any]:
    flops_peak, bw_peak = peaks()
    for _ in range(max(3, warmup)):
        engine.run(plan)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record(engine.stream)
    for i in range(steps):
        engine.update(plan)
        engine.run_async()
        if i:
            engine.run_async_wait()
    engine.run_async_wait()
    e1.record(engine.stream)
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / steps
    engine.check_status()
    # experts that got rows in the last iteration (fewest of all layers): their weights have to be read
    counts = [c for c in getattr(engine, "moe_counts_of", []) if c is not None and c.numel()]
    engine._experts_used = min((int((c > 0).sum()) for c in counts), default=0)
    engine._expert_rows = min((int(c.sum()) for c in counts), default=0)      # (fewer than chosen with identity experts)
    # one op at a time, best of three iterations
    best: Dict[int, float] = {}
    for _ in range(3):
        engine.update(plan)
        engine._last_sym = dict(engine._staged["sym"])
        engine.run_async(timed=True)
        engine.run_async_wait()
        for i, (_, _, a, b) in enumerate(engine.timeline()):
            best[i] = min(best.get(i, 1e9), b - a)
    table: Dict[str, List[float]] = {}
    for i, op in enumerate(engine.graph.ops):
        fl, by = op_work(engine, op, spans)
        if fl == 0 and by == 0:
            continue
        name = op.name.split(".")[-1]
        if op.name.startswith("R") and name in ("in", "o", "gate_up", "down"):
            spec = engine.model.layers[engine.model.runs[op.layer].layer].mixer.kind
            name = f"{spec[:6]}.{name}" if name in ("in", "o") else name
        r = table.setdefault(name, [0, 0.0, 0.0])
        r[0] += 1
        r[1] += best[i]
        r[2] += max(fl / flops_peak, by / bw_peak) * 1e6
    T = sum(n for _, n in spans)
    return {"ms": round(ms, 3), "tokens_per_s": round(T / ms * 1e3),
            "ops": {k: {"us": round(us / n, 1), "of_roofline": round(roof / us, 3)} for k, (n, us, roof) in table.items()}}


def run(sizes: List[str], steps: int, warmup: int, only: str = "", model: str = "volarax") -> Dict[str, Any]:
    device = torch.device("cuda", torch.cuda.current_device())
    out: Dict[str, Any] = {}
    for size in sizes:
        for label, spans in WORKLOADS:
            if only and only not in label:
                continue
            pages = sum((c + n + 15) // 16 for c, n in spans) + 8
            for kind in ["llama"] + model.split(","):
                engine = make_engine(kind, SIZES[size], spans, device, pages)
                res = measure(engine, make_plan(engine, spans, pages), spans, steps, warmup)
                engine.finalize()
                del engine
                torch.cuda.empty_cache()
                out[f"{size} {label} {kind}"] = res
    return out


def report(out: Dict[str, Any]) -> str:
    lines = [f"{LAYERS} layers, random weights, one GPU; kernel columns: us per launch (fraction of roofline)", ""]
    for key, r in out.items():
        ops = ", ".join(f"{k} {v['us']} ({v['of_roofline']})" for k, v in r["ops"].items())
        lines.append(f"{key}: {r['ms']} ms, {r['tokens_per_s']} tokens/s\n    {ops}")
    return "\n".join(lines)
