"""Gupizen on the CPU: configuration, weights, work lists, the oracle's own sensitivity, and the serving loop on the CPU
backend against the plain oracle. The GPU counterpart is test_gupizen_gpu.py."""
import json
import math

import numpy as np
import pytest
import torch

import gupizen_cases as cases
import gupizen_oracle as oracle
from nanoflow_b200.config import builtin_config, folder_config, load_config
from nanoflow_b200.models import gupizen
from nanoflow_b200.models.registry import family_of
from nanoflow_b200.models.safetensors_io import write_safetensors
from nanoflow_b200.ops import reference as ref
from nanoflow_b200.replay import TraceReplay
from nanoflow_b200.runtime.cpu_layer_list import CpuLayerListEngine
from nanoflow_b200.runtime.layer_list import delta_item_floats, query_items, rotations
from nanoflow_b200.serving import DistKVPool, RequestManager, Scheduler, StateSlotPool
from nanoflow_b200.serving.loop import ServingLoop
from volarax_cases import prompt, row_errors

TOL = 5e-5


def cpu_engine(raw, tensors, **kw):
    cfg = cases.engine_config(raw, dtype="float32", **kw)
    return CpuLayerListEngine(cfg, gupizen.weights_from_tensors(cfg.model, tensors.__getitem__), num_pages=cfg.engine.num_pages)


def portions(rp, tokens, sizes, rid="a"):
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(k, len(sizes) - 1)], len(tokens) - at)
        out.append(rp.step([{"id": rid, "tokens": tokens[at:at + n], "want": list(range(n))}], [rid] if at + n == len(tokens) else []))
        at, k = at + n, k + 1
    return np.concatenate(out)


def row_max(got, want):
    return float(row_errors(got, want).max())


# ---- configuration and weights ---------------------------------------------------------------------------
def test_config_is_read_from_the_dictionary():
    raw = cases.CASES["mixed"]
    m = cases.engine_config(raw).model
    assert family_of(raw).name == "gupizen" and m.output_norms and not m.parallel and not m.embed_norm and m.norm_kind == "rms"
    assert (m.hidden_size, m.vocab_size, m.embed_scale, m.norm_eps, m.input_conv) == (104, 211, 2.0, 1e-5, 4)
    a, b, f = m.layers[0].mixer.left, m.layers[0].mixer.right, m.layers[0].mlp
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.talk, a.qk_norm) == (6, 2, 24, 40, 20, True, False)
    assert (a.rotary.dims, a.rotary.base, a.rotary.values, a.rotary.scaling.factor) == (16, 1000.0, True, 3.0)
    assert (b.width, b.blocks, b.conv, b.cols) == (72, 3, 3, 72)
    d = m.layers[2].mixer
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.decay_rank, d.gate_rank) == (6, 3, 24, 40, 4, 9, 13)
    assert (f.experts, f.top, f.score, f.expert.ff, f.expert.gated) == (10, 3, "softmax", 24, False)
    assert [r.layer for r in m.runs] == [0, 1, 2, 1, 2, 3] and [r.step for r in m.runs] == [None, None, None, 1, None, None]
    assert m.has_state and m.kv_window == 48 and m.tied_head
    assert cases.engine_config(cases.CASES["delta_first"]).model.layers[1].mixer.left.rotary.scaling is None
    for bad, what in ((lambda r: r["layers"][0].update(type="gru"), "unknown layer type"),
                      (lambda r: r["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward"),
                      (lambda r: r["layers"][0]["mixer"]["left"].update(kv_heads=4), "evenly"),
                      (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=26), "do not fit"),
                      (lambda r: r["layers"][0]["mixer"]["left"].update(vdim=39), "even size"),
                      (lambda r: r["layers"][0]["mixer"]["right"].update(blocks=5), "does not form"),
                      (lambda r: r["layers"][0]["mixer"]["right"].update(conv=9), "taps"),
                      (lambda r: r["canon"].update(taps=9), "taps"),
                      (lambda r: r["layers"][2]["mixer"].update(kv_heads=4), "evenly"),
                      (lambda r: r["layers"][0]["mlp"]["router"].update(top=11), "cannot be chosen"),
                      (lambda r: r["loop"].update(stop=5), "loop"),
                      (lambda r: r["layers"][2]["mixer"].pop("gate_rank"), "gate_rank")):
        broken = json.loads(json.dumps(raw))
        bad(broken)
        with pytest.raises(ValueError, match=what):
            cases.engine_config(broken)


def test_sizes_that_only_the_tensors_say_come_from_the_folder(tmp_path):
    hf = json.loads(json.dumps(cases.CASES["mixed"]))
    t = cases.tensors(hf)
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    for lay in hf["layers"]:
        lay["mixer"].pop("decay_rank", None)
        lay["mixer"].pop("gate_rank", None)
    (tmp_path / "config.json").write_text(json.dumps(hf))
    cfg = load_config(str(tmp_path))
    assert [(s.decay_rank, s.gate_rank) for s in cfg.model.run_specs("delta")] == [(9, 13)] * 2 and cfg.model.dtype == torch.bfloat16
    cfg = folder_config(str(tmp_path), dtype="float32")
    w = family_of(hf).load_folder(cfg, str(tmp_path), "cpu")
    rp = TraceReplay(CpuLayerListEngine(cfg, w, num_pages=16), 16, 2)
    toks = prompt(20, hf["vocab"], 0)
    assert row_max(portions(rp, toks, [20]), oracle.forward(cases.CASES["mixed"], t, toks)) < TOL
    t["l0.canon1"] = t["l0.canon1"][:, :3].contiguous()
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    with pytest.raises(ValueError, match="l0.canon1"):
        gupizen.load_weights(cfg.model, str(tmp_path))
    del t["l2.mix.dt_bias"]
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    with pytest.raises((KeyError, ValueError)):
        gupizen.load_weights(cfg.model, str(tmp_path))


def test_tensor_names_cover_what_the_oracle_reads():
    for raw in cases.CASES.values():
        t = gupizen.random_tensors(raw)
        assert set(t) == set(gupizen.tensor_shapes(raw))
        oracle.forward(raw, t, [1, 2, 3])          # every name it asks for exists, every shape fits


def test_builtin_sizes():
    m = builtin_config("gupizen-8B").model
    dense = builtin_config("llama3-8B").model
    assert m.matmul_flops_per_token() == pytest.approx(dense.matmul_flops_per_token(), rel=0.25)
    assert m.kv_bytes_per_token_local() == 16 * 2 * 8 * 128 * 2 and m.kv_window == 1024
    pair = 4096 * 4 + 2 * 3 * 4096 * 2
    delta = 32 * 128 * 128 * 4 + 2 * 3 * 3 * 4096 * 2
    assert m.state_bytes_per_slot() == 16 * (pair + delta) + 32 * 2 * (2 * 3 * 4096 * 2)
    assert builtin_config("gupizen-tiny", global_batch_size=64).engine.pipeline_type == "NON_OVERLAP_LOCAL"
    w = gupizen.random_weights(builtin_config("gupizen-tiny").model, builtin_config("gupizen-tiny").raw["model"])
    assert w.lm_head is w.embed and w.nbytes() < 8 << 20       # tied tables and parts of one matrix count once


def test_rotation_frequencies_match_the_oracle():
    """Wavelengths below, between and above the two bounds, and exactly the plain ones without scaling."""
    for raw in cases.CASES.values():
        for lay in raw["layers"]:
            if lay["type"] == "parallel":
                a = lay["mixer"]["left"]
                spec = cases.engine_config(cases.config([lay])).model.layers[0].mixer.left
                keys, values = rotations(spec)
                want = oracle.scaled_frequencies(a["rot"]["dims"], a["rot"]["base"], a["rot"]["scaling"])
                assert np.allclose(keys, want, rtol=1e-12)
                assert np.allclose(values, oracle.frequencies(a["vdim"], a["rot"]["base"]), rtol=1e-12)
    s = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": 60.0}
    plain, scaled = oracle.frequencies(16, 1000.0), oracle.scaled_frequencies(16, 1000.0, s)
    kinds = ["kept" if 2 * math.pi / f < 12 else "slowed" if 2 * math.pi / f > 60 else "ramp" for f in plain]
    assert set(kinds) == {"kept", "slowed", "ramp"}
    for f, g, k in zip(plain, scaled, kinds):
        assert g == f if k == "kept" else g == f / 3 if k == "slowed" else f / 3 < g < f


# ---- routing and work lists ----------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top", [(10, 3), (7, 1), (6, 6), (40, 5)])
def test_reference_routing_matches_the_oracle(E, top):
    g = torch.Generator().manual_seed(E)
    z, bias = torch.randn(50, E, generator=g) * 3, torch.randn(E, generator=g)
    idx, w = ref.moe_route(z, bias, top, 1, 1, 1.0, "softmax")
    want_idx, want_w = oracle.route(z + bias, top)
    assert torch.equal(idx, want_idx) and torch.allclose(w, want_w, rtol=1e-5)


def test_query_tiles_cover_the_portions():
    qo = np.asarray([0, 1, 2, 19, 21, 37], dtype=np.int32)      # two single tokens, portions of 17, 2, 16
    assert query_items(qo, 2, 16).tolist() == [[2, 2, 16], [2, 18, 1], [3, 19, 2], [4, 21, 16]]


def test_chunk_scratch_covers_two_head_sizes():
    spec = lambda d, v: cases.engine_config(cases.config([cases.delta(dim=d, vdim=v)])).model.layers[0].mixer
    assert delta_item_floats(spec(24, 40)) == delta_item_floats(spec(64, 64)) < delta_item_floats(spec(72, 8)) == \
        delta_item_floats(spec(128, 128))


# ---- the oracle notices -----------------------------------------------------------------------------------------
def test_every_mechanism_shows_in_the_logits(monkeypatch):
    """A mistake in any mechanism moves the oracle's logits far more than the tests tolerate."""
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw, 3)
    toks = prompt(70, raw["vocab"], 3)
    want = oracle.forward(raw, t, toks)
    names = ("head_weights", "mix_heads", "rotate", "scaled_frequencies", "causal_conv", "gated_scan", "side_by_side", "delta_rule",
             "unit", "channel_decay", "route", "gelu_erf", "gelu_tanh", "layer_order", "centred_weight_norm", "input_conv", "block_gate")
    real = {k: getattr(oracle, k) for k in names}
    faults = {
        "window one too wide": ("head_weights", lambda q, k, s, sink, w: real["head_weights"](q, k, s, sink, w + 1)),
        "window one too narrow": ("head_weights", lambda q, k, s, sink, w: real["head_weights"](q, k, s, sink, w - 1)),
        "no sink": ("head_weights", lambda q, k, s, sink, w: real["head_weights"](q, k, s, torch.full_like(sink, -1e9), w)),
        "wrong key head": ("head_weights", lambda q, k, *a: real["head_weights"](q, k.flip(1), *a)),
        "heads not mixed": ("mix_heads", lambda w, talk: w),
        "mixing transposed": ("mix_heads", lambda w, talk: real["mix_heads"](w, talk.T)),
        "outputs not turned back": ("rotate", lambda x, f, sign=1: x if sign < 0 else real["rotate"](x, f)),
        "other direction": ("rotate", lambda x, f, sign=1: real["rotate"](x, f, -sign)),
        "frequencies not scaled": ("scaled_frequencies", lambda n, base, s: oracle.frequencies(n, base)),
        "filters reversed": ("causal_conv", lambda x, w, b=None: real["causal_conv"](x, w.flip(1), b)),
        "no input convolution": ("input_conv", lambda h, w: h),
        "recurrence lost in the middle": ("gated_scan", lambda u, r, i, lam: torch.cat(
            [real["gated_scan"](u[:33], r[:33], i[:33], lam), real["gated_scan"](u[33:], r[33:], i[33:], lam)])),
        "recurrent inputs not scaled": ("gated_scan", lambda u, r, i, lam: real["gated_scan"](
            u / torch.sqrt(1 - torch.exp(-16 * r * torch.nn.functional.softplus(lam))), r, i, lam)),
        "gates of other blocks": ("block_gate", lambda u, w, b: real["block_gate"](u, w.flip(0), b)),
        "outputs not normed": ("side_by_side", lambda a, b, wa, wb, eps: 0.5 * (a + b)),
        "state lost in the middle": ("delta_rule", lambda q, k, v, g, b: (torch.cat(
            [real["delta_rule"](q[:33], k[:33], v[:33], g[:33], b[:33])[0], real["delta_rule"](q[33:], k[33:], v[33:], g[33:], b[33:])[0]]),
            None)),
        "read before the write": ("delta_rule", lambda q, k, v, g, b: (torch.cat(
            [torch.zeros_like(v[:1]), real["delta_rule"](torch.cat([q[1:], q[:1]]), k, v, g, b)[0][:-1]]), None)),
        "keys not of unit length": ("unit", lambda x: x),
        "decay per head": ("channel_decay", lambda h, w, H: real["channel_decay"](h, w, H).mean(-1, keepdim=True).expand(
            -1, -1, w["dt_bias"].numel() // H)),
        "equal shares": ("route", lambda z, top: (real["route"](z, top)[0], torch.full((z.shape[0], top), 1 / top, dtype=z.dtype))),
        "next expert": ("route", lambda z, top: (real["route"](z, top + 1)[0][:, 1:], real["route"](z, top)[1])),
        "other gelu": ("gelu_erf", lambda x: torch.relu(x)),
        "no gelu branch": ("gelu_tanh", lambda x: x),
        "embedding not added again": ("layer_order", lambda c: [(i, False) for i, _ in real["layer_order"](c)]),
        "one pass too few": ("layer_order", lambda c: real["layer_order"](c)[:3] + real["layer_order"](c)[5:]),
        "norm weights around zero": ("centred_weight_norm", lambda x, w, eps: oracle.rms_norm(x, eps, w)),
    }
    for what, (name, f) in faults.items():
        monkeypatch.setattr(oracle, name, f)
        e = row_errors(oracle.forward(raw, t, toks), want)
        monkeypatch.setattr(oracle, name, real[name])
        assert not float(e.max()) <= 0.02, what


# ---- the CPU backend against the oracle ------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_cpu_backend_matches_the_oracle_however_the_prompt_is_cut(name):
    raw = cases.CASES[name]
    t = cases.tensors(raw)
    toks = prompt(60, raw["vocab"], 3)
    want = oracle.forward(raw, t, toks)
    for sizes in ([60], [33, 1], [2, 17, 3, 16, 1]):
        rp = TraceReplay(cpu_engine(raw, t), 64, 4)
        assert row_max(portions(rp, toks, sizes), want) < TOL


def test_batches_over_reused_pages_and_slots():
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw)
    rp = TraceReplay(cpu_engine(raw, t, pages=12), 12, 3)
    rng = np.random.default_rng(0)
    prompts = {f"r{i}": prompt(int(n), raw["vocab"], i) for i, n in enumerate((50, 9, 33, 60, 4, 21))}
    todo, live, got = list(prompts), {}, {rid: [] for rid in prompts}
    while todo or live:
        while todo and len(live) < 3:
            live[todo.pop(0)] = 0
        entries, end = [], []
        for rid in list(live):
            if len(live) > 1 and rng.random() < 0.2:
                continue                                     # sits out this step
            p, at = prompts[rid], live[rid]
            n = min(int(rng.choice([1, 1, 2, 7, 18])), len(p) - at)
            entries.append({"id": rid, "tokens": p[at:at + n].tolist(), "want": list(range(n))})
            live[rid] = at + n
            if live[rid] == len(p):
                end.append(rid)
                del live[rid]
        if entries:
            out, at = rp.step(entries, end), 0
            for e in entries:
                got[e["id"]].append(out[at:at + len(e["tokens"])])
                at += len(e["tokens"])
    for rid, p in prompts.items():
        assert row_max(np.concatenate(got[rid]), oracle.forward(raw, t, p)) < TOL
    assert rp.pool.num_free_pages == 12 and rp.slots.num_free == 3


def test_pages_that_leave_every_window_are_given_back():
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw)
    rp = TraceReplay(cpu_engine(raw, t, pages=6), 6, 1)       # the prompt alone would take 10
    toks = prompt(150, raw["vocab"], 9)
    assert row_max(portions(rp, toks, [30, 20, 1, 2, 40, 30, 17, 1]), oracle.forward(raw, t, toks)) < TOL


@pytest.mark.parametrize("name,pages,preempt", [("mixed", 40, False), ("delta_first", 40, False), ("mixed", 7, True)])
def test_greedy_generation_through_the_serving_loop(name, pages, preempt):
    """Chunked prompts beside decoding, more requests than slots; with a pool that is too small for what was admitted,
    a running request loses pages and slot and is computed again."""
    raw = cases.CASES[name]
    t = cases.tensors(raw, seed=5)
    prompts = [prompt(n, raw["vocab"], 10 + n) for n in ((14, 15, 13) if preempt else (3, 41, 17, 1, 58))]
    n_out = 24 if preempt else 9
    eng = cpu_engine(raw, t, batch=64 if preempt else 24, requests=3, pages=pages)
    rm = RequestManager(vocab_size=raw["vocab"])
    for p in prompts:
        rm.add_request(len(p), n_out, 0.0, prompt=p)
    rm.finalize_stats()
    m = eng.model
    pool, state = DistKVPool(m.run_layers, 1, m.head_dim, pages, 16, 1), StateSlotPool(3)
    sch = Scheduler(pool, rm.avaliable_request_queue, global_batch_size=64 if preempt else 24, max_batch_size=3,
                    average_prefill_length=1 if preempt else rm.average_prefill_length,
                    average_decode_length=1 if preempt else n_out, group_size=1, state_pool=state, kv_window=m.kv_window)
    st = ServingLoop(eng, sch, rm, est_cycle_time=1.0).run()
    assert pool.num_free_pages == pages and state.num_free == 3 and (sch.preemptions > 0) == preempt
    outs = {}
    for r in st.retired:
        outs.setdefault(r.req_idx, []).append(r)
    for i, p in enumerate(prompts):
        # a preempted request continues as a new one whose prompt holds what it had generated
        r = max(outs[i], key=lambda r: len(r.prompt))
        assert np.concatenate([r.prompt, r.output]).tolist() == p.tolist() + oracle.generate(raw, t, p.tolist(), n_out)
