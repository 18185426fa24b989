"""Gimudra on the CPU: configuration, weights, page release, the oracle's own sensitivity, and the serving loop on the CPU
backend against the plain oracle. The GPU counterpart is test_gimudra_gpu.py."""
import json
import math

import numpy as np
import pytest
import torch

import gimudra_cases as cases
import gimudra_oracle as oracle
from nanoflow_b200.config import builtin_config, folder_config, load_config
from nanoflow_b200.models import gimudra
from nanoflow_b200.models.registry import family_of
from nanoflow_b200.models.safetensors_io import write_safetensors
from nanoflow_b200.ops import reference as ref
from nanoflow_b200.replay import TraceReplay
from nanoflow_b200.runtime.cpu_layer_list import CpuLayerListEngine
from nanoflow_b200.runtime.layer_list import by_keys, query_items
from nanoflow_b200.serving import DistKVPool, RequestManager, Scheduler, StateSlotPool
from nanoflow_b200.serving.loop import ServingLoop
from volarax_cases import prompt, row_errors

TOL = 5e-5


def cpu_engine(raw, tensors, **kw):
    cfg = cases.engine_config(raw, dtype="float32", **kw)
    return CpuLayerListEngine(cfg, gimudra.weights_from_tensors(cfg.model, tensors.__getitem__), num_pages=cfg.engine.num_pages)


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
    assert family_of(raw).name == "gimudra" and not m.output_norms and not m.parallel and not m.embed_norm and m.norm_kind == "rms"
    assert (m.hidden_size, m.vocab_size, m.embed_scale, m.norm_eps, m.sinusoid) == (104, 211, 2.0, 1e-5, 10000.0)
    assert m.layer_scale and m.depth_average and (m.input_conv, m.input_conv_mlp) == (2, False) and m.has_state
    a, b = m.layers[0].mixer, m.layers[2].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.kv_from, a.sink, a.qk_norm, a.window) == (6, 2, 24, 40, 20, None, False, False, None)
    assert (b.chunk, b.kv_from, b.bias, b.distance_bias, b.proj_heads, a.proj_heads) == (48, 0, True, True, 6, 10)
    f = m.layers[0].mlp
    assert (f.experts, f.identity, f.outputs, f.top, f.groups, f.keep, f.scale, f.score, f.group_score, f.expert.act.name) == \
        (9, 3, 12, 4, 3, 2, 1.7, "softmax_all", "max", "relu2")
    assert (m.layers[2].mlp.groups, m.layers[2].mlp.keep, m.layers[3].mlp) == (1, 1, None)
    assert m.layers[1].mlp.bias and m.layers[1].mlp.act.name == "silu"
    assert cases.engine_config(cases.CASES["wide_heads"]).model.layers[1].mixer.chunk is None
    for bad, what in ((lambda r: r["layers"][0].update(type="gru"), "unknown layer type"),
                      (lambda r: r["layers"][0]["mlp"].update(kind="other"), "unknown feed-forward"),
                      (lambda r: r["layers"][0]["mixer"].update(kv_heads=4), "evenly"),
                      (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "positive"),
                      (lambda r: r["layers"][2]["mixer"].update(kv_from=3), "nothing to lend|no keys"),
                      (lambda r: r["layers"][4]["mixer"].update(kv_from=2), "no keys"),
                      (lambda r: r["layers"][2]["mixer"].update(vdim=48), "other sizes"),
                      (lambda r: r["layers"][0]["mlp"]["router"].update(identity=2), "do not form"),
                      (lambda r: r["layers"][0]["mlp"]["router"].update(top=9), "cannot be chosen")):
        broken = json.loads(json.dumps(raw))
        bad(broken)
        with pytest.raises(ValueError, match=what):
            cases.engine_config(broken)


def test_a_model_folder_is_loaded_by_its_names(tmp_path):
    hf = json.loads(json.dumps(cases.CASES["mixed"]))
    t = cases.tensors(hf)
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(hf))
    assert load_config(str(tmp_path)).model.dtype == torch.bfloat16
    cfg = folder_config(str(tmp_path), dtype="float32")
    w = family_of(hf).load_folder(cfg, str(tmp_path), "cpu")
    rp = TraceReplay(CpuLayerListEngine(cfg, w, num_pages=16), 16, 2)
    toks = prompt(25, hf["vocab"], 0)
    assert row_max(portions(rp, toks, [25]), oracle.forward(hf, t, toks)) < TOL
    t["l1.dwa"] = t["l1.dwa"][:2].contiguous()
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    with pytest.raises(ValueError, match="l1.dwa"):
        gimudra.load_weights(cfg.model, str(tmp_path))
    del t["l0.mix.r2"]
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    with pytest.raises(KeyError, match="l0.mix.r2"):
        gimudra.load_weights(cfg.model, str(tmp_path))


def test_tensor_names_cover_what_the_oracle_reads():
    for raw in cases.CASES.values():
        t = gimudra.random_tensors(raw)
        assert set(t) == set(gimudra.tensor_shapes(raw))
        oracle.forward(raw, t, [1, 2, 3])          # every name it asks for exists, every shape fits


def test_builtin_sizes():
    m = builtin_config("gimudra-8B").model
    dense = builtin_config("llama3-8B").model
    assert m.matmul_flops_per_token() == pytest.approx(dense.matmul_flops_per_token(), rel=0.25)
    own = sum(s.kv_from is None for s in m.run_specs("attention"))
    assert own == 17 and m.kv_bytes_per_token_local() == own * 2 * 8 * 128 * 2
    assert m.state_bytes_per_slot() == 32 * 2 * 4096 * 2           # the last row of every mixer's input, in two halves
    assert builtin_config("gimudra-tiny", global_batch_size=64).engine.pipeline_type == "NON_OVERLAP_LOCAL"
    w = gimudra.random_weights(builtin_config("gimudra-tiny").model, builtin_config("gimudra-tiny").raw["model"])
    assert w.nbytes() < 8 << 20


def test_first_position_that_any_layer_sees():
    m = cases.engine_config(cases.CASES["mixed"]).model                  # chunks of 20, 33, 48, 64, 50
    for p in range(400):
        want = min(p // c * c for c in (20, 33, 48, 64, 50))
        assert m.first_seen(p) == want <= m.first_seen(p + 1)
    assert cases.engine_config(cases.CASES["wide_heads"]).model.first_seen(399) == 0


def test_work_items_are_ordered_by_the_keys_they_see():
    """Two prompts from their start and one that goes on behind the start of a chunk."""
    qo = np.asarray([0, 1, 41, 81, 121])
    pos = np.concatenate([[500], np.arange(40), np.arange(40), np.arange(90, 130)])
    items = by_keys(query_items(qo, 1, 16), pos, lambda p: p // 100 * 100)
    assert sorted(map(tuple, items.tolist())) == sorted(map(tuple, query_items(qo, 1, 16).tolist()))
    seen = [int(pos[t + n - 1]) - int(pos[t]) // 100 * 100 for _, t, n in items]
    assert seen == sorted(seen)
    assert by_keys(query_items(qo, 4, 16), pos, lambda p: 0).shape == (0, 3)


# ---- single mechanisms of the CPU backend -------------------------------------------------------------------------
@pytest.mark.parametrize("E,identity,groups,keep,top", [(9, 3, 3, 2, 4), (7, 0, 1, 1, 1), (3, 4, 7, 4, 3), (6, 2, 2, 1, 4), (5, 5, 2, 1, 5)])
def test_reference_routing_matches_the_oracle(E, identity, groups, keep, top):
    g = torch.Generator().manual_seed(E)
    z, corr = torch.randn(50, E + identity, generator=g) * 3, torch.rand(E + identity, generator=g) - 2.0
    idx, w = ref.moe_route(z, corr, top, groups, keep, 1.3, "softmax_all", "max")
    want_idx, want_w = oracle.route(z, corr, {"groups": {"count": groups, "keep": keep}, "top": top, "scale": 1.3})
    assert torch.equal(idx, want_idx) and torch.allclose(w, want_w, rtol=1e-5)


def test_groups_left_out_lose_even_to_negative_choice_scores():
    """The best group counts by its largest score alone, and nobody outside it is chosen though all scores are below zero."""
    s = torch.tensor([[0.40, 0.05, 0.30, 0.25]])
    idx, w = ref.moe_route(torch.log(s), torch.full((4,), -3.0), 2, 2, 1, 2.0, "softmax_all", "max")
    assert idx.tolist() == [[0, 1]] and torch.allclose(w, torch.tensor([[0.8, 0.1]]))
    idx, _ = ref.moe_route(torch.log(s), torch.full((4,), -3.0), 2, 2, 1, 2.0, "softmax_all")
    assert idx.tolist() == [[2, 3]]                                       # by the sum of two it would be the other group


def test_sinusoid_of_an_odd_width():
    got, want = ref.sinusoid(np.arange(300), 51, 10000.0), oracle.sinusoid(300, 51, torch.float64)
    assert torch.allclose(got.double(), want, atol=1e-6)
    assert math.isclose(float(want[7, 2]), math.sin(7 * 10000 ** (-2 / 51))) and math.isclose(float(want[7, 3]), math.cos(7 * 10000 ** (-2 / 51)))


# ---- the oracle notices -----------------------------------------------------------------------------------------
def test_every_mechanism_shows_in_the_logits(monkeypatch):
    """A mistake in any mechanism moves the oracle's logits far more than the tests tolerate."""
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw, 3)
    toks = prompt(130, raw["vocab"], 3)
    want = oracle.forward(raw, t, toks)
    names = ("sinusoid", "token_shift", "distance_bias", "same_chunk", "attend", "keys_and_values", "project", "kept_groups", "route",
             "identity_expert", "squared_relu", "silu", "layer_scale", "depth_average", "rms_norm", "embed")
    real = {k: getattr(oracle, k) for k in names}
    by = lambda w, T: torch.arange(T)[:, None] - torch.arange(T)[None, :]

    def shifted_chunk(by):
        def f(T, size):
            i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
            return (j <= i) & ((i + by) // size == (j + by) // size)
        return f

    faults = {
        "positions one off": ("sinusoid", lambda T, W, dt: real["sinusoid"](T + 1, W, dt)[1:]),
        "sine and cosine swapped": ("sinusoid", lambda T, W, dt: real["sinusoid"](T, W, dt).reshape(T, -1, 2).flip(-1).reshape(T, -1)),
        "position vector scaled too": ("embed", lambda tok, tab, s: tab[torch.as_tensor(tok)] * s + s * real["sinusoid"](len(tok), tab.shape[1], tab.dtype)),
        "no shift": ("token_shift", lambda h, a: h),
        "shift from the next but one": ("token_shift", lambda h, a: h + (torch.cat([h[:1] * 0, h[:1] * 0, h[:-2]]) - h) * a),
        "shift of the shifted": ("token_shift", lambda h, a: real["token_shift"](real["token_shift"](h, a), a)),
        "previous row lost in the middle": ("token_shift", lambda h, a: torch.cat([real["token_shift"](h[:65], a), real["token_shift"](h[65:], a)])),
        "no distance bias": ("distance_bias", lambda T, a, b: 0.0),
        "bias grows linearly": ("distance_bias", lambda T, a, b: a[:, None, None] * b[:, None, None] * by(None, T).clamp(min=0)),
        "distance one off": ("distance_bias", lambda T, a, b: real["distance_bias"](T + 1, a, b)[:, 1:, :-1]),
        "base two logarithm": ("distance_bias", lambda T, a, b: real["distance_bias"](T, a, b) / math.log(2)),
        "chunks one late": ("same_chunk", shifted_chunk(-1)),
        "chunks one early": ("same_chunk", shifted_chunk(1)),
        "no chunks": ("same_chunk", lambda T, size: real["same_chunk"](T, None)),
        "a window instead": ("same_chunk", lambda T, size: real["same_chunk"](T, None) & (by(None, T) < size)),
        "wrong key head": ("attend", lambda q, k, v, *a: real["attend"](q, k.flip(1), v, *a)),
        "wrong value head": ("attend", lambda q, k, v, *a: real["attend"](q, k, v.flip(1), *a)),
        "no projection biases": ("project", lambda h, w, n: h @ w[n].T),
        "groups not limited": ("kept_groups", lambda c, g: c),
        "groups left out count as zero": ("kept_groups", lambda c, g: real["kept_groups"](c, g).masked_fill(
            real["kept_groups"](c, g) == -math.inf, 0.0)),
        "weights with the correction": ("route", lambda z, c, r: (real["route"](z, c, r)[0], (torch.softmax(z, -1) + c).gather(
            1, real["route"](z, c, r)[0]) * r["scale"])),
        "weights normed": ("route", lambda z, c, r: (real["route"](z, c, r)[0], r["scale"] * real["route"](z, c, r)[1] /
                                                     real["route"](z, c, r)[1].sum(-1, keepdim=True))),
        "weights not scaled": ("route", lambda z, c, r: (real["route"](z, c, r)[0], real["route"](z, c, r)[1] / r["scale"])),
        "no correction": ("route", lambda z, c, r: real["route"](z, 0 * c, r)),
        "identity experts give nothing": ("identity_expert", lambda h: 0 * h),
        "relu not squared": ("squared_relu", torch.relu),
        "other gate": ("silu", torch.relu),
        "outputs not scaled": ("layer_scale", lambda y, a: y),
        "no average": ("depth_average", lambda x, w: x[-1]),
        "embedding left out of the average": ("depth_average", lambda x, w: real["depth_average"](x[1:], w[1:])),
        "average in reverse": ("depth_average", lambda x, w: real["depth_average"](x, w.flip(0))),
        "eps outside the root": ("rms_norm", lambda x, eps, w: x / (x.pow(2).mean(-1, keepdim=True).sqrt() + 100 * eps) * (w + 0.05)),
    }
    for what, (name, f) in faults.items():
        monkeypatch.setattr(oracle, name, f)
        e = row_errors(oracle.forward(raw, t, toks), want)
        monkeypatch.setattr(oracle, name, real[name])
        assert not float(e.max()) <= 0.02, what
    for i, j in ((2, 1), (3, 0)):                        # keys and values of another layer
        other = json.loads(json.dumps(raw))
        other["layers"][i]["mixer"]["kv_from"] = j
        assert float(row_errors(oracle.forward(other, t, toks), want).max()) > 0.02


# ---- the CPU backend against the oracle ------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_cpu_backend_matches_the_oracle_however_the_prompt_is_cut(name):
    raw = cases.CASES[name]
    t = cases.tensors(raw)
    toks = prompt(70, raw["vocab"], 3)
    want = oracle.forward(raw, t, toks)
    for sizes in ([70], [33, 1], [2, 17, 3, 16, 1]):
        rp = TraceReplay(cpu_engine(raw, t), 64, 4)
        assert row_max(portions(rp, toks, sizes), want) < TOL


def test_batches_over_reused_pages_and_slots():
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw)
    rp = TraceReplay(cpu_engine(raw, t, pages=13), 13, 3)
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
    assert rp.pool.num_free_pages == 13 and rp.slots.num_free == 3


def test_pages_of_past_chunks_are_given_back():
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw)
    rp = TraceReplay(cpu_engine(raw, t, pages=8), 8, 1)       # the prompt alone would take 13
    toks = prompt(200, raw["vocab"], 9)
    assert row_max(portions(rp, toks, [30, 20, 1, 2, 40, 30, 17, 33, 1]), oracle.forward(raw, t, toks)) < TOL


@pytest.mark.parametrize("name,pages,preempt", [("mixed", 40, False), ("even", 40, False), ("mixed", 7, True)])
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
                    average_decode_length=1 if preempt else n_out, group_size=1, state_pool=state, first_seen=m.first_seen)
    st = ServingLoop(eng, sch, rm, est_cycle_time=1.0).run()
    assert pool.num_free_pages == pages and state.num_free == 3 and (sch.preemptions > 0) == preempt
    outs = {}
    for r in st.retired:
        outs.setdefault(r.req_idx, []).append(r)
    for i, p in enumerate(prompts):
        # a preempted request continues as a new one whose prompt holds what it had generated
        r = max(outs[i], key=lambda r: len(r.prompt))
        assert np.concatenate([r.prompt, r.output]).tolist() == p.tolist() + oracle.generate(raw, t, p.tolist(), n_out)
