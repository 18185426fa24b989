"""Zubedra on the CPU: configuration, weights, work lists, the oracle's own sensitivity, and the serving loop on the CPU
backend against the plain oracle. The GPU counterpart is test_zubedra_gpu.py."""
import json

import numpy as np
import pytest
import torch

import zubedra_cases as cases
import zubedra_oracle as oracle
from nanoflow_b200.config import builtin_config, folder_config, load_config
from nanoflow_b200.models import zubedra
from nanoflow_b200.models.registry import family_of
from nanoflow_b200.models.safetensors_io import read_safetensors, write_safetensors
from nanoflow_b200.ops import reference as ref
from nanoflow_b200.replay import TraceReplay
from nanoflow_b200.runtime.cpu_layer_list import CpuLayerListEngine
from nanoflow_b200.runtime.layer_list import chunk_work, query_items
from nanoflow_b200.serving import DistKVPool, RequestManager, Scheduler, StateSlotPool
from nanoflow_b200.serving.loop import ServingLoop
from volarax_cases import prompt, row_errors

TOL = 2e-5


def cpu_engine(raw, tensors, **kw):
    cfg = cases.engine_config(raw, dtype="float32", **kw)
    return CpuLayerListEngine(cfg, zubedra.weights_from_tensors(cfg.model, tensors.__getitem__), num_pages=cfg.engine.num_pages)


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
    assert family_of(raw).name == "zubedra" and m.parallel and not m.output_norms and not m.embed_norm
    assert (m.hidden_size, m.vocab_size, m.embed_scale, m.logit_scale, m.norm_eps) == (104, 211, 3.0, 0.6, 1e-5)
    a, w, f = m.layers[0].mixer, m.layers[1].mixer, m.layers[0].mlp
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.softcap, a.value_mix) == (6, 2, 24, 40, 6.0, True)
    assert (w.heads, w.dim, w.rank) == (3, 24, 9) and m.layers[2].mixer.softcap is None and not m.layers[2].mixer.value_mix
    assert (f.experts, f.top, f.groups, f.keep, f.scale) == (10, 3, 5, 3, 1.7)
    assert (f.expert.ff, f.expert.act.limit, f.shared.ff, f.shared.act.limit) == (24, 1.2, 40, 0.8)
    assert m.has_state and m.kv_window == 0 and m.first_value_run == 0
    assert cases.engine_config(cases.CASES["recurrent_first"]).model.first_value_run == 2
    for bad, what in ((lambda r: r["layers"][0].update(type="gru"), "unknown layer type"),
                      (lambda r: r["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward"),
                      (lambda r: r["layers"][0]["mixer"].update(kv_heads=4), "evenly"),
                      (lambda r: r["layers"][0]["mlp"]["router"].update(top=7), "cannot be chosen"),
                      (lambda r: r["layers"][0]["mlp"]["router"]["groups"].update(count=3), "do not form"),
                      (lambda r: r["layers"][0]["mixer"].update(vdim=16), "mix values"),
                      (lambda r: r["layers"][1]["mixer"].pop("decay_rank"), "decay_rank")):
        broken = json.loads(json.dumps(raw))
        bad(broken)
        with pytest.raises(ValueError, match=what):
            cases.engine_config(broken)


def test_sizes_that_only_the_tensors_say_come_from_the_folder(tmp_path):
    hf = json.loads(json.dumps(cases.CASES["mixed"]))
    t = cases.tensors(hf)
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    back = read_safetensors(str(tmp_path / "model.safetensors"))
    assert back.keys() == t.keys() and all(torch.equal(back[k], t[k]) and back[k].shape == t[k].shape for k in t)
    for lay in hf["layers"]:
        lay["mixer"].pop("decay_rank", None)
    (tmp_path / "config.json").write_text(json.dumps(hf))
    cfg = load_config(str(tmp_path))
    assert [s.rank for s in cfg.model.run_specs("wkv")] == [9, 9] and cfg.model.dtype == torch.bfloat16
    cfg = folder_config(str(tmp_path), dtype="float32")
    w = family_of(hf).load_folder(cfg, str(tmp_path), "cpu")
    rp = TraceReplay(CpuLayerListEngine(cfg, w, num_pages=16), 16, 2)
    toks = prompt(20, hf["vocab"], 0)
    assert row_max(portions(rp, toks, [20]), oracle.forward(cases.CASES["mixed"], t, toks)) < TOL
    del t["l1.mix.u"]
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    with pytest.raises(KeyError, match="l1.mix.u"):
        zubedra.load_weights(cfg.model, str(tmp_path))


def test_tensor_names_cover_what_the_oracle_reads():
    for raw in cases.CASES.values():
        t = zubedra.random_tensors(raw)
        assert set(t) == set(zubedra.tensor_shapes(raw))
        oracle.forward(raw, t, [1, 2, 3])          # every name it asks for exists, every shape fits


def test_builtin_sizes():
    m = builtin_config("zubedra-8B").model
    dense = builtin_config("llama3-8B").model
    assert m.matmul_flops_per_token() == pytest.approx(dense.matmul_flops_per_token(), rel=0.2)
    assert m.param_count() > 4 * dense.param_count() and m.kv_bytes_per_token_local() == 16 * 2 * 8 * 128 * 2
    assert m.state_bytes_per_slot() == 16 * (64 * 64 * 64 * 4 + 2 * 4096 * 2)
    assert builtin_config("zubedra-tiny", global_batch_size=64).engine.pipeline_type == "NON_OVERLAP_LOCAL"


# ---- routing ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,groups,keep,top", [(10, 5, 3, 3), (7, 7, 2, 1), (6, 1, 1, 6), (40, 4, 2, 5)])
def test_reference_routing_matches_the_oracle(E, groups, keep, top):
    g = torch.Generator().manual_seed(E)
    z, corr = torch.randn(50, E, generator=g), torch.randn(E, generator=g)
    idx, w = ref.moe_route(z, corr, top, groups, keep, 1.7)
    want_idx, want_w = oracle.route(torch.sigmoid(z), corr, {"groups": {"count": groups, "keep": keep}, "top": top, "scale": 1.7})
    assert torch.equal(idx, want_idx) and torch.allclose(w, want_w, rtol=1e-5)


def test_groups_left_out_lose_even_to_negative_choice_scores():
    s = torch.tensor([[0.9, 0.1, 0.6, 0.5]])
    corr = torch.tensor([-3.0, -3.0, -2.9, -2.9])          # group 1 wins with negative scores; group 0 has the best expert
    idx, w = oracle.route(s, corr, {"groups": {"count": 2, "keep": 1}, "top": 2, "scale": 1.0})
    assert idx.tolist() == [[2, 3]] and torch.allclose(w, torch.tensor([[0.6 / 1.1, 0.5 / 1.1]]))
    assert ref.moe_route(torch.logit(s), corr, 2, 2, 1, 1.0)[0].tolist() == [[2, 3]]


# ---- work lists ---------------------------------------------------------------------------------------------------
def test_wkv_chunks_cover_portions_in_order_and_the_rest_goes_token_by_token():
    qo = np.asarray([0, 1, 2, 132, 134, 198, 300], dtype=np.int32)      # two single tokens, portions of 130, 2, 64, 102
    items, seq = chunk_work(qo, 2, 100)
    assert seq.size == 0 and items.tolist() == [[2, 2, 64, 0], [2, 66, 64, 1], [2, 130, 2, 2], [3, 132, 2, 0], [4, 134, 64, 0],
                                                [5, 198, 64, 0], [5, 262, 38, 1]]
    items, seq = chunk_work(qo, 2, 5)
    assert seq.tolist() == [5] and items.shape == (5, 4)
    items, seq = chunk_work(qo, 2, 0)
    assert seq.tolist() == [2, 3, 4, 5] and items.shape == (0, 4)
    assert query_items(qo, 2, 42).tolist() == [[2, 2, 42], [2, 44, 42], [2, 86, 42], [2, 128, 4], [3, 132, 2], [4, 134, 42],
                                               [4, 176, 22], [5, 198, 42], [5, 240, 42], [5, 282, 18]]


# ---- the oracle notices -----------------------------------------------------------------------------------------
def test_every_mechanism_shows_in_the_logits(monkeypatch):
    """A mistake in any mechanism moves the oracle's logits far more than the tests tolerate."""
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw, 3)
    toks = prompt(70, raw["vocab"], 3)
    want = oracle.forward(raw, t, toks)
    real = {k: getattr(oracle, k) for k in ("causal_sink_attention", "mix_values", "token_shift", "wkv_recurrence", "route",
                                            "capped_mlp", "soft_cap")}
    late = lambda q, k, v, scale, cap, sink: real["causal_sink_attention"](q, torch.cat([k[:1], k[:-1]]), v, scale, cap, sink)
    no_sink = lambda q, k, v, scale, cap, sink: real["causal_sink_attention"](q, k, v, scale, cap, torch.full_like(sink, -1e9))
    heads = lambda q, k, v, *a: real["causal_sink_attention"](q, k.flip(1), v.flip(1), *a)
    faults = {
        "key of the token before": ("causal_sink_attention", late), "no sink": ("causal_sink_attention", no_sink),
        "wrong key head": ("causal_sink_attention", heads), "no cap": ("soft_cap", lambda s, cap: s),
        "values not mixed": ("mix_values", lambda v, first, lam: v),
        "no previous token": ("token_shift", lambda h, before=None: torch.zeros_like(h)),
        "state lost in the middle": ("wkv_recurrence", lambda r, k, v, w, u: (torch.cat(
            [real["wkv_recurrence"](r[:33], k[:33], v[:33], w[:33], u)[0], real["wkv_recurrence"](r[33:], k[33:], v[33:], w[33:], u)[0]]), None)),
        "bonus kept in the state": ("wkv_recurrence", lambda r, k, v, w, u: real["wkv_recurrence"](r, k, v, w, torch.ones_like(u))),
        "weights with the correction": ("route", lambda s, c, r: (real["route"](s, c, r)[0], real["route"](s + c, 0 * c, r)[1])),
        "choice without the correction": ("route", lambda s, c, r: real["route"](s, 0 * c, r)),
        "groups ignored": ("route", lambda s, c, r: real["route"](s, c, {k: v for k, v in r.items() if k != "groups"})),
        "no limit": ("capped_mlp", lambda h, g, u, d, limit: real["capped_mlp"](h, g, u, d, 1e9)),
    }
    for what, (name, f) in faults.items():
        monkeypatch.setattr(oracle, name, f)
        e = row_errors(oracle.forward(raw, t, toks), want)
        monkeypatch.setattr(oracle, name, real[name])
        assert float(e.max()) > 0.02, what


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


@pytest.mark.parametrize("name,pages,preempt", [("mixed", 40, False), ("recurrent_first", 40, False), ("mixed", 7, True)])
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
