"""Volarax on the CPU: configuration, weights, caches, work lists, and the serving loop on the CPU backend against
the plain oracle. The GPU counterpart is test_volarax_gpu.py."""
import io
import json

import numpy as np
import pytest
import torch

import volarax_cases as cases
import volarax_oracle as oracle
from nanoflow_b200.config import builtin_config, folder_config, load_config, make_config, parse_config
from nanoflow_b200.models import volarax
from nanoflow_b200.models.registry import family, family_of
from nanoflow_b200.models.safetensors_io import read_safetensors, write_safetensors
from nanoflow_b200.replay import TraceReplay
from nanoflow_b200.runtime.cpu_layer_list import CpuLayerListEngine
from nanoflow_b200.runtime.layer_list import mlstm_segments, route_attention
from nanoflow_b200.serving import (DistKVCache, DistKVPool, Portion, RequestManager, Scheduler, StateSlotPool,
                                   StateSlotsExhausted, plan_portions)
from nanoflow_b200.serving.loop import ServingLoop

TOL = 2e-5


def cpu_engine(raw, tensors, **kw):
    cfg = cases.engine_config(raw, dtype="float32", **kw)
    return CpuLayerListEngine(cfg, volarax.weights_from_tensors(cfg.model, tensors.__getitem__), num_pages=cfg.engine.num_pages)


def replay_portions(rp, tokens, sizes, rid="a", want_all=True):
    """Feed ``tokens`` in portions of the given sizes (the last one repeats); logits of every position."""
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(k, len(sizes) - 1)], len(tokens) - at)
        last = at + n == len(tokens)
        out.append(rp.step([{"id": rid, "tokens": tokens[at:at + n], "want": list(range(n))}], [rid] if last else []))
        at, k = at + n, k + 1
    return np.concatenate(out)


# ---- configuration and weights ---------------------------------------------------------------------------
def test_registry_picks_the_family_and_rejects_unknown_names():
    assert family_of(cases.CASES["mixed"]).name == "volarax"
    assert family_of({"architectures": ["LlamaForCausalLM"], "num_attention_heads": 4}).name == "llama"
    assert family_of({"architectures": ["SomethingElse"], "num_attention_heads": 4}).name == "llama"
    with pytest.raises(ValueError, match="unknown architecture"):
        family_of({"architecture": "Nope"})
    assert family("volarax").runs_float32 and not family("llama").runs_float32


def test_config_is_read_from_the_dictionary():
    raw = cases.CASES["mixed"]
    m = cases.engine_config(raw).model
    assert [(r.layer, r.step) for r in m.runs] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert [(r.layer, r.step) for r in m.runs] == [t for t in oracle.layer_order(raw)]
    assert m.kv_window == 37 and m.has_state and m.hidden_size == 104 and m.norm_eps == 1e-5
    assert m.layers[2].mixer.heads == 5 and m.layers[2].mixer.window == 20 and m.layers[3].mlp is None
    assert cases.engine_config(cases.CASES["wide_heads"]).model.kv_window == 0
    for bad, what in ((lambda r: r["layers"][0].update(type="gru"), "unknown layer type"),
                      (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
                      (lambda r: r["loop"].update(stop=9), "does not fit"),
                      (lambda r: r["layers"][1]["mixer"].update(gate_cap=0.0), "gate_cap"),
                      (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "window")):
        broken = json.loads(json.dumps(raw))
        bad(broken)
        with pytest.raises(ValueError, match=what):
            cases.engine_config(broken)


def test_builtin_architectures_and_model_folders(tmp_path):
    raw = make_config("volarax-tiny", global_batch_size=64)
    assert parse_config(raw).engine.pipeline_type == "NON_OVERLAP_LOCAL"
    m = builtin_config("volarax-8B").model
    assert 8.0e9 < m.param_count() < 9.0e9 and m.kv_window == 1024
    with pytest.raises(ValueError, match="one GPU"):
        parse_config(raw, tp=2)
    hf = cases.CASES["mixed"]
    (tmp_path / "config.json").write_text(json.dumps(hf))
    t = cases.tensors(hf)
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    back = read_safetensors(str(tmp_path / "model.safetensors"))
    assert back.keys() == t.keys() and all(torch.equal(back[k], t[k]) and back[k].dtype == t[k].dtype for k in t)
    cfg = load_config(str(tmp_path))
    w = family_of(hf).load_folder(cfg, str(tmp_path), "cpu")
    assert w.layers[0].mixer.w_in.dtype == torch.bfloat16 and w.layers[0].norm_in.w.dtype == torch.float32
    assert folder_config(str(tmp_path), dtype="float32").model.dtype == torch.float32
    del t["l1.mix.i.b"]
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    with pytest.raises(KeyError, match="l1.mix.i.b"):
        volarax.load_weights(cfg.model, str(tmp_path))


def test_tensor_names_cover_what_the_oracle_reads():
    for raw in cases.CASES.values():
        t = volarax.random_tensors(raw)
        assert set(t) == set(volarax.tensor_shapes(raw))
        oracle.forward(raw, t, [1, 2, 3])          # every name it asks for exists, every shape fits


# ---- caches ------------------------------------------------------------------------------------------------
def test_pages_behind_the_window_are_given_back_and_used_again():
    pool = DistKVPool(1, 1, 8, 8, 16, 1)
    kv = DistKVCache(pool)
    kv.allocate_tokens(50)
    first = kv.indices.tolist()
    assert kv.trim(15) == 0 and kv.trim(16) == 1 and kv.trim(47) == 1 and kv.first_page_slot == 2
    assert kv.indices.tolist() == first[2:] and kv.num_pages == 2 and pool.num_free_pages == 6
    other = DistKVCache(pool)
    other.allocate_tokens(20)
    assert set(other.indices.tolist()) == set(first[:2])
    kv.allocate_tokens(30)                              # 80 tokens: slots 2..4 held
    assert kv.seqlen == 80 and kv.num_pages == 3 and kv.last_page_offset == 16
    kv.release()
    other.release()
    assert pool.num_free_pages == 8 and kv.first_page_slot == 0


def test_state_slots_follow_the_request():
    pool, slots = DistKVPool(1, 1, 8, 4, 16, 1), StateSlotPool(2)
    a, b, c = (DistKVCache(pool, slots) for _ in range(3))
    a.allocate_tokens(3)
    b.allocate_tokens(3)
    assert (a.state_slot, b.state_slot) == (0, 1)
    with pytest.raises(StateSlotsExhausted):
        c.allocate_tokens(1)
    assert c.num_pages == 0 and pool.num_free_pages == 2
    assert [a.state_ref(), a.state_ref(), a.state_ref()] == [0, 1, 0]      # the half flips with every step
    a.release()
    with pytest.raises(Exception):
        c.allocate_tokens(1000)                          # no pages: the slot is not kept either
    assert slots.num_free == 1 and c.state_slot == -1
    c.allocate_tokens(1)
    assert c.state_slot == 0 and c.state_ref() == 0
    with pytest.raises(ValueError):
        slots.free(7)


def test_plan_of_given_portions_keeps_the_order_of_wanted_rows():
    pool = DistKVPool(1, 1, 8, 32, 16, 1)
    kvs = [DistKVCache(pool) for _ in range(3)]
    for kv, n in zip(kvs, (5, 20, 1)):
        kv.allocate_tokens(n)
    plan = plan_portions([Portion(kvs[0], np.arange(5), [4, 0]), Portion(kvs[1], np.asarray([7]), [0]),
                          Portion(kvs[2], np.asarray([9]), [])])
    assert plan.num_decode == 2 and plan.num_tokens == 7 and plan.qo_indptr.tolist() == [0, 1, 2, 7]
    assert plan.host_ids.tolist() == [7, 9, 0, 1, 2, 3, 4] and plan.positions.tolist() == [19, 0, 0, 1, 2, 3, 4]
    assert plan.sample_rows.tolist() == [6, 2, 0] and plan.token_req.tolist() == [0, 1, 2, 2, 2, 2, 2]
    assert np.diff(plan.kv_indptr).tolist() == [2, 1, 1]


# ---- work lists -----------------------------------------------------------------------------------------------
def _plan(starts_and_lens, window=0):
    pool = DistKVPool(1, 1, 8, 512, 16, 1)
    parts = []
    for s, n in starts_and_lens:
        kv = DistKVCache(pool)
        if s:
            kv.allocate_tokens(s)
        if window:
            kv.trim(s - window + 1)
        kv.allocate_tokens(n)
        parts.append(Portion(kv, np.zeros(n, dtype=np.int32)))
    return plan_portions(parts)


@pytest.mark.parametrize("window", [0, 1, 16, 37])
def test_every_token_attends_on_exactly_one_path_and_its_keys_are_expanded(window):
    plan = _plan([(40, 1), (0, 130), (77, 20), (64, 3), (15, 40), (9, 1)], window)
    w = route_attention(plan, window, True, 64, 17)
    seen = list(w["abs"])
    for b, t0, n in w["items"]:
        assert 0 < n <= 128
        seen += range(t0, t0 + n)
        pages = w["xpage"][w["xptr"][b]:w["xptr"][b + 1]]
        q0, q1 = plan.qo_indptr[b], plan.qo_indptr[b + 1]
        lo = max(0, plan.positions[q0] - window + 1) if window else 0
        slots = np.arange(lo // 16, plan.positions[q1 - 1] // 16 + 1)
        assert pages.tolist() == plan.kv_indices[plan.kv_indptr[b] + slots - plan.kv_first[b]].tolist()
    assert sorted(seen) == list(range(plan.num_tokens))
    # nothing fits: everything stays in latent space
    assert route_attention(plan, window, True, 1, 17)["abs"].tolist() == list(range(plan.num_tokens))
    assert route_attention(plan, window, False, 64, 17)["abs"].size == plan.num_tokens


def test_mlstm_segments_cover_portions_in_order():
    for lens, ctas in (([5], 4), ([4096], 64), ([1000, 3, 700], 8), ([64] * 60, 1), ([2], 200)):
        qo = np.concatenate([[0, 1, 2], 2 + np.cumsum(lens)]).astype(np.int32)
        segs = mlstm_segments(qo, 2, ctas, 148)
        assert segs.shape[0] <= max(len(lens), 48)
        at = 2
        for b, t0, n, k in segs:
            assert t0 == at and n > 0 and (k == 0) == (t0 == qo[b]) and t0 + n <= qo[b + 1]
            assert t0 + n == qo[b + 1] or n % 64 == 0
            at += n
        assert at == qo[-1]
    assert mlstm_segments(np.asarray([0, 1, 2], dtype=np.int32), 2, 8, 148).shape == (0, 4)
    assert mlstm_segments(np.asarray([0, 4096], dtype=np.int32), 0, 64, 148).shape[0] > 1


# ---- the CPU backend against the oracle ------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_cpu_backend_matches_the_oracle_however_the_prompt_is_cut(name):
    raw = cases.CASES[name]
    t = cases.tensors(raw)
    toks = cases.prompt(60, raw["vocab"], 3)
    want = oracle.forward(raw, t, toks)
    for sizes in ([60], [33, 1], [2, 17, 3, 16, 1]):
        rp = TraceReplay(cpu_engine(raw, t), 64, 4)
        assert row_max(replay_portions(rp, toks, sizes), want) < TOL


def row_max(got, want):
    return float(cases.row_errors(got, want).max())


def test_replay_of_mixed_batches_reuses_pages_and_slots(tmp_path):
    """Requests come and go over a pool that holds only what is live; each one's logits are those of the oracle."""
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw)
    rp = TraceReplay(cpu_engine(raw, t, pages=12), 12, 3)
    rng = np.random.default_rng(0)
    todo = [(f"r{i}", cases.prompt(int(n), raw["vocab"], i)) for i, n in enumerate((50, 9, 33, 70, 4, 21))]
    live, got = {}, {rid: [] for rid, _ in todo}
    prompts = dict(todo)
    while todo or live:
        while todo and len(live) < 3:
            rid, p = todo.pop(0)
            live[rid] = 0
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
        if not entries:
            continue
        out = rp.step(entries, end)
        at = 0
        for e in entries:
            got[e["id"]].append(out[at:at + len(e["tokens"])])
            at += len(e["tokens"])
    for rid, p in prompts.items():
        assert row_max(np.concatenate(got[rid]), oracle.forward(raw, t, p)) < TOL
    assert rp.pool.num_free_pages == 12 and rp.slots.num_free == 3


def serve_cpu(raw, t, prompts, n_out, *, batch, pages, slots, requests=4, eos=None):
    cfg_kw = dict(batch=batch, requests=requests, pages=pages)
    eng = cpu_engine(raw, t, **cfg_kw)
    eng.eng.state_slots = slots
    rm = RequestManager(vocab_size=raw["vocab"])
    for p in prompts:
        rm.add_request(len(p), n_out, 0.0, prompt=p)
    rm.finalize_stats()
    m = eng.model
    pool = DistKVPool(m.run_layers, 1, m.head_dim, pages, 16, 1)
    state = StateSlotPool(slots) if m.has_state else None
    sch = Scheduler(pool, rm.avaliable_request_queue, global_batch_size=batch, max_batch_size=requests,
                    average_prefill_length=rm.average_prefill_length, average_decode_length=n_out, group_size=1,
                    state_pool=state, kv_window=m.kv_window, eos_token_id=eos, stop_on_eos=eos is not None)
    st = ServingLoop(eng, sch, rm, est_cycle_time=1.0).run()
    assert pool.num_free_pages == pages and (state is None or state.num_free == slots)
    return st, sch


@pytest.mark.parametrize("name", ["mixed", "recurrent_first", "all_looped"])
def test_greedy_generation_through_the_serving_loop(name):
    """Chunked prompts beside decoding, more requests than slots, window pages released on the way."""
    raw = cases.CASES[name]
    t = cases.tensors(raw, seed=5)
    prompts = [cases.prompt(n, raw["vocab"], 10 + n) for n in (3, 41, 17, 1, 58)]
    st, sch = serve_cpu(raw, t, prompts, 9, batch=24, pages=24, slots=3, requests=3)
    assert len(st.retired) == len(prompts)
    for r in st.retired:
        assert r.output == oracle.generate(raw, t, prompts[r.req_idx].tolist(), 9)


def test_preempted_requests_start_over_from_a_zero_state():
    """A pool too small for what was admitted takes pages and slot away from a running request; recomputed, it
    generates what it would have generated."""
    raw = cases.CASES["wide_heads"]                          # no window: pages only grow
    t = cases.tensors(raw, seed=2)
    prompts = [cases.prompt(n, raw["vocab"], n) for n in (14, 15, 13)]
    eng = cpu_engine(raw, t, batch=64, requests=3, pages=5)
    rm = RequestManager(vocab_size=raw["vocab"])
    for p in prompts:
        rm.add_request(len(p), 20, 0.0, prompt=p)
    rm.finalize_stats()
    pool, state = DistKVPool(eng.model.run_layers, 1, 200, 5, 16, 1), StateSlotPool(3)
    sch = Scheduler(pool, rm.avaliable_request_queue, global_batch_size=64, max_batch_size=3, average_prefill_length=1,
                    average_decode_length=1, group_size=1, state_pool=state, kv_window=eng.model.kv_window)
    st = ServingLoop(eng, sch, rm, est_cycle_time=1.0).run()
    assert sch.preemptions > 0 and pool.num_free_pages == 5 and state.num_free == 3
    outs = {}
    for r in st.retired:
        outs.setdefault(r.req_idx, []).append(r)
    for i, p in enumerate(prompts):
        # a preempted request continues as a new one whose prompt holds what it had generated
        r = max(outs[i], key=lambda r: len(r.prompt))
        full = np.concatenate([r.prompt, r.output]).tolist()
        assert full == p.tolist() + oracle.generate(raw, t, p.tolist(), 20)


def test_replay_command_line_parses_and_refuses(monkeypatch, tmp_path):
    from nanoflow_b200 import replay
    import nanoflow_b200.ops.build as build
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw)
    monkeypatch.setattr(build, "build_runtime", lambda: None)
    monkeypatch.setattr(replay, "build_replay", lambda model, dtype, n, r: TraceReplay(cpu_engine(raw, t), 64, r))
    toks = cases.prompt(12, raw["vocab"], 1).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:9], "want": [8, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[9:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[10:], "want": [1]}], "end": ["x"]}]
    out = io.StringIO()
    rc = replay.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"],
                     io.StringIO("\n".join(json.dumps(s) for s in steps)), out)
    assert rc == 0 and out.getvalue().split("\n")[:3] == ["done 0", "done 1", "done 2"]
    want = oracle.forward(raw, t, toks)
    a = np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, -1)
    b = np.fromfile(tmp_path / "2.f32", "<f4").reshape(1, -1)
    assert row_max(np.concatenate([a, b]), want[[8, 2, 11]]) < TOL and not (tmp_path / "1.f32").exists()

    def refuse(*a):
        raise NotImplementedError("no 32-bit")
    monkeypatch.setattr(replay, "build_replay", refuse)
    assert replay.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"], io.StringIO(""), out) == 3
