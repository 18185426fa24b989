"""CPU backend of layer-list models: executes a scheduler :class:`BatchPlan` with plain PyTorch fp32 ops.

The data flow is that of the GPU engine (paged latent pool and page tables with released leading pages, state
slots with two halves for the small vectors, weights in kernel layout with their padding, token feedback), so
the scheduler, the caches and the weight packing can be tested end to end without a GPU. It is a test and
development backend, chosen explicitly (``serve.py --backend cpu``); the GPU engine never falls back to it.
"""
from __future__ import annotations

from typing import List, Optional

import numpy as np
import torch

from ..config import NanoflowConfig
from ..models.layer_list import LayerListConfig, LayerListWeights, parts_of, round8
from ..ops import reference as ref
from ..serving.scheduler import BatchPlan
from .layer_list import DELTA_UNIT_EPS, rotations


class CpuLayerListEngine:
    def __init__(self, cfg: NanoflowConfig, weights: LayerListWeights, num_pages: int = 256):
        self.cfg, self.eng = cfg, cfg.engine
        self.model: LayerListConfig = cfg.model
        if self.model.dtype != torch.float32:
            raise ValueError("the CPU backend computes in float32: load the model with dtype float32")
        self.w, self.num_pages = weights, num_pages
        m = self.model
        self.num_slots = (self.eng.state_slots or self.eng.max_batch_size) if m.has_state else 0
        self.pools, self.state, self.conv_state = [], [], []
        n = self.num_slots
        for r in m.runs:
            parts = parts_of(m.layers[r.layer].mixer)
            shapes = [m.pool_shape(s) for s in parts if m.pool_shape(s) is not None]
            self.pools.append(torch.zeros(num_pages, *shapes[0]) if shapes else None)
            self.state.append(tuple(torch.zeros(n, *shape) for s in parts for shape, _ in m.state_shapes(s)))
            self.conv_state.append([torch.zeros(n, *m.conv_state_shape()) for _ in range(2)] if m.input_conv else None)
            src = getattr(m.layers[r.layer].mixer, "kv_from", None)
            if src is not None:                              # lent keys and values (no loops: runs are layers)
                self.pools[-1] = self.pools[src]
        self.v_first: Optional[torch.Tensor] = None
        self.sampled = torch.zeros(self.eng.max_sample_rows or self.eng.max_batch_size, dtype=torch.int32)
        self._staged: Optional[BatchPlan] = None
        self._inflight: List[np.ndarray] = []
        self._last = np.zeros(0, dtype=np.int32)
        self._logits: Optional[torch.Tensor] = None

    # ---- one iteration --------------------------------------------------------------------------------
    def _norm(self, x, n):
        m = self.model
        y = x * n.w[:m.hidden_size] if n.kind == "scale" else \
            ref.layernorm(x, n.w[:m.hidden_size], None if n.b is None else n.b[:m.hidden_size], m.norm_eps) if m.norm_kind == "layer" else \
            ref.rmsnorm(x, n.w[:m.hidden_size], m.norm_eps)
        return torch.nn.functional.pad(y, (0, m.width_p - m.hidden_size))

    def _input_conv(self, r, sublayer, h, w, plan):
        return h if w is None else ref.short_conv(h, w, self.conv_state[r][sublayer], plan.positions, plan.qo_indptr,
                                                  plan.state_ref, residual=True)

    def _latent_attention(self, r, s, lw, h, plan):
        m = self.model
        dq, dv = m.head_pads(s)
        proj = h @ lw.w_in.t()
        T = h.shape[0]
        ref.latent_append(proj[:, s.heads * dq:s.heads * dq + s.kv_rank], lw.dkv_norm, self.pools[r], plan.positions,
                          plan.token_req, plan.kv_indptr, plan.kv_indices, plan.kv_first, m.norm_eps)
        q = torch.einsum("thd,hrd->thr", proj[:, :s.heads * dq].reshape(T, s.heads, dq), lw.w_qk.reshape(s.heads, -1, dq))
        o = ref.latent_attention(q, self.pools[r], plan.positions, plan.token_req, plan.kv_indptr, plan.kv_indices,
                                 plan.kv_first, scale=s.scale, window=s.window or 0, sinks=lw.sinks)
        a = torch.einsum("thr,hvr->thv", o, lw.w_ov.reshape(s.heads, dv, -1)).reshape(T, -1)
        return a @ lw.w_o.t()

    def _mlstm(self, r, s, lw, h, plan):
        H, d, v, T = s.heads, round8(s.dim), round8(s.vdim), h.shape[0]
        proj = h @ lw.w_in.t()
        q, k, vv, g, gates = proj.split([H * d, H * d, H * v, H * v, proj.shape[1] - 2 * H * (d + v)], dim=1)
        o = ref.mlstm(q.reshape(T, H, d) * s.dim ** -0.5, k.reshape(T, H, d), vv.reshape(T, H, v), gates[:, :H] + lw.i_b,
                      gates[:, H:2 * H] + lw.f_b, s.gate_cap, self.state[r], plan.positions, plan.qo_indptr, plan.state_ref)
        return ref.head_norm_gate(o, g.reshape(T, H, v), lw.norm.reshape(H, v), s.vdim, self.model.norm_eps).reshape(T, -1) @ \
            lw.w_o.t()

    def _attention(self, r, s, lw, h, plan):
        m, T = self.model, h.shape[0]
        H, G, hd = s.heads, s.kv_heads, m.attn_hd(s)
        proj = h @ lw.w_in.t() if lw.b_in is None else h @ lw.w_in.t() + lw.b_in
        q, k, v = proj.split([H * hd, G * hd, G * hd], dim=1) if s.kv_from is None else (proj, None, None)
        if s.value_mix and r == m.first_value_run:
            self.v_first = v
        elif s.value_mix:
            v = (1.0 - lw.value_lambda) * v + lw.value_lambda * self.v_first
        pages = (plan.positions, plan.token_req, plan.kv_indptr, plan.kv_indices, plan.kv_first)
        turns = rotations(s)
        turn = lambda x, n, i, sign=1.0: x if x is None or len(turns) <= i else \
            ref.turn_pairs(x.reshape(T, n, hd), plan.positions, turns[i], sign).reshape(T, -1)
        q, k, v = turn(q, H, 0), turn(k, G, 0), turn(v, G, 1)
        if k is not None:
            q = ref.gqa_append(q, k, v, lw.q_norm, lw.k_norm, self.pools[r], *pages, heads=H, kv_heads=G, dim=s.dim,
                               eps=m.norm_eps)
        if s.talk:
            o = ref.talk_attention(q.reshape(T, H, hd), self.pools[r], *pages, scale=s.scale, talk=lw.talk, window=s.window or 0,
                                   sinks=lw.sinks)
        else:
            o = ref.gqa_attention(q.reshape(T, H, hd), self.pools[r], *pages, scale=s.scale, softcap=s.softcap or 0.0,
                                  window=s.window or 0, sinks=lw.sinks, dist=lw.dist, chunk=s.chunk or 0)
        o = turn(o, H, 1, -1.0)
        return o.reshape(T, -1) @ lw.w_o.t()

    def _wkv(self, r, s, lw, h, plan):
        m, T, H, d = self.model, h.shape[0], s.heads, round8(s.dim)
        S, before = self.state[r]
        mix = ref.token_shift(h, lw.mu, before, plan.positions, plan.qo_indptr, plan.state_ref)
        proj = [(mix[:, j] @ w.t()).reshape(T, H, d) for j, w in enumerate(lw.w_in.chunk(4))]
        x = torch.tanh(mix[:, 4] @ lw.w_down.t()) @ lw.w_up.t() + lw.w_bias
        o = ref.wkv(proj[0], proj[1], proj[2], x.reshape(T, H, d), lw.u.reshape(H, d), S, plan.positions, plan.qo_indptr,
                    plan.state_ref)
        return ref.head_norm_silu(o, proj[3], lw.norm.reshape(H, d), s.dim, m.norm_eps).reshape(T, -1) @ lw.w_o.t()

    def _rglru(self, r, s, lw, h, plan):
        T, n, bp = h.shape[0], s.cols, s.block_p
        S, before = self.state[r]
        step = (plan.positions, plan.qo_indptr, plan.state_ref)
        y, x = (h @ lw.w_in.t() + lw.b_in).split([n, n], dim=1)
        u = ref.short_conv(x, lw.conv, before, *step, bias=lw.conv_b)
        gates = torch.einsum("tbk,bok->tbo", u.reshape(T, s.blocks, bp), lw.w_gates.reshape(s.blocks, 2 * bp, bp))
        o = ref.rglru(u, y, gates[:, :, :bp].reshape(T, n) + lw.r_b, gates[:, :, bp:].reshape(T, n) + lw.i_b, lw.log_a, S, *step)
        return o @ lw.w_o.t()

    def _pair(self, r, s, lw, h, plan):
        m = self.model
        rms = lambda y, w: ref.rmsnorm(y[:, :m.hidden_size], w[:m.hidden_size], m.norm_eps)
        y = 0.5 * (rms(self._attention(r, s.left, lw.left, h, plan), lw.left_norm) +
                   rms(self._rglru(r, s.right, lw.right, h, plan), lw.right_norm))
        return torch.nn.functional.pad(y, (0, m.width_p - m.hidden_size))

    def _delta(self, r, s, lw, h, plan):
        T, H, G, d, v, rp = h.shape[0], s.heads, s.kv_heads, round8(s.dim), round8(s.vdim), s.rank_p
        S, before = self.state[r]
        step = (plan.positions, plan.qo_indptr, plan.state_ref)
        qkv, down, gate, beta = (h @ lw.w_in.t()).split([2 * G * d + H * v, rp, rp, round8(H)], dim=1)
        q, k, vv = ref.short_conv(qkv, lw.conv, before, *step, act="silu").split([G * d, G * d, H * v], dim=1)
        x = down @ lw.w_decay.t() + lw.dt_bias
        o = ref.delta(q.reshape(T, G, d), k.reshape(T, G, d), vv.reshape(T, H, v), x.reshape(T, H, d), lw.rate, beta[:, :H], S,
                      *step, q_scale=s.dim ** -0.5, eps=DELTA_UNIT_EPS)
        o = ref.head_norm_gate(o, (gate @ lw.w_gate.t()).reshape(T, H, v), lw.norm.expand(H, v), s.vdim, self.model.norm_eps)
        return o.reshape(T, -1) @ lw.w_o.t()

    # ---- feed-forwards ----------------------------------------------------------------------------------
    def _dense(self, s, lw, h):
        a = s.act
        return ref.gated_mlp(h, lw.w_gate, lw.w_up, lw.w_down, a.name, biases=(lw.b_gate, lw.b_up, lw.b_down), limit=a.limit,
                             alpha=a.alpha, shift=a.shift)

    def _moe(self, s, lw, h):
        logits = h @ lw.router.t()
        idx, weight = ref.moe_route(logits[:, :s.outputs], lw.correction, s.top, s.groups, s.keep, s.scale, s.score, s.group_score)
        mats = [None if t is None else t.chunk(s.experts) for t in (lw.w_gate, lw.w_up, lw.w_down)]
        a, out = s.expert.act, torch.zeros_like(h)
        for e in range(s.experts):
            t, k = (idx == e).nonzero(as_tuple=True)
            if t.numel():
                y = ref.linear_act(h[t] @ mats[1][e].t(), a.name) @ mats[2][e].t() if not s.expert.gated else \
                    ref.gated_mlp(h[t], mats[0][e], mats[1][e], mats[2][e], a.name, limit=a.limit, alpha=a.alpha, shift=a.shift)
                out.index_add_(0, t, y * weight[t, k][:, None])
        if s.identity:
            out += (weight * (idx >= s.experts)).sum(-1, keepdim=True) * h
        if s.shared is not None:
            out += torch.sigmoid(logits[:, s.experts:s.experts + 1]) * self._dense(s.shared, lw.shared, h)
        return out

    def update(self, plan: BatchPlan) -> None:
        self._staged = plan

    def run_async(self) -> None:
        plan, self._staged = self._staged, None
        m, w = self.model, self.w
        ids = torch.from_numpy(plan.host_ids).long().clone()
        fb = torch.from_numpy(plan.feedback_src).long()
        ids[fb >= 0] = self.sampled[fb[fb >= 0]].long()
        W = m.hidden_size
        after = lambda y, n: y if n is None else self._norm(y[:, :W], n)
        x = start = after(w.embed[ids] * m.embed_scale, w.embed_norm)
        if m.sinusoid:
            x = start = x + torch.nn.functional.pad(ref.sinusoid(plan.positions, W, m.sinusoid), (0, m.width_p - W))
        results = [x]
        for r, run in enumerate(m.runs):
            spec, lw = m.layers[run.layer], w.layers[run.layer]
            if run.step is not None:
                x = x + (start if m.loop_add == "embedding" else w.loop_steps[run.step])
            h = self._input_conv(r, 0, self._norm(x[:, :W], lw.norm_in), lw.conv_in, plan)
            y = MIXERS[spec.mixer.kind](self, r, spec.mixer, lw.mixer, h, plan)
            if spec.mlp is None:
                x = x + after(y, lw.norm_out)
            elif m.parallel:
                x = x + (y + FEED_FORWARDS[spec.mlp.kind](self, spec.mlp, lw.mlp, h))
            else:
                x = x + after(y, lw.norm_out)
                h = self._input_conv(r, 1, self._norm(x[:, :W], lw.mlp_in), lw.conv_mlp, plan)
                x = x + after(FEED_FORWARDS[spec.mlp.kind](self, spec.mlp, lw.mlp, h), lw.mlp_out)
            if m.depth_average:
                results.append(x)
                x = sum(a * y for a, y in zip(lw.depth, results))
        rows = torch.from_numpy(plan.sample_rows).long()
        self._logits = (self._norm(x[rows][:, :m.hidden_size], w.final_norm) @ w.lm_head.t())[:, :m.vocab_size]
        toks = self._logits.argmax(dim=-1).int()
        self.sampled[:toks.numel()] = toks
        self._inflight.append(toks.numpy().copy())

    def run_async_wait(self) -> np.ndarray:
        self._last = self._inflight.pop(0)
        return self._last

    def run(self, plan: BatchPlan) -> np.ndarray:
        self.update(plan)
        self.run_async()
        return self.run_async_wait()

    def last_logits(self, n: int) -> torch.Tensor:
        return self._logits[:n]

    def getPipelineOutput(self) -> np.ndarray:
        return self._last

    @property
    def in_flight(self) -> int:
        return len(self._inflight)

    def check_status(self) -> None:
        pass

    def finalize(self) -> None:
        self._inflight.clear()


MIXERS = {"latent_attention": CpuLayerListEngine._latent_attention, "mlstm": CpuLayerListEngine._mlstm,
          "attention": CpuLayerListEngine._attention, "wkv": CpuLayerListEngine._wkv,
          "rglru": CpuLayerListEngine._rglru, "delta": CpuLayerListEngine._delta, "pair": CpuLayerListEngine._pair}
FEED_FORWARDS = {"dense": CpuLayerListEngine._dense, "moe": CpuLayerListEngine._moe}
