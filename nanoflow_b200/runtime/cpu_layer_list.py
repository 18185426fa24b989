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
from ..models.layer_list import LayerListConfig, LayerListWeights, round8
from ..ops import reference as ref
from ..serving.scheduler import BatchPlan
from .layer_list import PAGE


class CpuLayerListEngine:
    def __init__(self, cfg: NanoflowConfig, weights: LayerListWeights, num_pages: int = 256):
        self.cfg, self.eng = cfg, cfg.engine
        self.model: LayerListConfig = cfg.model
        if self.model.dtype != torch.float32:
            raise ValueError("the CPU backend computes in float32: load the model with dtype float32")
        self.w, self.num_pages = weights, num_pages
        m = self.model
        self.num_slots = (self.eng.state_slots or self.eng.max_batch_size) if m.has_state else 0
        self.pools, self.state = [], []
        for r in m.runs:
            s = m.layers[r.layer].mixer
            latent = s.kind == "latent_attention"
            self.pools.append(torch.zeros(num_pages, PAGE, m.latent_ld(s)) if latent else None)
            d, v, n = round8(s.dim), round8(s.vdim), self.num_slots
            self.state.append(None if latent else (torch.zeros(n, s.heads, d, v), torch.zeros(n, s.heads, 2, d),
                                                   torch.zeros(n, s.heads, 2)))
        self.sampled = torch.zeros(self.eng.max_sample_rows or self.eng.max_batch_size, dtype=torch.int32)
        self._staged: Optional[BatchPlan] = None
        self._inflight: List[np.ndarray] = []
        self._last = np.zeros(0, dtype=np.int32)
        self._logits: Optional[torch.Tensor] = None

    # ---- one iteration --------------------------------------------------------------------------------
    def _norm(self, x, n):
        m = self.model
        y = ref.layernorm(x, n.w[:m.hidden_size], n.b[:m.hidden_size], m.norm_eps) if m.norm_kind == "layer" else \
            ref.rmsnorm(x, n.w[:m.hidden_size], m.norm_eps)
        return torch.nn.functional.pad(y, (0, m.width_p - m.hidden_size))

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

    def update(self, plan: BatchPlan) -> None:
        self._staged = plan

    def run_async(self) -> None:
        plan, self._staged = self._staged, None
        m, w = self.model, self.w
        ids = torch.from_numpy(plan.host_ids).long().clone()
        fb = torch.from_numpy(plan.feedback_src).long()
        ids[fb >= 0] = self.sampled[fb[fb >= 0]].long()
        x = self._norm(w.embed[ids][:, :m.hidden_size], w.embed_norm)
        for r, run in enumerate(m.runs):
            spec, lw = m.layers[run.layer], w.layers[run.layer]
            if run.step is not None:
                x = x + w.loop_steps[run.step]
            mix = self._latent_attention if spec.mixer.kind == "latent_attention" else self._mlstm
            y = mix(r, spec.mixer, lw.mixer, self._norm(x[:, :m.hidden_size], lw.norm_in), plan)
            x = x + self._norm(y[:, :m.hidden_size], lw.norm_out)
            if spec.mlp is not None:
                h = self._norm(x[:, :m.hidden_size], lw.mlp_in)
                y = ref.gated_mlp(h, lw.w_gate, lw.w_up, lw.w_down, spec.mlp.act)
                x = x + self._norm(y[:, :m.hidden_size], lw.mlp_out)
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
