"""Engine of layer-list models (:mod:`..models.layer_list`): buffers, caches and the op graph of one iteration.

Everything around the graph (staging of the batch metadata, launches, token feedback on the device,
status word) is :class:`.engine.Engine`; this module says what an iteration consists of. One nano-batch,
one GPU, one stream. Per layer run:

* the packed input projection of the mixer (gate pre-activations leave it in fp32);
* latent attention: latents normed into the paged pool, then two ways to attend, chosen per portion when the
  batch is staged. Single tokens and short portions (and everything in 32-bit) stay in latent space: the
  queries are multiplied by their heads' key matrices (one block-diagonal GEMM), the kernel reads the cached
  rows as keys and values at once, and a second block-diagonal GEMM applies the value matrices. Longer
  portions gather the latents they can see, expand them to keys and values of all heads with one GEMM, and
  run the tcgen05 prefill kernel over those;
* grouped-query attention: queries and keys normed or rotated, values mixed or rotated, both appended to the paged
  pool (or those of an earlier layer read from its pool); single tokens on the split-KV decode kernel, portions on the
  tcgen05 prefill kernel, both with capped scores, sinks, distance biases and chunks (in 32-bit, and for head sizes and
  options those are not built for, one simple kernel); attention with mixed heads on kernels of its own;
* mLSTM: one kernel for requests with one token, one for longer portions, then head norm and output gate;
* WKV: every stream's mix with the previous token (kept per request), the four projections as one block-diagonal
  product, the low-rank decay, one kernel for single tokens and one for portions (chunks, or token by token),
  both with head norm and gate;
* real-gated linear recurrent unit: short convolution, both gates as one block-diagonal product, one kernel for the
  recurrence and the product with the GELU branch;
* delta rule: short convolutions of queries, keys and values as one, low-rank decays and gates, one kernel for single
  tokens and one for portions, both with head norm and gate;
* two mixers side by side: one input projection for both;
* output projection;
* feed-forward: gated, or a mixture of experts (router product, routing, rows in expert order, two products per
  expert, the shared expert, or experts that hand on the input);
* one kernel for: norm or scale of the sublayer's output, of a pair's outputs, or of the weighted sum of experts and shared
  expert, residual sum in fp32, the step vector of a loop pass or the embedding row (with its position vector), the
  weighted sum with the results of earlier layers, and the norm the next sublayer reads; a convolution over time after
  it where the model has one.

A new kind of mixer needs a spec and weights in ``models/layer_list.py`` and a builder in ``MIXERS``, a new kind of
feed-forward one in ``FEED_FORWARDS``.
"""
from __future__ import annotations

from ctypes import c_void_p
from typing import Dict, List, Optional, Tuple

import numpy as np
import torch

from .. import ops
from ..models.layer_list import (DELTA_CHUNK_DIM, PAGE, PREFILL_HEAD_DIM, WKV_CHUNK_DIM, ActSpec, LayerListConfig, NormWeights, parts_of,
                                 round8)
from ..ops import ACTS, CONV_ACTS, LIN_ACTS, NORMS, ROUTER_SCORES, dtype_code
from ..ops.layer_list import mlstm_scratch_floats
from ..serving.scheduler import BatchPlan
from .engine import DECODE_MAX_CHUNKS, DECODE_SPLIT_ROWS, GEMM_WS_BYTES, Engine, MetaLayout
from .graph import (ArgmaxParams, AttnParams, DeltaParams, GemmParams, GqaAppendParams, GqaAttnParams, HeadNormGateParams,
                    LatentAppendParams, LatentAttnParams, LatentGatherParams, MemcpyParams, MlstmParams, MoeGemmParams,
                    MoePermuteParams, MoeRouteParams, OpGraph, ResidualNormParams, RgLruParams, RopeTableParams,
                    ShortConvParams, TalkAttnParams, TokenShiftParams, WkvParams)
from .pipeline import _ptr

QUERY_TILE = 128             # query tokens per work item of the prefill attention kernel
MLSTM_CHUNK = 64             # tokens per chunk of the chunked mLSTM kernel
MLSTM_COLS = 64              # columns of the state per CTA of that kernel
SEGMENT_ITEMS = 48           # most segments that prompt portions are cut into for the mLSTM kernel
CHUNK = 64                   # tokens per chunk of the chunked WKV and delta-rule kernels
SPARE_CHUNKS = 64        # chunks beyond whole ones that their scratch has room for; further portions go token by token


TALK_TILE = 16               # query tokens per work item of the prefill kernel for mixed heads
DELTA_UNIT_EPS = 1e-6        # of the unit vectors of the delta rule


class PathGroup:
    """Latent-attention layers that share their work lists: same window, same choice of paths."""

    def __init__(self, index: int, window: int, expands: bool):
        self.index, self.window, self.expands = index, window, expands

    def name(self, what: str) -> str:
        return f"{what}{self.index}"


class LayerListEngine(Engine):
    model: LayerListConfig

    # ---- set-up -------------------------------------------------------------------------------------
    def _setup(self, num_pages: Optional[int]) -> None:
        m, e = self.model, self.eng
        if len(self.nano_sizes) != 1 or e.overlap:
            raise ValueError("layer-list models run in one nano-batch on one stream (pipeline_type NON_OVERLAP_LOCAL)")
        if e.offload:
            raise ValueError("KV offload is not built for layer-list models")
        T, B = e.global_batch_size, e.max_batch_size
        self.T, self.B = T, B
        self.S_cap = e.max_sample_rows or B
        self.code = dtype_code(m.dtype)
        self.gemm_kernel = "nfk_gemm_f32" if m.dtype == torch.float32 else "nfk_gemm_bf16"
        self.num_slots = (e.state_slots or B) if m.has_state else 0
        self.groups: List[PathGroup] = []
        for s in m.run_specs("latent_attention"):
            key = (s.window or 0, m.expands(s))
            if not any((g.window, g.expands) == key for g in self.groups):
                self.groups.append(PathGroup(len(self.groups), *key))
        # query heads per KV head of the attention layers on the tcgen05 prefill kernel: a work list for each
        self.attn_groups = sorted({s.group for s in m.run_specs("attention") if m.attn_on_tensor_cores(s)})
        self.chunk_cap = 0
        if m.dtype == torch.bfloat16 and (any(round8(s.dim) <= WKV_CHUNK_DIM for s in m.run_specs("wkv")) or
                                          any(self._delta_in_chunks(s) for s in m.run_specs("delta"))):
            self.chunk_cap = T // CHUNK + min(B, SPARE_CHUNKS)
        self.x_pages = self._expand_pages()
        self._alloc_state()
        self.num_pages = int(num_pages or e.num_pages or self._derive_num_pages(T, B))
        extra = {"kv_first": B, "state_ref": B}
        for g in self.groups:
            extra[g.name("abs")] = T
            if g.expands:
                extra.update({g.name("xptr"): B + 1, g.name("xpage"): self.x_pages, g.name("xitem"): 3 * (T // QUERY_TILE + B + 1)})
        for n in self.attn_groups:
            extra[f"gitem{n}"] = 3 * (T // (QUERY_TILE // n) + B + 1)
        if m.run_specs("mlstm"):
            extra["segs"] = 4 * max(B, SEGMENT_ITEMS)
        if any(s.talk for s in m.run_specs("attention")):
            extra["titem"] = 3 * (T // TALK_TILE + B + 1)
        if m.run_specs("wkv") or m.run_specs("delta"):
            extra.update(chunk_items=4 * max(1, self.chunk_cap), chunk_seq=B)
        if m.run_specs("wkv") or m.run_specs("delta"):
            extra["pre_reqs"] = B
        self._make_metadata(MetaLayout(T, B, self.nano_sizes, self.num_pages, 0, self.S_cap, extra))
        self.meta = {n: self._meta_view(n) for n in self.layout.off}
        self._alloc_buffers()
        if e.autotune_gemm and m.dtype == torch.bfloat16:
            self._autotune()
        self.graph = self._build_graph()

    def _expand_pages(self) -> int:
        """Pages of latents that one iteration can expand to keys and values."""
        if not any(g.expands for g in self.groups):
            return 0
        rows = self.eng.expand_rows
        if rows <= 0:
            window = max(g.window for g in self.groups if g.expands)
            if any(g.expands and g.window == 0 for g in self.groups):
                window = 8192
            rows = self.T + 8 * (window + 2 * PAGE)
        return max(2, (rows + PAGE - 1) // PAGE)

    def _alloc_state(self) -> None:
        m, dev = self.model, self.device
        n = self.num_slots
        z = lambda *shape, dtype=torch.float32: torch.zeros(*shape, dtype=dtype, device=dev)
        # per run: the state of its recurrent mixer, and the last inputs of the two sublayers' input convolutions
        self.state: List[Tuple[torch.Tensor, ...]] = []
        self.conv_state: List[Tuple[Optional[torch.Tensor], ...]] = []
        for r in m.runs:
            lay = m.layers[r.layer]
            self.state.append(tuple(z(n, *shape, dtype=dt) for s in parts_of(lay.mixer) for shape, dt in m.state_shapes(s)))
            conv = lambda used: z(n, *m.conv_state_shape(), dtype=m.dtype) if m.input_conv and used else None
            self.conv_state.append((conv(True), conv(m.conv_mlp(lay))))

    def _widths(self) -> Dict[str, int]:
        """Columns of the shared activation buffers (the widest layer's)."""
        m = self.model
        w = dict(proj=8, gates=8, attn=8, q_lat=0, o_lat=0, o_rec=8, act=8, kv=0, cg=0, qn=0, v_first=0, mix=0, lora=0,
                 router=0, e_in=0, e_act=0, e_out=0, e_top=0, conv=0, aux=0, beta=0)
        up = lambda k, n: w.__setitem__(k, max(w[k], n))
        for lay in m.layers:
            s = lay.mixer
            if s.kind == "pair":
                a, b, hd = s.left, s.right, m.attn_hd(s.left)
                up("proj", (a.heads + 2 * a.kv_heads) * hd + 2 * b.cols)
                up("qn", a.heads * hd)
                up("attn", a.heads * hd)
                up("conv", b.cols)
                up("gates", 2 * b.cols)
                up("aux", b.cols)
            elif s.kind == "rglru":
                up("proj", 2 * s.cols)
                up("conv", s.cols)
                up("gates", 2 * s.cols)
                up("attn", s.cols)
            elif s.kind == "delta":
                d, v = round8(s.dim), round8(s.vdim)
                qkv = 2 * s.kv_heads * d + s.heads * v
                up("proj", qkv + 2 * s.rank_p)
                up("conv", qkv)
                up("beta", round8(s.heads))
                up("gates", s.heads * d)
                up("aux", s.heads * v)
                up("o_rec", s.heads * v)
                up("attn", s.heads * v)
            elif s.kind == "latent_attention":
                dq, dv = m.head_pads(s)
                ld = m.latent_ld(s)
                up("proj", s.heads * dq + round8(s.kv_rank))
                up("attn", s.heads * dv)
                up("q_lat", s.heads * ld)
                if m.expands(s):
                    up("kv", s.heads * 2 * PREFILL_HEAD_DIM)
                    up("cg", ld)
            elif s.kind == "attention":
                hd = m.attn_hd(s)
                up("proj", s.proj_heads * hd)
                if moves_queries(s):
                    up("qn", s.heads * hd)
                up("attn", s.heads * hd)
                if s.value_mix:
                    up("v_first", s.kv_heads * hd)
            elif s.kind == "wkv":
                d = round8(s.dim)
                up("mix", 5 * m.width_p)
                up("proj", 4 * s.heads * d)
                up("lora", round8(s.rank))
                up("gates", s.heads * d)
                up("o_rec", s.heads * d)
                up("attn", s.heads * d)
            else:
                d, v = round8(s.dim), round8(s.vdim)
                up("proj", s.heads * 2 * (d + v))
                up("gates", round8(2 * s.heads))
                up("o_rec", s.heads * v)
                up("attn", s.heads * v)
            f = lay.mlp
            if f is not None and f.kind == "dense":
                up("act", round8(f.ff))
            elif f is not None:
                up("router", round8(f.router_cols))
                up("e_in", f.top * m.width_p)
                up("e_act", f.top * round8(f.expert.ff))
                up("e_out", f.top * m.width_p)
                up("e_top", f.top)
                if f.shared is not None:
                    up("act", round8(f.shared.ff))
        return w

    def _derive_num_pages(self, T: int, B: int) -> int:
        m, e = self.model, self.eng
        free, total = torch.cuda.mem_get_info(self.device)
        w = self._widths()
        es = m.elem_bytes
        act = T * (4 * m.width_p + es * (3 * m.width_p + w["proj"] + w["attn"] + 2 * w["q_lat"] + w["act"] + w["qn"] +
                                         w["v_first"] + w["mix"] + w["lora"] + w["e_in"] + w["e_act"] + w["e_out"] + w["conv"] +
                                         w["aux"] + 2 * m.width_p) +
                   4 * (w["gates"] + w["o_rec"] + w["router"] + w["beta"] + 5 * w["e_top"] + 2 * sum((len(k) + 7) // 8 * 8 for k in self._rotations())))
        act += self._decode_ws_floats() * 4 + self._chunk_scratch_floats() * 4
        act += 4 * T * m.width_p * len(m.runs) if m.depth_average else 0
        act += self.x_pages * PAGE * (w["kv"] + w["cg"]) * es + self.S_cap * (es * m.width_p + 4 * m.vocab_p)
        budget = free - total * (1.0 - e.gpu_mem_fraction) - act - (1 << 30)
        per_page = max(1, m.kv_bytes_per_token_local()) * PAGE
        n = int(min(budget // per_page, 1 << 22))
        if n < 64:
            raise RuntimeError(f"not enough GPU memory for a page pool ({free >> 20} MiB free)")
        return n

    def _rotations(self) -> List[tuple]:
        """The distinct lists of frequencies of the model."""
        return sorted({key for s in self.model.run_specs("attention") for key in rotations(s)})

    def _decode_ws_floats(self) -> int:
        """Partial results of split-KV decode attention."""
        hd = max([self.model.attn_hd(s) for s in self.model.run_specs("attention") if self.model.attn_on_tensor_cores(s)],
                 default=0)
        return DECODE_SPLIT_ROWS * DECODE_MAX_CHUNKS * (hd + 2) if hd else 0

    def _chunk_scratch_floats(self) -> int:
        sizes = [(s.heads, round8(s.dim)) for s in self.model.run_specs("wkv")]
        floats = [h * (d * d + d) for h, d in sizes if d <= WKV_CHUNK_DIM]
        floats += [s.heads * delta_item_floats(s) for s in self.model.run_specs("delta") if self._delta_in_chunks(s)]
        return self.chunk_cap * max(floats, default=0)

    def _delta_in_chunks(self, s) -> bool:
        return self.model.dtype == torch.bfloat16 and max(round8(s.dim), round8(s.vdim)) <= DELTA_CHUNK_DIM

    def _talk_kernels(self, s, talk: torch.Tensor) -> Tuple[bool, bool]:
        """Whether single tokens and portions of an attention layer with mixed heads run on the kernels made for them."""
        if self.model.dtype != torch.bfloat16:
            return False, False
        keys = min(s.window or self.num_pages * PAGE, self.num_pages * PAGE)
        fits = ops.lib().nfk_talk_attn_fits(s.heads, s.kv_heads, self.model.attn_hd(s), keys)
        exact = torch.equal(talk.to(torch.bfloat16).float(), talk)      # it enters their products in bf16
        return bool(fits & 2) and exact, bool(fits & 1) and exact

    def _alloc_buffers(self) -> None:
        m, T, dev = self.model, self.T, self.device
        dt, f32, w = m.dtype, torch.float32, self._widths()
        P = lambda rows, cols, dtype=dt, name="": self._plain(rows, cols, dtype=dtype, name=name)
        self.x = P(T, m.width_p, f32, "x")
        self.h = P(T, m.width_p, dt, "h")
        self.y = P(T, m.width_p, dt, "y")
        self.h_raw = P(T, m.width_p, dt, "h_raw") if m.input_conv else None      # before the input convolution
        # the embedding output and every layer's result, where later layers read them
        self.hist = self._plain(len(m.runs) * T, m.width_p, dtype=f32, name="results").view(len(m.runs), T, m.width_p) \
            if m.depth_average else None
        self.pos_freq = None
        if m.sinusoid:
            i = torch.arange((m.hidden_size + 1) // 2 + 1, dtype=torch.float64)
            f = m.sinusoid ** (-2.0 * i / m.hidden_size)
            self.pos_freq = torch.stack([f.float(), (f - f.float().double()).float()], dim=1).contiguous().to(dev)
        pairs = any(lay.mixer.kind == "pair" for lay in m.layers)
        self.y2 = P(T, m.width_p, dt, "y2") if m.parallel or m.run_moes() or pairs else None
        flat = lambda k, dtype, rows=T: P(1, max(8, rows * w[k]), dtype, k).view(-1)
        self.flat = {"proj": flat("proj", dt), "attn": flat("attn", dt), "act": flat("act", dt), "gates": flat("gates", f32),
                     "o_rec": flat("o_rec", f32), "q_lat": flat("q_lat", dt), "o_lat": flat("q_lat", dt),
                     "kv": flat("kv", dt, self.x_pages * PAGE), "cg": flat("cg", dt, self.x_pages * PAGE),
                     "router": flat("router", f32), "beta": flat("beta", f32)}
        self.flat.update({k: flat(k, dt) for k in ("qn", "v_first", "mix", "lora", "e_in", "e_act", "e_out", "conv", "aux")})
        # (cos, sin) of every token's angles, one table per distinct list of frequencies
        self.angles: Dict[tuple, Tuple[torch.Tensor, torch.Tensor]] = {}
        for key in self._rotations():
            f = torch.zeros(max(8, (len(key) + 7) // 8 * 8), dtype=f32, device=dev)
            f[:len(key)] = torch.tensor(key, dtype=torch.float64)
            self.angles[key] = (f, torch.zeros(T, f.numel(), 2, dtype=f32, device=dev))
        i32 = torch.int32
        self.moe_ids = {k: flat("e_top", f32 if k == "weight" else i32) for k in ("expert", "rank", "slot", "weight")}
        self.moe_gate = P(1, T, f32, "moe_gate").view(-1)
        # one counter per expert and layer run, cleared from zeros at the start of an iteration
        moes = [m.layers[r.layer].mlp for r in m.runs]
        sizes = [f.experts if f is not None and f.kind == "moe" else 0 for f in moes]
        self.moe_counts = torch.zeros(max(1, sum(sizes)), dtype=i32, device=dev)
        self.moe_zeros = torch.zeros_like(self.moe_counts)
        self.moe_counts_of = [c for c in self.moe_counts[:sum(sizes)].split(sizes)] if sum(sizes) else [None] * len(sizes)
        self.decode_ws = torch.empty(max(8, self._decode_ws_floats()), dtype=f32, device=dev)
        self.chunk_ws = torch.empty(max(8, self._chunk_scratch_floats()), dtype=f32, device=dev)
        self.h_s = P(self.S_cap, m.width_p, dt, "sample_h")
        self.logits = P(self.S_cap, m.vocab_p, f32, "logits")
        self.pools = [next((p for s in parts_of(m.layers[r.layer].mixer) for p in [self._pool(s)] if p is not None), None)
                      for r in m.runs]
        for r, run in enumerate(m.runs):                 # lent keys and values (no loops: runs are layers)
            src = getattr(m.layers[run.layer].mixer, "kv_from", None)
            if src is not None:
                self.pools[r] = self.pools[src]
        self.arange = torch.arange(self.x_pages + 1, dtype=torch.int32, device=dev)
        heads = max([s.heads * (m.latent_ld(s) + 2) for s in m.run_specs("latent_attention")], default=0)
        self.latent_ws = torch.empty(max(8, 160 * heads), dtype=f32, device=dev)
        seg = max([mlstm_scratch_floats(SEGMENT_ITEMS, s.heads, round8(s.dim), round8(s.vdim), T) +
                   mlstm_scratch_floats(self.B, s.heads, 8, 8, T, False) for s in m.run_specs("mlstm")], default=0)
        self.seg_ws = torch.empty(max(8, seg if dt == torch.bfloat16 else 8), dtype=f32, device=dev)
        self.gemm_ws = torch.zeros(GEMM_WS_BYTES // 4, dtype=f32, device=dev) if dt == torch.bfloat16 else None
        self.taps = P(len(m.runs) * T, m.width_p, f32, "taps").view(len(m.runs), T, m.width_p) \
            if self.eng.tap_residual else None

        class _Bufs:                      # the members Engine reads
            pass
        self.bufs = _Bufs()
        self.bufs.sampled = self._plain(self.S_cap, dtype=torch.int32, name="sampled")
        self.bufs.status = torch.zeros(1, dtype=torch.int32, device=dev)
        self.bufs.logits = self.logits

    def _pool(self, s) -> Optional[torch.Tensor]:
        shape = self.model.pool_shape(s)
        return None if shape is None else torch.zeros(self.num_pages, *shape, dtype=self.model.dtype, device=self.device)

    def view(self, name: str, cols: int, rows: Optional[int] = None) -> torch.Tensor:
        rows = rows or self.T
        return self.flat[name][:rows * cols].view(rows, cols)

    # ---- graph --------------------------------------------------------------------------------------
    def _build_graph(self) -> OpGraph:
        m, w = self.model, self.w
        g = self.g = OpGraph()
        self.last_op: Optional[int] = None
        T = g.symbol("T")
        for s in ("nb0_T", "nb0_items", "nb0_dec_begin", "nb0_dec_count", "n_sample", "n_dec", "n_pre"):
            g.symbol(s)
        lay = self.layout
        self._op("meta_h2d", MemcpyParams(dst=_ptr(self.meta_dev), src=c_void_p(0), elem_bytes=4, count=lay.fixed_words),
                 dyn=[("src", g.symbol("meta_src"))])
        self._op("kv_indices_h2d", MemcpyParams(dst=c_void_p(self.meta_dev.data_ptr() + 4 * lay.off["kv_indices"]),
                                                src=c_void_p(0), elem_bytes=4, count=0),
                 dyn=[("src", g.symbol("kv_src")), ("count", g.symbol("kv_words"))])
        if m.run_moes():
            self._op("moe_counts", MemcpyParams(dst=_ptr(self.moe_counts), src=_ptr(self.moe_zeros), elem_bytes=4,
                                                count=self.moe_counts.numel()))
        for i, (freq, table) in enumerate(self.angles.values()):
            self._op(f"angles{i}", RopeTableParams(cos_sin=_ptr(table), inv_freq=_ptr(freq), positions=_ptr(self.meta["positions"]),
                                                   T=0, half=freq.numel()), dyn=[("T", T)])
        # what joins the stream before each run: a step vector, or the embedding row
        step = lambda r: None if m.runs[r].step is None else "embedding" if m.loop_add == "embedding" else \
            w.loop_steps[m.runs[r].step]
        self._residual("embedding", None, w.embed_norm, w.layers[m.runs[0].layer].norm_in, step(0), embed=True, feeds=(0, 0),
                       average=-1 if m.depth_average else None)
        for r, run in enumerate(m.runs):
            spec, lw = m.layers[run.layer], w.layers[run.layer]
            last = r + 1 == len(m.runs)
            nxt = None if last else w.layers[m.runs[r + 1].layer].norm_in
            add = None if last else step(r + 1)
            more = MIXERS[spec.mixer.kind](self, r, run.layer, spec.mixer, lw.mixer) or {}
            y, out = self.y, lw.norm_out                   # what joins the stream at the end of the layer
            if spec.mlp is not None:
                if not m.parallel:
                    self._residual(f"R{r}.mid", self.y, lw.norm_out, lw.mlp_in, None, layer=r, more=more, feeds=(r, 1))
                    out = lw.mlp_out
                more = FEED_FORWARDS[spec.mlp.kind](self, r, run.layer, spec.mlp, lw.mlp)
                if not m.parallel:
                    y = more.pop("y2", None) if "y2_gate" not in more else None
            average = r if m.depth_average else None
            if last and self.taps is None:
                # only the sampled rows go on
                self._residual("final", y, out, w.final_norm, None, sampled=True, more=more, average=average)
            else:
                tap_add = add if self.taps is None else None
                go_on = not last and self.taps is None
                self._residual(f"R{r}.out", y, out, nxt if go_on else None, tap_add, layer=r, more=more,
                               feeds=(r + 1, 0) if go_on else None, average=average)
                if self.taps is not None:
                    self._op(f"R{r}.tap", MemcpyParams(dst=_ptr(self.taps[r]), src=_ptr(self.x), elem_bytes=4 * m.width_p,
                                                       count=0), dyn=[("count", T)], layer=r)
                    if last:
                        self._residual("final", None, None, w.final_norm, None, sampled=True)
                    else:
                        self._residual(f"R{r}.next", None, None, nxt, add, layer=r, feeds=(r + 1, 0))
        S = g.symbol("n_sample")
        self._gemm("lm_head", self.h_s, w.lm_head, None, rows=S, d32=self.logits)
        self._op("argmax", ArgmaxParams(idx_out=_ptr(self.bufs.sampled), val_out=c_void_p(0), logits=_ptr(self.logits),
                                        rows=0, cols=m.vocab_size, ld=self.logits.stride(0), col_offset=0, dtype=ops.F32),
                 dyn=[("rows", S)])
        self._op("tokens_d2h", MemcpyParams(dst=c_void_p(0), src=_ptr(self.bufs.sampled), elem_bytes=4, count=0),
                 dyn=[("dst", g.symbol("tokens_dst")), ("count", S)])
        self._op("status_d2h", MemcpyParams(dst=c_void_p(0), src=_ptr(self.bufs.status), elem_bytes=4, count=1),
                 dyn=[("dst", g.symbol("status_dst"))])
        return g

    def _op(self, name, params, *, dyn=(), kernel=None, layer=-1) -> None:
        self.last_op = self.g.add(name, params, "gemm", deps=[] if self.last_op is None else [self.last_op], dyn=dyn,
                                  kernel=kernel, layer=layer, nano=0)

    def _residual(self, name, y, norm_in: Optional[NormWeights], norm_out: Optional[NormWeights], add, *, embed=False,
                  sampled=False, layer=-1, more: Optional[dict] = None, feeds: Optional[Tuple[int, int]] = None,
                  average: Optional[int] = None) -> None:
        """``more``: what a sublayer adds to the sum besides ``y``: ``y2`` with ``y2_gate`` per row, and expert rows
        (``e_out``, ``e_slot``, ``e_weight``, ``e_top``), under the same norm; or ``pair``: the norms of ``y`` and ``y2``
        whose mean is the output. ``add``: a vector, or "embedding". ``feeds``: the run and sublayer (mixer 0, feed-forward
        1) that reads the normed stream, through its input convolution if it has one: single tokens get it here, portions
        by an op of its own. ``average``: the run whose result this is (-1: the embedding output); the weighted sum of all
        results so far goes on."""
        m = self.model
        kind = lambda norm: NORMS[norm.kind or m.norm_kind]
        p = ResidualNormParams()
        conv, state = None, None
        if feeds is not None:
            lw = self.w.layers[m.runs[feeds[0]].layer]
            conv, state = (lw.conv_mlp if feeds[1] else lw.conv_in), self.conv_state[feeds[0]][feeds[1]]
        p.x, p.ld_x = _ptr(self.x), self.x.stride(0)
        again = isinstance(add, str)
        if embed or again:
            p.table_add = int(again)
            p.table, p.ld_table, p.vocab = _ptr(self.w.embed), self.w.embed.stride(0), m.vocab_size
            p.host_ids, p.feedback_src = _ptr(self.meta["host_ids"]), _ptr(self.meta["feedback_src"])
            p.prev_tokens = _ptr(self.bufs.sampled)
            p.src_scale = m.embed_scale
        if embed and self.pos_freq is not None:
            p.pos_freq, p.positions = _ptr(self.pos_freq), _ptr(self.meta["positions"])
        if average is not None:
            if average >= 0:
                p.hist, p.hist_w = _ptr(self.hist), _ptr(self.w.layers[m.runs[average].layer].depth)
                p.hist_n, p.hist_stride = average + 1, self.hist.stride(0)
            if average + 1 < len(m.runs):
                p.hist_out = _ptr(self.hist[average + 1])
        if y is not None and not embed:
            p.y, p.ld_y = _ptr(y), y.stride(0)
        if norm_in is not None:
            p.in_w, p.in_b, p.in_kind = _ptr(norm_in.w), _ptr(norm_in.b), kind(norm_in)
        more = more or {}
        if more.get("y2") is not None:
            p.y2, p.ld_y2, p.y2_gate = _ptr(more["y2"]), more["y2"].stride(0), _ptr(more.get("y2_gate"))
        if more.get("e_out") is not None:
            p.e_out, p.ld_e, p.e_rows = _ptr(more["e_out"]), more["e_out"].stride(0), more["e_out"].shape[0]
            p.e_slot, p.e_weight, p.e_top = _ptr(more["e_slot"]), _ptr(more["e_weight"]), more["e_top"]
        if more.get("pair") is not None:
            p.pair_w, p.pair_w2 = _ptr(more["pair"][0]), _ptr(more["pair"][1])
        elif norm_in is not None and (p.y2 or p.e_out):
            p.norm_sum = 1
        p.add = None if again else _ptr(add)
        if norm_out is not None:
            h = self.h_s if sampled else self.h if conv is None else self.h_raw
            p.h, p.ld_h, p.out_w, p.out_b, p.out_kind = _ptr(h), h.stride(0), _ptr(norm_out.w), _ptr(norm_out.b), kind(norm_out)
        if sampled:
            p.rows_idx, p.in_rows = _ptr(self.meta["sample_rows"]), self.T
        p.cols, p.eps, p.dtype, p.status = m.hidden_size, m.norm_eps, self.code, _ptr(self.bufs.status)
        dyn = [("rows", "n_sample" if sampled else "T")]
        if conv is not None:
            p.conv_w, p.conv_out, p.conv_state = _ptr(conv), _ptr(self.h), _ptr(state)
            p.state_slot, p.positions = _ptr(self.meta["state_ref"]), _ptr(self.meta["positions"])
            p.conv_taps, p.conv_ld, p.num_slots = conv.shape[0], conv.shape[1], self.num_slots
            dyn.append(("conv_rows", "n_dec"))
        self._op(name, p, dyn=dyn, layer=layer)
        if conv is not None:
            self._short_conv(f"R{feeds[0]}.input_conv{feeds[1]}", self.h_raw, self.h, conv, state, residual=True, portions=True,
                             layer=feeds[0])

    def _short_conv(self, name, x, out, w, state, *, bias=None, act=None, residual=False, portions=False,
                    layer=-1) -> None:
        """``portions``: only the rows behind the single tokens."""
        meta, m = self.meta, self.model
        p = ShortConvParams(x=_ptr(x), ld_x=x.stride(0), out=_ptr(out), ld_out=out.stride(0), w=_ptr(w), bias=_ptr(bias),
                            state=_ptr(state), state_slot=_ptr(meta["state_ref"]), positions=_ptr(meta["positions"]),
                            token_req=_ptr(meta["token_req"]), qo_indptr=_ptr(meta["qo_indptr"]), row_begin=0, T=0,
                            cols=w.shape[1], taps=w.shape[0], act=CONV_ACTS[act], residual=int(residual),
                            num_slots=self.num_slots, dtype=self.code, status=_ptr(self.bufs.status))
        self._op(name, p, dyn=[("T", "T")] + ([("row_begin", "n_dec")] if portions else []), layer=layer)

    def _gemm(self, name, a, wt, out, *, rows: str, up=None, act: ActSpec = ActSpec("silu"), lin_act=None, bias=None, up_bias=None,
              d32=None, f32_col0=0, groups=1, group_k=0, k=0, key="", layer=-1) -> None:
        """out[rows, N] = a @ wt^T. ``d32``: columns from ``f32_col0`` on leave as fp32; ``groups`` > 1:
        block-diagonal (each group of rows of ``wt`` sees ``k`` columns of ``a``, ``group_k`` apart)."""
        p = GemmParams()
        p.A, p.B, p.B2, p.D = _ptr(a), _ptr(wt), _ptr(up), _ptr(out)
        p.lda, p.ldb, p.ldd = a.stride(0), wt.stride(0), (out.stride(0) if out is not None else wt.shape[0])
        p.N, p.K = wt.shape[0], k or wt.shape[1]
        p.epilogue, p.lin_act, p.bias, p.bias2 = (1 if up is not None else 0), LIN_ACTS[lin_act], _ptr(bias), _ptr(up_bias)
        p.act, p.act_limit, p.act_alpha, p.act_shift = ACTS[act.name], act.limit, act.alpha, act.shift
        if d32 is not None:
            p.D32, p.ld32, p.f32_col0 = _ptr(d32), d32.stride(0), f32_col0
        p.groups, p.group_k = groups, group_k
        p.status = _ptr(self.bufs.status)
        if self.gemm_ws is not None:
            p.workspace, p.workspace_bytes = _ptr(self.gemm_ws), self.gemm_ws.numel() * 4
        shape = self.eng.gemm_shapes.get(key)
        if shape is not None:
            p.tile_m, p.tile_n, p.cta_group = shape["tile_m"], shape["tile_n"], shape["cta_group"]
            p.split_k, p.stream_k = shape["split_k"], shape["stream_k"]
        self._op(name, p, dyn=[("M", rows)], kernel=self.gemm_kernel, layer=layer)

    # ---- mixers: read self.h, leave their output projection in self.y ---------------------------------
    def _latent_attention(self, r: int, layer: int, s, lw) -> None:
        m, g, T = self.model, self.g, "T"
        dq, dv = m.head_pads(s)
        H, ld, pool = s.heads, m.latent_ld(s), self.pools[r]
        pg = next(x for x in self.groups if (x.window, x.expands) == (s.window or 0, m.expands(s)))
        meta, st = self.meta, _ptr(self.bufs.status)
        proj = self.view("proj", H * dq + round8(s.kv_rank))
        self._gemm(f"R{r}.in", self.h, lw.w_in, proj, rows=T, key=f"l{layer}.in", layer=r)
        ap = LatentAppendParams(src=c_void_p(proj.data_ptr() + H * dq * proj.element_size()), ld_src=proj.stride(0),
                                w=_ptr(lw.dkv_norm), pool=_ptr(pool), ld=ld, positions=_ptr(meta["positions"]),
                                token_req=_ptr(meta["token_req"]), kv_indptr=_ptr(meta["kv_indptr"]),
                                kv_indices=_ptr(meta["kv_indices"]), kv_first=_ptr(meta["kv_first"]), T=0, rank=s.kv_rank,
                                page_size=PAGE, num_pages=self.num_pages, eps=m.norm_eps, dtype=self.code, status=st)
        self._op(f"R{r}.latent_append", ap, dyn=[("T", T)], layer=r)
        # in latent space
        rows, n_abs = g.symbol(pg.name("abs_rows")), g.symbol(pg.name("n_abs"))
        q_lat, o_lat, attn = self.view("q_lat", H * ld), self.view("o_lat", H * ld), self.view("attn", H * dv)
        self._gemm(f"R{r}.q_latent", proj, lw.w_qk, q_lat, rows=rows, groups=H, group_k=dq, layer=r)
        lp = LatentAttnParams(q=_ptr(q_lat), ld_q=q_lat.stride(0), pool=_ptr(pool), ld=ld, out=_ptr(o_lat),
                              ld_out=o_lat.stride(0), tokens=_ptr(meta[pg.name("abs")]), positions=_ptr(meta["positions"]),
                              token_req=_ptr(meta["token_req"]), kv_indptr=_ptr(meta["kv_indptr"]),
                              kv_indices=_ptr(meta["kv_indices"]), kv_first=_ptr(meta["kv_first"]), sinks=_ptr(lw.sinks),
                              n_tokens=0, heads=H, page_size=PAGE, num_pages=self.num_pages, window=s.window or 0,
                              scale=s.scale, dtype=self.code, impl=0, splits=1, workspace=_ptr(self.latent_ws),
                              workspace_floats=self.latent_ws.numel(), status=st)
        self._op(f"R{r}.latent_attn", lp, dyn=[("n_tokens", n_abs), ("splits", g.symbol(pg.name("splits")))], layer=r)
        self._gemm(f"R{r}.v_latent", o_lat, lw.w_ov, attn, rows=rows, groups=H, group_k=ld, layer=r)
        # expanded keys and values
        if pg.expands:
            n_x = g.symbol(pg.name("n_xpages"))
            kv_cols = H * 2 * PREFILL_HEAD_DIM
            cg, kv = self.view("cg", ld, self.x_pages * PAGE), self.view("kv", kv_cols, self.x_pages * PAGE)
            mp = LatentGatherParams(pool=_ptr(pool), out=_ptr(cg), page_ids=_ptr(meta[pg.name("xpage")]), ld=ld, n_pages=0,
                                    page_size=PAGE, num_pages=self.num_pages, dtype=self.code, status=st)
            self._op(f"R{r}.latent_gather", mp, dyn=[("n_pages", n_x)], layer=r)
            self._gemm(f"R{r}.expand", cg, lw.w_kv, kv, rows=g.symbol(pg.name("x_rows")), layer=r)
            pp = AttnParams()
            pp.q, pp.out, pp.kv_pool = _ptr(proj), _ptr(attn), _ptr(kv)
            pp.qo_indptr, pp.kv_indptr = _ptr(meta["qo_indptr"]), _ptr(meta[pg.name("xptr")])
            pp.kv_indices, pp.kv_last_page_len = _ptr(self.arange), _ptr(meta["kv_last_page_len"])
            pp.q_heads = pp.kv_heads = H
            pp.head_dim, pp.page_size, pp.num_pages, pp.sm_scale = PREFILL_HEAD_DIM, PAGE, self.x_pages, s.scale
            pp.items, pp.status = _ptr(meta[pg.name("xitem")]), st
            pp.window, pp.sinks = s.window or 0, _ptr(lw.sinks)
            pp.kv_ld, pp.k_col, pp.v_col = kv_cols, 0, H * PREFILL_HEAD_DIM
            pp.q_rows, pp.ld_q = self.T, proj.stride(0)
            self._op(f"R{r}.attn_prefill", pp, kernel="nfk_attn_prefill_ws", dyn=[("num_items", g.symbol(pg.name("n_xitems")))],
                     layer=r)
        self._gemm(f"R{r}.o", attn, lw.w_o, self.y, rows=T, key=f"l{layer}.o", layer=r)

    def _mlstm(self, r: int, layer: int, s, lw) -> None:
        m, T, meta = self.model, "T", self.meta
        H, d, v = s.heads, round8(s.dim), round8(s.vdim)
        main = H * 2 * (d + v)
        proj, gates = self.view("proj", main), self.view("gates", round8(2 * H))
        o_rec, attn = self.view("o_rec", H * v), self.view("attn", H * v)
        self._gemm(f"R{r}.in", self.h, lw.w_in, proj, rows=T, d32=gates, f32_col0=main, key=f"l{layer}.in", layer=r)
        S, n, mx = self.state[r]

        def params() -> MlstmParams:
            return MlstmParams(
                qkv=_ptr(proj), ld_qkv=proj.stride(0), q_off=0, k_off=H * d, v_off=2 * H * d, gates=_ptr(gates),
                ld_gates=gates.stride(0), i_bias=_ptr(lw.i_b), f_bias=_ptr(lw.f_b), S=_ptr(S), n=_ptr(n), m=_ptr(mx),
                out=_ptr(o_rec), ld_out=o_rec.stride(0), positions=_ptr(meta["positions"]),
                qo_indptr=_ptr(meta["qo_indptr"]), state_slot=_ptr(meta["state_ref"]), req_begin=0, req_count=0, heads=H,
                dim=d, vdim=v, num_slots=self.num_slots, gate_cap=s.gate_cap, q_scale=s.dim ** -0.5, dtype=self.code,
                impl=0, items=_ptr(meta["segs"]), num_items=0, num_tokens=0, scratch=_ptr(self.seg_ws),
                scratch_floats=self.seg_ws.numel(), status=_ptr(self.bufs.status))

        self._op(f"R{r}.mlstm_decode", params(), kernel="nfk_mlstm_decode", dyn=[("req_count", "n_dec")], layer=r)
        self._op(f"R{r}.mlstm_prefill", params(), kernel="nfk_mlstm_prefill",
                 dyn=[("req_begin", "n_dec"), ("req_count", "n_pre"), ("num_items", self.g.symbol("n_segs")),
                      ("num_tokens", T)], layer=r)
        g_cols = c_void_p(proj.data_ptr() + (2 * H * d + H * v) * proj.element_size())
        hp = HeadNormGateParams(o=_ptr(o_rec), ld_o=o_rec.stride(0), g=g_cols, ld_g=proj.stride(0), w=_ptr(lw.norm),
                                out=_ptr(attn), ld_out=attn.stride(0), T=0, heads=H, vdim=s.vdim, vdim_p=v, eps=m.norm_eps,
                                dtype=self.code)
        self._op(f"R{r}.head_norm", hp, dyn=[("T", T)], layer=r)
        self._gemm(f"R{r}.o", attn, lw.w_o, self.y, rows=T, key=f"l{layer}.o", layer=r)

    def _attention(self, r: int, layer: int, s, lw, proj=None) -> None:
        """``proj``: the projected queries, keys and values, if they are there already."""
        m, g, T, meta, st = self.model, self.g, "T", self.meta, _ptr(self.bufs.status)
        H, G, hd, pool = s.heads, s.kv_heads, m.attn_hd(s), self.pools[r]
        attn = self.view("attn", H * hd)
        if proj is None:
            proj = self.view("proj", s.proj_heads * hd)
            self._gemm(f"R{r}.in", self.h, lw.w_in, proj, rows=T, bias=lw.b_in, key=f"l{layer}.in", layer=r)
        # queries that nothing is done to stay in the projection's rows
        q, ld_q = (self.view("qn", H * hd), 0) if moves_queries(s) else (proj, proj.stride(0))
        mode = 0 if not s.value_mix else 1 if r == m.first_value_run else 2
        ap = GqaAppendParams(src=_ptr(proj), ld_src=proj.stride(0), q_off=0, k_off=H * hd, v_off=(H + G) * hd, q_out=None if ld_q else _ptr(q),
                             q_w=_ptr(lw.q_norm), k_w=_ptr(lw.k_norm), v_first=_ptr(self.flat["v_first"]), v_mode=mode,
                             v_lambda=lw.value_lambda, pool=_ptr(pool), positions=_ptr(meta["positions"]),
                             token_req=_ptr(meta["token_req"]), kv_indptr=_ptr(meta["kv_indptr"]),
                             kv_indices=_ptr(meta["kv_indices"]), kv_first=_ptr(meta["kv_first"]), T=0, heads=H, kv_heads=G,
                             hd=hd, dim=s.dim, page_size=PAGE, num_pages=self.num_pages, eps=m.norm_eps, dtype=self.code,
                             status=st)
        turns = rotations(s)
        if turns:
            ap.rot, ap.rot_pairs, ap.rot_ld = _ptr(self.angles[turns[0]][1]), len(turns[0]), self.angles[turns[0]][0].numel()
        if len(turns) > 1:
            v_rot, v_pairs, v_ld = _ptr(self.angles[turns[1]][1]), len(turns[1]), self.angles[turns[1]][0].numel()
            ap.v_rot, ap.v_pairs, ap.v_ld = v_rot, v_pairs, v_ld
        else:
            v_rot, v_pairs, v_ld = None, 0, 0
        if s.kv_from is None:
            self._op(f"R{r}.gqa_append", ap, dyn=[("T", T)], layer=r)
        if s.talk:
            def params() -> TalkAttnParams:
                return TalkAttnParams(
                    q=_ptr(q), pool=_ptr(pool), out=_ptr(attn), positions=_ptr(meta["positions"]),
                    token_req=_ptr(meta["token_req"]), kv_indptr=_ptr(meta["kv_indptr"]), kv_indices=_ptr(meta["kv_indices"]),
                    kv_first=_ptr(meta["kv_first"]), sinks=_ptr(lw.sinks), talk=_ptr(lw.talk), v_rot=v_rot, v_pairs=v_pairs,
                    v_ld=v_ld, token_begin=0, n_tokens=0, heads=H, kv_heads=G, hd=hd, page_size=PAGE, num_pages=self.num_pages,
                    window=s.window or 0, scale=s.scale, dtype=self.code, status=st, items=_ptr(meta["titem"]))

            dec, pre = self._talk_kernels(s, lw.talk)
            self._op(f"R{r}.talk_decode", params(), kernel="nfk_talk_attn_decode" if dec else "nfk_talk_attn",
                     dyn=[("n_tokens", "n_dec")] + ([("max_keys", g.symbol(f"keys{s.window or 0}"))] if dec else []), layer=r)
            if pre:
                self._op(f"R{r}.talk_prefill", params(), kernel="nfk_talk_attn_prefill",
                         dyn=[("num_items", g.symbol("n_titems"))], layer=r)
            else:
                self._op(f"R{r}.talk_prefill", params(), kernel="nfk_talk_attn",
                         dyn=[("token_begin", "n_dec"), ("n_tokens", g.symbol("pre_tokens"))], layer=r)
        elif m.attn_on_tensor_cores(s):
            def params() -> AttnParams:
                p = AttnParams()
                p.q, p.ld_q, p.out, p.kv_pool = _ptr(q), ld_q, _ptr(attn), _ptr(pool)
                p.kv_first, p.dist, p.chunk = _ptr(meta["kv_first"]), _ptr(lw.dist), s.chunk or 0
                p.qo_indptr, p.kv_indptr = _ptr(meta["qo_indptr"]), _ptr(meta["kv_indptr"])
                p.kv_indices, p.kv_last_page_len = _ptr(meta["kv_indices"]), _ptr(meta["kv_last_page_len"])
                p.q_heads, p.kv_heads, p.head_dim, p.page_size, p.num_pages = H, G, hd, PAGE, self.num_pages
                p.sm_scale, p.softcap, p.sinks, p.precise, p.status = s.scale, s.softcap or 0.0, _ptr(lw.sinks), 1, st
                return p

            d = params()
            d.workspace, d.max_chunks = _ptr(self.decode_ws), 1
            self._op(f"R{r}.attn_decode", d, kernel="nfk_attn_decode",
                     dyn=[("req_count", "n_dec"), ("chunk_pages", g.symbol("dec_chunk_pages")),
                          ("max_chunks", g.symbol("dec_max_chunks"))], layer=r)
            p = params()
            p.items = _ptr(meta[f"gitem{s.group}"])
            self._op(f"R{r}.attn_prefill", p, kernel="nfk_attn_prefill_ws",
                     dyn=[("num_items", g.symbol(f"n_gitems{s.group}"))], layer=r)
        else:
            gp = GqaAttnParams(q=_ptr(q), ld_q=ld_q, dist=_ptr(lw.dist), chunk=s.chunk or 0, pool=_ptr(pool), out=_ptr(attn), positions=_ptr(meta["positions"]),
                               token_req=_ptr(meta["token_req"]), kv_indptr=_ptr(meta["kv_indptr"]),
                               kv_indices=_ptr(meta["kv_indices"]), kv_first=_ptr(meta["kv_first"]), sinks=_ptr(lw.sinks),
                               token_begin=0, n_tokens=0, heads=H, kv_heads=G, hd=hd, page_size=PAGE,
                               num_pages=self.num_pages, window=s.window or 0, scale=s.scale, softcap=s.softcap or 0.0, dtype=self.code,
                               status=st)
            self._op(f"R{r}.attn", gp, dyn=[("n_tokens", T)], layer=r)
        self._gemm(f"R{r}.o", attn, lw.w_o, self.y, rows=T, key=f"l{layer}.o", layer=r)

    def _wkv(self, r: int, layer: int, s, lw) -> None:
        m, T, meta, st = self.model, "T", self.meta, _ptr(self.bufs.status)
        H, d, wp = s.heads, round8(s.dim), m.width_p
        S, before = self.state[r]
        mix, proj, lora = self.view("mix", 5 * wp), self.view("proj", 4 * H * d), self.view("lora", round8(s.rank))
        decay, attn = self.view("gates", H * d), self.view("attn", H * d)
        ts = TokenShiftParams(h=_ptr(self.h), ld_h=wp, out=_ptr(mix), mu=_ptr(lw.mu), state=_ptr(before),
                              state_slot=_ptr(meta["state_ref"]), positions=_ptr(meta["positions"]),
                              token_req=_ptr(meta["token_req"]), qo_indptr=_ptr(meta["qo_indptr"]), T=0, n_mix=5,
                              num_slots=self.num_slots, dtype=self.code, status=st)
        self._op(f"R{r}.token_shift", ts, dyn=[("T", T)], layer=r)
        self._gemm(f"R{r}.in", mix, lw.w_in, proj, rows=T, groups=4, group_k=wp, k=wp, key=f"l{layer}.in", layer=r)
        self._gemm(f"R{r}.decay_down", mix[:, 4 * wp:], lw.w_down, lora, rows=T, lin_act="tanh", key=f"l{layer}.decay_down", layer=r)
        self._gemm(f"R{r}.decay_up", lora, lw.w_up, None, rows=T, d32=decay, bias=lw.w_bias, key=f"l{layer}.decay_up", layer=r)

        def params() -> WkvParams:
            return WkvParams(rkvg=_ptr(proj), ld=proj.stride(0), r_off=0, k_off=H * d, v_off=2 * H * d, g_off=3 * H * d,
                             x=_ptr(decay), ld_x=decay.stride(0), u=_ptr(lw.u), norm=_ptr(lw.norm), S=_ptr(S), y=_ptr(attn),
                             ld_y=attn.stride(0), positions=_ptr(meta["positions"]), qo_indptr=_ptr(meta["qo_indptr"]),
                             state_slot=_ptr(meta["state_ref"]), req_begin=0, req_count=0, heads=H, dim=d, dim_real=s.dim,
                             num_slots=self.num_slots, eps=m.norm_eps, dtype=self.code, o=_ptr(self.flat["o_rec"]),
                             items=_ptr(meta["chunk_items"]), scratch=_ptr(self.chunk_ws), scratch_floats=self.chunk_ws.numel(),
                             status=st)

        self._op(f"R{r}.wkv_decode", params(), kernel="nfk_wkv_decode", dyn=[("req_count", "n_dec")], layer=r)
        chunked = self.chunk_cap > 0 and d <= WKV_CHUNK_DIM
        p = params()
        p.seq_reqs = _ptr(meta["chunk_seq" if chunked else "pre_reqs"])
        dyn = [("num_seq", self.g.symbol("n_chunk_seq" if chunked else "n_pre"))]
        if chunked:
            dyn.append(("num_items", self.g.symbol("n_chunks")))
        self._op(f"R{r}.wkv_prefill", p, kernel="nfk_wkv_prefill", dyn=dyn, layer=r)
        self._gemm(f"R{r}.o", attn, lw.w_o, self.y, rows=T, key=f"l{layer}.o", layer=r)

    def _rglru(self, r: int, layer: int, s, lw, proj=None, act=None, out=None) -> None:
        """``proj``: the two projected branches, if they are there already; ``act``, ``out``: where the recurrence's result
        and its output projection go."""
        T, meta, n, bp = "T", self.meta, s.cols, s.block_p
        S, before = self.state[r]
        if proj is None:
            proj = self.view("proj", 2 * n)
            self._gemm(f"R{r}.in", self.h, lw.w_in, proj, rows=T, bias=lw.b_in, key=f"l{layer}.in", layer=r)
        act = self.view("attn", n) if act is None else act
        u, gates = self.view("conv", n), self.view("gates", 2 * n)
        self._short_conv(f"R{r}.rec_conv", proj[:, n:], u, lw.conv, before, bias=lw.conv_b, layer=r)
        self._gemm(f"R{r}.rec_gates", u, lw.w_gates, None, rows=T, d32=gates, groups=s.blocks, group_k=bp, k=bp, layer=r)

        def params() -> RgLruParams:
            return RgLruParams(u=_ptr(u), ld_u=u.stride(0), y=_ptr(proj), ld_y=proj.stride(0), gates=_ptr(gates),
                               ld_g=gates.stride(0), r_b=_ptr(lw.r_b), i_b=_ptr(lw.i_b), log_a=_ptr(lw.log_a), S=_ptr(S),
                               out=_ptr(act), ld_out=act.stride(0), positions=_ptr(meta["positions"]),
                               qo_indptr=_ptr(meta["qo_indptr"]), state_slot=_ptr(meta["state_ref"]), req_begin=0, req_count=0,
                               cols=n, block=bp, num_slots=self.num_slots, dtype=self.code, status=_ptr(self.bufs.status))

        self._op(f"R{r}.rglru_decode", params(), kernel="nfk_rglru_decode", dyn=[("req_count", "n_dec")], layer=r)
        self._op(f"R{r}.rglru_prefill", params(), kernel="nfk_rglru_prefill",
                 dyn=[("req_begin", "n_dec"), ("req_count", "n_pre")], layer=r)
        self._gemm(f"R{r}.rec_o", act, lw.w_o, self.y if out is None else out, rows=T, key=f"l{layer}.rec_o", layer=r)

    def _pair(self, r: int, layer: int, s, lw) -> dict:
        n = lw.left.w_in.shape[0]
        proj = self.view("proj", lw.w_in.shape[0])
        self._gemm(f"R{r}.in", self.h, lw.w_in, proj, rows="T", bias=lw.b_in, key=f"l{layer}.in", layer=r)
        self._attention(r, layer, s.left, lw.left, proj[:, :n])
        self._rglru(r, layer, s.right, lw.right, proj[:, n:], self.view("aux", s.right.cols), self.y2)
        return {"y2": self.y2, "pair": (lw.left_norm, lw.right_norm)}

    def _delta(self, r: int, layer: int, s, lw) -> None:
        T, meta, st = "T", self.meta, _ptr(self.bufs.status)
        H, G, d, v, rp = s.heads, s.kv_heads, round8(s.dim), round8(s.vdim), s.rank_p
        S, before = self.state[r]
        qkv = 2 * G * d + H * v
        proj, conv, beta = self.view("proj", qkv + 2 * rp), self.view("conv", qkv), self.view("beta", round8(H))
        decay, gate, attn = self.view("gates", H * d), self.view("aux", H * v), self.view("attn", H * v)
        self._gemm(f"R{r}.in", self.h, lw.w_in, proj, rows=T, d32=beta, f32_col0=qkv + 2 * rp, key=f"l{layer}.in", layer=r)
        self._short_conv(f"R{r}.qkv_conv", proj, conv, lw.conv, before, act="silu", layer=r)
        self._gemm(f"R{r}.decay_up", proj[:, qkv:qkv + rp], lw.w_decay, None, rows=T, d32=decay, key=f"l{layer}.decay_up", layer=r)
        self._gemm(f"R{r}.gate_up2", proj[:, qkv + rp:], lw.w_gate, gate, rows=T, key=f"l{layer}.gate_up2", layer=r)

        def params() -> DeltaParams:
            return DeltaParams(qkv=_ptr(conv), ld=conv.stride(0), q_off=0, k_off=G * d, v_off=2 * G * d, x=_ptr(decay),
                               ld_x=decay.stride(0), beta=_ptr(beta), ld_b=beta.stride(0), g=_ptr(gate), ld_g=gate.stride(0),
                               rate=_ptr(lw.rate), dt_bias=_ptr(lw.dt_bias), norm=_ptr(lw.norm), S=_ptr(S), y=_ptr(attn),
                               ld_y=attn.stride(0), positions=_ptr(meta["positions"]), qo_indptr=_ptr(meta["qo_indptr"]),
                               state_slot=_ptr(meta["state_ref"]), req_begin=0, req_count=0, heads=H, kv_heads=G, dim=d, vdim=v,
                               vdim_real=s.vdim, num_slots=self.num_slots, q_scale=s.dim ** -0.5, unit_eps=DELTA_UNIT_EPS,
                               eps=self.model.norm_eps, dtype=self.code, seq_reqs=_ptr(meta["pre_reqs"]), num_seq=0,
                               o=_ptr(self.flat["o_rec"]), items=_ptr(meta["chunk_items"]), scratch=_ptr(self.chunk_ws),
                               scratch_floats=self.chunk_ws.numel(), status=st)

        self._op(f"R{r}.delta_decode", params(), kernel="nfk_delta_decode", dyn=[("req_count", "n_dec")], layer=r)
        p, dyn = params(), [("num_seq", "n_pre")]
        if self._delta_in_chunks(s):
            p.seq_reqs = _ptr(meta["chunk_seq"])
            dyn = [("num_seq", self.g.symbol("n_chunk_seq")), ("num_items", self.g.symbol("n_chunks")),
                   ("num_portions", self.g.symbol("n_chunk_reqs"))]
        self._op(f"R{r}.delta_prefill", p, kernel="nfk_delta_prefill", dyn=dyn, layer=r)
        self._gemm(f"R{r}.o", attn, lw.w_o, self.y, rows=T, key=f"l{layer}.o", layer=r)

    # ---- feed-forwards: read self.h; return what joins the stream (see _residual) -------------------------
    def _dense(self, r: int, layer: int, s, lw, key="") -> dict:
        act = self.view("act", round8(s.ff))
        out = self.y2 if self.y2 is not None else self.y
        self._gemm(f"R{r}.{key}gate_up", self.h, lw.w_gate, act, rows="T", up=lw.w_up, act=s.act, bias=lw.b_gate, up_bias=lw.b_up,
                   key=f"l{layer}.{key}gate_up", layer=r)
        self._gemm(f"R{r}.{key}down", act, lw.w_down, out, rows="T", bias=lw.b_down, key=f"l{layer}.{key}down", layer=r)
        return {"y2": out}

    def _moe(self, r: int, layer: int, s, lw) -> dict:
        m, T, st, wp, ids = self.model, "T", _ptr(self.bufs.status), self.model.width_p, self.moe_ids
        rows = self.g.symbol(f"e_rows{s.top}")                 # tokens x experts per token
        logits, counts, cap = self.view("router", lw.router.shape[0]), self.moe_counts_of[r], self.T * s.top
        flat = lambda k, cols: self.flat[k][:cap * cols].view(cap, cols)
        e_in, e_act, e_out = flat("e_in", wp), flat("e_act", round8(s.expert.ff)), flat("e_out", wp)
        self._gemm(f"R{r}.router", self.h, lw.router, None, rows=T, d32=logits, key=f"l{layer}.router", layer=r)
        rp = MoeRouteParams(logits=_ptr(logits), ld=logits.stride(0), correction=_ptr(lw.correction), expert=_ptr(ids["expert"]),
                            weight=_ptr(ids["weight"]), rank=_ptr(ids["rank"]), counts=_ptr(counts), gate=_ptr(self.moe_gate),
                            T=0, experts=s.experts, top=s.top, groups=s.groups, keep=s.keep,
                            gate_col=s.experts if s.shared is not None else -1, scale=s.scale, score=ROUTER_SCORES[s.score],
                            identity=s.identity, group_max=int(s.group_score == "max"))
        self._op(f"R{r}.moe_route", rp, dyn=[("T", T)], layer=r)
        pp = MoePermuteParams(h=_ptr(self.h), ld_h=wp, out=_ptr(e_in), ld_out=wp, expert=_ptr(ids["expert"]),
                              rank=_ptr(ids["rank"]), counts=_ptr(counts), slot=_ptr(ids["slot"]), T=0, top=s.top,
                              experts=s.experts, cols=wp, dtype=self.code)
        self._op(f"R{r}.moe_permute", pp, dyn=[("T", T)], layer=r)

        def product(name, a, b, b2, out, n, lin_act=None) -> None:
            act = s.expert.act
            p = MoeGemmParams(A=_ptr(a), B=_ptr(b), B2=_ptr(b2), D=_ptr(out), counts=_ptr(counts), lda=a.stride(0),
                              ldb=b.stride(0), ldd=out.stride(0), rows=0, experts=s.experts, N=n, K=b.shape[1],
                              act=ACTS.get(act.name, 0), act_limit=act.limit, act_alpha=act.alpha, act_shift=act.shift,
                              dtype=self.code, num_ctas=0, status=st, lin_act=LIN_ACTS[lin_act])
            self._op(f"R{r}.{name}", p, dyn=[("rows", rows)], layer=r)

        if s.expert.gated:
            product("moe_gate_up", e_in, lw.w_gate, lw.w_up, e_act, round8(s.expert.ff))
        else:
            product("moe_up", e_in, lw.w_up, None, e_act, round8(s.expert.ff), s.expert.act.name)
        product("moe_down", e_act, lw.w_down, None, e_out, wp)
        out = dict(e_out=e_out, e_slot=ids["slot"], e_weight=ids["weight"], e_top=s.top)
        if s.identity:
            out.update(y2=self.h, y2_gate=self.moe_gate)
        if s.shared is not None:
            out.update(self._dense(r, layer, s.shared, lw.shared, key="shared_"), y2_gate=self.moe_gate)
        return out

    # ---- GEMM shapes ----------------------------------------------------------------------------------
    def _autotune(self) -> None:
        """Measured shapes for the dense products of every distinct layer at the full batch size."""
        from ..ops import autotune
        m, T, done = self.model, self.T, {}
        self.h.normal_()
        for k in ("attn", "act", "lora", "aux"):
            self.flat[k].normal_()
        for i, lay in enumerate(m.layers):
            lw = self.w.layers[i]
            mixer = lw.mixer.left if lay.mixer.kind == "pair" else lw.mixer
            specs = [("o", None, mixer.w_o, None, None)]
            if lay.mixer.kind == "pair":
                rec = lw.mixer.right.w_o
                specs += [("in", self.h, lw.mixer.w_in, None, self.flat["proj"]),
                          ("rec_o", self.view("aux", rec.shape[1]), rec, None, None)]
            elif lay.mixer.kind == "delta":
                specs += [("in", self.h, lw.mixer.w_in, None, self.flat["proj"]),
                          ("decay_up", self.h[:, :lay.mixer.rank_p], lw.mixer.w_decay, None, self.flat["proj"]),
                          ("gate_up2", self.h[:, :lay.mixer.rank_p], lw.mixer.w_gate, None, self.flat["proj"])]
            elif lay.mixer.kind == "wkv":          # (its input projection is block-diagonal: left to the cost model)
                lora = self.view("lora", lw.mixer.w_down.shape[0])
                specs += [("decay_down", self.h, lw.mixer.w_down, None, self.flat["proj"]),
                          ("decay_up", lora, lw.mixer.w_up, None, self.flat["proj"])]
            else:
                specs.append(("in", self.h, lw.mixer.w_in, None, self.flat["proj"]))
            if lay.mlp is not None and lay.mlp.kind == "moe":
                specs.append(("router", self.h, lw.mlp.router, None, self.flat["proj"]))
            f, key = (lw.mlp, "") if lay.mlp is None or lay.mlp.kind == "dense" else (lw.mlp.shared, "shared_")
            if f is not None:
                specs += [(key + "gate_up", self.h, f.w_gate, f.w_up, self.flat["act"]), (key + "down", None, f.w_down, None, None)]
            for key, a, wt, up, out in specs:
                name = f"l{i}.{key}"
                if name in self.eng.gemm_shapes:
                    continue
                if a is None:
                    a = self.view("attn" if key == "o" else "act", wt.shape[1])
                n = wt.shape[0]
                if out is not None and T * n > out.numel():
                    n = out.numel() // T // 8 * 8          # the fp32 gate columns have no place in the bf16 buffer
                    wt = wt[:n]
                dst = self.y if out is None else out[:T * n].view(T, n)
                sig = (key, n, wt.shape[1], up is not None)
                if sig not in done:
                    done[sig] = autotune.tune_gemm(a, [wt], dst, weights_up=None if up is None else [up], workspace=self.gemm_ws)
                res = done[sig]
                self.eng.gemm_shapes[name] = dict(res["best"])
                self.gemm_tuning[name] = dict(M=T, best=res["best"], us=res["us"], auto_us=res["auto_us"])
        torch.cuda.synchronize(self.device)
        for t in (self.h, self.y, *self.flat.values()):
            t.zero_()

    # ---- per iteration ----------------------------------------------------------------------------------
    def _stage_model(self, plan: BatchPlan, put, sym: Dict[str, int]) -> None:
        if plan.num_tail_decode:
            raise ValueError("layer-list models take their decode requests at the front of the batch")
        m, D, P, B = self.model, plan.num_decode, len(plan.prefill), plan.num_requests
        put("kv_first", plan.kv_first)
        put("state_ref", plan.state_ref)
        sym["n_dec"], sym["n_pre"] = D, P
        qo, span = plan.qo_indptr, np.diff(plan.qo_indptr)
        if m.run_specs("mlstm"):
            segs = mlstm_segments(qo, D, self._segment_ctas(), ops.sm_count(self.device))
            put("segs", segs.reshape(-1))
            sym["n_segs"] = segs.shape[0]
        if "chunk_items" in self.meta:
            items, seq = chunk_work(qo, D, self.chunk_cap)
            put("chunk_items", items.reshape(-1))
            put("chunk_seq", seq)
            sym["n_chunks"], sym["n_chunk_seq"], sym["n_chunk_reqs"] = items.shape[0], seq.size, P - seq.size
        if "titem" in self.meta:
            items = query_items(qo, D, TALK_TILE)
            put("titem", items.reshape(-1))
            sym["n_titems"], sym["pre_tokens"] = items.shape[0], plan.num_tokens - int(qo[D])
            seen = int(plan.positions[:D].max()) + 1 if D else 1
            for w in {s.window or 0 for s in m.run_specs("attention")}:
                sym[f"keys{w}"] = min(w or seen, seen)
        if "pre_reqs" in self.meta:
            put("pre_reqs", np.arange(D, D + P, dtype=np.int32))
        for n in self.attn_groups:
            items = by_keys(query_items(qo, D, QUERY_TILE // n), plan.positions, m.first_seen)
            put(f"gitem{n}", items.reshape(-1))
            sym[f"n_gitems{n}"] = items.shape[0]
        if self.attn_groups:
            chunks = [s.chunk for s in m.run_specs("attention") if m.attn_on_tensor_cores(s)]
            seen = plan.max_kv_pages if None in chunks else min(plan.max_kv_pages, max(chunks) // PAGE + 2)
            sym["dec_chunk_pages"], sym["dec_max_chunks"] = self._attn_split(D, seen)
        for top in {f.top for f in m.run_moes()}:
            sym[f"e_rows{top}"] = plan.num_tokens * top
        for g in self.groups:
            work = route_attention(plan, g.window, g.expands, self.x_pages, self.eng.expand_min_tokens)
            put(g.name("abs"), work["abs"])
            n_abs = int(work["abs"].size)
            sym[g.name("n_abs")] = n_abs
            sym[g.name("abs_rows")] = int(work["abs"].max()) + 1 if n_abs else 0
            ctx = plan.max_kv_pages * PAGE
            sym[g.name("splits")] = self._latent_splits(n_abs, min(ctx, g.window + PAGE) if g.window else ctx)
            if g.expands:
                put(g.name("xptr"), work["xptr"])
                put(g.name("xpage"), work["xpage"])
                put(g.name("xitem"), work["items"].reshape(-1))
                sym[g.name("n_xpages")] = int(work["xpage"].size)
                sym[g.name("x_rows")] = int(work["xpage"].size) * PAGE
                sym[g.name("n_xitems")] = int(work["items"].shape[0])

    def _attn_split(self, n_dec: int, pages: int) -> Tuple[int, int]:
        """(pages per key range, ranges) of decode attention, so that a few long contexts still occupy the SMs."""
        specs = [s for s in self.model.run_specs("attention") if self.model.attn_on_tensor_cores(s)]
        work = n_dec * min(s.kv_heads for s in specs)
        target = 4 * ops.sm_count(self.device)
        if work == 0 or work >= target or pages <= 16 or n_dec * max(s.heads for s in specs) > DECODE_SPLIT_ROWS:
            return 0, 1
        chunk = max(8, -(-pages // min(DECODE_MAX_CHUNKS, -(-target // work))))
        return chunk, max(1, -(-pages // chunk))

    def _segment_ctas(self) -> int:
        """CTAs of the chunked mLSTM kernel per segment (of the layer with the fewest)."""
        return min(s.heads * ((s.vdim + MLSTM_COLS - 1) // MLSTM_COLS) for s in self.model.run_specs("mlstm"))

    def _latent_splits(self, n_abs: int, ctx: int) -> int:
        """Key ranges per token, so that a few tokens still occupy the SMs (at least four 64-key tiles each)."""
        if n_abs == 0:
            return 1
        groups = max((s.heads + 31) // 32 for s in self.model.run_specs("latent_attention"))
        return int(max(1, min(16, ctx // 256, ops.sm_count(self.device) // (n_abs * groups))))

    def last_logits(self, n: int) -> torch.Tensor:
        """fp32 logits [n, vocab] of the first ``n`` sampled rows of the last iteration."""
        torch.cuda.synchronize(self.device)
        return self.logits[:n, :self.model.vocab_size]


MIXERS = {"latent_attention": LayerListEngine._latent_attention, "mlstm": LayerListEngine._mlstm,
          "attention": LayerListEngine._attention, "wkv": LayerListEngine._wkv, "rglru": LayerListEngine._rglru,
          "delta": LayerListEngine._delta, "pair": LayerListEngine._pair}
FEED_FORWARDS = {"dense": LayerListEngine._dense, "moe": LayerListEngine._moe}


def delta_item_floats(s) -> int:
    """Scratch of a chunk and head of the chunked delta-rule kernels (nfk_delta_item_floats)."""
    n = 64 if max(round8(s.dim), round8(s.vdim)) <= 64 else 128
    return (6 * CHUNK * (n + 8) + 2 * CHUNK * (CHUNK + 8)) // 2 + n + n // 32 * CHUNK * 36


def moves_queries(s) -> bool:
    """Whether an attention layer's queries pass through the append kernel."""
    return s.qk_norm or s.rotary is not None or s.talk


def rotations(s) -> List[tuple]:
    """Frequencies by which an attention layer turns queries and keys, and if it does, values."""
    if s.rotary is None:
        return []
    keys = tuple(s.rotary.frequencies(s.rotary.dims, True))
    return [keys, tuple(s.rotary.frequencies(s.vdim, False))] if s.rotary.values else [keys]


# --------------------------------------------------------------------------------------------------
# Work lists (host side, no GPU needed)
# --------------------------------------------------------------------------------------------------
def mlstm_segments(qo_indptr: np.ndarray, n_dec: int, ctas_per_segment: int, sms: int) -> np.ndarray:
    """Rows (request, first token, tokens, segment) for the chunked mLSTM kernel. A portion is one segment unless
    the portions alone leave SMs idle; then long ones are cut into equal runs of whole chunks, enough of them to
    keep the last wave short (segments cost an extra pass over the keys and values)."""
    reqs = np.arange(n_dec, qo_indptr.size - 1)
    lens = np.diff(qo_indptr)[n_dec:]
    if reqs.size == 0:
        return np.zeros((0, 4), dtype=np.int32)
    target = 4 * sms // max(1, ctas_per_segment)
    seg_len = int(lens.max())
    if 2 * reqs.size * ctas_per_segment < 3 * sms and reqs.size < min(target, SEGMENT_ITEMS):
        room = min(target, SEGMENT_ITEMS) - reqs.size
        seg_len = max(4 * MLSTM_CHUNK, -(-int(lens.sum()) // room))
        seg_len = (seg_len + MLSTM_CHUNK - 1) // MLSTM_CHUNK * MLSTM_CHUNK
    out = []
    for b, n in zip(reqs, lens):
        for k, t in enumerate(range(0, int(n), seg_len)):
            out.append((b, qo_indptr[b] + t, min(seg_len, n - t), k))
    return np.asarray(out, dtype=np.int32)


def chunk_work(qo_indptr: np.ndarray, n_dec: int, chunk_cap: int) -> Tuple[np.ndarray, np.ndarray]:
    """Rows (request, first token, tokens, chunk of the portion) for the chunked WKV and delta-rule kernels, and the requests whose
    portions do not fit what is left of ``chunk_cap`` chunks: those go token by token."""
    rows, seq = [], []
    for b in range(n_dec, qo_indptr.size - 1):
        t0, n = int(qo_indptr[b]), int(qo_indptr[b + 1] - qo_indptr[b])
        if len(rows) + -(-n // CHUNK) > chunk_cap:
            seq.append(b)
            continue
        rows += [(b, t0 + c, min(CHUNK, n - c), c // CHUNK) for c in range(0, n, CHUNK)]
    return np.asarray(rows, dtype=np.int32).reshape(-1, 4), np.asarray(seq, dtype=np.int32)


def query_items(qo_indptr: np.ndarray, n_dec: int, tile: int) -> np.ndarray:
    """Rows (request, first token, tokens) of the prefill attention kernel."""
    rows = []
    for b in range(n_dec, qo_indptr.size - 1):
        q0, q1 = int(qo_indptr[b]), int(qo_indptr[b + 1])
        rows += [(b, t, min(tile, q1 - t)) for t in range(q0, q1, tile)]
    return np.asarray(rows, dtype=np.int32).reshape(-1, 3)


def by_keys(items: np.ndarray, positions: np.ndarray, first_seen) -> np.ndarray:
    """Work items in the order of how many keys they see: the prefill kernel deals out the last ones first."""
    if items.shape[0] == 0:
        return items
    first, last = positions[items[:, 1]], positions[items[:, 1] + items[:, 2] - 1]
    return items[np.argsort(last - np.asarray([first_seen(int(p)) for p in first]), kind="stable")]


def route_attention(plan: BatchPlan, window: int, expands: bool, page_cap: int, min_tokens: int) -> dict:
    """Which tokens attend in latent space (``abs``) and, for the portions that do not, the latent pages to
    expand (``xpage``, per-request ranges ``xptr`` of the expanded pages) and the prefill kernel's work items.
    A portion whose pages do not fit what is left of ``page_cap`` stays in latent space."""
    D, B, qo = plan.num_decode, plan.num_requests, plan.qo_indptr
    if not expands:
        return dict(abs=np.arange(plan.num_tokens, dtype=np.int32))
    toks = [np.arange(qo[D], dtype=np.int32)]
    pages, items = [], []
    xptr = np.zeros(B + 1, dtype=np.int32)
    used = 0
    for b in range(D, B):
        q0, q1 = int(qo[b]), int(qo[b + 1])
        start, end = int(plan.positions[q0]), int(plan.positions[q1 - 1])
        lo = max(0, start - window + 1) if window else 0
        first, n = lo // PAGE, end // PAGE - lo // PAGE + 1
        if q1 - q0 < min_tokens or used + n > page_cap:
            toks.append(np.arange(q0, q1, dtype=np.int32))
        else:
            p0 = int(plan.kv_indptr[b]) + first - int(plan.kv_first[b])
            pages.append(plan.kv_indices[p0:p0 + n])
            t = np.arange(q0, q1, QUERY_TILE, dtype=np.int32)
            items.append(np.stack([np.full_like(t, b), t, np.minimum(QUERY_TILE, q1 - t)], axis=1))
            used += n
        xptr[b + 1] = used
    cat = lambda parts, empty: np.concatenate(parts).astype(np.int32, copy=False) if parts else empty
    return dict(abs=np.concatenate(toks), xptr=xptr, xpage=cat(pages, np.zeros(0, dtype=np.int32)),
                items=cat(items, np.zeros((0, 3), dtype=np.int32)))
