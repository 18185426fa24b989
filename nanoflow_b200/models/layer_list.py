"""Models described as an explicit list of layers: configuration, weights in kernel layout, random weights.

A layer is a mixer (one of the registered kinds below, with its own sizes) and optionally a feed-forward
(gated, or a mixture of gated experts), one after the other or side by side on one normed input; a contiguous range of layers may run several times in a row with the same weights, each
pass with a cache or state of its own. :class:`LayerListConfig` plays the part :class:`~..config.ModelConfig`
plays for the Llama family; :class:`LayerListWeights` that of ``RankWeights``. Designs map their
``config.json`` and tensor names onto these (``models/volarax.py``, ``models/zubedra.py``).

Kernel layout of the weights: every matrix ``[N, K]`` with both sizes padded with zeros to multiples of 8
(per head where a matrix is per head), projections of one input packed into one matrix, norm weights,
biases and other vectors in fp32. Padded rows produce zero columns and padded columns meet zero
activations, so no kernel needs to know about them.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

import torch

PREFILL_HEAD_DIM = 128        # head size of the tcgen05 prefill attention kernel
ATTN_HEAD_DIMS = (64, 128)    # head sizes of the tensor-core attention kernels over pages of keys and values
ATTN_MAX_GROUP = 16           # query heads per KV head that the decode kernel takes
WKV_CHUNK_DIM = 128           # largest head size of the chunked WKV kernels
MOE_MAX_EXPERTS, MOE_MAX_TOP = 1024, 32
LATENT_LDS = (64, 128, 192, 256, 384, 512)   # row sizes the tensor-core latent attention kernel is built for


def round8(n: int) -> int:
    return (n + 7) // 8 * 8


def _positive(where: str, **values) -> None:
    for name, v in values.items():
        if not v > 0:
            raise ValueError(f"{where}: {name} must be positive, not {v}")


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention over a cached low-rank latent per token. ``window`` None = no window."""
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: Optional[int] = None
    sink: bool = True
    kind = "latent_attention"

    def check(self, where: str) -> None:
        _positive(where, heads=self.heads, dim=self.dim, vdim=self.vdim, kv_rank=self.kv_rank)
        if self.window is not None:
            _positive(where, window=self.window)

    def matrix_params(self, w: int) -> int:
        return w * (self.heads * self.dim + self.kv_rank) + self.kv_rank * self.heads * (self.dim + self.vdim) + \
            self.heads * self.vdim * w


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention without positions: RMS norm over whole query and key rows, optionally capped scores
    and a sink per head. ``value_mix``: values are mixed with those of the first layer that has it set."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float] = None
    sink: bool = True
    value_mix: bool = False
    kind = "attention"

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads

    def check(self, where: str) -> None:
        _positive(where, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.softcap is not None:
            _positive(where, softcap=self.softcap)
        if self.heads % self.kv_heads:
            raise ValueError(f"{where}: {self.heads} query heads do not share {self.kv_heads} key/value heads evenly")

    def matrix_params(self, w: int) -> int:
        return w * (self.heads * (self.dim + self.vdim) + self.kv_heads * (self.dim + self.vdim))


@dataclass(frozen=True)
class MlstmSpec:
    """Matrix-memory recurrence with capped exponential input and sigmoid forget gates."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    kind = "mlstm"

    def check(self, where: str) -> None:
        _positive(where, heads=self.heads, dim=self.dim, vdim=self.vdim, gate_cap=self.gate_cap)

    def matrix_params(self, w: int) -> int:
        return w * self.heads * (2 * self.dim + 3 * self.vdim + 2)


@dataclass(frozen=True)
class WkvSpec:
    """Matrix-memory recurrence with a decay per key channel that depends on the token (through a low-rank
    projection) and a bonus for the current token; its inputs are mixes of a token with the one before."""
    heads: int
    dim: int
    rank: int
    kind = "wkv"

    @property
    def vdim(self) -> int:
        return self.dim

    def check(self, where: str) -> None:
        _positive(where, heads=self.heads, dim=self.dim, rank=self.rank)

    def matrix_params(self, w: int) -> int:
        return 5 * w * self.heads * self.dim + self.rank * (w + self.heads * self.dim)


@dataclass(frozen=True)
class ActSpec:
    """Activation of a gated feed-forward with its constants (those of "capped", see the GEMM epilogue)."""
    name: str
    limit: float = 0.0
    alpha: float = 1.0
    shift: float = 0.0


@dataclass(frozen=True)
class MlpSpec:
    ff: int
    act: ActSpec
    kind = "dense"

    def check(self, where: str) -> None:
        _positive(where, ff=self.ff)

    def matrix_params(self, w: int) -> int:
        return 3 * w * self.ff

    active_params = matrix_params


@dataclass(frozen=True)
class MoeSpec:
    """Mixture of gated experts: sigmoid scores, a correction added for the choice, experts in ``groups`` of which
    only the best ``keep`` can be chosen, the ``top`` chosen scores normed and times ``scale``. ``shared``: an
    expert that runs for every token, times a sigmoid gate of its own."""
    expert: MlpSpec
    experts: int
    top: int
    scale: float
    groups: int = 1
    keep: int = 1
    shared: Optional[MlpSpec] = None
    kind = "moe"

    def check(self, where: str) -> None:
        _positive(where, experts=self.experts, top=self.top, groups=self.groups, keep=self.keep)
        self.expert.check(where)
        if self.shared is not None:
            self.shared.check(where + " (shared expert)")
        if self.experts % self.groups or self.keep > self.groups:
            raise ValueError(f"{where}: {self.experts} experts do not form {self.groups} groups of which {self.keep} are kept")
        if self.top > self.keep * (self.experts // self.groups):
            raise ValueError(f"{where}: {self.top} experts per token cannot be chosen from {self.keep} groups")
        if self.experts > MOE_MAX_EXPERTS or self.top > MOE_MAX_TOP:
            raise ValueError(f"{where}: at most {MOE_MAX_EXPERTS} experts and {MOE_MAX_TOP} per token are built")

    @property
    def router_cols(self) -> int:
        return self.experts + (1 if self.shared is not None else 0)

    def matrix_params(self, w: int) -> int:
        return w * self.router_cols + self.experts * self.expert.matrix_params(w) + \
            (self.shared.matrix_params(w) if self.shared else 0)

    def active_params(self, w: int) -> int:
        return w * self.router_cols + self.top * self.expert.matrix_params(w) + \
            (self.shared.matrix_params(w) if self.shared else 0)


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any
    mlp: Any = None


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``step`` is the pass whose step vector joins the stream right before it."""
    layer: int
    step: Optional[int] = None


@dataclass
class LayerListConfig:
    name: str
    hidden_size: int
    vocab_size: int
    layers: List[LayerSpec]
    norm_kind: str = "layer"            # "layer" or "rms"
    norm_eps: float = 1e-5
    embed_norm: bool = True             # norm of the embedding row
    output_norms: bool = True           # norm of every sublayer's output before it joins the stream
    parallel: bool = False              # mixer and feed-forward read one normed input and join the stream together
    embed_scale: float = 1.0
    logit_scale: float = 1.0            # folded into the final norm's weight
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    eos_token_id: int = -1
    bos_token_id: int = -1
    dtype: torch.dtype = torch.bfloat16              # storage of weights, activations and caches
    tp: int = 1

    def __post_init__(self):
        _positive(self.name, hidden_size=self.hidden_size, vocab_size=self.vocab_size, layers=len(self.layers),
                  norm_eps=self.norm_eps)
        if self.tp != 1:
            raise ValueError("layer-list models run on one GPU (tensor parallelism is not built for them)")
        if self.norm_kind not in ("layer", "rms"):
            raise ValueError(f"unknown norm '{self.norm_kind}'")
        if self.loop is not None:
            start, stop, times = self.loop
            if not (0 <= start < stop <= len(self.layers)) or times < 1:
                raise ValueError(f"loop {self.loop} does not fit {len(self.layers)} layers")
        if self.parallel and self.output_norms:
            raise ValueError("norms of sublayer outputs are not built for parallel layers")
        for i, lay in enumerate(self.layers):
            lay.mixer.check(f"layer {i}")
            if lay.mlp is not None:
                lay.mlp.check(f"layer {i}")
                if lay.mlp.kind == "moe" and self.output_norms:
                    raise ValueError(f"layer {i}: norms of sublayer outputs are not built for a mixture of experts")
        mixed = {(l.mixer.kv_heads, l.mixer.vdim) for l in self.layers if getattr(l.mixer, "value_mix", False)}
        if len(mixed) > 1:
            raise ValueError(f"layers that mix values need the same key/value heads and value size, not {sorted(mixed)}")
        self.runs: List[LayerRun] = []
        for i in range(len(self.layers)):
            if self.loop is None or not self.loop[0] <= i < self.loop[1]:
                self.runs.append(LayerRun(i))
            elif i == self.loop[0]:
                for t in range(self.loop[2]):
                    self.runs += [LayerRun(j, t if j == i else None) for j in range(*self.loop[:2])]

    # ---- what the scheduler, the page pool and the benchmarks ask for --------------------------------
    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def run_layers(self) -> int:
        return len(self.runs)

    num_kv_heads = 1          # pages are counted in tokens, whatever a layer keeps per token
    group_size = 1

    @property
    def head_dim(self) -> int:
        return max([l.mixer.kv_rank for l in self.layers if l.mixer.kind == "latent_attention"] +
                   [max(l.mixer.dim, l.mixer.vdim) for l in self.layers if l.mixer.kind == "attention"], default=0)

    @property
    def width_p(self) -> int:
        return round8(self.hidden_size)

    @property
    def vocab_p(self) -> int:
        return round8(self.vocab_size)

    def run_specs(self, kind: str) -> List[Any]:
        return [self.layers[r.layer].mixer for r in self.runs if self.layers[r.layer].mixer.kind == kind]

    def run_moes(self) -> List[MoeSpec]:
        mlps = [self.layers[r.layer].mlp for r in self.runs]
        return [f for f in mlps if f is not None and f.kind == "moe"]

    @property
    def kv_window(self) -> int:
        """Positions back that any token sees at most (itself included); 0 = no bound."""
        specs = self.run_specs("latent_attention")
        if not specs or self.run_specs("attention") or any(s.window is None for s in specs):
            return 0
        return max(s.window for s in specs)

    @property
    def has_state(self) -> bool:
        return bool(self.run_specs("mlstm") or self.run_specs("wkv"))

    @property
    def first_value_run(self) -> int:
        """The run whose values later value-mixing layers read, -1 if there is none."""
        for r, run in enumerate(self.runs):
            if getattr(self.layers[run.layer].mixer, "value_mix", False):
                return r
        return -1

    @property
    def elem_bytes(self) -> int:
        return 4 if self.dtype == torch.float32 else 2

    def latent_ld(self, spec: LatentAttentionSpec) -> int:
        """Elements of one cached latent row."""
        if self.dtype == torch.bfloat16:
            for ld in LATENT_LDS:
                if spec.kv_rank <= ld:
                    return ld
        return round8(spec.kv_rank)

    def expands(self, spec: LatentAttentionSpec) -> bool:
        """Whether long prompt portions expand the latents into keys and values for the prefill kernel."""
        return self.dtype == torch.bfloat16 and max(spec.dim, spec.vdim) <= PREFILL_HEAD_DIM

    def head_pads(self, spec: LatentAttentionSpec) -> Tuple[int, int]:
        """Columns per head of queries and of attention outputs."""
        return (PREFILL_HEAD_DIM, PREFILL_HEAD_DIM) if self.expands(spec) else (round8(spec.dim), round8(spec.vdim))

    def attn_hd(self, spec: AttentionSpec) -> int:
        """Columns per head of queries, keys, values and outputs."""
        n = max(spec.dim, spec.vdim)
        if self.dtype == torch.bfloat16:
            for hd in ATTN_HEAD_DIMS:
                if n <= hd:
                    return hd
        return round8(n)

    def attn_on_tensor_cores(self, spec: AttentionSpec) -> bool:
        return self.dtype == torch.bfloat16 and self.attn_hd(spec) in ATTN_HEAD_DIMS and spec.group <= ATTN_MAX_GROUP

    def kv_bytes_per_token_local(self, dtype_bytes: int = 0) -> int:
        elems = sum(self.latent_ld(s) for s in self.run_specs("latent_attention")) + \
            sum(2 * s.kv_heads * self.attn_hd(s) for s in self.run_specs("attention"))
        return elems * (dtype_bytes or self.elem_bytes)

    def state_bytes_per_slot(self) -> int:
        n = 0
        for s in self.run_specs("wkv"):
            n += s.heads * round8(s.dim) ** 2 * 4 + 2 * self.width_p * self.elem_bytes
        for s in self.run_specs("mlstm"):
            d, v = round8(s.dim), round8(s.vdim)
            n += s.heads * (d * v + 2 * d + 2) * 4
        return n

    def param_count(self) -> int:
        w = self.hidden_size
        return sum(l.mixer.matrix_params(w) + (l.mlp.matrix_params(w) if l.mlp is not None else 0) for l in self.layers) + \
            2 * self.vocab_size * w

    def matmul_flops_per_token(self) -> float:
        w = self.hidden_size
        lays = [self.layers[r.layer] for r in self.runs]
        return 2.0 * sum(l.mixer.matrix_params(w) + (l.mlp.active_params(w) if l.mlp is not None else 0) for l in lays)


# --------------------------------------------------------------------------------------------------
# Weights
# --------------------------------------------------------------------------------------------------
@dataclass
class NormWeights:
    w: torch.Tensor                      # fp32, padded with zeros
    b: Optional[torch.Tensor] = None


@dataclass
class LatentAttentionWeights:
    w_in: torch.Tensor                   # queries (per head padded) | latent
    dkv_norm: torch.Tensor               # fp32 [kv_rank]
    w_qk: torch.Tensor                   # [heads * ld, dim_p]: query -> latent space, block per head
    w_ov: torch.Tensor                   # [heads * vdim_p, ld]: latent-space output -> values, block per head
    w_kv: Optional[torch.Tensor]         # [heads * 128 | heads * 128, ld]: latent -> keys | values of all heads
    w_o: torch.Tensor
    sinks: Optional[torch.Tensor]        # fp32 [heads]


@dataclass
class MlstmWeights:
    w_in: torch.Tensor                   # q | k | v | output gate | input and forget gates
    i_b: torch.Tensor
    f_b: torch.Tensor
    norm: torch.Tensor                   # fp32 [heads * vdim_p]
    w_o: torch.Tensor


@dataclass
class AttentionWeights:
    w_in: torch.Tensor                   # queries | keys | values, per head padded
    q_norm: torch.Tensor                 # fp32 [heads * hd]
    k_norm: torch.Tensor                 # fp32 [kv_heads * hd]
    w_o: torch.Tensor
    sinks: Optional[torch.Tensor]        # fp32 [heads]
    value_lambda: float


@dataclass
class WkvWeights:
    mu: torch.Tensor                     # fp32 [5, width_p]: r, k, v, g, decay
    w_in: torch.Tensor                   # r | k | v | g, each [heads * dim_p, width_p]
    w_down: torch.Tensor                 # [rank_p, width_p], then tanh
    w_up: torch.Tensor                   # [heads * dim_p, rank_p]
    w_bias: torch.Tensor                 # [heads * dim_p]
    u: torch.Tensor                      # fp32 [heads * dim_p]
    norm: torch.Tensor                   # fp32 [heads * dim_p]
    w_o: torch.Tensor


@dataclass
class MlpWeights:
    w_gate: torch.Tensor
    w_up: torch.Tensor
    w_down: torch.Tensor


@dataclass
class MoeWeights:
    router: torch.Tensor                 # experts | gate of the shared expert, rows padded to a multiple of 8
    correction: Optional[torch.Tensor]   # fp32 [experts]
    w_gate: torch.Tensor                 # [experts * ff_p, width_p]
    w_up: torch.Tensor
    w_down: torch.Tensor                 # [experts * width_p, ff_p]
    shared: Optional[MlpWeights]


@dataclass
class LayerListLayer:
    mixer: Any
    norm_in: NormWeights
    norm_out: Optional[NormWeights] = None
    mlp_in: Optional[NormWeights] = None         # not in parallel layers
    mlp_out: Optional[NormWeights] = None
    mlp: Any = None


@dataclass
class LayerListWeights:
    embed: torch.Tensor                  # [vocab, width_p]
    embed_norm: Optional[NormWeights]
    final_norm: NormWeights
    lm_head: torch.Tensor                # [vocab_p, width_p]
    layers: List[LayerListLayer] = field(default_factory=list)
    loop_steps: Optional[torch.Tensor] = None      # fp32 [times, width_p]
    rank: int = 0
    tp: int = 1

    def nbytes(self) -> int:
        total, stack = 0, [self]
        while stack:
            o = stack.pop()
            if isinstance(o, torch.Tensor):
                total += o.numel() * o.element_size()
            elif isinstance(o, list):
                stack += o
            elif hasattr(o, "__dataclass_fields__"):
                stack += [getattr(o, f) for f in o.__dataclass_fields__]
        return total


def pad_to(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """``t`` in the corner of a zero tensor of ``shape``."""
    if tuple(t.shape) == tuple(shape):
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def pad_heads(t: torch.Tensor, heads: int, dim: int, dim_p: int) -> torch.Tensor:
    """Rows grouped by head, each group padded from ``dim`` to ``dim_p`` rows."""
    return pad_to(t.reshape(heads, dim, *t.shape[1:]), heads, dim_p, *t.shape[1:]).reshape(heads * dim_p, *t.shape[1:])


def pack_latent_attention(cfg: LayerListConfig, spec: LatentAttentionSpec, q, dkv, dkv_norm, uk, uv, sink, o,
                          device) -> LatentAttentionWeights:
    """Plain matrices ([out, in], heads one after the other) -> kernel layout."""
    H, wp, ld = spec.heads, cfg.width_p, cfg.latent_ld(spec)
    dq, dv = cfg.head_pads(spec)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    w_in = torch.cat([pad_heads(q, H, spec.dim, dq), pad_to(dkv, round8(spec.kv_rank), dkv.shape[1])])
    qk = pad_to(uk.reshape(H, spec.dim, spec.kv_rank).transpose(1, 2), H, ld, dq).reshape(H * ld, dq)
    ov = pad_to(pad_heads(uv, H, spec.vdim, dv), H * dv, ld)
    kv = None
    if cfg.expands(spec):
        kv = mv(torch.cat([pad_to(pad_heads(uk, H, spec.dim, dq), H * dq, ld), ov]))
    w_o = pad_to(o.reshape(-1, H, spec.vdim), wp, H, dv).reshape(wp, H * dv)
    return LatentAttentionWeights(
        w_in=mv(pad_to(w_in, w_in.shape[0], wp)), dkv_norm=dkv_norm.to(device=device, dtype=torch.float32).contiguous(),
        w_qk=mv(qk), w_ov=mv(ov), w_kv=kv, w_o=mv(w_o),
        sinks=None if sink is None else sink.to(device=device, dtype=torch.float32).contiguous())


def pack_mlstm(cfg: LayerListConfig, spec: MlstmSpec, q, k, v, g, i, f, i_b, f_b, norm, o, device) -> MlstmWeights:
    H, wp, d, vd = spec.heads, cfg.width_p, round8(spec.dim), round8(spec.vdim)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    gates = torch.cat([i, f])
    w_in = torch.cat([pad_heads(q, H, spec.dim, d), pad_heads(k, H, spec.dim, d), pad_heads(v, H, spec.vdim, vd),
                      pad_heads(g, H, spec.vdim, vd), pad_to(gates, round8(2 * H), gates.shape[1])])
    w_o = pad_to(o.reshape(-1, H, spec.vdim), wp, H, vd).reshape(wp, H * vd)
    return MlstmWeights(w_in=mv(pad_to(w_in, w_in.shape[0], wp)), i_b=f32(i_b), f_b=f32(f_b),
                        norm=f32(pad_heads(norm, H, spec.vdim, vd)), w_o=mv(w_o))


def pack_attention(cfg: LayerListConfig, spec: AttentionSpec, q, k, v, q_norm, k_norm, sink, o, value_lambda: float,
                   device) -> AttentionWeights:
    H, G, wp, hd = spec.heads, spec.kv_heads, cfg.width_p, cfg.attn_hd(spec)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    w_in = torch.cat([pad_heads(q, H, spec.dim, hd), pad_heads(k, G, spec.dim, hd), pad_heads(v, G, spec.vdim, hd)])
    w_o = pad_to(o.reshape(-1, H, spec.vdim), wp, H, hd).reshape(wp, H * hd)
    return AttentionWeights(w_in=mv(pad_to(w_in, w_in.shape[0], wp)), q_norm=f32(pad_heads(q_norm, H, spec.dim, hd)),
                            k_norm=f32(pad_heads(k_norm, G, spec.dim, hd)), w_o=mv(w_o),
                            sinks=None if sink is None else f32(sink), value_lambda=float(value_lambda))


def pack_wkv(cfg: LayerListConfig, spec: WkvSpec, mu, r, k, v, g, w1, w2, w0, u, norm, o, device) -> WkvWeights:
    """``mu``: the five mixing vectors in the order r, k, v, g, decay."""
    H, wp, d, rp = spec.heads, cfg.width_p, round8(spec.dim), round8(spec.rank)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    heads = lambda t: pad_heads(t, H, spec.dim, d)
    w_in = torch.cat([heads(t) for t in (r, k, v, g)])
    w_o = pad_to(o.reshape(-1, H, spec.dim), wp, H, d).reshape(wp, H * d)
    return WkvWeights(mu=f32(torch.stack([pad_to(t, wp) for t in mu])), w_in=mv(pad_to(w_in, w_in.shape[0], wp)),
                      w_down=mv(pad_to(w1, rp, wp)), w_up=mv(pad_to(heads(w2), H * d, rp)), w_bias=mv(heads(w0)),
                      u=f32(heads(u.reshape(-1))), norm=f32(heads(norm)), w_o=mv(w_o))


def pack_mlp(cfg: LayerListConfig, ff: int, gate, up, down, device) -> MlpWeights:
    fp, wp = round8(ff), cfg.width_p
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    return MlpWeights(mv(pad_to(gate, fp, wp)), mv(pad_to(up, fp, wp)), mv(pad_to(down, wp, fp)))


def pack_moe(cfg: LayerListConfig, spec: MoeSpec, router, correction, expert, shared, shared_gate, device) -> MoeWeights:
    """``expert(e, part)``: a matrix of expert ``e`` (part "gate", "up" or "down"); ``shared``: the shared expert's three
    matrices, or None; ``shared_gate`` [1, width]."""
    fp, wp = round8(spec.expert.ff), cfg.width_p

    def stack(part, rows, cols):
        out = torch.zeros(spec.experts * rows, cols, dtype=cfg.dtype, device=device)
        for e in range(spec.experts):
            t = expert(e, part)
            out[e * rows:e * rows + t.shape[0], :t.shape[1]] = t.to(device=device, dtype=cfg.dtype)
        return out

    rows = [router] if spec.shared is None else [router, shared_gate]
    return MoeWeights(
        router=pad_to(torch.cat(rows), round8(spec.router_cols), wp).to(device=device, dtype=cfg.dtype).contiguous(),
        correction=None if correction is None else correction.to(device=device, dtype=torch.float32).contiguous(),
        w_gate=stack("gate", fp, wp), w_up=stack("up", fp, wp), w_down=stack("down", wp, fp),
        shared=None if spec.shared is None else pack_mlp(cfg, spec.shared.ff, *shared, device))


def pack_norm(cfg: LayerListConfig, w, b, device) -> NormWeights:
    f = lambda t: None if t is None else pad_to(t.to(device=device, dtype=torch.float32), cfg.width_p).contiguous()
    return NormWeights(f(w), f(b))
