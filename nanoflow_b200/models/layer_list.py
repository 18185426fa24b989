"""Models described as an explicit list of layers: configuration, weights in kernel layout, random weights.

A layer is a mixer (one of the registered kinds below, with its own sizes) and optionally a gated
feed-forward; a contiguous range of layers may run several times in a row with the same weights, each
pass with a cache or state of its own. :class:`LayerListConfig` plays the part :class:`~..config.ModelConfig`
plays for the Llama family; :class:`LayerListWeights` that of ``RankWeights``. Designs map their
``config.json`` and tensor names onto these (``models/volarax.py``).

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
LATENT_LDS = (64, 128, 192, 256, 384, 512)   # row sizes the tensor-core latent attention kernel is built for


def round8(n: int) -> int:
    return (n + 7) // 8 * 8


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


@dataclass(frozen=True)
class MlstmSpec:
    """Matrix-memory recurrence with capped exponential input and sigmoid forget gates."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    kind = "mlstm"


@dataclass(frozen=True)
class MlpSpec:
    ff: int
    act: str


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any
    mlp: Optional[MlpSpec] = None


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``step`` is the pass whose step vector joins the stream right before it."""
    layer: int
    step: Optional[int] = None


def _positive(where: str, **values) -> None:
    for name, v in values.items():
        if not v > 0:
            raise ValueError(f"{where}: {name} must be positive, not {v}")


@dataclass
class LayerListConfig:
    name: str
    hidden_size: int
    vocab_size: int
    layers: List[LayerSpec]
    norm_kind: str = "layer"            # "layer" (weight and bias) or "rms"
    norm_eps: float = 1e-5
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
        for i, lay in enumerate(self.layers):
            m = lay.mixer
            _positive(f"layer {i}", heads=m.heads, dim=m.dim, vdim=m.vdim)
            if m.kind == "latent_attention":
                _positive(f"layer {i}", kv_rank=m.kv_rank)
                if m.window is not None:
                    _positive(f"layer {i}", window=m.window)
            else:
                _positive(f"layer {i}", gate_cap=m.gate_cap)
            if lay.mlp is not None:
                _positive(f"layer {i}", ff=lay.mlp.ff)
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

    num_kv_heads = 1          # one latent row per token, whatever the number of query heads
    group_size = 1

    @property
    def head_dim(self) -> int:
        return max([l.mixer.kv_rank for l in self.layers if l.mixer.kind == "latent_attention"], default=0)

    @property
    def width_p(self) -> int:
        return round8(self.hidden_size)

    @property
    def vocab_p(self) -> int:
        return round8(self.vocab_size)

    def run_specs(self, kind: str) -> List[Any]:
        return [self.layers[r.layer].mixer for r in self.runs if self.layers[r.layer].mixer.kind == kind]

    @property
    def kv_window(self) -> int:
        """Positions back that any token sees at most (itself included); 0 = no bound."""
        specs = self.run_specs("latent_attention")
        if not specs or any(s.window is None for s in specs):
            return 0
        return max(s.window for s in specs)

    @property
    def has_state(self) -> bool:
        return bool(self.run_specs("mlstm"))

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

    def kv_bytes_per_token_local(self, dtype_bytes: int = 0) -> int:
        return sum(self.latent_ld(s) for s in self.run_specs("latent_attention")) * (dtype_bytes or self.elem_bytes)

    def state_bytes_per_slot(self) -> int:
        n = 0
        for s in self.run_specs("mlstm"):
            d, v = round8(s.dim), round8(s.vdim)
            n += s.heads * (d * v + 2 * d + 2) * 4
        return n

    def _matrix_params(self, lay: LayerSpec) -> int:
        w, m = self.hidden_size, lay.mixer
        if m.kind == "latent_attention":
            n = w * (m.heads * m.dim + m.kv_rank) + m.kv_rank * m.heads * (m.dim + m.vdim) + m.heads * m.vdim * w
        else:
            n = w * m.heads * (2 * m.dim + 3 * m.vdim + 2)
        return n + (3 * w * lay.mlp.ff if lay.mlp is not None else 0)

    def param_count(self) -> int:
        return sum(self._matrix_params(l) for l in self.layers) + 2 * self.vocab_size * self.hidden_size

    def matmul_flops_per_token(self) -> float:
        return 2.0 * sum(self._matrix_params(self.layers[r.layer]) for r in self.runs)


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
class LayerListLayer:
    mixer: Any
    norm_in: NormWeights
    norm_out: NormWeights
    mlp_in: Optional[NormWeights] = None
    mlp_out: Optional[NormWeights] = None
    w_gate: Optional[torch.Tensor] = None
    w_up: Optional[torch.Tensor] = None
    w_down: Optional[torch.Tensor] = None


@dataclass
class LayerListWeights:
    embed: torch.Tensor                  # [vocab, width_p]
    embed_norm: NormWeights
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


def pack_mlp(cfg: LayerListConfig, ff: int, gate, up, down, device):
    fp, wp = round8(ff), cfg.width_p
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    return mv(pad_to(gate, fp, wp)), mv(pad_to(up, fp, wp)), mv(pad_to(down, wp, fp))


def pack_norm(cfg: LayerListConfig, w, b, device) -> NormWeights:
    f = lambda t: None if t is None else pad_to(t.to(device=device, dtype=torch.float32), cfg.width_p).contiguous()
    return NormWeights(f(w), f(b))
