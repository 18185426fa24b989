"""Models described as an explicit list of layers: configuration, weights in kernel layout, random weights.

A layer is a mixer (one of the registered kinds below, with its own sizes, or two of them side by side) and optionally
a feed-forward (gated, or a mixture of experts), one after the other or side by side on one normed input; what a
sublayer reads may first pass a short convolution over time, and what goes on to the next layer may be a weighted sum of
all results so far. A contiguous range of layers may run several times in a row
with the same weights, each pass with a cache or state of its own. :class:`LayerListConfig` plays the part
:class:`~..config.ModelConfig` plays for the Llama family; :class:`LayerListWeights` that of ``RankWeights``. Designs map
their ``config.json`` and tensor names onto these (``models/volarax.py``, ``models/zubedra.py``, ``models/gupizen.py``,
``models/gimudra.py``).

Kernel layout of the weights: every matrix ``[N, K]`` with both sizes padded with zeros to multiples of 8
(per head where a matrix is per head), projections of one input packed into one matrix, norm weights,
biases and other vectors in fp32. Padded rows produce zero columns and padded columns meet zero
activations, so no kernel needs to know about them.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

import torch

PREFILL_HEAD_DIM = 128        # head size of the tcgen05 prefill attention kernel
ATTN_HEAD_DIMS = (64, 128)    # head sizes of the tensor-core attention kernels over pages of keys and values
ATTN_MAX_GROUP = 16           # query heads per KV head that the decode kernel takes
WKV_CHUNK_DIM = 128           # largest head size of the chunked WKV kernels
DELTA_CHUNK_DIM = 128         # ... and of the chunked delta-rule kernels
PAGE = 16                     # tokens per cache page
MOE_MAX_EXPERTS, MOE_MAX_TOP = 1024, 32
LINEAR_ACTS = ("gelu", "relu2")     # activations of products without a gate
CONV_MAX_TAPS = 8             # taps of the short convolution kernel
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
class RotaryScaling:
    """Rotations with a wavelength above ``original / low`` are slowed by ``factor``, those below ``original / high`` are
    kept, with a ramp in between (the scaling of Llama 3.1)."""
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first ``dims`` dimensions of queries and keys, neighbours 2i and 2i + 1 in a pair.
    ``values``: the values turn with their position too (all dimensions, unscaled), and every output turns back by the
    query's, so that it depends on distances only."""
    dims: int
    base: float
    scaling: Optional[RotaryScaling] = None
    values: bool = False

    def frequencies(self, n: int, scaled: bool) -> List[float]:
        """Radians per position of the n / 2 pairs."""
        out, s = [], self.scaling if scaled else None
        for i in range(n // 2):
            f = self.base ** (-2.0 * i / n)
            if s is not None:
                length = 2.0 * math.pi / f
                if length > s.original / s.low:
                    f /= s.factor
                elif length >= s.original / s.high:
                    ramp = (s.original / length - s.low) / (s.high - s.low)
                    f = (1.0 - ramp) * f / s.factor + ramp * f
            out.append(f)
        return out


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention, with options: RMS norm over whole query and key rows, rotary positions, a sliding window,
    capped scores, a sink per head. ``value_mix``: values are mixed with those of the first layer that has it set.
    ``talk``: the heads' softmax weights are mixed by a matrix before they meet the values. ``bias``: the projections of
    queries, keys and values have biases. ``distance_bias``: scores lose a ln(1 + b distance), two numbers per head.
    ``chunk``: positions see only those of their own run of so many. ``kv_from``: the layer whose cached keys and values
    are used instead of own ones."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float] = None
    sink: bool = True
    value_mix: bool = False
    qk_norm: bool = True
    rotary: Optional[RotarySpec] = None
    window: Optional[int] = None
    talk: bool = False
    bias: bool = False
    distance_bias: bool = False
    chunk: Optional[int] = None
    kv_from: Optional[int] = None
    kind = "attention"

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads

    def check(self, where: str) -> None:
        _positive(where, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.softcap is not None:
            _positive(where, softcap=self.softcap)
        if self.window is not None:
            _positive(where, window=self.window)
        if self.heads % self.kv_heads:
            raise ValueError(f"{where}: {self.heads} query heads do not share {self.kv_heads} key/value heads evenly")
        if self.rotary is not None:
            _positive(where, rotary_base=self.rotary.base)
            if self.rotary.dims < 0 or self.rotary.dims % 2 or self.rotary.dims > self.dim:
                raise ValueError(f"{where}: {self.rotary.dims} rotated dimensions do not fit heads of {self.dim}")
            if self.rotary.values and self.vdim % 2:
                raise ValueError(f"{where}: rotated values need an even size, not {self.vdim}")
            if self.rotary.scaling is not None:
                s = self.rotary.scaling
                _positive(where, factor=s.factor, low=s.low, original=s.original, high_over_low=s.high - s.low)
        if self.talk and (self.softcap is not None or self.value_mix):
            raise ValueError(f"{where}: capped scores and mixed values are not built for mixed heads")
        if self.chunk is not None:
            _positive(where, chunk=self.chunk)
        if self.distance_bias and self.softcap is not None:
            raise ValueError(f"{where}: capped scores with a distance bias are not built")
        if self.chunk is not None and self.window is not None:
            raise ValueError(f"{where}: chunks with a window are not built")
        if self.talk and (self.distance_bias or self.chunk is not None):
            raise ValueError(f"{where}: distance biases and chunks are not built for mixed heads")
        if self.kv_from is not None and (self.qk_norm or self.rotary is not None or self.value_mix or self.talk):
            raise ValueError(f"{where}: another layer's keys and values are not built with norms, rotations, mixed values or heads")

    def first_seen(self, position: int) -> int:
        """The first position that a token sees."""
        if self.window is not None:
            return max(0, position - self.window + 1)
        return position // self.chunk * self.chunk if self.chunk is not None else 0

    @property
    def proj_heads(self) -> int:
        """Heads that the input projection forms."""
        return self.heads + (2 * self.kv_heads if self.kv_from is None else 0)

    def matrix_params(self, w: int) -> int:
        own = self.kv_heads * (self.dim + self.vdim) if self.kv_from is None else 0
        return w * (self.heads * (self.dim + self.vdim) + own)


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
class RgLruSpec:
    """Real-gated linear recurrent unit (one number of state per channel) behind a short convolution, times a GELU branch;
    the gates are block-diagonal projections of the convolution's output."""
    width: int
    blocks: int
    conv: int
    kind = "rglru"

    @property
    def block_p(self) -> int:
        """Columns per block."""
        return round8(self.width // self.blocks)

    @property
    def cols(self) -> int:
        return self.blocks * self.block_p

    def check(self, where: str) -> None:
        _positive(where, width=self.width, blocks=self.blocks, conv=self.conv)
        if self.width % self.blocks:
            raise ValueError(f"{where}: a width of {self.width} does not form {self.blocks} blocks")
        if self.conv > CONV_MAX_TAPS:
            raise ValueError(f"{where}: at most {CONV_MAX_TAPS} taps are built, not {self.conv}")

    def matrix_params(self, w: int) -> int:
        return 3 * w * self.width + 2 * self.width * (self.width // self.blocks)


@dataclass(frozen=True)
class DeltaSpec:
    """Delta-rule recurrence: a matrix state per head with a decay per key channel and token, from which what the key
    recalls is replaced by the value; short convolutions on queries, keys and values. ``decay_rank``, ``gate_rank``: of
    the low-rank projections of decays and output gates."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int
    kind = "delta"

    @property
    def rank_p(self) -> int:
        return round8(max(self.decay_rank, self.gate_rank))

    def check(self, where: str) -> None:
        _positive(where, heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, conv=self.conv,
                  decay_rank=self.decay_rank, gate_rank=self.gate_rank)
        if self.heads % self.kv_heads:
            raise ValueError(f"{where}: {self.heads} heads do not share {self.kv_heads} query/key heads evenly")
        if self.conv > CONV_MAX_TAPS:
            raise ValueError(f"{where}: at most {CONV_MAX_TAPS} taps are built, not {self.conv}")

    def matrix_params(self, w: int) -> int:
        return w * (2 * self.kv_heads * self.dim + 2 * self.heads * self.vdim + self.heads + self.decay_rank + self.gate_rank) + \
            self.heads * (self.decay_rank * self.dim + self.gate_rank * self.vdim)


@dataclass(frozen=True)
class PairSpec:
    """An attention and a linear recurrent unit side by side on one input: half the sum of their RMS-normed outputs."""
    left: AttentionSpec
    right: RgLruSpec
    kind = "pair"

    def check(self, where: str) -> None:
        if self.left.kind != "attention" or self.right.kind != "rglru":
            raise ValueError(f"{where}: a pair of {self.left.kind} and {self.right.kind} is not built")
        if self.left.value_mix:
            raise ValueError(f"{where}: mixed values are not built inside a pair")
        self.left.check(where + " (left)")
        self.right.check(where + " (right)")

    def matrix_params(self, w: int) -> int:
        return self.left.matrix_params(w) + self.right.matrix_params(w)


def parts_of(spec) -> Tuple[Any, ...]:
    """The mixers a layer's mixer consists of."""
    return (spec.left, spec.right) if spec.kind == "pair" else (spec,)


@dataclass(frozen=True)
class ActSpec:
    """Activation of a feed-forward with its constants (those of "capped", see the GEMM epilogue)."""
    name: str
    limit: float = 0.0
    alpha: float = 1.0
    shift: float = 0.0


@dataclass(frozen=True)
class MlpSpec:
    """``gated``: act(gate) * up; else act(up). ``bias``: all projections have biases."""
    ff: int
    act: ActSpec
    gated: bool = True
    bias: bool = False
    kind = "dense"

    def check(self, where: str) -> None:
        _positive(where, ff=self.ff)

    def matrix_params(self, w: int) -> int:
        return (3 if self.gated else 2) * w * self.ff

    active_params = matrix_params


@dataclass(frozen=True)
class MoeSpec:
    """Mixture of experts, of which a token uses ``top``. ``score`` "sigmoid": sigmoid scores, a correction added for the
    choice, the chosen scores normed and times ``scale``; "softmax": softmax over the chosen logits times ``scale``;
    "softmax_all": softmax over all logits, a correction added for the choice, the chosen scores times ``scale``.
    Experts in ``groups`` of which only the best ``keep`` can be chosen; a group counts by its two largest choice scores or
    (``group_score`` "max") its largest. ``shared``: an expert that runs for every token, times a sigmoid gate of its own.
    ``identity``: so many router outputs behind the experts' stand for the input itself."""
    expert: MlpSpec
    experts: int
    top: int
    scale: float
    groups: int = 1
    keep: int = 1
    shared: Optional[MlpSpec] = None
    score: str = "sigmoid"
    identity: int = 0
    group_score: str = "top2"
    kind = "moe"

    @property
    def outputs(self) -> int:
        """Experts to choose from, those that only hand on the input included."""
        return self.experts + self.identity

    def check(self, where: str) -> None:
        _positive(where, experts=self.experts, top=self.top, groups=self.groups, keep=self.keep)
        self.expert.check(where)
        if self.shared is not None:
            self.shared.check(where + " (shared expert)")
        if self.identity < 0 or (self.identity and self.shared is not None):
            raise ValueError(f"{where}: identity experts beside a shared expert are not built")
        if self.group_score not in ("top2", "max"):
            raise ValueError(f"{where}: unknown group score '{self.group_score}'")
        if self.expert.bias or (self.shared is not None and self.shared.bias):
            raise ValueError(f"{where}: experts with biases are not built")
        if self.outputs % self.groups or self.keep > self.groups:
            raise ValueError(f"{where}: {self.outputs} experts do not form {self.groups} groups of which {self.keep} are kept")
        if self.top > self.keep * (self.outputs // self.groups):
            raise ValueError(f"{where}: {self.top} experts per token cannot be chosen from {self.keep} groups")
        if self.score not in ("sigmoid", "softmax", "softmax_all"):
            raise ValueError(f"{where}: unknown router score '{self.score}'")
        if self.expert.gated == (self.expert.act.name in LINEAR_ACTS):
            raise ValueError(f"{where}: activation '{self.expert.act.name}' is not built for this kind of expert")
        if self.shared is not None and not self.shared.gated:
            raise ValueError(f"{where}: a shared expert without a gate product is not built")
        if self.outputs > MOE_MAX_EXPERTS or self.top > MOE_MAX_TOP:
            raise ValueError(f"{where}: at most {MOE_MAX_EXPERTS} experts and {MOE_MAX_TOP} per token are built")

    @property
    def router_cols(self) -> int:
        return self.outputs + (1 if self.shared is not None else 0)

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
    """One execution of a layer: ``step`` is the pass whose step vector (or the embedding output, see ``loop_add``) joins
    the stream right before it."""
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
    input_conv: int = 0                 # taps of the convolution over time that a sublayer's input passes (0: none)
    input_conv_mlp: bool = True         # ... a feed-forward's too
    sinusoid: float = 0.0               # base of the sinusoidal position vector that joins the embedding row (0: none)
    layer_scale: bool = False           # every sublayer's output is scaled per column before it joins the stream
    depth_average: bool = False         # a weighted sum of the embedding output and all layers' results goes on
    tied_head: bool = False             # the embedding table is the output matrix
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    loop_add: str = "steps"             # what joins the stream ahead of a pass: a vector per pass, or "embedding": what the
                                        # layers started from, ahead of every pass but the first
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
        if self.loop_add not in ("steps", "embedding"):
            raise ValueError(f"unknown loop addition '{self.loop_add}'")
        if self.loop_add == "embedding" and self.embed_norm and self.loop is not None:
            raise ValueError("a normed embedding output that joins every pass of a loop is not built")
        if not 0 <= self.input_conv <= CONV_MAX_TAPS:
            raise ValueError(f"at most {CONV_MAX_TAPS} taps of the input convolution are built, not {self.input_conv}")
        if self.input_conv and self.parallel:
            raise ValueError("input convolutions are not built for parallel layers")
        if self.layer_scale and (self.parallel or self.output_norms):
            raise ValueError("scaled sublayer outputs are not built for parallel layers or normed outputs")
        if self.depth_average and self.loop is not None:
            raise ValueError("averages over depth are not built for loops")
        if self.sinusoid and (self.sinusoid < 0 or self.embed_norm or (self.loop is not None and self.loop_add == "embedding")):
            raise ValueError("position vectors need a positive base, and are not built with normed or repeated embeddings")
        for i, lay in enumerate(self.layers):
            lay.mixer.check(f"layer {i}")
            if lay.mixer.kind == "pair" and (self.parallel or not self.output_norms or self.norm_kind != "rms"):
                raise ValueError(f"layer {i}: mixers side by side need RMS norms of sublayer outputs")
            if lay.mlp is not None:
                lay.mlp.check(f"layer {i}")
            src = getattr(lay.mixer, "kv_from", None)
            if src is not None:
                s = self.layers[src].mixer if 0 <= src < i else None
                if s is None or s.kind != "attention" or s.kv_from is not None:
                    raise ValueError(f"layer {i}: layer {src} has no keys and values to lend")
                if (s.kv_heads, s.dim, s.vdim) != (lay.mixer.kv_heads, lay.mixer.dim, lay.mixer.vdim):
                    raise ValueError(f"layer {i}: the keys and values of layer {src} have other sizes")
                if self.loop is not None:
                    raise ValueError(f"layer {i}: lent keys and values are not built for loops")
        mixed = {(l.mixer.kv_heads, l.mixer.vdim) for l in self.layers if getattr(l.mixer, "value_mix", False)}
        if len(mixed) > 1:
            raise ValueError(f"layers that mix values need the same key/value heads and value size, not {sorted(mixed)}")
        self.runs: List[LayerRun] = []
        for i in range(len(self.layers)):
            if self.loop is None or not self.loop[0] <= i < self.loop[1]:
                self.runs.append(LayerRun(i))
            elif i == self.loop[0]:
                for t in range(self.loop[2]):
                    joins = self.loop_add == "steps" or t > 0
                    self.runs += [LayerRun(j, t if j == i and joins else None) for j in range(*self.loop[:2])]

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
        mixers = [s for l in self.layers for s in parts_of(l.mixer)]
        return max([s.kv_rank for s in mixers if s.kind == "latent_attention"] +
                   [max(s.dim, s.vdim) for s in mixers if s.kind == "attention"], default=0)

    @property
    def width_p(self) -> int:
        return round8(self.hidden_size)

    @property
    def vocab_p(self) -> int:
        return round8(self.vocab_size)

    def run_specs(self, kind: str) -> List[Any]:
        return [s for r in self.runs for s in parts_of(self.layers[r.layer].mixer) if s.kind == kind]

    def run_moes(self) -> List[MoeSpec]:
        mlps = [self.layers[r.layer].mlp for r in self.runs]
        return [f for f in mlps if f is not None and f.kind == "moe"]

    @property
    def kv_window(self) -> int:
        """Positions back that any token sees at most (itself included); 0 = no bound."""
        specs = self.run_specs("latent_attention") + self.run_specs("attention")
        if not specs or any(s.window is None for s in specs):
            return 0
        return max(s.window for s in specs)

    def first_seen(self, position: int) -> int:
        """The first position that any layer sees from ``position``; tokens after it see none before."""
        latent, attn = self.run_specs("latent_attention"), self.run_specs("attention")
        firsts = [0 if s.window is None else max(0, position - s.window + 1) for s in latent] + [s.first_seen(position) for s in attn]
        return min(firsts, default=0)

    @property
    def has_state(self) -> bool:
        return any(self.run_specs(kind) for kind in ("mlstm", "wkv", "rglru", "delta")) or self.input_conv > 1

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
        return self.dtype == torch.bfloat16 and self.attn_hd(spec) in ATTN_HEAD_DIMS and spec.group <= ATTN_MAX_GROUP and \
            spec.window is None and not spec.talk and spec.rotary is None

    def kv_bytes_per_token_local(self, dtype_bytes: int = 0) -> int:
        elems = sum(self.latent_ld(s) for s in self.run_specs("latent_attention")) + \
            sum(2 * s.kv_heads * self.attn_hd(s) for s in self.run_specs("attention") if s.kv_from is None)
        return elems * (dtype_bytes or self.elem_bytes)

    def pool_shape(self, spec) -> Optional[Tuple[int, ...]]:
        """Shape of one page of a mixer's cache (None: it keeps none)."""
        if spec.kind == "latent_attention":
            return (PAGE, self.latent_ld(spec))
        own = spec.kind == "attention" and spec.kv_from is None
        return (2, spec.kv_heads, PAGE, self.attn_hd(spec)) if own else None

    def state_shapes(self, spec) -> List[Tuple[Tuple[int, ...], torch.dtype]]:
        """What a request keeps of a recurrent mixer, as (shape, type) without the leading slots. Small vectors come in two
        halves, of which a step reads one and writes the other (see ``DistKVCache.state_ref``)."""
        f32 = torch.float32
        if spec.kind == "mlstm":
            d, v = round8(spec.dim), round8(spec.vdim)
            return [((spec.heads, d, v), f32), ((spec.heads, 2, d), f32), ((spec.heads, 2), f32)]
        if spec.kind == "wkv":
            d = round8(spec.dim)
            return [((spec.heads, d, d), f32), ((2, self.width_p), self.dtype)]
        if spec.kind == "rglru":
            return [((spec.cols,), f32), ((2, max(1, spec.conv - 1), spec.cols), self.dtype)]
        if spec.kind == "delta":
            d, v = round8(spec.dim), round8(spec.vdim)
            return [((spec.heads, d, v), f32),
                    ((2, max(1, spec.conv - 1), 2 * spec.kv_heads * d + spec.heads * v), self.dtype)]
        return []

    def conv_state_shape(self) -> Tuple[int, ...]:
        """The last inputs of a sublayer's input convolution, in two halves."""
        return (2, max(1, self.input_conv - 1), self.width_p)

    def conv_mlp(self, layer: LayerSpec) -> bool:
        """Whether a layer's feed-forward reads through an input convolution."""
        return bool(self.input_conv) and self.input_conv_mlp and layer.mlp is not None

    def state_bytes_per_slot(self) -> int:
        n = 0
        for r in self.runs:
            lay = self.layers[r.layer]
            for s in parts_of(lay.mixer):
                n += sum(math.prod(shape) * (4 if dt == torch.float32 else 2) for shape, dt in self.state_shapes(s))
            if self.input_conv:
                n += (2 if self.conv_mlp(lay) else 1) * math.prod(self.conv_state_shape()) * self.elem_bytes
        return n

    def param_count(self) -> int:
        w = self.hidden_size
        return sum(l.mixer.matrix_params(w) + (l.mlp.matrix_params(w) if l.mlp is not None else 0) for l in self.layers) + \
            (1 if self.tied_head else 2) * self.vocab_size * w

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
    kind: Optional[str] = None           # other than the model's: "scale" only multiplies by the weights


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
    w_in: torch.Tensor                   # queries | keys | values, per head padded (queries only with lent keys and values)
    q_norm: Optional[torch.Tensor]       # fp32 [heads * hd]
    k_norm: Optional[torch.Tensor]       # fp32 [kv_heads * hd]
    w_o: torch.Tensor
    sinks: Optional[torch.Tensor]        # fp32 [heads]
    value_lambda: float
    talk: Optional[torch.Tensor] = None  # fp32 [heads, heads]
    b_in: Optional[torch.Tensor] = None  # bias of w_in
    dist: Optional[torch.Tensor] = None  # fp32 [heads, 2]: factor and rate of the distance bias


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
class RgLruWeights:
    w_in: torch.Tensor                   # GELU branch | convolved branch, [2 cols, width_p]
    b_in: torch.Tensor                   # [2 cols]
    conv: torch.Tensor                   # fp32 [taps, cols]
    conv_b: torch.Tensor                 # fp32 [cols]
    w_gates: torch.Tensor                # per block: recurrence gate | input gate, [blocks * 2 block_p, block_p]
    r_b: torch.Tensor                    # fp32 [cols]
    i_b: torch.Tensor                    # fp32 [cols]
    log_a: torch.Tensor                  # fp32 [cols]: log of the decay at a recurrence gate of one
    w_o: torch.Tensor


@dataclass
class DeltaWeights:
    w_in: torch.Tensor                   # q | k | v | decay down | gate down | beta
    conv: torch.Tensor                   # fp32 [taps, q | k | v]
    w_decay: torch.Tensor                # [heads * dim_p, rank_p]
    w_gate: torch.Tensor                 # [heads * vdim_p, rank_p]
    dt_bias: torch.Tensor                # fp32 [heads * dim_p]
    rate: torch.Tensor                   # fp32 [heads]: exp(A_log)
    norm: torch.Tensor                   # fp32 [vdim_p]
    w_o: torch.Tensor


@dataclass
class PairWeights:
    w_in: torch.Tensor                   # input projections of both mixers
    b_in: torch.Tensor
    left: Any
    right: Any
    left_norm: torch.Tensor              # fp32 [width_p]
    right_norm: torch.Tensor


@dataclass
class MlpWeights:
    w_gate: torch.Tensor
    w_up: torch.Tensor
    w_down: torch.Tensor
    b_gate: Optional[torch.Tensor] = None
    b_up: Optional[torch.Tensor] = None
    b_down: Optional[torch.Tensor] = None


@dataclass
class MoeWeights:
    router: torch.Tensor                 # experts | identity experts | gate of the shared expert, rows padded to a multiple of 8
    correction: Optional[torch.Tensor]   # fp32 [experts | identity experts]: added for the choice, or to the logits of a softmax router
    w_gate: Optional[torch.Tensor]       # [experts * ff_p, width_p], None in experts without a gate product
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
    conv_in: Optional[torch.Tensor] = None       # fp32 [taps, width_p]: input convolutions of the two sublayers
    conv_mlp: Optional[torch.Tensor] = None
    depth: Optional[torch.Tensor] = None         # fp32: weights of the embedding output and all results up to this layer's


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
        total, stack, seen = 0, [self], set()
        while stack:
            o = stack.pop()
            if isinstance(o, torch.Tensor):
                if o.untyped_storage().data_ptr() not in seen:       # parts of one matrix, tied tables
                    seen.add(o.untyped_storage().data_ptr())
                    total += o.untyped_storage().nbytes()
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
                   device, talk=None, biases=None, dist=None) -> AttentionWeights:
    """``k``, ``v`` None: lent by another layer. ``biases``: of queries, keys and values; ``dist`` [heads, 2]."""
    H, G, wp, hd = spec.heads, spec.kv_heads, cfg.width_p, cfg.attn_hd(spec)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    def rows(q, k, v):
        parts = [pad_heads(q, H, spec.dim, hd)]
        return torch.cat(parts if k is None else parts + [pad_heads(k, G, spec.dim, hd), pad_heads(v, G, spec.vdim, hd)])

    w_in = rows(q, k, v)
    w_o = pad_to(o.reshape(-1, H, spec.vdim), wp, H, hd).reshape(wp, H * hd)
    return AttentionWeights(w_in=mv(pad_to(w_in, w_in.shape[0], wp)),
                            q_norm=None if q_norm is None else f32(pad_heads(q_norm, H, spec.dim, hd)),
                            k_norm=None if k_norm is None else f32(pad_heads(k_norm, G, spec.dim, hd)), w_o=mv(w_o),
                            sinks=None if sink is None else f32(sink), value_lambda=float(value_lambda),
                            talk=None if talk is None else f32(talk), b_in=None if biases is None else mv(rows(*biases)),
                            dist=None if dist is None else f32(dist))


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


def pack_conv(cfg: LayerListConfig, w, cols: int, device) -> torch.Tensor:
    """[channels, taps] -> fp32 [taps, cols]."""
    return pad_to(w.to(device=device, dtype=torch.float32).t(), w.shape[1], cols).contiguous()


def pack_rglru(cfg: LayerListConfig, spec: RgLruSpec, y, y_b, x, x_b, conv, conv_b, ra, ra_b, ri, ri_b, lam, o,
               device) -> RgLruWeights:
    """``lam``: the recurrence decays by exp(-8 softplus(lam)) per token at a gate of one."""
    n, b, bp, wp = spec.blocks, spec.width // spec.blocks, spec.block_p, cfg.width_p
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    ch = lambda t: pad_heads(t, n, b, bp)
    w_in = torch.cat([ch(y), ch(x)])
    gates = torch.cat([pad_to(ra, n, bp, bp), pad_to(ri, n, bp, bp)], dim=1).reshape(n * 2 * bp, bp)
    w_o = pad_to(o.reshape(-1, n, b), wp, n, bp).reshape(wp, n * bp)
    log_a = -8.0 * torch.nn.functional.softplus(lam.double())
    return RgLruWeights(w_in=mv(pad_to(w_in, w_in.shape[0], wp)), b_in=mv(torch.cat([ch(y_b), ch(x_b)])),
                        conv=pack_conv(cfg, ch(conv), spec.cols, device), conv_b=f32(ch(conv_b)), w_gates=mv(gates),
                        r_b=f32(ch(ra_b.reshape(-1))), i_b=f32(ch(ri_b.reshape(-1))), log_a=f32(ch(log_a)), w_o=mv(w_o))


def pack_delta(cfg: LayerListConfig, spec: DeltaSpec, q, k, v, q_conv, k_conv, v_conv, beta, a_log, a1, a2, dt_bias, g1, g2,
               norm, o, device) -> DeltaWeights:
    H, G, wp, d, vd, rp = spec.heads, spec.kv_heads, cfg.width_p, round8(spec.dim), round8(spec.vdim), spec.rank_p
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
    qk, vh = (lambda t: pad_heads(t, G, spec.dim, d)), (lambda t: pad_heads(t, H, spec.vdim, vd))
    w_in = torch.cat([qk(q), qk(k), vh(v), pad_to(a1, rp, a1.shape[1]), pad_to(g1, rp, g1.shape[1]),
                      pad_to(beta, round8(H), beta.shape[1])])
    conv = torch.cat([qk(q_conv), qk(k_conv), vh(v_conv)])
    w_o = pad_to(o.reshape(-1, H, spec.vdim), wp, H, vd).reshape(wp, H * vd)
    return DeltaWeights(w_in=mv(pad_to(w_in, w_in.shape[0], wp)), conv=pack_conv(cfg, conv, conv.shape[0], device),
                        w_decay=mv(pad_to(pad_heads(a2, H, spec.dim, d), H * d, rp)),
                        w_gate=mv(pad_to(vh(g2), H * vd, rp)), dt_bias=f32(pad_heads(dt_bias, H, spec.dim, d)),
                        rate=f32(torch.exp(a_log.double())), norm=f32(pad_to(norm, vd)), w_o=mv(w_o))


def pack_pair(cfg: LayerListConfig, spec: PairSpec, left: AttentionWeights, right: RgLruWeights, left_norm, right_norm,
              device) -> PairWeights:
    """One matrix for both mixers' input projections, of which theirs become parts."""
    w_in, n = torch.cat([left.w_in, right.w_in]), left.w_in.shape[0]
    b_in = torch.cat([torch.zeros(n, dtype=right.b_in.dtype, device=right.b_in.device), right.b_in])
    left.w_in, right.w_in, right.b_in = w_in[:n], w_in[n:], b_in[n:]
    f32 = lambda t: pad_to(t.to(device=device, dtype=torch.float32), cfg.width_p).contiguous()
    return PairWeights(w_in=w_in, b_in=b_in, left=left, right=right, left_norm=f32(left_norm), right_norm=f32(right_norm))


def pack_mlp(cfg: LayerListConfig, ff: int, gate, up, down, device, biases=None) -> MlpWeights:
    """``biases``: of the three products."""
    fp, wp = round8(ff), cfg.width_p
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    b = [None] * 3 if biases is None else [mv(pad_to(t, n)) for t, n in zip(biases, (fp, fp, wp))]
    return MlpWeights(mv(pad_to(gate, fp, wp)), mv(pad_to(up, fp, wp)), mv(pad_to(down, wp, fp)), *b)


def pack_moe(cfg: LayerListConfig, spec: MoeSpec, router, correction, expert, shared, shared_gate, device) -> MoeWeights:
    """``expert(e, part)``: a matrix of expert ``e`` (part "gate" if it has one, "up" or "down"); ``shared``: the shared expert's three
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
        w_gate=stack("gate", fp, wp) if spec.expert.gated else None, w_up=stack("up", fp, wp), w_down=stack("down", wp, fp),
        shared=None if spec.shared is None else pack_mlp(cfg, spec.shared.ff, *shared, device))


def pack_norm(cfg: LayerListConfig, w, b, device, kind: Optional[str] = None) -> NormWeights:
    f = lambda t: None if t is None else pad_to(t.to(device=device, dtype=torch.float32), cfg.width_p).contiguous()
    return NormWeights(f(w), f(b), kind)
