"""Gupizen: a small decoder that mixes two kinds of layers: windowed rotary attention with rotated values, sinks and mixed
heads beside a real-gated linear recurrent unit, and delta-rule recurrences with a decay per channel. A looped range of
layers starts every pass but the first from the embeddings again, every sublayer reads its input through a short
convolution, and the feed-forwards are mixtures of experts without gates.

Only what is particular to the design is here: its ``config.json`` keys, its tensor names, the choices it
makes among the mechanisms of :mod:`.layer_list`, and random weights of its shape. Engine, caches and
kernels are those of every layer-list model (``runtime/layer_list.py``).
"""
from __future__ import annotations

import copy
import json
import os
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch

from .layer_list import (ActSpec, AttentionSpec, DeltaSpec, LayerListConfig, LayerListLayer, LayerListWeights, LayerSpec, MlpSpec,
                         MoeSpec, PairSpec, RgLruSpec, RotaryScaling, RotarySpec, pack_attention, pack_conv, pack_delta, pack_moe,
                         pack_norm, pack_pair, pack_rglru, pad_to)
from .safetensors_io import read_safetensors, read_shapes

ARCHITECTURE = "Gupizen"
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def _rotary(r: Dict[str, Any]) -> RotarySpec:
    s = r.get("scaling")
    scaling = None if not s else RotaryScaling(float(s["factor"]), float(s["low"]), float(s["high"]), float(s["original"]))
    return RotarySpec(int(r["dims"]), float(r["base"]), scaling, values=True)


def _mixer(kind: str, m: Dict[str, Any], where: str):
    if kind == "parallel":
        a, b, mask = m["left"], m["right"], m["left"].get("mask")
        return PairSpec(
            AttentionSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                          scale=float(a["scale"]), qk_norm=False, rotary=_rotary(a["rot"]),
                          window=None if mask is None else int(mask["size"]), talk=True),
            RgLruSpec(width=int(b["width"]), blocks=int(b["blocks"]), conv=int(b["conv"])))
    if kind == "channel_delta":
        if "decay_rank" not in m or "gate_rank" not in m:
            raise ValueError(f"{where}: the ranks of the decay and gate projections are missing ('decay_rank', 'gate_rank'; a "
                             "model folder's tensors say them)")
        return DeltaSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         conv=int(m["conv"]), decay_rank=int(m["decay_rank"]), gate_rank=int(m["gate_rank"]))
    raise ValueError(f"{where}: unknown layer type '{kind}'")


def _mlp(f: Optional[Dict[str, Any]], where: str) -> Optional[MoeSpec]:
    if f is None:
        return None
    if f.get("kind", "moe") != "moe":
        raise ValueError(f"{where}: unknown feed-forward '{f['kind']}'")
    r = f["router"]
    return MoeSpec(expert=MlpSpec(int(f["expert"]["ff"]), ActSpec("gelu"), gated=False), experts=int(r["experts"]),
                   top=int(r["top"]), scale=1.0, score="softmax")


def complete(raw: Dict[str, Any], folder: str) -> Dict[str, Any]:
    """``config.json`` with the sizes that only the checkpoint's tensors give."""
    raw = copy.deepcopy(raw)
    shapes = read_shapes(os.path.join(folder, "model.safetensors"))
    for i, lay in enumerate(raw["layers"]):
        if lay["type"] == "channel_delta":
            for key, part in (("decay_rank", "a1"), ("gate_rank", "g1")):
                name = f"l{i}.mix.{part}"
                if name not in shapes:
                    raise KeyError(f"{folder}: tensor '{name}' is missing")
                lay["mixer"][key] = int(shapes[name][0])
    return raw


def parse_model(raw: Dict[str, Any], *, tp: int = 1, run_layers: int = 0, name: str = "") -> LayerListConfig:
    """``config.json`` -> :class:`LayerListConfig`. ``dtype`` ("bfloat16" / "float32") and the mixers' ``decay_rank`` and
    ``gate_rank`` are this framework's own keys."""
    layers: List[LayerSpec] = [LayerSpec(_mixer(lay["type"], lay["mixer"], f"layer {i}"), _mlp(lay.get("mlp"), f"layer {i}"))
                               for i, lay in enumerate(raw["layers"])]
    loop = raw.get("loop")
    cfg = LayerListConfig(
        name=name or ARCHITECTURE, hidden_size=int(raw["width"]), vocab_size=int(raw["vocab"]), layers=layers,
        norm_kind="rms", norm_eps=float(raw["norm"]["eps"]), embed_norm=False, output_norms=True,
        embed_scale=float(raw["embedding"]["scale"]), input_conv=int(raw["canon"]["taps"]), tied_head=True,
        loop=None if not loop else (int(loop["start"]), int(loop["stop"]), int(loop["times"])), loop_add="embedding",
        eos_token_id=int(raw.get("eos_token_id", -1)), bos_token_id=int(raw.get("bos_token_id", -1)),
        dtype=DTYPES[raw.get("dtype", "bfloat16")], tp=tp)
    if run_layers not in (0, cfg.run_layers, cfg.num_layers):
        raise ValueError("run_layer cannot be changed for a model whose layers are listed")
    return cfg


def tensor_shapes(raw: Dict[str, Any]) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of the checkpoint's tensors."""
    W, V, taps = int(raw["width"]), int(raw["vocab"]), int(raw["canon"]["taps"])
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "final.norm": (W,)}
    for i, lay in enumerate(raw["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,), p + "canon1": (W, taps)})
        if lay["type"] == "parallel":
            a, b, q = m["left"], m["right"], p + "mix.left."
            H, G, d, v = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            out.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * v, W), q + "talk": (H, H), q + "sink": (H,),
                        q + "o": (W, H * v), q + "out": (W,)})
            q, R, n = p + "mix.right.", b["width"], b["blocks"]
            out.update({q + "y": (R, W), q + "y.b": (R,), q + "x": (R, W), q + "x.b": (R,), q + "conv": (R, b["conv"]),
                        q + "conv.b": (R,), q + "lam": (R,), q + "o": (W, R), q + "out": (W,)})
            for gate in ("ra", "ri"):
                out.update({q + gate: (n, R // n, R // n), f"{q}{gate}.b": (n, R // n)})
        else:
            q, H, G, d, v, c = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for s, rows in (("q", G * d), ("k", G * d), ("v", H * v)):
                out.update({q + s: (rows, W), f"{q}{s}.conv": (rows, c)})
            out.update({q + "b": (H, W), q + "A_log": (H,), q + "norm": (v,), q + "a1": (m["decay_rank"], W),
                        q + "a2": (H * d, m["decay_rank"]), q + "dt_bias": (H * d,), q + "g1": (m["gate_rank"], W),
                        q + "g2": (H * v, m["gate_rank"]), q + "o": (W, H * v)})
        f = lay.get("mlp")
        if f is not None:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "canon2": (W, taps), p + "mlp.router": (E, W),
                        p + "mlp.router.b": (E,)})
            for e in range(E):
                out.update({f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
    return out


def weights_from_tensors(cfg: LayerListConfig, get: Callable[[str], torch.Tensor], device="cpu") -> LayerListWeights:
    """Checkpoint tensors by name -> kernel layout on ``device``."""
    norm = lambda n: pack_norm(cfg, 1.0 + get(n).float(), None, device)        # stored as the distance from one
    conv = lambda n: pack_conv(cfg, get(n), cfg.width_p, device)
    embed = pad_to(get("embed"), cfg.vocab_p, cfg.width_p).to(device=device, dtype=cfg.dtype).contiguous()
    w = LayerListWeights(embed=embed, embed_norm=None, final_norm=norm("final.norm"), lm_head=embed)
    for i, lay in enumerate(cfg.layers):
        if lay.mixer.kind == "pair":
            a, b = (lambda n: get(f"l{i}.mix.left.{n}")), (lambda n: get(f"l{i}.mix.right.{n}"))
            left = pack_attention(cfg, lay.mixer.left, a("q"), a("k"), a("v"), None, None, a("sink"), a("o"), 0.0, device, a("talk"))
            right = pack_rglru(cfg, lay.mixer.right, b("y"), b("y.b"), b("x"), b("x.b"), b("conv"), b("conv.b"), b("ra"),
                               b("ra.b"), b("ri"), b("ri.b"), b("lam"), b("o"), device)
            mix = pack_pair(cfg, lay.mixer, left, right, a("out"), b("out"), device)
        else:
            g = lambda n: get(f"l{i}.mix.{n}")
            mix = pack_delta(cfg, lay.mixer, g("q"), g("k"), g("v"), g("q.conv"), g("k.conv"), g("v.conv"), g("b"), g("A_log"),
                             g("a1"), g("a2"), g("dt_bias"), g("g1"), g("g2"), g("norm"), g("o"), device)
        out = LayerListLayer(mixer=mix, norm_in=norm(f"l{i}.norm1"), norm_out=norm(f"l{i}.norm1b"), conv_in=conv(f"l{i}.canon1"))
        if lay.mlp is not None:
            f = lambda n: get(f"l{i}.mlp.{n}")
            out.mlp_in, out.mlp_out, out.conv_mlp = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b"), conv(f"l{i}.canon2")
            out.mlp = pack_moe(cfg, lay.mlp, f("router"), f("router.b"), lambda e, part: f(f"e{e}.{part}"), None, None, device)
        w.layers.append(out)
    return w


def load_weights(cfg: LayerListConfig, path: str, device="cpu") -> LayerListWeights:
    """``path``: a folder with ``config.json`` and ``model.safetensors``."""
    tensors = read_safetensors(os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json")) as f:
        shapes = tensor_shapes(complete(json.load(f), path))
    for name, shape in shapes.items():
        if name not in tensors:
            raise KeyError(f"{path}: tensor '{name}' is missing")
        if tuple(tensors[name].shape) != tuple(shape):
            raise ValueError(f"{path}: tensor '{name}' has shape {tuple(tensors[name].shape)}, expected {tuple(shape)}")
    return weights_from_tensors(cfg, tensors.__getitem__, device)


def _random(name: str, shape: Tuple[int, ...], g: torch.Generator, device, dtype) -> torch.Tensor:
    """Matrices scaled by 1/sqrt(inputs), norms near the identity, head mixing near the identity, decays from quick to
    slow."""
    last, owner = name.rsplit(".", 1)[-1], name.rsplit(".", 2)[-2] if name.count(".") else ""
    uniform = lambda lo, hi: (torch.rand(shape, generator=g, device=device, dtype=torch.float32) * (hi - lo) + lo).to(dtype)
    t = torch.empty(shape, dtype=dtype, device=device).normal_(generator=g)
    if last in ("norm", "out") and owner != "final":                 # plain weights
        return 1.0 + 0.1 * t
    if last.startswith("norm"):                                      # distance from one
        return 0.1 * t
    if last == "lam":
        return uniform(-5.0, 1.0)
    if last == "A_log":
        return uniform(0.0, 1.5)
    if last == "dt_bias":
        return uniform(-6.0, 0.0)
    if last == "talk":
        return 0.2 * t + torch.eye(shape[0], device=device).to(dtype)
    if last == "sink":
        return t
    if last == "b" and len(shape) == 1 or name.endswith((".ra.b", ".ri.b")):
        return 0.1 * t
    return t * (0.05 if name == "embed" else shape[-1] ** -0.5)


def random_tensors(raw: Dict[str, Any], seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Checkpoint-named random tensors of the design's shapes."""
    g = torch.Generator(device=device).manual_seed(seed)
    return {name: _random(name, shape, g, device, torch.float32).to(dtype) for name, shape in tensor_shapes(raw).items()}


def random_weights(cfg: LayerListConfig, raw: Dict[str, Any], device="cpu", seed: int = 0) -> LayerListWeights:
    """Random weights made on ``device``, one tensor at a time."""
    shapes = tensor_shapes(raw)
    g = torch.Generator(device=device).manual_seed(seed)
    return weights_from_tensors(cfg, lambda name: _random(name, shapes[name], g, device, cfg.dtype), device)


def builtin(width: int, vocab: int, pattern: str, *, heads: int, kv_heads: int, dim: int, vdim: int, window: int, rec_width: int,
            rec_blocks: int, d_heads: int, d_kv_heads: int, d_dim: int, d_vdim: int, rank: int, experts: int, top: int, ff: int,
            rot_dims: int = 0, taps: int = 4, conv: int = 4, loop=None, base: float = 500000.0, eps: float = 1e-5) -> Dict[str, Any]:
    """A ``config.json`` dictionary from a layer pattern ("p": attention beside a recurrence, "d": delta rule; both with the
    mixture of experts)."""
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "mask": {"size": window},
            "rot": {"dims": rot_dims or dim, "base": base,
                    "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    mixers = {"p": ("parallel", {"left": left, "right": {"width": rec_width, "blocks": rec_blocks, "conv": conv}}),
              "d": ("channel_delta", {"heads": d_heads, "kv_heads": d_kv_heads, "dim": d_dim, "vdim": d_vdim, "conv": conv,
                                      "decay_rank": rank, "gate_rank": rank})}
    out = {"architecture": ARCHITECTURE, "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": width ** 0.5},
           "canon": {"taps": taps},
           "layers": [{"type": mixers[c][0], "mixer": copy.deepcopy(mixers[c][1]), "mlp": copy.deepcopy(mlp)} for c in pattern]}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out
