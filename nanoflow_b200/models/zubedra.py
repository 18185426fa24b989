"""Zubedra: a small decoder that mixes grouped-query attention without positions (normed queries and keys, capped
scores, a sink per head, values mixed with those of the first such layer) and WKV recurrences. In every layer the
mixer and a mixture of capped gated experts read one normed input side by side.

Only what is particular to the design is here: its ``config.json`` keys, its tensor names, the choices it
makes among the mechanisms of :mod:`.layer_list`, and random weights of its shape. Engine, caches and
kernels are those of every layer-list model (``runtime/layer_list.py``).
"""
from __future__ import annotations

import copy
import json
import os
from typing import Any, Callable, Dict, List, Tuple

import torch

from .layer_list import (ActSpec, AttentionSpec, LayerListConfig, LayerListLayer, LayerListWeights, LayerSpec, MlpSpec,
                         MoeSpec, WkvSpec, pack_attention, pack_moe, pack_norm, pack_wkv, pad_to)
from .safetensors_io import read_safetensors, read_shapes

ARCHITECTURE = "Zubedra"
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}
ACT_ALPHA, ACT_SHIFT = 1.702, 1.0          # g sigmoid(1.702 g) (u + 1)
MIXES = ("r", "k", "v", "g", "w")


def _mixer(kind: str, m: Dict[str, Any], where: str):
    if kind == "attention":
        cap = m.get("softcap")
        return AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                             scale=float(m["scale"]), softcap=None if cap is None else float(cap),
                             value_mix=bool(m.get("v_mix", False)))
    if kind == "wkv":
        if "decay_rank" not in m:
            raise ValueError(f"{where}: the rank of the decay projection is missing ('decay_rank'; a model folder's "
                             "tensors say it)")
        return WkvSpec(heads=int(m["heads"]), dim=int(m["dim"]), rank=int(m["decay_rank"]))
    raise ValueError(f"{where}: unknown layer type '{kind}'")


def _expert(e: Dict[str, Any]) -> MlpSpec:
    return MlpSpec(int(e["ff"]), ActSpec("capped", limit=float(e["limit"]), alpha=ACT_ALPHA, shift=ACT_SHIFT))


def _mlp(f: Dict[str, Any], where: str):
    if f is None:
        return None
    if f.get("kind", "moe") != "moe":
        raise ValueError(f"{where}: unknown feed-forward '{f['kind']}'")
    r, groups, shared = f["router"], f["router"].get("groups") or {}, f.get("shared")
    return MoeSpec(expert=_expert(f["expert"]), experts=int(r["experts"]), top=int(r["top"]), scale=float(r["scale"]),
                   groups=int(groups.get("count", 1)), keep=int(groups.get("keep", 1)),
                   shared=None if shared is None else _expert(shared))


def complete(raw: Dict[str, Any], folder: str) -> Dict[str, Any]:
    """``config.json`` with the sizes that only the checkpoint's tensors give."""
    raw = copy.deepcopy(raw)
    shapes = read_shapes(os.path.join(folder, "model.safetensors"))
    for i, lay in enumerate(raw["layers"]):
        if lay["type"] == "wkv":
            name = f"l{i}.mix.w1"
            if name not in shapes:
                raise KeyError(f"{folder}: tensor '{name}' is missing")
            lay["mixer"]["decay_rank"] = int(shapes[name][0])
    return raw


def parse_model(raw: Dict[str, Any], *, tp: int = 1, run_layers: int = 0, name: str = "") -> LayerListConfig:
    """``config.json`` -> :class:`LayerListConfig`. ``dtype`` ("bfloat16" / "float32") and the mixers' ``decay_rank`` are
    this framework's own keys."""
    layers: List[LayerSpec] = [LayerSpec(_mixer(lay["type"], lay["mixer"], f"layer {i}"), _mlp(lay.get("mlp"), f"layer {i}"))
                               for i, lay in enumerate(raw["layers"])]
    cfg = LayerListConfig(
        name=name or ARCHITECTURE, hidden_size=int(raw["width"]), vocab_size=int(raw["vocab"]), layers=layers,
        norm_kind="layer", norm_eps=float(raw["norm"]["eps"]), embed_norm=False, output_norms=False, parallel=True,
        embed_scale=float(raw["embedding"]["scale"]), logit_scale=float(raw["logit_scale"]),
        eos_token_id=int(raw.get("eos_token_id", -1)), bos_token_id=int(raw.get("bos_token_id", -1)),
        dtype=DTYPES[raw.get("dtype", "bfloat16")], tp=tp)
    if run_layers not in (0, cfg.run_layers, cfg.num_layers):
        raise ValueError("run_layer cannot be changed for a model whose layers are listed")
    return cfg


def tensor_shapes(raw: Dict[str, Any]) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of the checkpoint's tensors."""
    W, V = int(raw["width"]), int(raw["vocab"])
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}

    def mlp(p, f):
        out.update({p + "gate": (f, W), p + "up": (f, W), p + "down": (W, f)})

    for i, lay in enumerate(raw["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, d = m["heads"], m["dim"]
        out[p + "norm1"] = (W,)
        if lay["type"] == "attention":
            G, v = m["kv_heads"], m["vdim"]
            out.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.v": (G * v, W), p + "mix.o": (W, H * v),
                        p + "mix.q.norm": (H * d,), p + "mix.k.norm": (G * d,), p + "mix.sink": (H,)})
            if m.get("v_mix"):
                out[p + "mix.vmix"] = ()
        else:
            r = m["decay_rank"]
            out.update({f"{p}mix.mu.{s}": (W,) for s in MIXES})
            out.update({f"{p}mix.{s}": (H * d, W) for s in "rkvg"})
            out.update({p + "mix.w1": (r, W), p + "mix.w2": (H * d, r), p + "mix.w0": (H * d,), p + "mix.u": (H, d),
                        p + "mix.norm": (H * d,), p + "mix.o": (W, H * d)})
        f = lay.get("mlp")
        if f is not None:
            E = f["router"]["experts"]
            out.update({p + "mlp.router": (E, W), p + "mlp.correction": (E,)})
            for e in range(E):
                mlp(f"{p}mlp.e{e}.", f["expert"]["ff"])
            if f.get("shared") is not None:
                mlp(p + "mlp.shared.", f["shared"]["ff"])
                out[p + "mlp.shared.sg"] = (1, W)
    return out


def weights_from_tensors(cfg: LayerListConfig, get: Callable[[str], torch.Tensor], device="cpu") -> LayerListWeights:
    """Checkpoint tensors by name -> kernel layout on ``device``."""
    norm = lambda n, scale=1.0: pack_norm(cfg, get(n).float() * scale, None, device)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    w = LayerListWeights(embed=mv(pad_to(get("embed"), cfg.vocab_size, cfg.width_p)), embed_norm=None,
                         final_norm=norm("final.norm", cfg.logit_scale),
                         lm_head=mv(pad_to(get("head"), cfg.vocab_p, cfg.width_p)))
    first = cfg.first_value_run                # no loops here: runs are layers
    for i, lay in enumerate(cfg.layers):
        g = lambda n: get(f"l{i}.mix.{n}")
        if lay.mixer.kind == "attention":
            mixes = lay.mixer.value_mix and i != first
            mix = pack_attention(cfg, lay.mixer, g("q"), g("k"), g("v"), g("q.norm"), g("k.norm"), g("sink"), g("o"),
                                 g("vmix").item() if mixes else 0.0, device)
        else:
            mix = pack_wkv(cfg, lay.mixer, [g("mu." + s) for s in MIXES], g("r"), g("k"), g("v"), g("g"), g("w1"), g("w2"),
                           g("w0"), g("u"), g("norm"), g("o"), device)
        out = LayerListLayer(mixer=mix, norm_in=norm(f"l{i}.norm1"))
        if lay.mlp is not None:
            f = lambda n: get(f"l{i}.mlp.{n}")
            shared = lay.mlp.shared is not None
            out.mlp = pack_moe(cfg, lay.mlp, f("router"), f("correction"), lambda e, part: f(f"e{e}.{part}"),
                               [f("shared." + part) for part in ("gate", "up", "down")] if shared else None,
                               f("shared.sg") if shared else None, device)
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
    """Matrices scaled by 1/sqrt(inputs), norm weights around 1, mixing weights in [0, 1], decays from quick to slow."""
    last = name.rsplit(".", 1)[-1]
    if ".mu." in name or last == "vmix":
        return torch.rand(shape, generator=g, device=device, dtype=torch.float32).to(dtype)
    if last == "w0":
        return (torch.rand(shape, generator=g, device=device, dtype=torch.float32) * 5.0 - 5.0).to(dtype)
    t = torch.empty(shape, dtype=dtype, device=device).normal_(generator=g)
    if last in ("norm", "norm1"):
        return 1.0 + 0.1 * t
    if last in ("u", "sink"):
        return t
    if last == "correction":
        return 0.1 * t
    return t * (0.05 if name == "embed" else shape[1] ** -0.5)


def random_tensors(raw: Dict[str, Any], seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Checkpoint-named random tensors of the design's shapes."""
    g = torch.Generator(device=device).manual_seed(seed)
    return {name: _random(name, shape, g, device, torch.float32).to(dtype) for name, shape in tensor_shapes(raw).items()}


def random_weights(cfg: LayerListConfig, raw: Dict[str, Any], device="cpu", seed: int = 0) -> LayerListWeights:
    """Random weights made on ``device``, one tensor at a time."""
    shapes = tensor_shapes(raw)
    g = torch.Generator(device=device).manual_seed(seed)
    return weights_from_tensors(cfg, lambda name: _random(name, shapes[name], g, device, cfg.dtype), device)


def builtin(width: int, vocab: int, pattern: str, *, heads: int, kv_heads: int, dim: int, vdim: int, softcap: float,
            w_heads: int, w_dim: int, rank: int, experts: int, top: int, ff: int, groups: int, keep: int, shared_ff: int,
            limit: float = 7.0, router_scale: float = 2.0, eps: float = 1e-5) -> Dict[str, Any]:
    """A ``config.json`` dictionary from a layer pattern ("a": attention, "w": WKV; both with the mixture of experts)."""
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared_ff, "limit": limit},
           "router": {"experts": experts, "top": top, "scale": router_scale, "groups": {"count": groups, "keep": keep}}}
    mixers = {"a": ("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5,
                                  "softcap": softcap, "v_mix": True}),
              "w": ("wkv", {"heads": w_heads, "dim": w_dim, "decay_rank": rank})}
    return {"architecture": ARCHITECTURE, "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": 1.0,
            "embedding": {"scale": width ** 0.5},
            "layers": [{"type": mixers[c][0], "mixer": dict(mixers[c][1]), "mlp": copy.deepcopy(mlp)} for c in pattern]}
