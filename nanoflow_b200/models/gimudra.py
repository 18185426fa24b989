"""Gimudra: a small decoder of grouped-query attention in chunks, whose scores lose the logarithm of the distance, with
dense feed-forwards or mixtures of experts some of which hand on their input. Later layers can use the keys and values of
an earlier one; mixers read a mix of each token with the one before; sublayer outputs are scaled per column; a weighted
sum of the embedding output and all layers' results goes on from layer to layer.

Only what is particular to the design is here: its ``config.json`` keys, its tensor names, the choices it
makes among the mechanisms of :mod:`.layer_list`, and random weights of its shape. Engine, caches and
kernels are those of every layer-list model (``runtime/layer_list.py``).
"""
from __future__ import annotations

import copy
import json
import os
from typing import Any, Callable, Dict, List, Optional, Sequence, Tuple

import torch

from .layer_list import (ActSpec, AttentionSpec, LayerListConfig, LayerListLayer, LayerListWeights, LayerSpec, MlpSpec, MoeSpec,
                         pack_attention, pack_conv, pack_mlp, pack_moe, pack_norm, pad_to)
from .safetensors_io import read_safetensors

ARCHITECTURE = "Gimudra"
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}
SINUSOID_BASE = 10000.0


def _mixer(kind: str, m: Dict[str, Any], where: str) -> AttentionSpec:
    if kind != "attention":
        raise ValueError(f"{where}: unknown layer type '{kind}'")
    mask, src = m.get("mask"), m.get("kv_from")
    return AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         scale=float(m["scale"]), sink=False, qk_norm=False, bias=True, distance_bias=True,
                         chunk=None if mask is None else int(mask["size"]), kv_from=None if src is None else int(src))


def _mlp(f: Optional[Dict[str, Any]], where: str):
    if f is None:
        return None
    if f["kind"] == "dense":
        return MlpSpec(int(f["ff"]), ActSpec("silu"), bias=True)
    if f["kind"] != "moe":
        raise ValueError(f"{where}: unknown feed-forward '{f['kind']}'")
    r, groups = f["router"], f["router"].get("groups") or {}
    count = int(groups.get("count", 1))
    return MoeSpec(expert=MlpSpec(int(f["expert"]["ff"]), ActSpec("relu2"), gated=False), experts=int(r["experts"]),
                   top=int(r["top"]), scale=float(r["scale"]), groups=count, keep=int(groups.get("keep", count)),
                   score="softmax_all", identity=int(r.get("identity") or 0), group_score="max")


def parse_model(raw: Dict[str, Any], *, tp: int = 1, run_layers: int = 0, name: str = "") -> LayerListConfig:
    """``config.json`` -> :class:`LayerListConfig`. ``dtype`` ("bfloat16" / "float32") is this framework's own key."""
    layers: List[LayerSpec] = [LayerSpec(_mixer(lay["type"], lay["mixer"], f"layer {i}"), _mlp(lay.get("mlp"), f"layer {i}"))
                               for i, lay in enumerate(raw["layers"])]
    cfg = LayerListConfig(
        name=name or ARCHITECTURE, hidden_size=int(raw["width"]), vocab_size=int(raw["vocab"]), layers=layers,
        norm_kind="rms", norm_eps=float(raw["norm"]["eps"]), embed_norm=False, output_norms=False,
        embed_scale=float(raw["embedding"]["scale"]), sinusoid=SINUSOID_BASE, layer_scale=True, depth_average=True,
        input_conv=2, input_conv_mlp=False,
        eos_token_id=int(raw.get("eos_token_id", -1)), bos_token_id=int(raw.get("bos_token_id", -1)),
        dtype=DTYPES[raw.get("dtype", "bfloat16")], tp=tp)
    if run_layers not in (0, cfg.run_layers, cfg.num_layers):
        raise ValueError("run_layer cannot be changed for a model whose layers are listed")
    return cfg


def tensor_shapes(raw: Dict[str, Any]) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of the checkpoint's tensors."""
    W, V = int(raw["width"]), int(raw["vocab"])
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, lay in enumerate(raw["layers"]):
        p, m, f = f"l{i}.", lay["mixer"], lay.get("mlp")
        H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "shift": (W,), p + "ls1": (W,), p + "dwa": (i + 2,)})
        out.update({p + "mix.q": (H * d, W), p + "mix.q.b": (H * d,), p + "mix.r1": (H,), p + "mix.r2": (H,), p + "mix.o": (W, H * v)})
        if m.get("kv_from") is None:
            out.update({p + "mix.k": (G * d, W), p + "mix.k.b": (G * d,), p + "mix.v": (G * v, W), p + "mix.v.b": (G * v,)})
        if f is None:
            continue
        out.update({p + "norm2": (W,), p + "ls2": (W,)})
        if f["kind"] == "dense":
            for part, rows, cols in (("gate", f["ff"], W), ("up", f["ff"], W), ("down", W, f["ff"])):
                out.update({f"{p}mlp.{part}": (rows, cols), f"{p}mlp.{part}.b": (rows,)})
            continue
        E, ff, outputs = f["router"]["experts"], f["expert"]["ff"], f["router"]["experts"] + (f["router"].get("identity") or 0)
        out.update({p + "mlp.router": (outputs, W), p + "mlp.correction": (outputs,)})
        for e in range(E):
            out.update({f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
    return out


def weights_from_tensors(cfg: LayerListConfig, get: Callable[[str], torch.Tensor], device="cpu") -> LayerListWeights:
    """Checkpoint tensors by name -> kernel layout on ``device``."""
    norm = lambda n, kind=None: pack_norm(cfg, get(n), None, device, kind)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    w = LayerListWeights(embed=mv(pad_to(get("embed"), cfg.vocab_size, cfg.width_p)), embed_norm=None,
                         final_norm=norm("final.norm"), lm_head=mv(pad_to(get("head"), cfg.vocab_p, cfg.width_p)))
    for i, lay in enumerate(cfg.layers):
        g = lambda n: get(f"l{i}.mix.{n}")
        own = lay.mixer.kv_from is None
        mix = pack_attention(cfg, lay.mixer, g("q"), g("k") if own else None, g("v") if own else None, None, None, None, g("o"), 0.0,
                             device, biases=[g("q.b")] + ([g("k.b"), g("v.b")] if own else [None, None]),
                             dist=torch.stack([g("r1").float(), g("r2").float()], dim=1))
        # h + (h' - h) s is h plus a convolution of h' and h with the filter (s, -s)
        shift = get(f"l{i}.shift").float()
        out = LayerListLayer(mixer=mix, norm_in=norm(f"l{i}.norm1"), norm_out=norm(f"l{i}.ls1", "scale"),
                             conv_in=pack_conv(cfg, torch.stack([shift, -shift], dim=1), cfg.width_p, device),
                             depth=get(f"l{i}.dwa").to(device=device, dtype=torch.float32).contiguous())
        if lay.mlp is not None:
            f = lambda n: get(f"l{i}.mlp.{n}")
            out.mlp_in, out.mlp_out = norm(f"l{i}.norm2"), norm(f"l{i}.ls2", "scale")
            if lay.mlp.kind == "dense":
                parts = ("gate", "up", "down")
                out.mlp = pack_mlp(cfg, lay.mlp.ff, *(f(p) for p in parts), device, biases=[f(p + ".b") for p in parts])
            else:
                out.mlp = pack_moe(cfg, lay.mlp, f("router"), f("correction"), lambda e, part: f(f"e{e}.{part}"), None, None, device)
        w.layers.append(out)
    return w


def load_weights(cfg: LayerListConfig, path: str, device="cpu") -> LayerListWeights:
    """``path``: a folder with ``config.json`` and ``model.safetensors``."""
    tensors = read_safetensors(os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json")) as f:
        shapes = tensor_shapes(json.load(f))
    for name, shape in shapes.items():
        if name not in tensors:
            raise KeyError(f"{path}: tensor '{name}' is missing")
        if tuple(tensors[name].shape) != tuple(shape):
            raise ValueError(f"{path}: tensor '{name}' has shape {tuple(tensors[name].shape)}, expected {tuple(shape)}")
    return weights_from_tensors(cfg, tensors.__getitem__, device)


def _random(name: str, shape: Tuple[int, ...], g: torch.Generator, device, dtype) -> torch.Tensor:
    """Matrices scaled by 1/sqrt(inputs), norms and scales around 1, shifts in [0, 1], decays of the distance bias positive;
    what goes on from a layer is mostly its own result."""
    last = name.rsplit(".", 1)[-1]
    if last in ("shift", "r1", "r2"):
        return torch.rand(shape, generator=g, device=device, dtype=torch.float32).to(dtype)
    t = torch.empty(shape, dtype=dtype, device=device).normal_(generator=g)
    if last in ("norm", "norm1", "norm2", "ls1", "ls2"):
        return 1.0 + 0.1 * t
    if last == "b":
        return 0.1 * t
    if last == "correction":                     # (scores are shares of one)
        return 0.1 / shape[0] * t
    if last == "dwa":
        t = 0.1 * t
        t[-1] += 1.0
        return t
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


def builtin(width: int, vocab: int, pattern: str, *, heads: int, kv_heads: int, dim: int, vdim: int, chunks: Sequence[int], ff: int,
            experts: int, top: int, e_ff: int, groups: int, keep: int, identity: int, router_scale: float = 2.5,
            eps: float = 1e-5) -> Dict[str, Any]:
    """A ``config.json`` dictionary from a layer pattern: "d" has a dense feed-forward, "m" and "s" a mixture of experts; "s"
    uses the keys and values of the last layer before it that has its own. ``chunks``: taken in turn."""
    layers, last = [], -1
    for i, c in enumerate(pattern):
        mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5,
                 "mask": {"size": chunks[i % len(chunks)]}}
        if c == "s":
            mixer["kv_from"] = last
        else:
            last = i
        mlp = {"kind": "dense", "ff": ff} if c == "d" else \
            {"kind": "moe", "expert": {"ff": e_ff},
             "router": {"experts": experts, "top": top, "identity": identity, "scale": router_scale,
                        "groups": {"count": groups, "keep": keep}}}
        layers.append({"type": "attention", "mixer": mixer, "mlp": copy.deepcopy(mlp)})
    return {"architecture": ARCHITECTURE, "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": width ** 0.5},
            "layers": layers}
