"""Volarax: a small decoder that mixes windowed latent attention without positions and mLSTM layers, with a
looped range of layers, norms around every sublayer and ReLU-gated feed-forwards.

Only what is particular to the design is here: its ``config.json`` keys, its tensor names, the choices it
makes among the mechanisms of :mod:`.layer_list`, and random weights of its shape. Engine, caches and
kernels are those of every layer-list model (``runtime/layer_list.py``).
"""
from __future__ import annotations

import json
import os
from typing import Any, Callable, Dict, List, Tuple

import torch

from .layer_list import (ActSpec, LatentAttentionSpec, LayerListConfig, LayerListLayer, LayerListWeights, LayerSpec, MlpSpec,
                         MlstmSpec, pack_latent_attention, pack_mlp, pack_mlstm, pack_norm, pad_to)
from .safetensors_io import read_safetensors

ARCHITECTURE = "Volarax"
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def _mixer(kind: str, m: Dict[str, Any], where: str):
    if kind == "latent_attention":
        mask = m.get("mask")
        return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                   scale=float(m["scale"]), window=None if mask is None else int(mask["size"]))
    if kind == "mlstm":
        return MlstmSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))
    raise ValueError(f"{where}: unknown layer type '{kind}'")


def parse_model(raw: Dict[str, Any], *, tp: int = 1, run_layers: int = 0, name: str = "") -> LayerListConfig:
    """``config.json`` -> :class:`LayerListConfig`. ``dtype`` ("bfloat16" / "float32") is this framework's own
    key: the storage the engine runs in."""
    layers: List[LayerSpec] = []
    for i, lay in enumerate(raw["layers"]):
        mlp = lay.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        layers.append(LayerSpec(_mixer(lay["type"], lay["mixer"], f"layer {i}"),
                                None if mlp is None else MlpSpec(int(mlp["ff"]), ActSpec("relu"))))
    loop = raw.get("loop")
    cfg = LayerListConfig(
        name=name or ARCHITECTURE, hidden_size=int(raw["width"]), vocab_size=int(raw["vocab"]), layers=layers,
        norm_kind="layer", norm_eps=float(raw["norm"]["eps"]),
        loop=None if not loop else (int(loop["start"]), int(loop["stop"]), int(loop["times"])),
        eos_token_id=int(raw.get("eos_token_id", -1)), bos_token_id=int(raw.get("bos_token_id", -1)),
        dtype=DTYPES[raw.get("dtype", "bfloat16")], tp=tp)
    if run_layers not in (0, cfg.run_layers, cfg.num_layers):
        raise ValueError("run_layer cannot be changed for a model whose layers are listed")
    return cfg


def tensor_shapes(raw: Dict[str, Any]) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of the checkpoint's tensors."""
    W, V = int(raw["width"]), int(raw["vocab"])
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "head": (V, W)}

    def norm(name):
        out[name] = out[name + ".b"] = (W,)

    norm("embed.norm")
    norm("final.norm")
    if raw.get("loop"):
        out["loop.step"] = (int(raw["loop"]["times"]), W)
    for i, lay in enumerate(raw["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, d, v = m["heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        norm(p + "norm1b")
        if lay["type"] == "latent_attention":
            r = m["kv_rank"]
            out.update({p + "mix.q": (H * d, W), p + "mix.dkv": (r, W), p + "mix.dkv.norm": (r,), p + "mix.uk": (H * d, r),
                        p + "mix.uv": (H * v, r), p + "mix.sink": (H,), p + "mix.o": (W, H * v)})
        else:
            out.update({p + "mix.q": (H * d, W), p + "mix.k": (H * d, W), p + "mix.v": (H * v, W), p + "mix.g": (H * v, W),
                        p + "mix.o": (W, H * v), p + "mix.norm": (H * v,), p + "mix.i": (H, W), p + "mix.i.b": (H,),
                        p + "mix.f": (H, W), p + "mix.f.b": (H,)})
        if lay.get("mlp") is not None:
            f = lay["mlp"]["ff"]
            norm(p + "norm2")
            norm(p + "norm2b")
            out.update({p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f)})
    return out


def weights_from_tensors(cfg: LayerListConfig, get: Callable[[str], torch.Tensor], device="cpu") -> LayerListWeights:
    """Checkpoint tensors by name -> kernel layout on ``device``."""
    norm = lambda n: pack_norm(cfg, get(n), get(n + ".b"), device)
    mv = lambda t: t.to(device=device, dtype=cfg.dtype).contiguous()
    w = LayerListWeights(embed=mv(pad_to(get("embed"), cfg.vocab_size, cfg.width_p)), embed_norm=norm("embed.norm"),
                         final_norm=norm("final.norm"), lm_head=mv(pad_to(get("head"), cfg.vocab_p, cfg.width_p)))
    if cfg.loop is not None:
        w.loop_steps = pad_to(get("loop.step").to(device=device, dtype=torch.float32), cfg.loop[2], cfg.width_p).contiguous()
    for i, lay in enumerate(cfg.layers):
        g = lambda n: get(f"l{i}.mix.{n}")
        if lay.mixer.kind == "latent_attention":
            mix = pack_latent_attention(cfg, lay.mixer, g("q"), g("dkv"), g("dkv.norm"), g("uk"), g("uv"), g("sink"),
                                        g("o"), device)
        else:
            mix = pack_mlstm(cfg, lay.mixer, g("q"), g("k"), g("v"), g("g"), g("i"), g("f"), g("i.b"), g("f.b"),
                             g("norm"), g("o"), device)
        out = LayerListLayer(mixer=mix, norm_in=norm(f"l{i}.norm1"), norm_out=norm(f"l{i}.norm1b"))
        if lay.mlp is not None:
            out.mlp_in, out.mlp_out = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b")
            out.mlp = pack_mlp(cfg, lay.mlp.ff, get(f"l{i}.mlp.gate"), get(f"l{i}.mlp.up"), get(f"l{i}.mlp.down"), device)
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


def random_tensors(raw: Dict[str, Any], seed: int = 0, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Checkpoint-named random tensors of the design's shapes: matrices scaled by 1/sqrt(inputs), norm
    weights around 1, forget-gate biases that let the state live for a while."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(raw).items():
        t = torch.empty(shape, dtype=torch.float32, device=device).normal_(generator=g)
        if name.endswith(".f.b"):
            t = 3.0 + t
        elif len(shape) == 2:
            t *= 1.0 if name in ("embed",) else 0.1 if name == "loop.step" else shape[1] ** -0.5
        elif name.endswith(".norm") or name.rsplit(".", 1)[-1] in ("norm1", "norm1b", "norm2", "norm2b"):
            t = 1.0 + 0.1 * t
        else:
            t *= 0.1
        out[name] = t.to(dtype)
    return out


def random_weights(cfg: LayerListConfig, raw: Dict[str, Any], device="cpu", seed: int = 0) -> LayerListWeights:
    """Random weights made on ``device``, one tensor at a time."""
    shapes = tensor_shapes(raw)
    g = torch.Generator(device=device).manual_seed(seed)

    def get(name):
        shape = shapes[name]
        t = torch.empty(shape, dtype=cfg.dtype, device=device)
        if len(shape) == 2:
            t.normal_(0.0, shape[1] ** -0.5, generator=g)
        else:
            t.normal_(0.0, 0.1, generator=g)
            if name.endswith(".f.b"):
                t += 3.0
            elif not name.endswith(".b") and "sink" not in name:
                t += 1.0
        return t

    return weights_from_tensors(cfg, get, device)


def builtin(width: int, vocab: int, pattern: List[str], *, heads: int, dim: int, vdim: int, kv_rank: int, window: int,
            m_heads: int, m_dim: int, m_vdim: int, ff: int, loop=None, eps: float = 1e-5, gate_cap: float = 15.0,
            m_ff: int = 0) -> Dict[str, Any]:
    """A ``config.json`` dictionary from a layer pattern ("a": latent attention + feed-forward, "m": mLSTM,
    with a feed-forward of ``m_ff`` if given)."""
    layers = []
    for c in pattern:
        if c == "a":
            layers.append({"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff},
                           "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": dim ** -0.5,
                                     "mask": {"size": window}}})
        else:
            layers.append({"type": "mlstm", "mlp": {"kind": "dense", "ff": m_ff} if m_ff else None,
                           "mixer": {"heads": m_heads, "dim": m_dim, "vdim": m_vdim, "gate_cap": gate_cap}})
    return {"architecture": ARCHITECTURE, "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}
