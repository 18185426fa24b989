"""Small Zubedra configurations and tensors for the tests, made from their own sizes and seeds."""
import torch

from nanoflow_b200.config import parse_config
from nanoflow_b200.models import zubedra


def moe(ff=24, experts=10, top=3, groups=5, keep=3, limit=1.2, scale=1.7, shared=40, shared_limit=0.8):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}},
            "shared": None if shared is None else {"ff": shared, "limit": shared_limit}}


_MOE = object()


def attn(heads=6, kv_heads=2, dim=24, vdim=40, scale=None, softcap=6.0, v_mix=True, mlp=_MOE):
    return {"type": "attention", "mlp": moe() if mlp is _MOE else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap, "v_mix": v_mix,
                      "scale": dim ** -0.5 if scale is None else scale}}


def wkv(heads=3, dim=24, rank=9, mlp=_MOE):
    return {"type": "wkv", "mlp": moe() if mlp is _MOE else mlp, "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}}


def config(layers, *, width=104, vocab=211, eps=1e-5, embed=3.0, logit=0.6):
    return {"architecture": "Zubedra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers,
            "embedding": {"scale": embed}, "logit_scale": logit}


CASES = {
    # every mechanism, sizes that are no powers of two, a head group of three, an attention layer that does not mix
    "mixed": config([attn(), wkv(), attn(v_mix=False, heads=4, kv_heads=4, dim=32, vdim=16, softcap=None), wkv(heads=1, dim=56),
                     attn()]),
    # recurrence first and last, no mixing source before the third layer, layers without a feed-forward
    "recurrent_first": config([wkv(heads=2, dim=32, rank=16, mlp=None), attn(heads=2, kv_heads=1, dim=32, vdim=32, v_mix=False),
                               attn(heads=2, kv_heads=1, dim=32, vdim=32), attn(heads=2, kv_heads=1, dim=32, vdim=32, mlp=None),
                               wkv(heads=2, dim=32, rank=16)], width=64, vocab=96, eps=1e-3, embed=1.0, logit=1.0),
    # odd sizes everywhere, one expert per token, groups of one expert, no shared expert, all groups kept
    "odd": config([attn(heads=5, kv_heads=5, dim=9, vdim=7, mlp=moe(ff=11, experts=7, top=1, groups=7, keep=2, shared=None)),
                   wkv(heads=3, dim=7, rank=3, mlp=moe(ff=5, experts=6, top=6, groups=1, keep=1, shared=9)),
                   attn(heads=5, kv_heads=5, dim=9, vdim=7, mlp=moe(ff=13, experts=9, top=4, groups=3, keep=3))],
                  width=50, vocab=67),
    # heads wider than the tensor-core kernels take, and more of them per key/value head
    "wide_heads": config([attn(heads=2, kv_heads=1, dim=136, vdim=144, mlp=moe(ff=72, experts=40, top=5, groups=4, keep=2)),
                          wkv(heads=1, dim=136, rank=24), attn(heads=18, kv_heads=1, dim=24, vdim=24, v_mix=False)], width=96,
                         vocab=128),
    # the head sizes of large models
    "large": config([attn(heads=16, kv_heads=2, dim=128, vdim=128, softcap=15.0, mlp=moe(ff=136, experts=64, top=8, groups=8, keep=4)),
                     wkv(heads=2, dim=128, rank=40), attn(heads=16, kv_heads=2, dim=96, vdim=128), wkv(heads=4, dim=64, rank=64)],
                    width=160, vocab=150),
}


def tensors(raw, seed=0, sharp=2.0):
    """Random tensors in which positions matter: normed queries are scaled up so that single keys stand out, sinks differ
    between heads, decays reach from quick to very slow, corrections are partly negative."""
    t = zubedra.random_tensors(raw, seed)
    g = torch.Generator().manual_seed(seed + 1)
    rnd = lambda name, scale: (torch.randn(t[name].shape, generator=g) * scale).bfloat16()
    t["embed"] = rnd("embed", 1.0)
    for i, lay in enumerate(raw["layers"]):
        p = f"l{i}."
        if lay["type"] == "attention":
            t[p + "mix.q.norm"] = (t[p + "mix.q.norm"].float() * sharp).bfloat16()
            t[p + "mix.sink"] = rnd(p + "mix.sink", 2.0)
            if p + "mix.vmix" in t:
                t[p + "mix.vmix"] = torch.tensor(0.3 + 0.1 * i).bfloat16()
        else:
            t[p + "mix.w0"] = (torch.rand(t[p + "mix.w0"].shape, generator=g) * 9.0 - 7.0).bfloat16()
        if lay.get("mlp") is not None:
            t[p + "mlp.correction"] = rnd(p + "mlp.correction", 0.8)
    return t


def engine_config(raw, *, dtype="bfloat16", batch=256, requests=4, sample_rows=0, pages=64, **pipeline):
    return parse_config({
        "model": dict(raw, dtype=dtype),
        "model_configs": {"gpu_num": 1, "frame_page_size": 16, "max_batch_size": requests, "num_pages": pages,
                          "max_sample_rows": sample_rows or batch},
        "pipeline_configs": {"global_batch_size": batch, "autotune_gemm": False, **pipeline},
        "serve_configs": {"model": "zubedra-test", "actual_gpu_num": 1, "pipeline_type": "NON_OVERLAP_LOCAL"}})
