"""Small Gimudra configurations and tensors for the tests, made from their own sizes and seeds."""
import torch

from nanoflow_b200.config import parse_config
from nanoflow_b200.models import gimudra


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=9, top=4, groups=(3, 2), identity=3, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "identity": identity, "scale": scale,
                       "groups": None if groups is None else dict(zip(("count", "keep"), groups))}}


def layer(heads=6, kv_heads=2, dim=24, vdim=40, chunk=20, scale=None, kv_from=None, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
             "mask": None if chunk is None else {"size": chunk}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def config(layers, *, width=104, vocab=211, eps=1e-5, embed=2.0):
    return {"architecture": "Gimudra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "layers": layers}


CASES = {
    # every mechanism, sizes that are no powers of two; lent keys and values from two layers, read with other masks and other
    # head counts; a layer without a feed-forward
    "mixed": config([layer(mlp=moe()), layer(chunk=33, mlp=dense()), layer(chunk=48, kv_from=0, mlp=moe(groups=None, identity=1)),
                     layer(kv_from=1, chunk=64, mlp=None), layer(heads=2, chunk=50, kv_from=0, mlp=dense(40))]),
    # sizes that are equal, chunks of one page and of one token, no identity experts, all groups kept, a scale of one
    "even": config([layer(heads=2, kv_heads=2, dim=32, vdim=32, chunk=16, scale=1.0, mlp=dense(64)),
                    layer(heads=2, kv_heads=2, dim=32, vdim=32, chunk=1, mlp=moe(32, 4, 2, (2, 2), 0, 1.0)),
                    layer(heads=2, kv_heads=2, dim=32, vdim=32, chunk=64, kv_from=0, mlp=moe(32, 4, 1, None, 0, 1.0))],
                   width=64, vocab=96, eps=1e-3, embed=1.0),
    # odd sizes everywhere (the width too), one key head, more identity experts than experts, all experts chosen
    "odd": config([layer(heads=5, kv_heads=1, dim=9, vdim=14, chunk=7, mlp=moe(11, 3, 3, (7, 4), 4)),
                   layer(heads=3, kv_heads=3, dim=7, vdim=5, chunk=31, mlp=moe(5, 6, 7, None, 1)),
                   layer(heads=5, kv_heads=1, dim=9, vdim=14, chunk=100, kv_from=0, mlp=dense(13))], width=51, vocab=67),
    # heads wider than the tensor-core kernels take, no mask in one layer, one expert per group
    "wide_heads": config([layer(heads=2, kv_heads=1, dim=136, vdim=144, chunk=40, mlp=moe(72, 30, 5, (40, 30), 10)),
                          layer(heads=2, kv_heads=1, dim=40, vdim=136, chunk=None, mlp=dense(136))], width=96, vocab=128),
    # the head sizes of large models, more query heads per key head than the decode kernel takes, long chunks
    "large": config([layer(heads=20, kv_heads=4, dim=128, vdim=96, chunk=100, mlp=moe(136, 56, 8, (8, 3), 8)),
                     layer(heads=34, kv_heads=2, dim=64, vdim=64, chunk=130, mlp=dense(264)),
                     layer(heads=16, kv_heads=1, dim=64, vdim=40, chunk=700, mlp=moe(72, 20, 3, (5, 2), 5)),
                     layer(heads=12, kv_heads=4, dim=128, vdim=96, chunk=77, kv_from=0, mlp=dense(136))], width=160, vocab=150),
}


def tensors(raw, seed=0, sharp=2.5):
    """Random tensors in which positions matter: queries are scaled up so that single keys stand out, distances cost from
    little to much, choice scores are below zero, every earlier result weighs in what goes on."""
    t = gimudra.random_tensors(raw, seed)
    g = torch.Generator().manual_seed(seed + 1)
    uni = lambda name, lo, hi: (torch.rand(t[name].shape, generator=g) * (hi - lo) + lo).bfloat16()
    rnd = lambda name, scale: (torch.randn(t[name].shape, generator=g) * scale).bfloat16()
    t["embed"] = rnd("embed", 1.0)
    for name in t:
        last = name.rsplit(".", 1)[-1]
        if last in ("ls1", "ls2"):
            t[name] = uni(name, 0.3, 1.5)
        elif last in ("norm1", "norm2") or name == "final.norm":
            t[name] = uni(name, 0.5, 1.5)
        elif last == "b":
            t[name] = rnd(name, 0.5)
        elif last == "q":
            t[name] = (t[name].float() * sharp).bfloat16()
        elif last == "r1":
            t[name] = uni(name, 0.0, 2.0)
        elif last == "r2":
            t[name] = torch.exp(torch.rand(t[name].shape, generator=g) * 5.0 - 4.0).bfloat16()
        elif last == "router":
            t[name] = (t[name].float() * 2.0).bfloat16()
        elif last == "correction":
            t[name] = uni(name, -2.0, -1.5)
        elif last == "dwa":
            t[name] = rnd(name, 0.3)
            t[name][-1] += 1.0
    return t


def engine_config(raw, *, dtype="bfloat16", batch=256, requests=4, sample_rows=0, pages=64, **pipeline):
    return parse_config({
        "model": dict(raw, dtype=dtype),
        "model_configs": {"gpu_num": 1, "frame_page_size": 16, "max_batch_size": requests, "num_pages": pages,
                          "max_sample_rows": sample_rows or batch},
        "pipeline_configs": {"global_batch_size": batch, "autotune_gemm": False, **pipeline},
        "serve_configs": {"model": "gimudra-test", "actual_gpu_num": 1, "pipeline_type": "NON_OVERLAP_LOCAL"}})
