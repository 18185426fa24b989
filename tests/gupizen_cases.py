"""Small Gupizen configurations and tensors for the tests, made from their own sizes and seeds."""
import torch

from nanoflow_b200.config import parse_config
from nanoflow_b200.models import gupizen


def moe(ff=24, experts=10, top=3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


_MOE = object()


def parallel(heads=6, kv_heads=2, dim=24, vdim=40, window=20, rot=16, base=1000.0, original=60.0, scaling=True, scale=None, width=72,
             blocks=3, conv=3, mlp=_MOE):
    s = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": original} if scaling else None
    return {"type": "parallel", "mlp": moe() if mlp is _MOE else mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                               "rot": {"dims": rot, "base": base, "scaling": s}, "scale": dim ** -0.5 if scale is None else scale},
                      "right": {"width": width, "blocks": blocks, "conv": conv}}}


def delta(heads=6, kv_heads=3, dim=24, vdim=40, conv=4, decay_rank=9, gate_rank=13, mlp=_MOE):
    return {"type": "channel_delta", "mlp": moe() if mlp is _MOE else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
                      "gate_rank": gate_rank}}


def config(layers, *, width=104, vocab=211, eps=1e-5, embed=2.0, taps=4, loop=None):
    out = {"architecture": "Gupizen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers,
           "embedding": {"scale": embed}, "canon": {"taps": taps}}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CASES = {
    # every mechanism, sizes that are no powers of two, shared key heads in both mixers, a loop of two kinds of layers
    "mixed": config([parallel(), parallel(heads=4, kv_heads=4, dim=32, vdim=16, window=33, rot=10, width=40, blocks=5), delta(),
                     parallel(window=48)], loop=(1, 3, 2)),
    # no loop, a window of one token, layers without a feed-forward, filters of two taps, one block, sizes that are equal
    "delta_first": config([delta(heads=2, kv_heads=2, dim=32, vdim=32, conv=2, decay_rank=8, gate_rank=8, mlp=None),
                           parallel(heads=2, kv_heads=1, dim=32, vdim=32, rot=32, window=1, scaling=False, width=64, blocks=1, conv=2),
                           parallel(heads=2, kv_heads=1, dim=32, vdim=32, rot=32, window=16, width=64, blocks=1, conv=2, mlp=None),
                           delta(heads=2, kv_heads=1, dim=32, vdim=32, conv=2)], width=64, vocab=96, eps=1e-3, embed=1.0, taps=2),
    # odd sizes everywhere, one expert per token or all of them, the whole model loops
    "odd": config([parallel(heads=5, kv_heads=5, dim=10, vdim=6, rot=6, window=17, width=35, blocks=5, conv=5, mlp=moe(11, 7, 2)),
                   delta(heads=3, kv_heads=1, dim=7, vdim=5, conv=3, decay_rank=3, gate_rank=1, mlp=moe(5, 6, 6)),
                   parallel(heads=5, kv_heads=1, dim=9, vdim=14, rot=2, window=31, width=11, blocks=11, conv=1)],
                  width=50, vocab=67, taps=3, loop=(0, 3, 2)),
    # heads wider than the tensor-core kernels take; a loop that runs once
    "wide_heads": config([parallel(heads=2, kv_heads=1, dim=136, vdim=144, rot=100, window=40, mlp=moe(72, 40, 5)),
                          delta(heads=2, kv_heads=1, dim=136, vdim=72, decay_rank=24, gate_rank=40),
                          delta(heads=1, kv_heads=1, dim=24, vdim=136)], width=96, vocab=128, loop=(0, 1, 1)),
    # the head sizes of large models, more heads than one CTA of a kernel takes
    "large": config([parallel(heads=20, kv_heads=4, dim=128, vdim=96, rot=64, window=100, width=256, blocks=2, conv=4, mlp=moe(136, 64, 8)),
                     delta(heads=2, kv_heads=2, dim=128, vdim=128, decay_rank=40, gate_rank=40),
                     parallel(heads=34, kv_heads=17, dim=64, vdim=64, rot=64, window=130, width=96, blocks=1),
                     delta(heads=4, kv_heads=2, dim=64, vdim=128)], width=160, vocab=150, loop=(1, 4, 2)),
}


def tensors(raw, seed=0, sharp=2.5):
    """Random tensors in which positions matter: queries are scaled up so that single keys stand out, sinks differ between
    heads, the mixing of heads is far from symmetric, decays reach from quick to very slow."""
    t = gupizen.random_tensors(raw, seed)
    g = torch.Generator().manual_seed(seed + 1)
    rnd = lambda name, scale: (torch.randn(t[name].shape, generator=g) * scale).bfloat16()
    uni = lambda name, lo, hi: (torch.rand(t[name].shape, generator=g) * (hi - lo) + lo).bfloat16()
    t["embed"] = rnd("embed", 1.0)
    for name in t:
        if name.rsplit(".", 1)[-1] in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            t[name] = rnd(name, 0.3)
    for i, lay in enumerate(raw["layers"]):
        p = f"l{i}.mix."
        if lay["type"] == "parallel":
            t[p + "left.q"] = (t[p + "left.q"].float() * sharp).bfloat16()
            t[p + "left.sink"] = rnd(p + "left.sink", 2.0)
            H = lay["mixer"]["left"]["heads"]
            t[p + "left.talk"] = (torch.eye(H) + torch.randn(H, H, generator=g) * 0.6).bfloat16()
            t[p + "right.lam"] = uni(p + "right.lam", -7.0, 1.0)
        else:
            t[p + "A_log"] = uni(p + "A_log", -1.0, 1.5)
            t[p + "dt_bias"] = uni(p + "dt_bias", -7.0, 0.5)
    return t


def engine_config(raw, *, dtype="bfloat16", batch=256, requests=4, sample_rows=0, pages=64, **pipeline):
    return parse_config({
        "model": dict(raw, dtype=dtype),
        "model_configs": {"gpu_num": 1, "frame_page_size": 16, "max_batch_size": requests, "num_pages": pages,
                          "max_sample_rows": sample_rows or batch},
        "pipeline_configs": {"global_batch_size": batch, "autotune_gemm": False, **pipeline},
        "serve_configs": {"model": "gupizen-test", "actual_gpu_num": 1, "pipeline_type": "NON_OVERLAP_LOCAL"}})
