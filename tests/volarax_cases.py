"""Small Volarax configurations and tensors for the tests, made from their own sizes and seeds."""
import numpy as np
import torch

from nanoflow_b200.config import parse_config
from nanoflow_b200.models import volarax


def attn(heads=3, dim=40, vdim=24, kv_rank=48, window=37, scale=None, ff=72):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank,
                      "scale": scale if scale is not None else dim ** -0.5,
                      "mask": None if window is None else {"size": window}}}


def mlstm(heads=3, dim=24, vdim=40, gate_cap=9.0, ff=None):
    return {"type": "mlstm", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def config(layers, *, width=104, vocab=211, loop=None, eps=1e-5):
    return {"architecture": "Volarax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop))}


CASES = {
    # every mechanism, sizes that are no powers of two, a loop in the middle
    "mixed": config([attn(), mlstm(), attn(window=20, heads=5, dim=16, vdim=56, kv_rank=72), mlstm(heads=1, dim=56, vdim=8)],
                    loop=(1, 3, 2)),
    # recurrent layer first and last, feed-forward behind the recurrence, no loop, equal sizes
    "recurrent_first": config([mlstm(heads=2, dim=32, vdim=32, ff=40), attn(heads=1, dim=32, vdim=32, kv_rank=32, ff=None),
                               mlstm(heads=2, dim=32, vdim=32)], width=64, vocab=96, eps=1e-3),
    # the whole model loops, odd widths, a window of one token, a window of exactly one page
    "all_looped": config([attn(window=1, dim=9, vdim=7, kv_rank=13, ff=11), attn(window=16), mlstm(heads=2, dim=7, vdim=5)],
                         width=50, vocab=67, loop=(0, 3, 3)),
    # no window, a loop that runs once, heads wider than the prefill kernel takes
    "wide_heads": config([attn(window=None, heads=2, dim=136, vdim=144, kv_rank=200, ff=64), attn(window=None, heads=17, kv_rank=64),
                          mlstm(heads=1, dim=72, vdim=136)], width=96, vocab=128, loop=(1, 2, 1)),
    # large recurrent and latent sizes
    "large": config([attn(heads=4, dim=128, vdim=128, kv_rank=320, window=150, ff=128),
                     mlstm(heads=2, dim=144, vdim=200, gate_cap=15.0), attn(heads=33, dim=24, vdim=16, kv_rank=512, window=64, ff=None),
                     mlstm(heads=2, dim=264, vdim=72)], width=160, vocab=150),
}


def tensors(raw, seed=0, sharp=2.5):
    """Random tensors in which positions matter: queries are scaled up so that single keys stand out, sinks differ
    between heads, forget gates reach from quick to very slow."""
    t = volarax.random_tensors(raw, seed)
    g = torch.Generator().manual_seed(seed + 1)
    for i, lay in enumerate(raw["layers"]):
        p = f"l{i}.mix."
        if lay["type"] == "latent_attention":
            t[p + "q"] = (t[p + "q"].float() * sharp).bfloat16()
            t[p + "sink"] = (torch.randn(t[p + "sink"].shape, generator=g) * 2.0).bfloat16()
        else:
            t[p + "f.b"] = (torch.rand(t[p + "f.b"].shape, generator=g) * 8.0).bfloat16()
            t[p + "i.b"] = (torch.randn(t[p + "i.b"].shape, generator=g) * 2.0).bfloat16()
    return t


def engine_config(raw, *, dtype="bfloat16", batch=256, requests=4, sample_rows=0, pages=64, **pipeline):
    return parse_config({
        "model": dict(raw, dtype=dtype),
        "model_configs": {"gpu_num": 1, "frame_page_size": 16, "max_batch_size": requests, "num_pages": pages,
                          "max_sample_rows": sample_rows or batch},
        "pipeline_configs": {"global_batch_size": batch, "autotune_gemm": False, **pipeline},
        "serve_configs": {"model": "volarax-test", "actual_gpu_num": 1, "pipeline_type": "NON_OVERLAP_LOCAL"}})


def prompt(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n, dtype=np.int32)


def row_errors(got, want):
    """Root mean square error of each row of logits over the rows' root mean square, after the mean is taken off."""
    got, want = torch.as_tensor(got).double(), torch.as_tensor(want).double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
