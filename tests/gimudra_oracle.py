"""Plain, slow restatement of the Gimudra decoder, the oracle of its tests.

One function per mechanism, whole sequences only, no cache, no batching, nothing shared with the package.
Everything runs in the dtype of the tensors it is given (the tests use float64, so that the oracle's own
rounding never matters). A model is ``(config, tensors)``: the parsed ``config.json`` and a dict of tensors
under their checkpoint names.
"""
import math

import torch


def rms_norm(x, eps, weight):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def silu(x):
    return x * torch.sigmoid(x)


def squared_relu(x):
    return torch.relu(x) ** 2


# ---- before the layers ------------------------------------------------------------------------------------------
def sinusoid(T, width, dtype, base=10000.0):
    """Row p: sine and cosine of p * base^(-2i / width), next to each other."""
    a = torch.arange(T, dtype=dtype)[:, None] * base ** (-torch.arange(0, width, 2, dtype=dtype) / width)
    return torch.stack([torch.sin(a), torch.cos(a)], dim=-1).reshape(T, -1)[:, :width]


def embed(tokens, table, scale):
    x = table[torch.as_tensor(tokens, dtype=torch.long)] * scale
    return x + sinusoid(x.shape[0], x.shape[1], x.dtype)


# ---- attention --------------------------------------------------------------------------------------------------
def token_shift(h, amount):
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * amount


def project(h, w, name):
    return h @ w[name].T + w[name + ".b"]


def distance_bias(T, r1, r2):
    """[H, T, T]: what query i's score of key j loses."""
    d = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * d)


def same_chunk(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & (i // size == j // size)


def attend(q, k, v, scale, r1, r2, size):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    s = torch.stack([q[:, h] @ k[:, h // (H // G)].T for h in range(H)]) * scale - distance_bias(T, r1, r2)
    p = torch.softmax(s.masked_fill(~same_chunk(T, size), -math.inf), dim=-1)
    return torch.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], dim=1)


def keys_and_values(h, w, spec):
    T, G = h.shape[0], spec["kv_heads"]
    return project(h, w, "k").reshape(T, G, -1), project(h, w, "v").reshape(T, G, -1)


def attention(h, w, spec, kv):
    T = h.shape[0]
    q = project(h, w, "q").reshape(T, spec["heads"], -1)
    size = (spec.get("mask") or {}).get("size")
    return attend(q, *kv, spec["scale"], w["r1"], w["r2"], size).reshape(T, -1) @ w["o"].T


# ---- feed-forwards ----------------------------------------------------------------------------------------------
def dense(h, w):
    return (silu(project(h, w, "gate")) * project(h, w, "up")) @ w["down"].T + w["down.b"]


def kept_groups(choice, groups):
    """Choice scores with those of all but the best groups at minus infinity; a group is as good as its best expert."""
    n = groups.get("count", 1)
    best = choice.reshape(choice.shape[0], n, -1)
    order = torch.argsort(best.amax(-1), dim=-1, descending=True, stable=True)[:, :groups.get("keep", n)]
    keep = torch.zeros(choice.shape[0], n, dtype=torch.bool).scatter_(1, order, True)
    return best.masked_fill(~keep[:, :, None], -math.inf).reshape(choice.shape)


def route(z, correction, router):
    """logits [T, experts + identity] -> (chosen [T, top], weights [T, top])."""
    s = torch.softmax(z, dim=-1)
    choice = kept_groups(s + correction, router.get("groups") or {})
    idx = torch.argsort(choice, dim=-1, descending=True, stable=True)[:, :router["top"]]
    return idx, s.gather(1, idx) * router["scale"]


def expert(h, w, e):
    return squared_relu(h @ w[f"e{e}.up"].T) @ w[f"e{e}.down"].T


def identity_expert(h):
    return h


def moe(h, w, spec):
    r = spec["router"]
    idx, weight = route(h @ w["router"].T, w["correction"], r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(idx[t].tolist(), weight[t]):
            row = h[t:t + 1]
            out[t] += a * (identity_expert(row) if e >= r["experts"] else expert(row, w, e))[0]
    return out


# ---- model ------------------------------------------------------------------------------------------------------
def layer_scale(y, amount):
    return y * amount


def depth_average(results, weights):
    """``results``: the embedding output and the results of all layers so far."""
    return sum(a * x for a, x in zip(weights, results))


def forward(config, tensors, tokens, dtype=torch.float64, residuals=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the stream that goes on after every layer."""
    w = {k: t.to(dtype) for k, t in tensors.items()}
    eps = config["norm"]["eps"]
    x = embed(tokens, w["embed"], config["embedding"]["scale"])
    results, kvs = [x], []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        sub = lambda part: {k[len(p + part) + 1:]: t for k, t in w.items() if k.startswith(p + part + ".")}
        h = token_shift(rms_norm(x, eps, w[p + "norm1"]), w[p + "shift"])
        mix, spec = sub("mix"), layer["mixer"]
        src = spec.get("kv_from")
        kvs.append(keys_and_values(h, mix, spec) if src is None else kvs[src])
        x = x + layer_scale(attention(h, mix, spec, kvs[i]), w[p + "ls1"])
        if layer.get("mlp") is not None:
            h = rms_norm(x, eps, w[p + "norm2"])
            y = dense(h, sub("mlp")) if layer["mlp"]["kind"] == "dense" else moe(h, sub("mlp"), layer["mlp"])
            x = x + layer_scale(y, w[p + "ls2"])
        results.append(x)
        x = depth_average(results, w[p + "dwa"])
        if residuals is not None:
            residuals.append(x.clone())
    return rms_norm(x, eps, w["final.norm"]) @ w["head"].T


def generate(config, tensors, prompt, n, dtype=torch.float64):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(config, tensors, toks, dtype)[-1].argmax()))
    return toks[len(prompt):]
