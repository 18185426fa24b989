"""Plain, slow restatement of the Zubedra decoder, the oracle of its tests.

One function per mechanism, whole sequences only, no cache, no batching, nothing shared with the package.
Everything runs in the dtype of the tensors it is given (the tests use float64, so that the oracle's own
rounding never matters). A model is ``(config, tensors)``: the parsed ``config.json`` and a dict of tensors
under their checkpoint names.
"""
import math

import torch


def rms_norm(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def centred_norm(x, weight, eps):
    """Layer norm without a bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


# ---- attention ------------------------------------------------------------------------------------------
def soft_cap(s, cap):
    return s if cap is None else cap * torch.tanh(s / cap)


def causal_sink_attention(q, k, v, scale, cap, sink):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim], sink [H]: head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            s = soft_cap((k[:i + 1, g] @ q[i, h]) * scale, cap)
            top = max(float(s.max()), float(sink[h]))
            e = torch.exp(s - top)
            out[i, h] = e @ v[:i + 1, g] / (e.sum() + math.exp(float(sink[h]) - top))
    return out


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attention(h, w, spec, eps, first_values=None):
    """``w``: the mixer's tensors by their short names. Returns (output, values as projected). ``first_values``:
    values of the first value-mixing layer, None in that layer itself and without value mixing."""
    T, H, G = h.shape[0], spec["heads"], spec["kv_heads"]
    q = rms_norm(h @ w["q"].T, eps, w["q.norm"]).reshape(T, H, spec["dim"])
    k = rms_norm(h @ w["k"].T, eps, w["k.norm"]).reshape(T, G, spec["dim"])
    plain = h @ w["v"].T
    v = plain if first_values is None else mix_values(plain, first_values, w["vmix"])
    o = causal_sink_attention(q, k, v.reshape(T, G, spec["vdim"]), spec["scale"], spec.get("softcap"), w["sink"])
    return o.reshape(T, -1) @ w["o"].T, plain


# ---- WKV recurrence -------------------------------------------------------------------------------------
def token_shift(h, before=None):
    """h of the previous token (zeros, or ``before``, ahead of the first one)."""
    first = torch.zeros_like(h[:1]) if before is None else before[None]
    return torch.cat([first, h[:-1]])


def wkv_recurrence(r, k, v, decay, u, state=None):
    """r, k, decay [T, H, d], v [T, H, d], u [H, d], state [H, d (keys), d (values)]."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=r.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=r.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = ((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(1)
        S = decay[t][:, :, None] * S + kv
    return out, S


def wkv(h, w, spec, eps):
    T, H, d = h.shape[0], spec["heads"], spec["dim"]
    shifted = token_shift(h)
    mix = {s: h + (shifted - h) * w["mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[s].T).reshape(T, H, d) for s in "rkv")
    z = mix["g"] @ w["g"].T
    gate = z * torch.sigmoid(z)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).reshape(T, H, d)
    o, _ = wkv_recurrence(r, k, v, decay, w["u"])
    return (rms_norm(o, eps).reshape(T, -1) * w["norm"] * gate) @ w["o"].T


# ---- mixture of experts -----------------------------------------------------------------------------------
def capped_mlp(h, w_gate, w_up, w_down, limit):
    g = torch.clamp(h @ w_gate.T, max=limit)
    u = torch.clamp(h @ w_up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w_down.T


def route(scores, correction, router):
    """scores [T, E] -> (chosen experts [T, top], their weights)."""
    choice = scores + correction
    groups = router.get("groups")
    chosen = []
    for t in range(scores.shape[0]):
        c = choice[t].tolist()
        E = len(c)
        allowed = list(range(E))
        if groups:
            n = E // groups["count"]
            strength = [sum(sorted(c[g * n:(g + 1) * n], reverse=True)[:2]) for g in range(groups["count"])]
            best = sorted(range(groups["count"]), key=lambda g: -strength[g])[:groups["keep"]]
            allowed = [e for e in allowed if e // n in best]
        chosen.append(sorted(allowed, key=lambda e: -c[e])[:router["top"]])
    idx = torch.tensor(chosen)
    s = torch.gather(scores, 1, idx)
    return idx, s / (s.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def moe(h, w, spec):
    idx, weight = route(torch.sigmoid(h @ w["router"].T), w["correction"], spec["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(idx[t].tolist(), weight[t]):
            out[t] += a * capped_mlp(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], spec["expert"]["limit"])[0]
    if spec.get("shared"):
        y = capped_mlp(h, w["shared.gate"], w["shared.up"], w["shared.down"], spec["shared"]["limit"])
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * y
    return out


# ---- model ---------------------------------------------------------------------------------------------------
def forward(config, tensors, tokens, dtype=torch.float64, residuals=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the stream after every layer."""
    w = {k: t.to(dtype) for k, t in tensors.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    first_values = None
    for i, layer in enumerate(config["layers"]):
        sub = lambda part: {k[len(f"l{i}.{part}."):]: t for k, t in w.items() if k.startswith(f"l{i}.{part}.")}
        h = centred_norm(x, w[f"l{i}.norm1"], eps)
        if layer["type"] == "attention":
            mixes = bool(layer["mixer"].get("v_mix"))
            y, plain = attention(h, sub("mix"), layer["mixer"], eps, first_values if mixes else None)
            if mixes and first_values is None:
                first_values = plain
        else:
            y = wkv(h, sub("mix"), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + moe(h, sub("mlp"), layer["mlp"])
        x = x + y
        if residuals is not None:
            residuals.append(x.clone())
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T * config["logit_scale"]


def generate(config, tensors, prompt, n, dtype=torch.float64):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(config, tensors, toks, dtype)[-1].argmax()))
    return toks[len(prompt):]
