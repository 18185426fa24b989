"""Plain, slow restatement of the Volarax decoder, the oracle of its tests.

One function per mechanism, whole sequences only, no cache, no batching, nothing shared with the
package. Everything runs in the dtype of the tensors it is given (the tests use float64, so that the
oracle's own rounding never matters). A model is ``(config, tensors)``: the parsed ``config.json`` and a
dict of tensors under their checkpoint names.
"""
import math

import torch


def rms_norm(x, eps, weight=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * weight + bias


def gated_mlp(h, w_gate, w_up, w_down):
    return (torch.relu(h @ w_gate.T) * (h @ w_up.T)) @ w_down.T


def latents(h, w_dkv, norm_weight, eps):
    return rms_norm(h @ w_dkv.T, eps, norm_weight)


def windowed_sink_attention(q, k, v, scale, window, sink):
    """q, k [T, H, dim], v [T, H, vdim], sink [H]; ``window`` None = all earlier tokens."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        j0 = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            s = (k[j0:i + 1, h] @ q[i, h]) * scale
            top = max(float(s.max()), float(sink[h]))
            e = torch.exp(s - top)
            out[i, h] = (e[:, None] * v[j0:i + 1, h]).sum(0) / (e.sum() + math.exp(float(sink[h]) - top))
    return out


def latent_attention(h, w, spec, eps):
    """``w``: the mixer's tensors by their short names."""
    T, H = h.shape[0], spec["heads"]
    q = (h @ w["q"].T).reshape(T, H, spec["dim"])
    c = latents(h, w["dkv"], w["dkv.norm"], eps)
    k = (c @ w["uk"].T).reshape(T, H, spec["dim"])
    v = (c @ w["uv"].T).reshape(T, H, spec["vdim"])
    mask = spec.get("mask")
    o = windowed_sink_attention(q, k, v, spec["scale"], None if mask is None else mask["size"], w["sink"])
    return o.reshape(T, -1) @ w["o"].T


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def log_sigmoid(x):
    return -torch.log1p(torch.exp(-x.abs())) + torch.minimum(x, torch.zeros_like(x))


def mlstm_recurrence(q, k, v, log_i, log_f, state=None):
    """q, k [T, H, dim] (q already scaled), v [T, H, vdim], gates [T, H]. Returns outputs [T, H, vdim] and
    the state (S, n, m) after the last token."""
    T, H, dim = q.shape
    if state is None:
        state = (torch.zeros(H, dim, v.shape[-1], dtype=q.dtype), torch.zeros(H, dim, dtype=q.dtype),
                 torch.zeros(H, dtype=q.dtype))
    S, n, m = state
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        m_new = torch.maximum(log_f[t] + m, log_i[t])
        keep, write = torch.exp(log_f[t] + m - m_new), torch.exp(log_i[t] - m_new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = m_new
        num = (S * q[t][:, :, None]).sum(1)
        den = torch.maximum((n * q[t]).sum(1).abs(), torch.exp(-m)) + 1e-6
        out[t] = num / den[:, None]
    return out, (S, n, m)


def mlstm(h, w, spec, eps):
    T, H, dim, vdim = h.shape[0], spec["heads"], spec["dim"], spec["vdim"]
    q = (h @ w["q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ w["k"].T).reshape(T, H, dim)
    v = (h @ w["v"].T).reshape(T, H, vdim)
    cap = spec["gate_cap"]
    log_i = soft_cap(h @ w["i"].T + w["i.b"], cap)
    log_f = log_sigmoid(soft_cap(h @ w["f"].T + w["f.b"], cap))
    o, _ = mlstm_recurrence(q, k, v, log_i, log_f)
    o = rms_norm(o, eps).reshape(T, -1) * w["norm"] * torch.sigmoid(h @ w["g"].T)
    return o @ w["o"].T


MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm}


def layer_order(config):
    """[(layer, pass whose step vector comes right before it, or None)] in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(config, tensors, tokens, dtype=torch.float64, residuals=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the stream after every layer run."""
    w = {k: t.to(dtype) for k, t in tensors.items()}
    eps = config["norm"]["eps"]
    norm = lambda x, name: layer_norm(x, w[name], w[name + ".b"], eps)
    x = norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], "embed.norm")
    for i, step in layer_order(config):
        if step is not None:
            x = x + w["loop.step"][step]
        spec = config["layers"][i]
        sub = {k[len(f"l{i}.mix."):]: t for k, t in w.items() if k.startswith(f"l{i}.mix.")}
        x = x + norm(MIXERS[spec["type"]](norm(x, f"l{i}.norm1"), sub, spec["mixer"], eps), f"l{i}.norm1b")
        if spec["mlp"] is not None:
            y = gated_mlp(norm(x, f"l{i}.norm2"), w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"])
            x = x + norm(y, f"l{i}.norm2b")
        if residuals is not None:
            residuals.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T


def generate(config, tensors, prompt, n, dtype=torch.float64):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(config, tensors, toks, dtype)[-1].argmax()))
    return toks[len(prompt):]
