"""Plain, slow restatement of the Gupizen decoder, the oracle of its tests.

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


def centred_weight_norm(x, weight, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms_norm(x, eps, 1 + weight)


def causal_conv(x, w, bias=None):
    """x [T, C], w [C, taps]: the last tap meets the current token."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = sum(w[:, j] * padded[j:j + x.shape[0]] for j in range(taps))
    return y if bias is None else y + bias


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def gelu_erf(x):
    return 0.5 * x * (1 + torch.erf(x / math.sqrt(2)))


# ---- rotary attention with mixed heads ------------------------------------------------------------------------
def frequencies(n, base):
    return [base ** (-2 * i / n) for i in range(n // 2)]


def scaled_frequencies(n, base, s):
    """Slow rotations are slowed further by ``factor``, with a ramp between the two bounds on the wavelength."""
    out = []
    for f in frequencies(n, base):
        length = 2 * math.pi / f
        if s is None or length < s["original"] / s["high"]:
            out.append(f)
        elif length > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            a = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
            out.append((1 - a) * f / s["factor"] + a * f)
    return out


def rotate(x, freqs, sign=1):
    """x [T, heads, n]: neighbours 2i, 2i + 1 of the first 2 len(freqs) columns turn by position * freqs[i]."""
    T, k = x.shape[0], len(freqs)
    a = sign * torch.arange(T, dtype=x.dtype)[:, None, None] * torch.tensor(freqs, dtype=x.dtype)
    u, v = x[..., 0:2 * k:2], x[..., 1:2 * k:2]
    out = x.clone()
    out[..., 0:2 * k:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:2 * k:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def head_weights(q, k, scale, sink, window):
    """[H, T, T] softmax weights with a sink in the denominator; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    s = torch.stack([q[:, h] @ k[:, h // (H // G)].T for h in range(H)]) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) if window is None else (j <= i) & (i - j < window)
    s = s.masked_fill(~seen, -math.inf)
    top = torch.maximum(s.amax(-1), sink[:, None])
    e = torch.exp(s - top[..., None])
    return e / (e.sum(-1) + torch.exp(sink[:, None] - top))[..., None]


def mix_heads(weights, talk):
    return torch.einsum("hg,gij->hij", talk, weights)


def talking_attention(q, k, v, scale, sink, window, talk):
    H, G = q.shape[1], k.shape[1]
    mixed = mix_heads(head_weights(q, k, scale, sink, window), talk)
    return torch.stack([mixed[h] @ v[:, h // (H // G)] for h in range(H)], dim=1)


def attention(h, w, spec):
    T, H, G = h.shape[0], spec["heads"], spec["kv_heads"]
    rot = spec["rot"]
    freqs = scaled_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    v_freqs = frequencies(spec["vdim"], rot["base"])
    q = rotate((h @ w["q"].T).reshape(T, H, -1), freqs)
    k = rotate((h @ w["k"].T).reshape(T, G, -1), freqs)
    v = rotate((h @ w["v"].T).reshape(T, G, -1), v_freqs)
    o = rotate(talking_attention(q, k, v, spec["scale"], w["sink"], spec["mask"]["size"], w["talk"]), v_freqs, -1)
    return o.reshape(T, -1) @ w["o"].T


# ---- real-gated linear recurrent unit -----------------------------------------------------------------------------
def block_gate(u, w, b):
    """u [T, width] in equal parts, each times its own matrix."""
    parts = u.reshape(u.shape[0], w.shape[0], -1)
    return torch.sigmoid(torch.einsum("tbi,boi->tbo", parts, w) + b).reshape(u.shape)


def gated_scan(u, r, i, lam, state=None):
    log_a = -8 * r * torch.nn.functional.softplus(lam)
    a = torch.exp(log_a)
    S = torch.zeros_like(u[0]) if state is None else state
    out = []
    for t in range(u.shape[0]):
        S = a[t] * S + torch.sqrt(1 - a[t] ** 2) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def recurrent_block(h, w):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    S = gated_scan(u, block_gate(u, w["ra"], w["ra.b"]), block_gate(u, w["ri"], w["ri.b"]), w["lam"])
    return (S * y) @ w["o"].T


def side_by_side(left, right, w_left, w_right, eps):
    return 0.5 * (rms_norm(left, eps, w_left) + rms_norm(right, eps, w_right))


# ---- gated delta rule with a decay per channel ---------------------------------------------------------------------
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H], state [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def channel_decay(h, w, heads):
    z = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
    return torch.exp(-torch.exp(w["A_log"])[:, None] * torch.nn.functional.softplus(z).reshape(h.shape[0], heads, -1))


def channel_delta(h, w, spec, eps):
    T, H, G = h.shape[0], spec["heads"], spec["kv_heads"]
    q, k, v = (silu(causal_conv(h @ w[s].T, w[s + ".conv"])) for s in "qkv")
    per_head = lambda x: x.reshape(T, G, -1).repeat_interleave(H // G, dim=1)
    q = unit(per_head(q)) * spec["dim"] ** -0.5
    k = unit(per_head(k))
    o, _ = delta_rule(q, k, v.reshape(T, H, -1), channel_decay(h, w, H), torch.sigmoid(h @ w["b"].T))
    gate = torch.sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(T, H, -1)
    return (rms_norm(o, eps, w["norm"]) * gate).reshape(T, -1) @ w["o"].T


# ---- mixture of experts -----------------------------------------------------------------------------------------------
def route(z, top):
    """logits [T, E] -> (chosen experts [T, top], softmax over the chosen logits)."""
    vals, idx = torch.sort(z, dim=-1, descending=True, stable=True)
    return idx[:, :top], torch.softmax(vals[:, :top], dim=-1)


def expert(h, w_up, w_down):
    return gelu_erf(h @ w_up.T) @ w_down.T


def moe(h, w, spec):
    idx, weight = route(h @ w["router"].T + w["router.b"], spec["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(idx[t].tolist(), weight[t]):
            out[t] += a * expert(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    return out


# ---- model ---------------------------------------------------------------------------------------------------------
def input_conv(h, w):
    return h + causal_conv(h, w)


def layer_order(config):
    """[(layer, whether the embedding output joins the stream right before it)]."""
    loop, n = config.get("loop"), len(config["layers"])
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, t > 0 and i == a) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body + [(i, False) for i in range(b, n)]


def forward(config, tensors, tokens, dtype=torch.float64, residuals=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the stream after every layer run."""
    w = {k: t.to(dtype) for k, t in tensors.items()}
    eps = config["norm"]["eps"]
    start = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    x = start
    for i, joins in layer_order(config):
        layer = config["layers"][i]
        sub = lambda part: {k[len(f"l{i}.{part}."):]: t for k, t in w.items() if k.startswith(f"l{i}.{part}.")}
        if joins:
            x = x + start
        h = input_conv(centred_weight_norm(x, w[f"l{i}.norm1"], eps), w[f"l{i}.canon1"])
        if layer["type"] == "parallel":
            y = side_by_side(attention(h, sub("mix.left"), layer["mixer"]["left"]), recurrent_block(h, sub("mix.right")),
                             w[f"l{i}.mix.left.out"], w[f"l{i}.mix.right.out"], eps)
        else:
            y = channel_delta(h, sub("mix"), layer["mixer"], eps)
        x = x + centred_weight_norm(y, w[f"l{i}.norm1b"], eps)
        if layer.get("mlp") is not None:
            h = input_conv(centred_weight_norm(x, w[f"l{i}.norm2"], eps), w[f"l{i}.canon2"])
            x = x + centred_weight_norm(moe(h, sub("mlp"), layer["mlp"]), w[f"l{i}.norm2b"], eps)
        if residuals is not None:
            residuals.append(x.clone())
    return centred_weight_norm(x, w["final.norm"], eps) @ w["embed"].T


def generate(config, tensors, prompt, n, dtype=torch.float64):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(config, tensors, toks, dtype)[-1].argmax()))
    return toks[len(prompt):]
