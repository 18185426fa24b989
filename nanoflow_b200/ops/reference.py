"""Plain PyTorch fp32 restatements of every kernel in :mod:`nanoflow_b200.ops`.

These are the oracles of the numerics tests and the building blocks of the CPU backend; they run on
any device and make no attempt to be fast. The paged-attention oracle plays the role of the
reference's ``cpu_reference::single_mha`` + ``append_paged_kv_cache`` (gemv/src/cpu_reference.h:47-167).
"""
from __future__ import annotations

from typing import Optional

import torch


def gemm(a, w, residual=None, beta=1.0, bias=None):
    out = a.float() @ w.float().t()
    if bias is not None:
        out = out + bias.float()
    if residual is not None:
        out = out + beta * residual.float()
    return out


def gemm_swiglu(a, w_gate, w_up):
    g = a.float() @ w_gate.float().t()
    u = a.float() @ w_up.float().t()
    return torch.nn.functional.silu(g) * u


def rmsnorm(x, w, eps):
    xf = x.float()
    return xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def silu_mul(gate, up):
    return torch.nn.functional.silu(gate.float()) * up.float()


def rope_inv_freq(head_dim: int, theta: float, scaling: Optional[dict] = None) -> torch.Tensor:
    """Rotary inverse frequencies, with Llama-3.1 style smoothing when ``scaling`` asks for it.

    The reference bakes the same smoothing into its kernel through constants derived in
    pipeline/include/config.h:101-110 and applied in pipeline/include/small_cuda_operator.cuh:36-44.
    """
    inv = 1.0 / (theta ** (torch.arange(0, head_dim, 2, dtype=torch.float64) / head_dim))
    if scaling and scaling.get("rope_type", scaling.get("type")) == "llama3":
        factor = float(scaling["factor"])
        lo = float(scaling.get("low_freq_factor", 1.0))
        hi = float(scaling.get("high_freq_factor", 4.0))
        old = float(scaling.get("original_max_position_embeddings", 8192))
        wavelen = 2 * torch.pi / inv
        smooth = (old / wavelen - lo) / (hi - lo)
        scaled = torch.where(wavelen > old / lo, inv / factor, inv)
        mid = (wavelen <= old / lo) & (wavelen >= old / hi)
        scaled = torch.where(mid, (1 - smooth) * inv / factor + smooth * inv, scaled)
        inv = scaled
    return inv.float()


def rope(x: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor) -> torch.Tensor:
    """x: [T, heads, head_dim]; rotate-half convention (pairs i, i + head_dim/2)."""
    xf = x.float()
    ang = positions.to(x.device).float()[:, None] * inv_freq.to(x.device).float()[None, :]  # [T, hd/2]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
    half = x.shape[-1] // 2
    lo, hi = xf[..., :half], xf[..., half:]
    return torch.cat([lo * cos - hi * sin, hi * cos + lo * sin], dim=-1)


def rope_append(qkv, kv_pool, inv_freq, positions, token_req, kv_indptr, kv_indices, *, q_heads,
                kv_heads, head_dim, q_off, k_off, v_off):
    """Returns rotated q [T, q_heads*hd] (fp32) and writes rotated k / v into kv_pool (in place)."""
    T = qkv.shape[0]
    page_size = kv_pool.shape[3]
    q = qkv[:, q_off:q_off + q_heads * head_dim].reshape(T, q_heads, head_dim)
    k = qkv[:, k_off:k_off + kv_heads * head_dim].reshape(T, kv_heads, head_dim)
    v = qkv[:, v_off:v_off + kv_heads * head_dim].reshape(T, kv_heads, head_dim)
    qr = rope(q, positions, inv_freq)
    kr = rope(k, positions, inv_freq)
    for t in range(T):
        b = int(token_req[t])
        pos = int(positions[t])
        page = int(kv_indices[int(kv_indptr[b]) + pos // page_size])
        slot = pos % page_size
        kv_pool[page, 0, :, slot, :] = kr[t].to(kv_pool.dtype)
        kv_pool[page, 1, :, slot, :] = v[t].to(kv_pool.dtype)
    return qr.reshape(T, q_heads * head_dim)


def gather_kv(kv_pool, kv_indptr, kv_indices, kv_last_page_len, b):
    """Contiguous K, V [kv_len, kv_heads, hd] (fp32) of request b from the paged pool."""
    pages = kv_indices[int(kv_indptr[b]):int(kv_indptr[b + 1])].long()
    page_size = kv_pool.shape[3]
    kv_len = (len(pages) - 1) * page_size + int(kv_last_page_len[b])
    k = kv_pool[pages, 0].permute(0, 2, 1, 3).reshape(-1, kv_pool.shape[2], kv_pool.shape[4])
    v = kv_pool[pages, 1].permute(0, 2, 1, 3).reshape(-1, kv_pool.shape[2], kv_pool.shape[4])
    return k[:kv_len].float(), v[:kv_len].float()


def paged_attention(q, kv_pool, qo_indptr, kv_indptr, kv_indices, kv_last_page_len, *, q_heads,
                    sm_scale=None, requests=None):
    """Causal attention of every query token against its request's paged KV.

    q: [T, q_heads*hd]. The last query token of request b sits at position kv_len-1.
    Returns fp32 [T, q_heads*hd]; rows of requests not in ``requests`` are left zero.
    """
    T = q.shape[0]
    kvh, hd = kv_pool.shape[2], kv_pool.shape[4]
    group = q_heads // kvh
    scale = sm_scale if sm_scale is not None else hd ** -0.5
    out = torch.zeros((T, q_heads * hd), dtype=torch.float32, device=q.device)
    B = len(qo_indptr) - 1
    for b in (requests if requests is not None else range(B)):
        t0, t1 = int(qo_indptr[b]), int(qo_indptr[b + 1])
        if t1 <= t0:
            continue
        k, v = gather_kv(kv_pool, kv_indptr, kv_indices, kv_last_page_len, b)
        kv_len = k.shape[0]
        qb = q[t0:t1].float().reshape(t1 - t0, q_heads, hd)
        kk = k.repeat_interleave(group, dim=1)  # [kv_len, q_heads, hd]
        vv = v.repeat_interleave(group, dim=1)
        s = torch.einsum("thd,khd->htk", qb, kk) * scale
        pos = kv_len - (t1 - t0) + torch.arange(t1 - t0, device=q.device)
        mask = torch.arange(kv_len, device=q.device)[None, :] <= pos[:, None]
        s = s.masked_fill(~mask[None], float("-inf"))
        p = torch.softmax(s, dim=-1)
        out[t0:t1] = torch.einsum("htk,khd->thd", p, vv).reshape(t1 - t0, q_heads * hd)
    return out


def argmax(logits, col_offset=0):
    return logits.float().argmax(dim=-1).int() + col_offset


# ---- layer-list models ---------------------------------------------------------------------------------
def layernorm(x, w, b, eps):
    return torch.nn.functional.layer_norm(x.float(), (x.shape[-1],), w.float(), None if b is None else b.float(), eps)


def gated_act(g, u, act: str, limit=0.0, alpha=1.0, shift=0.0):
    if act == "capped":
        g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        return g * torch.sigmoid(alpha * g) * (u + shift)
    f = {"silu": torch.nn.functional.silu, "relu": torch.relu,
         "gelu_tanh": lambda z: torch.nn.functional.gelu(z, approximate="tanh")}[act]
    return f(g) * u


def gated_mlp(h, w_gate, w_up, w_down, act: str, biases=(None, None, None), **constants):
    g, u = h.float() @ w_gate.float().t(), h.float() @ w_up.float().t()
    plus = lambda t, b: t if b is None else t + b.float()
    return plus(gated_act(plus(g, biases[0]), plus(u, biases[1]), act, **constants) @ w_down.float().t(), biases[2])


def linear_act(x, act: str):
    """Activation of a product without a gate."""
    return torch.nn.functional.gelu(x) if act == "gelu" else torch.relu(x) ** 2


def sinusoid(positions, width, base):
    """[T, width]: sine and cosine of position * base^(-2 i / width), next to each other."""
    f = float(base) ** (-torch.arange(0, width, 2, dtype=torch.float64) / width)
    a = torch.as_tensor(positions, dtype=torch.float64)[:, None] * f
    return torch.stack([torch.sin(a), torch.cos(a)], dim=-1).flatten(1)[:, :width].float()


def _pool_rows(positions, req, kv_indptr, kv_indices, kv_first, page_size):
    """Row numbers of ``positions`` of one request in a pool flattened to [pages * page_size, ...]."""
    slot = positions // page_size - int(kv_first[req])
    assert (slot >= 0).all() and (slot < int(kv_indptr[req + 1] - kv_indptr[req])).all(), "position without a page"
    pages = torch.as_tensor(kv_indices).long()[int(kv_indptr[req]) + slot]
    return pages * page_size + positions % page_size


def latent_append(src, w, pool, positions, token_req, kv_indptr, kv_indices, kv_first, eps):
    """Latents [T, rank] -> RMS norm -> page slots of pool [pages, page_size, ld] (in place)."""
    c = rmsnorm(src, w, eps)
    flat = pool.view(-1, pool.shape[-1])
    for t in range(src.shape[0]):
        row = _pool_rows(torch.as_tensor([int(positions[t])]), int(token_req[t]), kv_indptr, kv_indices, kv_first, pool.shape[1])
        flat[row, :src.shape[1]] = c[t].to(pool.dtype)


def latent_attention(q, pool, positions, token_req, kv_indptr, kv_indices, kv_first, *, scale, window=0, sinks=None):
    """q [T, H, ld] in latent space -> [T, H, ld]: the pool's rows are keys and values."""
    T, H, ld = q.shape
    out = torch.zeros(T, H, ld)
    flat = pool.view(-1, pool.shape[-1]).float()
    for t in range(T):
        pos = int(positions[t])
        keys = torch.arange(max(0, pos - window + 1) if window else 0, pos + 1)
        c = flat[_pool_rows(keys, int(token_req[t]), kv_indptr, kv_indices, kv_first, pool.shape[1])]
        s = q[t].float() @ c.t() * scale
        if sinks is not None:
            s = torch.cat([s, sinks.float()[:, None]], dim=1)
        p = torch.softmax(s, dim=-1)
        out[t] = p[:, :keys.numel()] @ c
    return out


def mlstm(q, k, v, i_pre, f_pre, cap, state, positions, qo_indptr, state_ref):
    """q (scaled), k [T, H, d], v [T, H, vd], gate pre-activations [T, H]; ``state`` = (S, n, m) of all slots, updated in
    place: requests at position 0 start from zero, half ``ref & 1`` of n and m is read, the other written."""
    S_all, n_all, m_all = state
    li = cap * torch.tanh(i_pre.float() / cap)
    lf = torch.nn.functional.logsigmoid(cap * torch.tanh(f_pre.float() / cap))
    out = torch.zeros(v.shape)
    for b in range(len(qo_indptr) - 1):
        t0, t1 = int(qo_indptr[b]), int(qo_indptr[b + 1])
        slot, half = int(state_ref[b]) >> 1, int(state_ref[b]) & 1
        S, n, m = S_all[slot].clone(), n_all[slot, :, half].clone(), m_all[slot, :, half].clone()
        if int(positions[t0]) == 0:
            S, n, m = torch.zeros_like(S), torch.zeros_like(n), torch.zeros_like(m)
        for t in range(t0, t1):
            mn = torch.maximum(lf[t] + m, li[t])
            keep, write = torch.exp(lf[t] + m - mn), torch.exp(li[t] - mn)
            S = keep[:, None, None] * S + write[:, None, None] * k[t].float()[:, :, None] * v[t].float()[:, None, :]
            n = keep[:, None] * n + write[:, None] * k[t].float()
            m = mn
            den = torch.maximum((n * q[t].float()).sum(-1).abs(), torch.exp(-m)) + 1e-6
            out[t] = torch.einsum("hdv,hd->hv", S, q[t].float()) / den[:, None]
        S_all[slot], n_all[slot, :, half ^ 1], m_all[slot, :, half ^ 1] = S, n, m
    return out


def head_norm_gate(o, g, w, vdim, eps):
    """o, g [T, H, vd_padded], w [H, vd_padded]: RMS norm over each head's ``vdim`` values, weight, sigmoid gate."""
    inv = torch.rsqrt(o.float().pow(2).sum(-1, keepdim=True) / vdim + eps)
    return o.float() * inv * w.float() * torch.sigmoid(g.float())


def turn_pairs(x, positions, freqs, sign=1.0):
    """x [T, heads, n]: neighbouring columns 2i, 2i + 1 turn by sign * position * freqs[i]."""
    n = len(freqs)
    a = sign * torch.as_tensor(positions, dtype=torch.float32)[:, None] * torch.tensor(freqs, dtype=torch.float32)
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v, out = x[..., 0:2 * n:2], x[..., 1:2 * n:2], x.clone()
    out[..., 0:2 * n:2], out[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    return out


def talk_attention(q, pool, positions, token_req, kv_indptr, kv_indices, kv_first, *, scale, talk, window=0, sinks=None):
    """q [T, H, hd] -> [T, H, hd]: the heads' softmax weights (exp(sink) in the denominator) are mixed by talk [H, H] before
    they meet the values."""
    T, H, hd = q.shape
    G, ps = pool.shape[2], pool.shape[3]
    out = torch.zeros(T, H, hd)
    for t in range(T):
        pos = int(positions[t])
        keys = torch.arange(max(0, pos - window + 1) if window else 0, pos + 1)
        rows = _pool_rows(keys, int(token_req[t]), kv_indptr, kv_indices, kv_first, ps)
        k, v = (pool[rows // ps, j, :, rows % ps].float() for j in (0, 1))          # [n, G, hd]
        s = torch.einsum("gmd,ngd->gmn", q[t].float().reshape(G, H // G, hd), k).reshape(H, -1) * scale
        if sinks is not None:
            s = torch.cat([s, sinks.float()[:, None]], dim=1)
        p = (talk.float() @ torch.softmax(s, dim=-1)[:, :keys.numel()]).reshape(G, H // G, -1)
        out[t] = torch.einsum("gmn,ngd->gmd", p, v).reshape(H, hd)
    return out


def short_conv(x, w, state, positions, qo_indptr, state_ref, bias=None, act=None, residual=False):
    """x [T, C], w [taps, C], ``state`` [slots, 2, max(1, taps - 1), C] holds each request's last inputs (half ``ref & 1`` is
    read, the other written)."""
    H, out = w.shape[0] - 1, torch.zeros_like(x, dtype=torch.float32)
    for b in range(len(qo_indptr) - 1):
        t0, t1, ref = int(qo_indptr[b]), int(qo_indptr[b + 1]), int(state_ref[b])
        before = state[ref >> 1, ref & 1, :H].float() if int(positions[t0]) else torch.zeros(H, x.shape[1])
        xs = torch.cat([before, x[t0:t1].float()])
        y = sum(w[j].float() * xs[j:j + t1 - t0] for j in range(H + 1))
        y = y if bias is None else y + bias
        y = torch.nn.functional.silu(y) if act == "silu" else y
        out[t0:t1] = y + x[t0:t1] if residual else y
        if H:
            state[ref >> 1, (ref & 1) ^ 1, :H] = xs[xs.shape[0] - H:].to(state.dtype)
    return out


def rglru(u, y, r, i, log_a, state, positions, qo_indptr, state_ref):
    """u, y (before the GELU), gate pre-activations r, i (biases included) [T, C], state [slots, C], updated in place."""
    la = log_a * torch.sigmoid(r)
    a, x = torch.exp(la), torch.sqrt(-torch.expm1(2.0 * la)) * torch.sigmoid(i) * u
    out = torch.zeros_like(x)
    for b in range(len(qo_indptr) - 1):
        t0, t1, slot = int(qo_indptr[b]), int(qo_indptr[b + 1]), int(state_ref[b]) >> 1
        S = state[slot].clone() if int(positions[t0]) else torch.zeros_like(state[slot])
        for t in range(t0, t1):
            S = a[t] * S + x[t]
            out[t] = S
        state[slot] = S
    return out * torch.nn.functional.gelu(y, approximate="tanh")


def delta(q, k, v, x, rate, beta, state, positions, qo_indptr, state_ref, *, q_scale, eps):
    """q, k [T, G, d], v [T, H, dv], x [T, H, d] (decay pre-activation, bias included), rate [H], beta [T, H]
    (pre-activation), state [slots, H, d, dv], updated in place."""
    H = v.shape[1]
    unit = lambda t: (t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + eps)).repeat_interleave(H // t.shape[1], dim=1)
    q, k, out = unit(q.float()) * q_scale, unit(k.float()), torch.zeros(v.shape)
    w, beta = torch.exp(-rate[:, None] * torch.nn.functional.softplus(x.float())), torch.sigmoid(beta.float())
    for b in range(len(qo_indptr) - 1):
        t0, t1, slot = int(qo_indptr[b]), int(qo_indptr[b + 1]), int(state_ref[b]) >> 1
        S = state[slot].clone() if int(positions[t0]) else torch.zeros_like(state[slot])
        for t in range(t0, t1):
            S = w[t][:, :, None] * S
            u = beta[t][:, None] * (v[t].float() - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
            out[t] = torch.einsum("hdv,hd->hv", S, q[t])
        state[slot] = S
    return out


def gqa_append(q, k, v, q_w, k_w, pool, positions, token_req, kv_indptr, kv_indices, kv_first, *, heads, kv_heads, dim, eps):
    """q [T, heads * hd], k, v [T, kv_heads * hd] (padding columns zero), norm weights or None: keys and values go to their
    page slots of pool [pages, 2, kv_heads, page_size, hd] (in place). Returns the normed queries."""
    def norm(x, w, n):
        return x if w is None else x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / n + eps) * w
    q, k = norm(q.float(), q_w, heads * dim), norm(k.float(), k_w, kv_heads * dim)
    T, ps, hd = k.shape[0], pool.shape[3], pool.shape[4]
    for t in range(T):
        row = int(_pool_rows(torch.as_tensor([int(positions[t])]), int(token_req[t]), kv_indptr, kv_indices, kv_first, ps))
        pool[row // ps, 0, :, row % ps] = k[t].reshape(kv_heads, hd).to(pool.dtype)
        pool[row // ps, 1, :, row % ps] = v[t].reshape(kv_heads, hd).to(pool.dtype)
    return q


def gqa_attention(q, pool, positions, token_req, kv_indptr, kv_indices, kv_first, *, scale, softcap=0.0, window=0, sinks=None,
                  dist=None, chunk=0):
    """q [T, H, hd] -> [T, H, hd] over the paged keys and values; capped scores, exp(sink) in the denominator, ``dist`` [H, 2]
    (a, b): scores lose a ln(1 + b distance); ``chunk``: only keys of the position's own run of so many."""
    T, H, hd = q.shape
    G, ps = pool.shape[2], pool.shape[3]
    out = torch.zeros(T, H, hd)
    for t in range(T):
        pos = int(positions[t])
        first = max(0, pos - window + 1) if window else pos // chunk * chunk if chunk else 0
        keys = torch.arange(first, pos + 1)
        rows = _pool_rows(keys, int(token_req[t]), kv_indptr, kv_indices, kv_first, ps)
        k, v = (pool[rows // ps, j, :, rows % ps].float() for j in (0, 1))          # [n, G, hd]
        s = torch.einsum("gmd,ngd->gmn", q[t].float().reshape(G, H // G, hd), k).reshape(H, -1) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if dist is not None:
            s = s - dist[:, :1] * torch.log1p(dist[:, 1:] * (pos - keys).float())
        if sinks is not None:
            s = torch.cat([s, sinks.float()[:, None]], dim=1)
        p = torch.softmax(s, dim=-1)[:, :keys.numel()].reshape(G, H // G, -1)
        out[t] = torch.einsum("gmn,ngd->gmd", p, v).reshape(H, hd)
    return out


def token_shift(h, mu, state, positions, qo_indptr, state_ref):
    """h [T, W], mu [n, W] -> [T, n, W]; ``state`` [slots, 2, W] holds each request's last row (half ``ref & 1`` is read,
    the other written)."""
    prev = torch.zeros_like(h)
    prev[1:] = h[:-1]
    for b in range(len(qo_indptr) - 1):
        t0, t1, ref = int(qo_indptr[b]), int(qo_indptr[b + 1]), int(state_ref[b])
        prev[t0] = state[ref >> 1, ref & 1] if int(positions[t0]) else 0.0
        state[ref >> 1, (ref & 1) ^ 1] = h[t1 - 1]
    return h[:, None] + (prev - h)[:, None] * mu[None]


def wkv(r, k, v, x, u, state, positions, qo_indptr, state_ref):
    """r, k, v, x [T, H, d] (x: log of the decay's negative log), u [H, d], state [slots, H, d, d], updated in place."""
    out = torch.zeros(v.shape)
    w = torch.exp(-torch.exp(x.float()))
    for b in range(len(qo_indptr) - 1):
        t0, t1, slot = int(qo_indptr[b]), int(qo_indptr[b + 1]), int(state_ref[b]) >> 1
        S = state[slot].clone() if int(positions[t0]) else torch.zeros_like(state[slot])
        for t in range(t0, t1):
            kv = k[t].float()[:, :, None] * v[t].float()[:, None, :]
            out[t] = torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t].float())
            S = w[t][:, :, None] * S + kv
        state[slot] = S
    return out


def head_norm_silu(o, g, w, dim, eps):
    """o, g, w [.., H, d_padded]: RMS norm over each head's ``dim`` values, weight, SiLU gate."""
    inv = torch.rsqrt(o.float().pow(2).sum(-1, keepdim=True) / dim + eps)
    return o.float() * inv * w.float() * torch.nn.functional.silu(g.float())


def moe_route(logits, correction, top, groups, keep, scale, score="sigmoid", group_score="top2"):
    """(experts [T, top], weights [T, top]) from router logits [T, E]. ``score`` "softmax": of the chosen logits, the
    correction included; "softmax_all": of all logits, the chosen ones not normed."""
    z = logits.float()
    s = torch.sigmoid(z) if score == "sigmoid" else torch.softmax(z, dim=-1) if score == "softmax_all" else z
    choice = s if correction is None else s + correction
    z = choice
    if groups > 1:
        c = choice.reshape(len(s), groups, -1)
        best = c.topk(min(2 if group_score == "top2" else 1, c.shape[-1]), dim=-1).values.sum(-1).topk(keep, dim=-1).indices
        allowed = torch.zeros(len(s), groups, dtype=torch.bool).scatter_(1, best, True)
        choice = c.masked_fill(~allowed[:, :, None], float("-inf")).reshape(len(s), -1)
    idx = choice.topk(top, dim=-1).indices
    if score == "softmax":
        return idx, torch.softmax(z.gather(1, idx), dim=-1) * scale
    w = s.gather(1, idx)
    if score == "softmax_all":
        return idx, w * scale
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20) * scale
