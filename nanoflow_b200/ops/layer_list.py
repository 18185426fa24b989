"""Python entry points for the layer-list kernels (residual step, attention, recurrences, mixture of experts, general
GEMM forms).

Like the functions of :mod:`nanoflow_b200.ops` they take torch CUDA tensors, check what the C ABI cannot and
launch on the current stream; engines do not call them but put the same parameter blocks into their op graph.
"""
from __future__ import annotations

from ctypes import byref, c_longlong
from typing import Optional

import torch

from . import (ACTS, CONV_ACTS, LIN_ACTS, NORMS, ROUTER_SCORES, AttnParams, DeltaParams, GemmParams, GqaAppendParams, GqaAttnParams, HeadNormGateParams,
               LatentAppendParams, LatentAttnParams, LatentGatherParams, MlstmParams, MoeGemmParams, MoePermuteParams,
               MoeRouteParams, ResidualNormParams, RgLruParams, ShortConvParams, TalkAttnParams, TokenShiftParams, WkvParams, _check, _i32, _p, _stream, dtype_code, lib)


def _f32(t: Optional[torch.Tensor], name: str) -> None:
    if t is not None and (t.dtype != torch.float32 or not t.is_cuda or t.stride(-1) != 1):
        raise RuntimeError(f"{name} must be a CUDA float32 tensor with unit inner stride")


def gemm(a: torch.Tensor, w: torch.Tensor, *, out: Optional[torch.Tensor] = None, up: Optional[torch.Tensor] = None,
         act: str = "silu", out32: Optional[torch.Tensor] = None, f32_col0: int = 0, groups: int = 1, group_k: int = 0,
         k: int = 0, lin_act: Optional[str] = None, bias=None, up_bias=None, limit: float = 0.0, alpha: float = 1.0, shift: float = 0.0,
         workspace: Optional[torch.Tensor] = None, status=None, **shape) -> Optional[torch.Tensor]:
    """a @ w^T in the storage type of the operands (bf16: tensor cores, fp32: FMA). ``up``: act(a @ w^T) * (a @ up^T).
    ``out32``: columns from ``f32_col0`` on are written there as fp32. ``groups``: block-diagonal product. ``lin_act``:
    activation of the finished columns; ``bias``, ``up_bias``: one per column; ``limit``, ``alpha``, ``shift``: constants of the "capped" gated form."""
    M, N, p = a.shape[0], w.shape[0], GemmParams()
    if a.dtype != w.dtype or a.stride(1) != 1 or w.stride(1) != 1:
        raise RuntimeError("gemm: operands of one type with unit inner stride expected")
    _f32(out32, "out32")
    if out is None and not (out32 is not None and f32_col0 == 0):
        out = torch.zeros(M, f32_col0 if out32 is not None else N, dtype=a.dtype, device=a.device)
    p.A, p.B, p.B2, p.D = _p(a), _p(w), _p(up), _p(out)
    p.lda, p.ldb, p.ldd = a.stride(0), w.stride(0), out.stride(0) if out is not None else N
    p.M, p.N, p.K = M, N, k or w.shape[1]
    p.epilogue, p.act, p.groups, p.group_k = (1 if up is not None else 0), ACTS[act], groups, group_k
    p.lin_act, p.bias, p.act_limit, p.act_alpha, p.act_shift = LIN_ACTS[lin_act], _p(bias), limit, alpha, shift
    p.bias2 = _p(up_bias)
    if out32 is not None:
        p.D32, p.ld32, p.f32_col0 = _p(out32), out32.stride(0), f32_col0
    if workspace is not None:
        p.workspace, p.workspace_bytes = _p(workspace), workspace.numel() * workspace.element_size()
    p.status = _p(status)
    for key, v in shape.items():
        setattr(p, key, v)
    name = "nfk_gemm_f32" if a.dtype == torch.float32 else "nfk_gemm_bf16"
    _check(getattr(lib(), name)(byref(p), _stream()), name)
    return out


def residual_norm(x: torch.Tensor, *, y=None, table=None, ids=None, feedback_src=None, prev_tokens=None, norm_in=None,
                  add=None, h=None, norm_out=None, rows_idx=None, src_scale: float = 1.0, y2=None, y2_gate=None, experts=None,
                  cols: int, eps: float, rows: Optional[int] = None, norm_sum: bool = False, pair=None, table_add: bool = False,
                  conv=None, pos=None, history=None, status=None) -> None:
    """x <- (table ? 0 : x) + norm_in(src_scale * (y or table[ids])) (+ y2_gate y2) (+ weighted rows of ``experts``:
    outputs, slots, weights) (+ add); h <- norm_out(x). Norms: (kind, weight, bias). ``norm_sum``: norm_in of the whole
    sum; ``pair``: two RMS weights, the source is the mean of the normed y and y2; ``table_add``: the embedding row joins
    the stream instead of being the source; ``conv``: (weights [taps, ld], output, state, state references, positions,
    rows): the input convolution of the first rows; ``pos``: (positions, frequencies [n, 2] as sums of two floats): the
    sinusoidal vector that joins the embedding row; ``history``: (earlier results [n, rows, ld], weights [n + 1] or None,
    where the sum goes or None): what goes on is the weighted sum of the results and this one."""
    p = ResidualNormParams()
    if pos is not None:
        _i32(pos[0], "positions"); _f32(pos[1], "frequencies")
        p.positions, p.pos_freq = _p(pos[0]), _p(pos[1])
    if history is not None:
        hist, hw, hout = history
        _f32(hist, "history"); _f32(hw, "history weights"); _f32(hout, "history output")
        p.hist, p.hist_w, p.hist_out = _p(hist), _p(hw), _p(hout)
        if hist is not None:
            p.hist_n, p.hist_stride = hist.shape[0], hist.stride(0)
            assert hist.stride(1) == x.stride(0)
    if conv is not None:
        w, out, state, ref, pos, n = conv
        _f32(w, "conv"); _i32(ref, "state references"); _i32(pos, "positions")
        p.conv_w, p.conv_out, p.conv_state, p.state_slot, p.positions = _p(w), _p(out), _p(state), _p(ref), _p(pos)
        p.conv_taps, p.conv_rows, p.conv_ld, p.num_slots = w.shape[0], n, w.shape[1], state.shape[0]
    p.norm_sum, p.table_add = int(norm_sum), int(table_add)
    if pair is not None:
        _f32(pair[0], "pair"); _f32(pair[1], "pair")
        p.pair_w, p.pair_w2 = _p(pair[0]), _p(pair[1])
    _f32(x, "x")
    p.x, p.ld_x = _p(x), x.stride(0)
    typed = next(t for t in (y, table, h, y2) if t is not None)
    p.src_scale = src_scale
    if y2 is not None:
        _f32(y2_gate, "y2_gate")
        p.y2, p.ld_y2, p.y2_gate = _p(y2), y2.stride(0), _p(y2_gate)
    if experts is not None:
        out, slot, weight = experts
        _i32(slot, "slots"); _f32(weight, "weights")
        p.e_out, p.ld_e, p.e_rows = _p(out), out.stride(0), out.shape[0]
        p.e_slot, p.e_weight, p.e_top = _p(slot), _p(weight), slot.shape[1]
    p.dtype = dtype_code(typed.dtype)
    if y is not None:
        p.y, p.ld_y = _p(y), y.stride(0)
    if table is not None:
        p.table, p.ld_table, p.vocab = _p(table), table.stride(0), table.shape[0]
        p.host_ids, p.feedback_src, p.prev_tokens = _p(ids), _p(feedback_src), _p(prev_tokens)
    if norm_in is not None:
        p.in_kind, p.in_w, p.in_b = NORMS[norm_in[0]], _p(norm_in[1]), _p(norm_in[2])
    p.add = _p(add)
    if h is not None:
        p.h, p.ld_h = _p(h), h.stride(0)
        if norm_out is not None:
            p.out_kind, p.out_w, p.out_b = NORMS[norm_out[0]], _p(norm_out[1]), _p(norm_out[2])
    if rows_idx is not None:
        _i32(rows_idx, "rows_idx")
        p.rows_idx, p.in_rows = _p(rows_idx), x.shape[0]
    p.rows = rows if rows is not None else (rows_idx.numel() if rows_idx is not None else x.shape[0])
    p.cols, p.eps, p.status = cols, eps, _p(status)
    _check(lib().nfk_residual_norm(byref(p), _stream()), "nfk_residual_norm")


def latent_append(src, w, pool, positions, token_req, kv_indptr, kv_indices, kv_first=None, *, rank: int, eps: float,
                  status=None) -> None:
    """RMS-normed latents of src[:, :rank] into their slots of pool [pages, page size, row size]."""
    _f32(w, "w")
    p = LatentAppendParams(src=_p(src), ld_src=src.stride(0), w=_p(w), pool=_p(pool), ld=pool.shape[2],
                           positions=_p(positions), token_req=_p(token_req), kv_indptr=_p(kv_indptr),
                           kv_indices=_p(kv_indices), kv_first=_p(kv_first), T=src.shape[0], rank=rank,
                           page_size=pool.shape[1], num_pages=pool.shape[0], eps=eps, dtype=dtype_code(pool.dtype),
                           status=_p(status))
    _check(lib().nfk_latent_append(byref(p), _stream()), "nfk_latent_append")


def pool_to_rows(pool: torch.Tensor) -> torch.Tensor:
    """A latent pool [pages, page size, row size] as plain rows in the same shape: bf16 pages whose row size is a multiple
    of 64 are stored in tiles of 8 rows x 64 columns (see kernels.h)."""
    n, ps, ld = pool.shape
    if pool.dtype != torch.bfloat16 or ld % 64 or ps % 8:
        return pool
    return pool.reshape(n, ps // 8, ld // 64, 8, 64).permute(0, 1, 3, 2, 4).reshape(n, ps, ld)


def rows_to_pool(rows: torch.Tensor) -> torch.Tensor:
    """The inverse of :func:`pool_to_rows`."""
    n, ps, ld = rows.shape
    if rows.dtype != torch.bfloat16 or ld % 64 or ps % 8:
        return rows
    return rows.reshape(n, ps // 8, 8, ld // 64, 64).permute(0, 1, 3, 2, 4).reshape(n, ps, ld)


def latent_gather(pool: torch.Tensor, page_ids: torch.Tensor, status=None) -> torch.Tensor:
    """Pages of a latent pool as plain rows [n * page size, row size]."""
    _i32(page_ids, "page_ids")
    out = torch.zeros(page_ids.numel() * pool.shape[1], pool.shape[2], dtype=pool.dtype, device=pool.device)
    p = LatentGatherParams(pool=_p(pool), out=_p(out), page_ids=_p(page_ids), ld=pool.shape[2], n_pages=page_ids.numel(),
                           page_size=pool.shape[1], num_pages=pool.shape[0], dtype=dtype_code(pool.dtype), status=_p(status))
    _check(lib().nfk_latent_gather(byref(p), _stream()), "nfk_latent_gather")
    return out


def latent_attention(q, pool, out, tokens, positions, token_req, kv_indptr, kv_indices, kv_first=None, *, heads: int,
                     scale: float, window: int = 0, sinks=None, impl: int = 0, splits: int = 1, workspace=None,
                     status=None) -> None:
    """Attention of the listed token rows over latent rows; q and out are [T, heads * row size]."""
    _i32(tokens, "tokens")
    _f32(sinks, "sinks")
    p = LatentAttnParams(q=_p(q), ld_q=q.stride(0), pool=_p(pool), ld=pool.shape[2], out=_p(out), ld_out=out.stride(0),
                         tokens=_p(tokens), positions=_p(positions), token_req=_p(token_req), kv_indptr=_p(kv_indptr),
                         kv_indices=_p(kv_indices), kv_first=_p(kv_first), sinks=_p(sinks), n_tokens=tokens.numel(),
                         heads=heads, page_size=pool.shape[1], num_pages=pool.shape[0], window=window, scale=scale,
                         dtype=dtype_code(pool.dtype), impl=impl, splits=splits, workspace=_p(workspace),
                         workspace_floats=0 if workspace is None else workspace.numel(), status=_p(status))
    _check(lib().nfk_latent_attn(byref(p), _stream()), "nfk_latent_attn")


def attn_prefill_rows(q, kv, out, qo_indptr, kv_indptr, page_ids, kv_last_page_len, items, *, heads: int, scale: float,
                      window: int = 0, sinks=None, k_col: int = 0, v_col: Optional[int] = None, status=None) -> None:
    """The tcgen05 prefill kernel over expanded rows: q [T, >= heads * 128], kv [rows, ...] with head h's key at column
    k_col + 128 h and value at v_col + 128 h; page id x of a request stands for rows 16 x ... of kv."""
    p = AttnParams()
    p.q, p.out, p.kv_pool = _p(q), _p(out), _p(kv)
    p.qo_indptr, p.kv_indptr, p.kv_indices = _p(qo_indptr), _p(kv_indptr), _p(page_ids)
    p.kv_last_page_len, p.items, p.num_items = _p(kv_last_page_len), _p(items), items.shape[0]
    p.q_heads = p.kv_heads = heads
    p.head_dim, p.page_size, p.num_pages, p.sm_scale = 128, 16, kv.shape[0] // 16, scale
    p.window, p.sinks, p.status = window, _p(sinks), _p(status)
    p.kv_ld, p.k_col, p.v_col = kv.stride(0), k_col, heads * 128 if v_col is None else v_col
    p.q_rows, p.ld_q = q.shape[0], q.stride(0)
    _check(lib().nfk_attn_prefill_ws(byref(p), _stream()), "nfk_attn_prefill_ws")


def mlstm(qkv, gates, i_bias, f_bias, state, out, positions, qo_indptr, state_ref, *, heads: int, dim: int, vdim: int,
          gate_cap: float, q_scale: float, req_begin: int = 0, req_count: Optional[int] = None, decode: bool = False,
          impl: int = 0, items=None, scratch=None, status=None) -> None:
    """qkv rows are q | k | v of all heads; ``state`` = (S, n, m) of all slots (see kernels.h); out fp32 [T, heads * vdim].
    ``decode``: every request has one token. ``items`` [n, 4]: segments for the chunked form."""
    for t, nm in ((gates, "gates"), (i_bias, "i_bias"), (f_bias, "f_bias"), (out, "out")):
        _f32(t, nm)
    S, n, m = state
    p = MlstmParams(qkv=_p(qkv), ld_qkv=qkv.stride(0), q_off=0, k_off=heads * dim, v_off=2 * heads * dim, gates=_p(gates),
                    ld_gates=gates.stride(0), i_bias=_p(i_bias), f_bias=_p(f_bias), S=_p(S), n=_p(n), m=_p(m), out=_p(out),
                    ld_out=out.stride(0), positions=_p(positions), qo_indptr=_p(qo_indptr), state_slot=_p(state_ref),
                    req_begin=req_begin, req_count=qo_indptr.numel() - 1 if req_count is None else req_count, heads=heads,
                    dim=dim, vdim=vdim, num_slots=S.shape[0], gate_cap=gate_cap, q_scale=q_scale,
                    dtype=dtype_code(qkv.dtype), impl=impl, items=_p(items), num_items=0 if items is None else items.shape[0],
                    num_tokens=qkv.shape[0],
                    scratch=_p(scratch), scratch_floats=0 if scratch is None else scratch.numel(), status=_p(status))
    name = "nfk_mlstm_decode" if decode else "nfk_mlstm_prefill"
    _check(getattr(lib(), name)(byref(p), _stream()), name)


def mlstm_scratch_floats(items: int, heads: int, dim: int, vdim: int, tokens: int, segmented: bool = True) -> int:
    gates = (tokens // 64 + items + 1) * heads * 192
    return gates + (items * heads * (dim * vdim + dim + 8) if segmented else 0)


def head_norm_gate(o, g, w, out, *, heads: int, vdim: int, eps: float) -> None:
    """out = RMS norm of each head's values * w * sigmoid(g); o fp32 [T, heads * padded vdim]."""
    _f32(o, "o"); _f32(w, "w")
    p = HeadNormGateParams(o=_p(o), ld_o=o.stride(0), g=_p(g), ld_g=g.stride(0), w=_p(w), out=_p(out), ld_out=out.stride(0),
                           T=o.shape[0], heads=heads, vdim=vdim, vdim_p=w.numel() // heads, eps=eps, dtype=dtype_code(out.dtype))
    _check(lib().nfk_head_norm_gate(byref(p), _stream()), "nfk_head_norm_gate")


def gqa_append(src, q_out, pool, positions, token_req, kv_indptr, kv_indices, kv_first=None, *, heads: int, dim: int,
               q_w=None, k_w=None, v_first=None, v_mode: int = 0, v_lambda: float = 0.0, eps: float, rot=None, v_rot=None,
               status=None) -> None:
    """src rows are q | k | v (heads padded to the pool's head size); normed keys and the values go to ``pool`` [pages, 2,
    kv_heads, page size, head size], normed queries to ``q_out`` (None: they stay where they are). ``rot``, ``v_rot``: (table of angles [T, n, 2], pairs per
    head) for queries and keys, and for values."""
    for t, nm in ((q_w, "q_w"), (k_w, "k_w"), (rot and rot[0], "rot"), (v_rot and v_rot[0], "v_rot")):
        _f32(t, nm)
    n, _, G, ps, hd = pool.shape
    p = GqaAppendParams(src=_p(src), ld_src=src.stride(0), q_off=0, k_off=heads * hd, v_off=(heads + G) * hd, q_out=_p(q_out),
                        q_w=_p(q_w), k_w=_p(k_w), v_first=_p(v_first), v_mode=v_mode, v_lambda=v_lambda, pool=_p(pool),
                        positions=_p(positions), token_req=_p(token_req), kv_indptr=_p(kv_indptr), kv_indices=_p(kv_indices),
                        kv_first=_p(kv_first), T=src.shape[0], heads=heads, kv_heads=G, hd=hd, dim=dim, page_size=ps,
                        num_pages=n, eps=eps, dtype=dtype_code(pool.dtype), status=_p(status))
    if rot is not None:
        p.rot, p.rot_ld, p.rot_pairs = _p(rot[0]), rot[0].shape[1], rot[1]
    if v_rot is not None:
        p.v_rot, p.v_ld, p.v_pairs = _p(v_rot[0]), v_rot[0].shape[1], v_rot[1]
    _check(lib().nfk_gqa_append(byref(p), _stream()), "nfk_gqa_append")


def gqa_attention(q, pool, out, positions, token_req, kv_indptr, kv_indices, kv_first=None, *, heads: int, scale: float,
                  softcap: float = 0.0, window: int = 0, sinks=None, token_begin: int = 0, n_tokens: Optional[int] = None,
                  dist=None, chunk: int = 0, ld_q: int = 0, status=None) -> None:
    """The simple kernel: any head size, bf16 or fp32; q, out [T, heads * head size]."""
    _f32(sinks, "sinks"); _f32(dist, "dist")
    n, _, G, ps, hd = pool.shape
    p = GqaAttnParams(q=_p(q), pool=_p(pool), out=_p(out), positions=_p(positions), token_req=_p(token_req),
                      kv_indptr=_p(kv_indptr), kv_indices=_p(kv_indices), kv_first=_p(kv_first), sinks=_p(sinks),
                      token_begin=token_begin, n_tokens=q.shape[0] - token_begin if n_tokens is None else n_tokens, heads=heads,
                      kv_heads=G, hd=hd, page_size=ps, num_pages=n, window=window, scale=scale, softcap=softcap,
                      dtype=dtype_code(pool.dtype), status=_p(status), dist=_p(dist), chunk=chunk, ld_q=ld_q)
    _check(lib().nfk_gqa_attn(byref(p), _stream()), "nfk_gqa_attn")


def paged_attention(q, pool, out, qo_indptr, kv_indptr, kv_indices, kv_last_page_len, *, heads: int, scale: float,
                    softcap: float = 0.0, sinks=None, items=None, req_count: int = 0, chunk_pages: int = 0,
                    max_chunks: int = 1, workspace=None, dist=None, chunk: int = 0, kv_first=None, ld_q: int = 0,
                    status=None) -> None:
    """The tensor-core kernels with capped scores, sinks, distance biases, chunks and probabilities in two parts: portions (``items`` [n, 3]: request,
    first token, tokens) on the prefill kernel, else single tokens of the first ``req_count`` requests."""
    _f32(sinks, "sinks"); _f32(dist, "dist")
    p = AttnParams()
    p.q, p.out, p.kv_pool = _p(q), _p(out), _p(pool)
    p.qo_indptr, p.kv_indptr, p.kv_indices = _p(qo_indptr), _p(kv_indptr), _p(kv_indices)
    p.kv_last_page_len, p.q_heads, p.kv_heads = _p(kv_last_page_len), heads, pool.shape[2]
    p.head_dim, p.page_size, p.num_pages, p.sm_scale = pool.shape[4], pool.shape[3], pool.shape[0], scale
    p.softcap, p.sinks, p.precise, p.status = softcap, _p(sinks), 1, _p(status)
    p.dist, p.chunk, p.kv_first, p.ld_q = _p(dist), chunk, _p(kv_first), ld_q
    if items is not None:
        p.items, p.num_items = _p(items), items.shape[0]
        _check(lib().nfk_attn_prefill_ws(byref(p), _stream()), "nfk_attn_prefill_ws")
        return
    p.req_count, p.chunk_pages, p.max_chunks, p.workspace = req_count, chunk_pages, max_chunks, _p(workspace)
    _check(lib().nfk_attn_decode(byref(p), _stream()), "nfk_attn_decode")


def talk_attention(q, pool, out, positions, token_req, kv_indptr, kv_indices, kv_first=None, *, heads: int, scale: float, talk,
                   window: int = 0, sinks=None, v_rot=None, token_begin: int = 0, n_tokens: Optional[int] = None,
                   items=None, max_keys: int = 0, status=None) -> None:
    """Attention whose heads' weights are mixed by ``talk`` [heads, heads]; q, out [T, heads * head size]. ``v_rot``: (table
    of angles [T, n, 2], pairs per head) by which outputs turn back. ``items`` [n, 3] (request, first token, at most 16
    tokens): the prefill kernel; ``max_keys``: the decode kernel; else the simple one (any head size, bf16 or fp32)."""
    _f32(sinks, "sinks"); _f32(talk, "talk")
    n, _, G, ps, hd = pool.shape
    p = TalkAttnParams(q=_p(q), pool=_p(pool), out=_p(out), positions=_p(positions), token_req=_p(token_req),
                       kv_indptr=_p(kv_indptr), kv_indices=_p(kv_indices), kv_first=_p(kv_first), sinks=_p(sinks),
                       talk=_p(talk), token_begin=token_begin, n_tokens=q.shape[0] - token_begin if n_tokens is None else n_tokens,
                       heads=heads, kv_heads=G, hd=hd, page_size=ps, num_pages=n, window=window, scale=scale,
                       dtype=dtype_code(pool.dtype), status=_p(status))
    if v_rot is not None:
        _f32(v_rot[0], "v_rot")
        p.v_rot, p.v_ld, p.v_pairs = _p(v_rot[0]), v_rot[0].shape[1], v_rot[1]
    name = "nfk_talk_attn"
    if items is not None:
        _i32(items, "items")
        p.items, p.num_items, name = _p(items), items.shape[0], "nfk_talk_attn_prefill"
    elif max_keys:
        p.max_keys, name = max_keys, "nfk_talk_attn_decode"
    _check(getattr(lib(), name)(byref(p), _stream()), name)


def short_conv(x, w, state, state_ref, positions, token_req, qo_indptr, *, bias=None, act: Optional[str] = None,
               residual: bool = False, row_begin: int = 0, status=None) -> torch.Tensor:
    """x [T, cols], w [taps, cols]; ``state`` [slots, 2, max(1, taps - 1), cols] in place (one half is read, the other
    written)."""
    _f32(w, "w"); _f32(bias, "bias")
    out = torch.zeros(x.shape[0], w.shape[1], dtype=x.dtype, device=x.device)
    p = ShortConvParams(x=_p(x), ld_x=x.stride(0), out=_p(out), ld_out=out.stride(0), w=_p(w), bias=_p(bias), state=_p(state),
                        state_slot=_p(state_ref), positions=_p(positions), token_req=_p(token_req), qo_indptr=_p(qo_indptr),
                        row_begin=row_begin, T=x.shape[0], cols=w.shape[1], taps=w.shape[0], act=CONV_ACTS[act],
                        residual=int(residual), num_slots=state.shape[0], dtype=dtype_code(x.dtype), status=_p(status))
    _check(lib().nfk_short_conv(byref(p), _stream()), "nfk_short_conv")
    return out


def rglru(u, y, gates, r_b, i_b, log_a, state, out, positions, qo_indptr, state_ref, *, block: int, req_begin: int = 0,
          req_count: Optional[int] = None, decode: bool = False, status=None) -> None:
    """u, y, out [T, cols], gates [T, 2 cols] (per block of channels: recurrence gates, input gates), ``state`` [slots, cols] in
    place. ``decode``: every request has one token."""
    for t, nm in ((gates, "gates"), (r_b, "r_b"), (i_b, "i_b"), (log_a, "log_a"), (state, "state")):
        _f32(t, nm)
    p = RgLruParams(u=_p(u), ld_u=u.stride(0), y=_p(y), ld_y=y.stride(0), gates=_p(gates), ld_g=gates.stride(0), r_b=_p(r_b),
                    i_b=_p(i_b), log_a=_p(log_a), S=_p(state), out=_p(out), ld_out=out.stride(0), positions=_p(positions),
                    qo_indptr=_p(qo_indptr), state_slot=_p(state_ref), req_begin=req_begin,
                    req_count=qo_indptr.numel() - 1 - req_begin if req_count is None else req_count, cols=state.shape[1],
                    block=block, num_slots=state.shape[0], dtype=dtype_code(u.dtype), status=_p(status))
    name = "nfk_rglru_decode" if decode else "nfk_rglru_prefill"
    _check(getattr(lib(), name)(byref(p), _stream()), name)


def delta(qkv, x, beta, g, rate, dt_bias, norm, state, y, positions, qo_indptr, state_ref, *, kv_heads: int, vdim_real: int,
          q_scale: float, eps: float, unit_eps: float = 1e-6, decode: int = 0, items=None, seq=None, status=None) -> None:
    """qkv rows are q | k (kv_heads each) | v, x [T, heads * dim], beta [T, >= heads], g [T, heads * vdim]; ``state`` [slots,
    heads, dim, vdim] in place. ``decode``: the first so many requests have one token each; else ``items`` [n, 4] in chunks
    and the requests ``seq`` token by token."""
    for t, nm in ((x, "x"), (beta, "beta"), (rate, "rate"), (dt_bias, "dt_bias"), (norm, "norm"), (state, "state")):
        _f32(t, nm)
    slots, heads, dim, vdim = state.shape
    o = torch.zeros(qkv.shape[0], heads * vdim, device=qkv.device)
    n = 0 if items is None else items.shape[0]
    lib().nfk_delta_item_floats.restype = c_longlong
    ws = torch.zeros(max(1, n) * heads * lib().nfk_delta_item_floats(dim, vdim), device=qkv.device)
    p = DeltaParams(qkv=_p(qkv), ld=qkv.stride(0), q_off=0, k_off=kv_heads * dim, v_off=2 * kv_heads * dim, x=_p(x),
                    ld_x=x.stride(0), beta=_p(beta), ld_b=beta.stride(0), g=_p(g), ld_g=g.stride(0), rate=_p(rate),
                    dt_bias=_p(dt_bias), norm=_p(norm), S=_p(state), y=_p(y), ld_y=y.stride(0), positions=_p(positions),
                    qo_indptr=_p(qo_indptr), state_slot=_p(state_ref), req_begin=0, req_count=decode, heads=heads,
                    kv_heads=kv_heads, dim=dim, vdim=vdim, vdim_real=vdim_real, num_slots=slots, q_scale=q_scale,
                    unit_eps=unit_eps, eps=eps, dtype=dtype_code(qkv.dtype), seq_reqs=_p(seq),
                    num_seq=0 if seq is None else seq.numel(), o=_p(o), items=_p(items), num_items=n, scratch=_p(ws),
                    scratch_floats=ws.numel(), status=_p(status),
                    num_portions=0 if items is None else int((items[:, 3] == 0).sum()))
    name = "nfk_delta_decode" if decode else "nfk_delta_prefill"
    _check(getattr(lib(), name)(byref(p), _stream()), name)


def moe_route(logits, correction, counts, *, top: int, experts: int, groups: int = 1, keep: int = 1, scale: float,
              gate_col: int = -1, score: str = "sigmoid", identity: int = 0, group_max: bool = False):
    """(experts [T, top], weights, ranks, gate [T]); ``counts`` [experts] is increased. ``identity``: outputs behind the
    experts that stand for the input; gate is then the sum of their weights."""
    _f32(logits, "logits"); _f32(correction, "correction"); _i32(counts, "counts")
    T, dev = logits.shape[0], logits.device
    idx, rank = (torch.zeros(T, top, dtype=torch.int32, device=dev) for _ in range(2))
    weight, gate = torch.zeros(T, top, device=dev), torch.zeros(T, device=dev)
    p = MoeRouteParams(logits=_p(logits), ld=logits.stride(0), correction=_p(correction), expert=_p(idx), weight=_p(weight),
                       rank=_p(rank), counts=_p(counts), gate=_p(gate), T=T, experts=experts, top=top, groups=groups, keep=keep,
                       gate_col=gate_col, scale=scale, score=ROUTER_SCORES[score], identity=identity, group_max=int(group_max))
    _check(lib().nfk_moe_route(byref(p), _stream()), "nfk_moe_route")
    return idx, weight, rank, gate


def moe_permute(h, expert, rank, counts):
    """(rows of h in expert order [T * top, cols], slots [T, top])."""
    T, top = expert.shape
    out = torch.zeros(T * top, h.shape[1], dtype=h.dtype, device=h.device)
    slot = torch.zeros(T, top, dtype=torch.int32, device=h.device)
    p = MoePermuteParams(h=_p(h), ld_h=h.stride(0), out=_p(out), ld_out=out.stride(0), expert=_p(expert), rank=_p(rank),
                         counts=_p(counts), slot=_p(slot), T=T, top=top, experts=counts.numel(), cols=h.shape[1],
                         dtype=dtype_code(h.dtype))
    _check(lib().nfk_moe_permute(byref(p), _stream()), "nfk_moe_permute")
    return out, slot


def moe_gemm(a, w, counts, *, up=None, act: str = "silu", limit: float = 0.0, alpha: float = 1.0, shift: float = 0.0,
             lin_act: Optional[str] = None, status=None) -> torch.Tensor:
    """Rows of ``a`` in expert order times their expert's matrix; w (and up) [experts * N, K]. ``lin_act``: activation
    without ``up``."""
    _i32(counts, "counts")
    E = counts.numel()
    n = w.shape[0] // E
    out = torch.zeros(a.shape[0], n, dtype=a.dtype, device=a.device)
    p = MoeGemmParams(A=_p(a), B=_p(w), B2=_p(up), D=_p(out), counts=_p(counts), lda=a.stride(0), ldb=w.stride(0),
                      ldd=out.stride(0), rows=a.shape[0], experts=E, N=n, K=w.shape[1], act=ACTS[act], act_limit=limit,
                      act_alpha=alpha, act_shift=shift, dtype=dtype_code(a.dtype), num_ctas=0, status=_p(status),
                      lin_act=LIN_ACTS[lin_act])
    _check(lib().nfk_moe_gemm(byref(p), _stream()), "nfk_moe_gemm")
    return out


def token_shift(h, mu, state, state_ref, positions, token_req, qo_indptr, status=None) -> torch.Tensor:
    """[T, n_mix * width]: every stream's mix of a row with the previous token's; ``state`` [slots, 2, width]."""
    _f32(mu, "mu")
    out = torch.zeros(h.shape[0], mu.shape[0] * h.shape[1], dtype=h.dtype, device=h.device)
    p = TokenShiftParams(h=_p(h), ld_h=h.stride(0), out=_p(out), mu=_p(mu), state=_p(state), state_slot=_p(state_ref),
                         positions=_p(positions), token_req=_p(token_req), qo_indptr=_p(qo_indptr), T=h.shape[0],
                         n_mix=mu.shape[0], num_slots=state.shape[0], dtype=dtype_code(h.dtype), status=_p(status))
    _check(lib().nfk_token_shift(byref(p), _stream()), "nfk_token_shift")
    return out


def wkv(rkvg, x, u, norm, state, y, positions, qo_indptr, state_ref, *, dim_real: int, eps: float, decode: int = 0,
        items=None, seq=None, status=None) -> None:
    """rkvg rows are r | k | v | g of all heads, x [T, heads * dim]; ``state`` [slots, heads, dim, dim] in place. ``decode``: the
    first so many requests have one token each; else ``items`` [n, 4] in chunks and the requests ``seq`` token by token."""
    for t, nm in ((x, "x"), (u, "u"), (norm, "norm"), (state, "state")):
        _f32(t, nm)
    _, heads, dim, _ = state.shape
    o = torch.zeros(rkvg.shape[0], heads * dim, device=rkvg.device)
    n = 0 if items is None else items.shape[0]
    ws = torch.zeros(max(1, n) * heads * (dim * dim + dim), device=rkvg.device)
    p = WkvParams(rkvg=_p(rkvg), ld=rkvg.stride(0), r_off=0, k_off=heads * dim, v_off=2 * heads * dim, g_off=3 * heads * dim,
                  x=_p(x), ld_x=x.stride(0), u=_p(u), norm=_p(norm), S=_p(state), y=_p(y), ld_y=y.stride(0),
                  positions=_p(positions), qo_indptr=_p(qo_indptr), state_slot=_p(state_ref), req_begin=0, req_count=decode,
                  heads=heads, dim=dim, dim_real=dim_real, num_slots=state.shape[0], eps=eps, dtype=dtype_code(rkvg.dtype),
                  seq_reqs=_p(seq), num_seq=0 if seq is None else seq.numel(), o=_p(o), items=_p(items), num_items=n,
                  scratch=_p(ws), scratch_floats=ws.numel(), status=_p(status))
    name = "nfk_wkv_decode" if decode else "nfk_wkv_prefill"
    _check(getattr(lib(), name)(byref(p), _stream()), name)
