"""Zubedra on the GPU: every kernel against the plain oracle of its mechanism, then the engine against the oracle
model in 32-bit (tight) and bf16, however prompts are cut and batched, and greedy generation through the serving
loop. All sizes and weights are the tests' own."""
import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

import zubedra_cases as cases
import zubedra_oracle as oracle
from nanoflow_b200 import ops
from nanoflow_b200.models import zubedra
from nanoflow_b200.models.registry import family
from nanoflow_b200.ops import layer_list as K
from nanoflow_b200.replay import TraceReplay
from nanoflow_b200.runtime.layer_list import query_items, chunk_work
from nanoflow_b200.serving import DistKVPool, RequestManager, Scheduler, StateSlotPool
from nanoflow_b200.serving.loop import ServingLoop
from volarax_cases import prompt, row_errors

BOTH = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.2e-2}


def i32(v):
    return torch.as_tensor(np.asarray(v), dtype=torch.int32).cuda()


def rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).cuda()


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).abs().max() / want.pow(2).mean().sqrt())


def off(got, want):
    """Largest error of an element over its size plus the typical one: rounding to bf16 makes at most 0.004 of it."""
    got, want = got.double().cpu(), want.double().cpu()
    return float(((got - want).abs() / (want.abs() + want.pow(2).mean().sqrt())).max())


ROUNDED = {torch.float32: 2e-5, torch.bfloat16: 5e-3}


# ---- GEMM forms -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("M,N,Kd", [(1, 8, 8), (70, 88, 136), (300, 520, 1000)])
def test_gemm_with_tanh_and_with_bias_in_fp32(dtype, M, N, Kd):
    a, w, b = rnd(M, Kd, seed=1, dtype=dtype), rnd(N, Kd, seed=2, dtype=dtype, scale=Kd ** -0.5), rnd(N, seed=3, dtype=dtype)
    z = a.double() @ w.double().T
    ws = torch.zeros(1 << 22, device="cuda")
    for kw in ({}, {"workspace": ws}, {"workspace": ws, "split_k": 2} if dtype == torch.bfloat16 and Kd >= 1000 else {}):
        assert rel(K.gemm(a, w, lin_act="tanh", **kw), torch.tanh(z)) < TOL[dtype]
        out32 = torch.zeros(M, N, device="cuda")
        K.gemm(a, w, bias=b, out32=out32, **kw)
        assert rel(out32, z + b.double()) < 2e-5


@pytest.mark.parametrize("dtype", BOTH)
def test_gated_gemm_with_capped_halves(dtype):
    a = rnd(70, 136, seed=1, dtype=dtype)
    g, u = (rnd(88, 136, seed=s, dtype=dtype, scale=2 * 136 ** -0.5) for s in (2, 3))
    zg, zu = (a.double() @ t.double().T for t in (g, u))
    zg, zu = zg.clamp(max=1.5), zu.clamp(-1.5, 1.5)
    want = zg * torch.sigmoid(1.3 * zg) * (zu + 0.5)
    assert rel(K.gemm(a, g, up=u, act="capped", limit=1.5, alpha=1.3, shift=0.5), want) < TOL[dtype] * 4


# ---- residual step ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("cols,top", [(5, 1), (104, 3), (4096, 8)])
def test_residual_step_sums_mixer_experts_and_shared_expert(dtype, cols, top):
    ld, rows, eps = (cols + 7) // 8 * 8, 21, 1e-3
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - cols)).contiguous()
    x, y, y2 = pad(rnd(rows, cols, seed=1)), pad(rnd(rows, cols, seed=2, dtype=dtype)), pad(rnd(rows, cols, seed=3, dtype=dtype))
    e = pad(rnd(rows * top, cols, seed=4, dtype=dtype))
    gate, wt = rnd(rows, seed=5), rnd(rows, top, seed=6)
    slot = i32(np.random.default_rng(0).permutation(rows * top).reshape(rows, top))
    w = pad(rnd(1, cols, seed=7))[0]
    d = lambda t: t.double()[..., :cols]
    want = d(x) + d(y) + gate.double()[:, None] * d(y2) + (wt.double()[..., None] * d(e)[slot.long()]).sum(1)
    kw = dict(y=y, y2=y2, y2_gate=gate, experts=(e, slot, wt), norm_out=("layer", w, None), cols=cols, eps=eps)
    idx, before, st = i32([20, 0, 5, 5]), x.clone(), ops.new_status()
    hs = torch.zeros(4, ld, dtype=dtype, device="cuda")
    K.residual_norm(x, h=hs, rows_idx=idx, status=st, **kw)
    want_h = oracle.centred_norm(want, d(w), eps)
    assert torch.equal(x, before) and rel(hs[:, :cols], want_h[idx.long()]) < TOL[dtype] * 4
    h = torch.zeros(rows, ld, dtype=dtype, device="cuda")
    K.residual_norm(x, h=h, status=st, **kw)
    ops.check_status(st)
    assert rel(x[:, :cols], want) < 2e-5 and rel(h[:, :cols], want_h) < TOL[dtype] * 4 and (h[:, cols:] == 0).all()


@pytest.mark.parametrize("dtype", BOTH)
def test_embedding_step_scales_the_row_in_fp32(dtype):
    table, w = rnd(67, 56, seed=1, dtype=dtype), rnd(56, seed=2)
    x, h = torch.full((3, 56), 9.0, device="cuda"), torch.zeros(3, 56, dtype=dtype, device="cuda")
    K.residual_norm(x, table=table, ids=i32([3, 66, 1]), src_scale=3.3, h=h, norm_out=("layer", w, None), cols=56, eps=1e-5)
    want = table.double()[[3, 66, 1]] * 3.3
    assert rel(x, want) < 1e-6 and rel(h, oracle.centred_norm(want, w.double(), 1e-5)) < TOL[dtype] * 4


# ---- attention -----------------------------------------------------------------------------------------------------
class PagedKv:
    """Sequences of keys and values in a paged pool, pages handed out in a shuffled order."""

    def __init__(self, lens, G, hd, dtype, seed=0):
        rng = np.random.default_rng(seed)
        self.lens, self.G, self.hd = lens, G, hd
        n = [(x + 15) // 16 for x in lens]
        ids = rng.permutation(sum(n) + 5)
        self.pool = torch.zeros(sum(n) + 5, 2, G, 16, hd, dtype=dtype, device="cuda")
        self.rows = [ids[sum(n[:b]):sum(n[:b + 1])] for b in range(len(lens))]
        self.indptr, self.indices = i32(np.concatenate([[0], np.cumsum(n)])), i32(np.concatenate(self.rows))
        self.last = i32([(x - 1) % 16 + 1 for x in lens])

    def fill(self, b, k, v):
        """k, v [len, G, columns]"""
        for t in range(self.lens[b]):
            page = int(self.rows[b][t // 16])
            self.pool[page, 0, :, t % 16, :k.shape[-1]] = k[t]
            self.pool[page, 1, :, t % 16, :v.shape[-1]] = v[t]


def attention_setup(dtype, group, G, dim, vdim, lens, spans, hd, seed=0, sharp=0):
    """Sequences of ``lens`` whose last ``spans`` tokens are the queries of a step. ``sharp`` > 0: for some queries one key
    (first, last, at a page border, in the middle) stands out, with a value of its own."""
    H, rng = group * G, np.random.default_rng(seed)
    pg = PagedKv(lens, G, hd, dtype, seed)
    T = sum(spans)
    q = torch.zeros(T, H, hd, dtype=dtype, device="cuda")
    pos, req, want, t0 = [], [], [], 0
    ks, vs = [], []
    for b, (n, m) in enumerate(zip(lens, spans)):
        k, v = rnd(n, G, dim, seed=seed + 10 * b + 1, dtype=dtype), rnd(n, G, vdim, seed=seed + 10 * b + 2, dtype=dtype)
        qq = rnd(m, H, dim, seed=seed + 10 * b + 3, dtype=dtype)
        for i in range(m if sharp else 0):
            p = n - m + i
            for h in range(H):
                j = int(rng.choice([0, p, max(0, p // 16 * 16 - 1), min(p, p // 16 * 16), p // 2]))
                qq[i, h] = (k[j, h // group].float() * sharp / k[j, h // group].float().norm()).to(dtype)
        pg.fill(b, k, v)
        q[t0:t0 + m, :, :dim] = qq
        ks.append(k.double().cpu())
        vs.append(v.double().cpu())
        pos += range(n - m, n)
        req += [b] * m
        t0 += m
    qo = np.concatenate([[0], np.cumsum(spans)]).astype(np.int32)
    return pg, q, ks, vs, i32(pos), i32(req), qo


def attention_want(q, ks, vs, pos, req, dim, scale, cap, sink):
    out = []
    for t in range(q.shape[0]):
        b, p = int(req[t]), int(pos[t])
        H, G = q.shape[1], ks[b].shape[1]
        k, v = ks[b][:p + 1], vs[b][:p + 1]
        s = torch.einsum("hd,nhd->hn", q[t, :, :dim].double().cpu(), k.repeat_interleave(H // G, dim=1)) * scale
        s = oracle.soft_cap(s, cap)
        if sink is not None:
            s = torch.cat([s, sink.double().cpu()[:, None]], dim=1)
        w = torch.softmax(s, dim=-1)[:, :p + 1]
        out.append(torch.einsum("hn,nhv->hv", w, v.repeat_interleave(H // G, dim=1)))
    return torch.stack(out)


@pytest.mark.parametrize("cap,with_sink", [(None, False), (4.0, True)])
@pytest.mark.parametrize("group,G,dim,vdim", [(1, 3, 24, 40), (3, 2, 64, 64), (5, 1, 128, 72), (8, 2, 96, 128), (16, 1, 128, 128),
                                              (7, 2, 40, 16)])
def test_attention_kernels(group, G, dim, vdim, cap, with_sink):
    """Decode with and without split key ranges, prefill, and the simple kernel on both."""
    H, scale, hd = group * G, 1.3 * dim ** -0.5, 64 if max(dim, vdim) <= 64 else 128
    sink = rnd(H, seed=77, scale=2.0) if with_sink else None
    lens = [1, 15, 16, 17, 64, 65, 300, 500]
    pg, q, ks, vs, pos, req, qo = attention_setup(torch.bfloat16, group, G, dim, vdim, lens, [1] * len(lens), hd, 5, sharp=12.0)
    want = attention_want(q, ks, vs, pos, req, dim, scale, cap, sink)
    ws = torch.zeros(len(lens) * H * 16 * (hd + 2), device="cuda")
    for chunk, mc in ((0, 1), (2, 16), (8, 4), (5, 2)):
        out, st = torch.full_like(q, 7.0), ops.new_status()
        K.paged_attention(q, pg.pool, out, i32(qo), pg.indptr, pg.indices, pg.last, heads=H, scale=scale, softcap=cap or 0.0,
                          sinks=sink, req_count=len(lens), chunk_pages=chunk, max_chunks=mc, workspace=ws, status=st)
        ops.check_status(st)
        assert off(out[..., :vdim], want) < 5e-3, (chunk, mc)
        assert (out[..., vdim:] == 0).all()
    lens, spans = [2, 20, 130, 300, 333], [2, 3, 130, 140, 2]
    pg, q, ks, vs, pos, req, qo = attention_setup(torch.bfloat16, group, G, dim, vdim, lens, spans, hd, 6, sharp=12.0)
    want = attention_want(q, ks, vs, pos, req, dim, scale, cap, sink)
    out, st = torch.full_like(q, 7.0), ops.new_status()
    K.paged_attention(q, pg.pool, out, i32(qo), pg.indptr, pg.indices, pg.last, heads=H, scale=scale, softcap=cap or 0.0,
                      sinks=sink, items=i32(query_items(qo, 0, 128 // group)), status=st)
    ops.check_status(st)
    assert off(out[..., :vdim], want) < 5e-3
    simple = torch.full_like(q, 7.0)
    K.gqa_attention(q, pg.pool, simple, pos, req, pg.indptr, pg.indices, heads=H, scale=scale, softcap=cap or 0.0, sinks=sink,
                    status=st)
    ops.check_status(st)
    assert off(simple[..., :vdim], want) < 5e-3


@pytest.mark.parametrize("group,G,dim,vdim", [(3, 2, 24, 40), (18, 1, 136, 144)])
def test_simple_attention_in_32_bit(group, G, dim, vdim):
    H, hd = group * G, (max(dim, vdim) + 7) // 8 * 8
    sink = rnd(H, seed=77, scale=2.0)
    pg, q, ks, vs, pos, req, qo = attention_setup(torch.float32, group, G, dim, vdim, [1, 130, 77], [1, 9, 2], hd, 7, sharp=9.0)
    out, st = torch.full_like(q, 7.0), ops.new_status()
    K.gqa_attention(q, pg.pool, out, pos, req, pg.indptr, pg.indices, heads=H, scale=0.2, softcap=3.0, sinks=sink, status=st)
    ops.check_status(st)
    assert rel(out[..., :vdim], attention_want(q, ks, vs, pos, req, dim, 0.2, 3.0, sink)) < 2e-5


@pytest.mark.parametrize("sink", [-60.0, 40.0])
def test_capped_scores_and_sinks_at_the_ends_of_their_range(sink):
    """Scores far beyond the cap are all equal to it; a sink far above them takes everything, one far below nothing."""
    H, hd, n = 4, 64, 200
    pg, q, ks, vs, pos, req, qo = attention_setup(torch.bfloat16, 2, 2, 64, 64, [n, n], [1, 70], hd, 8)
    sinks = torch.full((H,), sink, device="cuda")
    q *= 50.0
    want = attention_want(q, ks, vs, pos, req, 64, 1.0, 30.0, sinks)
    out, st = torch.zeros_like(q), ops.new_status()
    for kw in (dict(req_count=1), dict(items=i32(query_items(qo, 1, 64)))):
        K.paged_attention(q, pg.pool, out, i32(qo), pg.indptr, pg.indices, pg.last, heads=H, scale=1.0, softcap=30.0, sinks=sinks,
                          status=st, **kw)
    ops.check_status(st)
    assert torch.allclose(out.double().cpu(), want, rtol=1e-2, atol=0.01 * float(vs[0].std()) + 1e-3)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,dim,hd", [(6, 2, 24, 64), (1, 1, 7, 8), (16, 4, 128, 128)])
def test_append_norms_whole_rows_and_mixes_values(dtype, H, G, dim, hd):
    T, eps, lam = 19, 1e-2, 0.3
    hd = hd if dtype == torch.bfloat16 else (dim + 7) // 8 * 8
    pg = PagedKv([40, 33], G, hd, dtype, 3)
    padh = lambda t, n: torch.nn.functional.pad(t.reshape(-1, n, dim), (0, hd - dim)).reshape(-1, n * hd).contiguous()
    q, k, v, vf = (rnd(T, n * dim, seed=s, dtype=dtype) for s, n in ((1, H), (2, G), (3, G), (4, G)))
    qw, kw = rnd(H * dim, seed=5), rnd(G * dim, seed=6)
    src = torch.cat([padh(q, H), padh(k, G), padh(v, G)], dim=1)
    pos = i32(list(range(21, 33)) + list(range(7)))
    req = i32([0] * 12 + [1] * 7)
    wq = oracle.rms_norm(q.double().cpu(), eps, qw.double().cpu())
    wk = oracle.rms_norm(k.double().cpu(), eps, kw.double().cpu())
    for mode in (0, 1, 2):
        first, qo, st = padh(vf, G).clone(), torch.zeros(T, H * hd, dtype=dtype, device="cuda"), ops.new_status()
        K.gqa_append(src, qo, pg.pool, pos, req, pg.indptr, pg.indices, heads=H, dim=dim, q_w=padh(qw, H)[0], k_w=padh(kw, G)[0],
                     v_first=first, v_mode=mode, v_lambda=lam, eps=eps, status=st)
        ops.check_status(st)
        wv = v.double().cpu() if mode < 2 else oracle.mix_values(v.double().cpu(), vf.double().cpu(), lam)
        assert off(qo.reshape(T, H, hd)[..., :dim], wq.reshape(T, H, dim)) < ROUNDED[dtype]
        got = [torch.stack([pg.pool[int(pg.rows[int(b)][int(p) // 16]), j, :, int(p) % 16, :dim] for p, b in zip(pos, req)]) for j in (0, 1)]
        assert off(got[0], wk.reshape(T, G, dim)) < ROUNDED[dtype] and off(got[1], wv.reshape(T, G, dim)) < ROUNDED[dtype]
        assert torch.equal(first, padh(v if mode == 1 else vf, G)) and (qo.reshape(T, H, hd)[..., dim:] == 0).all()


# ---- WKV ---------------------------------------------------------------------------------------------------------------
class WkvCase:
    """Sequences fed to the kernels in steps; the outputs of all steps against the oracle's."""

    def __init__(self, lens, H, dim, dtype, seed=0, x_lo=-7.0, x_hi=1.5):
        self.lens, self.H, self.dim, self.dp, self.dtype = lens, H, dim, (dim + 7) // 8 * 8, dtype
        n = sum(lens)
        self.r, self.k, self.v, self.g = (rnd(n, H, dim, seed=seed + s, dtype=dtype) for s in range(4))
        g = torch.Generator().manual_seed(seed + 9)
        self.x = (torch.rand(n, H, dim, generator=g) * (x_hi - x_lo) + x_lo).cuda()
        self.u, self.norm = rnd(H, dim, seed=seed + 5), 1.0 + 0.2 * rnd(H, dim, seed=seed + 6)
        self.off = np.concatenate([[0], np.cumsum(lens)])
        self.state = torch.full((len(lens) + 2, H, self.dp, self.dp), 3.0, device="cuda")       # left over from others
        self.y = torch.zeros(n, H, dim, device="cuda")
        self.at = [0] * len(lens)

    def pad(self, t):
        return torch.nn.functional.pad(t, (0, self.dp - self.dim)).flatten(-2).contiguous()

    def step(self, tokens, how):
        """``tokens``: {sequence: count}. ``how``: "decode", "chunks", "seq", or "both" (a cap that sends some token by token)."""
        rows = np.concatenate([np.arange(self.off[b] + self.at[b], self.off[b] + self.at[b] + n) for b, n in tokens.items()])
        pos = np.concatenate([np.arange(self.at[b], self.at[b] + n) for b, n in tokens.items()])
        qo = np.concatenate([[0], np.cumsum(list(tokens.values()))]).astype(np.int32)
        sel = torch.from_numpy(rows).cuda()
        rkvg = torch.cat([self.pad(t[sel]) for t in (self.r, self.k, self.v, self.g)], dim=1)
        y = torch.zeros(len(rows), self.H * self.dp, dtype=self.dtype, device="cuda")
        kw, st = {}, ops.new_status()
        if how == "decode":
            kw["decode"] = len(tokens)
        else:
            items, seq = chunk_work(qo, 0, {"chunks": 1 << 20, "seq": 0, "both": 4}[how])
            kw = dict(items=i32(items) if items.size else None, seq=i32(seq) if seq.size else None)
        K.wkv(rkvg, self.pad(self.x[sel]), self.pad(self.u[None])[0], self.pad(self.norm[None])[0], self.state, y, i32(pos), i32(qo),
              i32([2 * (b + 1) + self.at[b] % 2 for b in tokens]), dim_real=self.dim, eps=1e-4, status=st, **kw)
        ops.check_status(st)
        y = y.reshape(-1, self.H, self.dp)
        assert (y[..., self.dim:] == 0).all()
        self.y[sel] = y[..., :self.dim].float()
        for b, n in tokens.items():
            self.at[b] += n

    def check(self):
        for b, n in enumerate(self.lens):
            s = slice(self.off[b], self.off[b] + self.at[b])
            d = lambda t: t[s].double().cpu()
            o, S = oracle.wkv_recurrence(d(self.r), d(self.k), d(self.v), torch.exp(-torch.exp(d(self.x))), self.u.double().cpu())
            g = d(self.g)
            want = oracle.rms_norm(o, 1e-4) * self.norm.double().cpu() * g * torch.sigmoid(g)
            assert off(self.y[s], want) < ROUNDED[self.dtype]
            got = self.state[b + 1, :, :self.dim, :self.dim]
            assert rel(got, S) < (1e-4 if self.dtype == torch.float32 else 1e-3)
        assert (self.state[0] == 3.0).all() and (self.state[-1] == 3.0).all()        # nobody else's slot


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,dim", [(3, 24), (1, 7), (2, 64), (2, 72), (1, 136)])
def test_wkv_token_by_token_and_single_tokens(dtype, H, dim):
    c = WkvCase([40, 9, 21], H, dim, dtype, seed=dim)
    c.step({0: 17, 2: 2}, "seq")
    for _ in range(6):
        c.step({0: 1, 1: 1, 2: 1}, "decode")
    c.step({2: 13, 1: 3, 0: 16}, "seq")
    c.step({0: 1}, "decode")
    c.check()


@pytest.mark.parametrize("H,dim", [(3, 24), (2, 64), (2, 72), (2, 128), (1, 8)])
def test_wkv_chunks(H, dim):
    """Portions that end inside, at and just behind a run of 16 and a chunk of 64, beside each other and after one another."""
    c = WkvCase([300, 150, 70], H, dim, torch.bfloat16, seed=dim + 1)
    c.step({0: 2, 1: 64}, "chunks")
    c.step({0: 63, 1: 15, 2: 17}, "chunks")
    c.step({0: 1, 1: 1, 2: 1}, "decode")
    c.step({1: 49, 0: 129, 2: 52}, "both")
    c.step({0: 100, 1: 16}, "chunks")
    c.step({0: 5, 1: 5}, "chunks")
    c.check()


@pytest.mark.parametrize("x_lo,x_hi", [(-12.0, -8.0), (0.5, 3.0), (-9.0, 6.0)])
def test_wkv_chunks_with_very_slow_and_very_quick_decays(x_lo, x_hi):
    """From states that hardly fade over 500 tokens to ones that are gone at once, also mixed within a head."""
    c = WkvCase([520], 2, 64, torch.bfloat16, seed=3, x_lo=x_lo, x_hi=x_hi)
    c.step({0: 500}, "chunks")
    c.step({0: 20}, "chunks")
    c.check()


def test_wkv_far_token_is_read_many_chunks_later():
    c = WkvCase([700], 1, 64, torch.bfloat16, seed=4, x_lo=-14.0, x_hi=-12.0)
    c.k *= 0.05
    c.k[3] = 4.0 * torch.sign(c.k[3].float()).to(c.dtype)
    c.r[640] = c.k[3]
    c.step({0: 130}, "chunks")
    c.step({0: 570}, "chunks")
    c.check()


@pytest.mark.parametrize("dtype", BOTH)
def test_token_shift_takes_the_previous_row_from_batch_state_or_nowhere(dtype):
    W, n = 56, 3
    h, mu = rnd(40, W, seed=1, dtype=dtype), rnd(n, W, seed=2)
    state = rnd(4, 2, W, seed=3, dtype=dtype)
    refs, got, at = {0: 2 * 2, 1: 2 * 0}, {}, {0: 0, 1: 0}
    seqs = {0: h[:25], 1: h[25:]}
    for tokens in ({0: 1}, {0: 4, 1: 7}, {1: 1, 0: 1}, {0: 19, 1: 7}):
        rows = torch.cat([seqs[b][at[b]:at[b] + m] for b, m in tokens.items()]).contiguous()
        pos = np.concatenate([np.arange(at[b], at[b] + m) for b, m in tokens.items()])
        qo = np.concatenate([[0], np.cumsum(list(tokens.values()))])
        st = ops.new_status()
        out = K.token_shift(rows, mu, state, i32([refs[b] for b in tokens]), i32(pos), i32(np.repeat(np.arange(len(tokens)), list(tokens.values()))),
                            i32(qo), status=st)
        ops.check_status(st)
        for j, (b, m) in enumerate(tokens.items()):
            got.setdefault(b, []).append(out[qo[j]:qo[j + 1]])
            at[b] += m
            refs[b] ^= 1
    for b, s in seqs.items():
        s = s.double()
        want = torch.cat([s + (oracle.token_shift(s) - s) * mu[i].double() for i in range(n)], dim=1)
        assert off(torch.cat(got[b]), want) < ROUNDED[dtype]


# ---- mixture of experts -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,groups,keep,top", [(10, 5, 3, 3), (7, 7, 2, 1), (6, 1, 1, 6), (40, 4, 2, 5), (256, 8, 4, 8), (64, 1, 1, 32)])
def test_routing(E, groups, keep, top):
    z, corr = rnd(70, E + 9, seed=E), rnd(E, seed=E + 1, scale=0.7)
    counts = torch.zeros(E, dtype=torch.int32, device="cuda")
    idx, w, rank, gate = K.moe_route(z, corr, counts, top=top, experts=E, groups=groups, keep=keep, scale=1.7, gate_col=E)
    s = torch.sigmoid(z[:, :E].double().cpu())
    want_idx, want_w = oracle.route(s, corr.double().cpu(), {"groups": {"count": groups, "keep": keep}, "top": top, "scale": 1.7})
    assert torch.equal(idx.cpu().long(), want_idx) and rel(w, want_w) < 1e-5
    assert rel(gate, torch.sigmoid(z[:, E].double())) < 1e-5
    assert torch.equal(counts.cpu(), torch.bincount(want_idx.flatten(), minlength=E).int())
    for e in range(E):
        ranks = rank[idx == e].sort().values.cpu()
        assert torch.equal(ranks, torch.arange(ranks.numel(), dtype=torch.int32))
    # equal scores: the lower index; groups left out lose even to negative choice scores
    counts.zero_()
    idx, *_ = K.moe_route(torch.zeros_like(z), None, counts, top=1, experts=E, scale=1.0)
    assert (idx == 0).all()


def test_groups_left_out_lose_even_to_negative_choice_scores():
    s = torch.tensor([[0.9, 0.1, 0.6, 0.5]])
    corr = torch.tensor([-3.0, -3.0, -2.9, -2.9]).cuda()
    counts = torch.zeros(4, dtype=torch.int32, device="cuda")
    idx, w, *_ = K.moe_route(torch.logit(s).cuda(), corr, counts, top=2, experts=4, groups=2, keep=1, scale=1.0)
    assert idx.tolist() == [[2, 3]] and torch.allclose(w.cpu(), torch.tensor([[0.6 / 1.1, 0.5 / 1.1]]))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,E,top,W,ff", [(1, 5, 2, 24, 16), (37, 10, 3, 104, 24), (700, 6, 2, 136, 200), (300, 70, 8, 256, 520),
                                          (130, 3, 1, 1000, 72)])
def test_products_per_expert(dtype, T, E, top, W, ff):
    """Unequal shares, also experts without rows, ranges that start anywhere, more and fewer rows than a tile."""
    h = rnd(T, W, seed=1, dtype=dtype)
    z = rnd(T, E, seed=2) + torch.linspace(4.0, -4.0, E, device="cuda")        # the first experts get most
    counts = torch.zeros(E, dtype=torch.int32, device="cuda")
    idx, w, rank, _ = K.moe_route(z, None, counts, top=top, experts=E, scale=1.0)
    rows, slot = K.moe_permute(h, idx, rank, counts)
    assert torch.equal(rows[slot.long()], h[:, None].expand(T, top, W)) and slot.flatten().sort().values.tolist() == list(range(T * top))
    wg, wu = (rnd(E * ff, W, seed=s, dtype=dtype, scale=2 * W ** -0.5) for s in (3, 4))
    wd = rnd(E * W, ff, seed=5, dtype=dtype, scale=ff ** -0.5)
    st = ops.new_status()
    act = K.moe_gemm(rows, wg, counts, up=wu, act="capped", limit=1.5, alpha=1.702, shift=1.0, status=st)
    out = K.moe_gemm(act, wd, counts, status=st)
    ops.check_status(st)
    own = torch.repeat_interleave(torch.arange(E), counts.cpu().long())
    a = rows.double().cpu()
    for e in set(own.tolist()):
        r = own == e
        m = lambda t, n: t.double().cpu()[e * n:(e + 1) * n]
        g, u = (a[r] @ m(wg, ff).T).clamp(max=1.5), (a[r] @ m(wu, ff).T).clamp(-1.5, 1.5)
        want = g * torch.sigmoid(1.702 * g) * (u + 1)
        assert rel(act[r.cuda()], want) < TOL[dtype] * 4
        assert rel(out[r.cuda()], act[r.cuda()].double().cpu() @ m(wd, W).T) < TOL[dtype] * 2


# ---- the engine ------------------------------------------------------------------------------------------------------
def make_replay(raw, t, dtype, *, pages=64, requests=4, batch=512, **pipeline):
    cfg = cases.engine_config(raw, dtype=dtype, batch=batch, requests=requests, pages=pages, **pipeline)
    eng = family("zubedra").engine(cfg, zubedra.weights_from_tensors(cfg.model, t.__getitem__, "cuda"))
    return TraceReplay(eng, pages, requests)


def portions(rp, tokens, sizes, rid="a"):
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(k, len(sizes) - 1)], len(tokens) - at)
        out.append(rp.step([{"id": rid, "tokens": tokens[at:at + n], "want": list(range(n))}],
                           [rid] if at + n == len(tokens) else []))
        at, k = at + n, k + 1
    rp.engine.check_status()
    return np.concatenate(out)


_want = {}


def wanted(name, seed, n):
    """Oracle logits of a case's prompt (computed once per test session)."""
    key = (name, seed, n)
    if key not in _want:
        raw = cases.CASES[name]
        t = cases.tensors(raw, seed)
        toks = prompt(n, raw["vocab"], seed + 100)
        _want[key] = (raw, t, toks, oracle.forward(raw, t, toks))
    return _want[key]


def assert_close(got, want, dtype):
    e = row_errors(got, want)
    # rounding is amplified now and then (a softmax near a tie, two experts with nearly equal choice scores); a wrong
    # key or a lost state shows as an error of order one at every position behind it
    top = e.sort().values[:max(1, int(0.98 * e.numel()))]
    if dtype == "float32":
        assert float(top[-1]) < 3e-5 and float(e.max()) < 1e-3, (float(top[-1]), float(e.max()), int(e.argmax()))
        return
    assert float(e.median()) < 0.03 and float(top[-1]) < 0.3, (float(e.median()), float(top[-1]), int(e.argmax()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(cases.CASES))
@pytest.mark.parametrize("sizes", [[230], [150, 1], [1], [2, 17, 3, 40, 16, 64, 2, 1, 30]], ids=["whole", "then_single", "single", "portions"])
def test_engine_matches_the_oracle(dtype, name, sizes):
    n = 230 if sizes != [1] else 90
    raw, t, toks, want = wanted(name, 1, 230)
    got = portions(make_replay(raw, t, dtype), toks[:n], sizes)
    assert_close(got, want[:n], dtype)


def test_logits_do_not_depend_on_how_a_prompt_is_cut():
    """bf16, beyond the oracle's tolerance: the same prompt in one portion and in many differs by rounding only."""
    raw, t, toks, _ = wanted("large", 1, 230)
    whole = portions(make_replay(raw, t, "bfloat16"), toks, [230])
    for sizes in ([2, 17, 3, 40, 16, 64, 2, 1, 30], [64], [100, 1]):
        e = row_errors(portions(make_replay(raw, t, "bfloat16"), toks, sizes), whole)
        assert float(e.median()) < 0.02 and float(e.sort().values[int(0.98 * e.numel())]) < 0.3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "large"])
def test_batches_of_unequal_requests_over_reused_pages_and_slots(dtype, name):
    """Requests of all lengths come and go in one small pool, portions beside single tokens: every request's logits
    are its own, whatever ran beside it and whoever had its pages and slot before."""
    raw = cases.CASES[name]
    t = cases.tensors(raw, 4)
    rp = make_replay(raw, t, dtype, pages=28, requests=3)
    rng = np.random.default_rng(1)
    lens = (120, 9, 61, 140, 1, 48, 90)
    prompts = {f"r{i}": prompt(n, raw["vocab"], i) for i, n in enumerate(lens)}
    todo, live, got = list(prompts), {}, {r: [] for r in prompts}
    while todo or live:
        while todo and len(live) < 3:
            live[todo.pop(0)] = 0
        entries, end = [], []
        for rid in list(live):
            if len(live) > 1 and rng.random() < 0.15:
                continue
            p, at = prompts[rid], live[rid]
            n = min(int(rng.choice([1, 1, 2, 3, 20, 45])), len(p) - at)
            entries.append({"id": rid, "tokens": p[at:at + n], "want": list(range(n))})
            live[rid] = at + n
            if live[rid] == len(p):
                end.append(rid)
                del live[rid]
        if entries:
            out, at = rp.step(entries, end), 0
            for e in entries:
                got[e["id"]].append(out[at:at + len(e["tokens"])])
                at += len(e["tokens"])
    rp.engine.check_status()
    assert rp.pool.num_free_pages == 28 and rp.slots.num_free == 3
    for rid, p in prompts.items():
        assert_close(np.concatenate(got[rid]), oracle.forward(raw, t, p), dtype)


def test_long_decoding_in_32_bit():
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw, 8)
    toks = prompt(700, raw["vocab"], 8)
    got = portions(make_replay(raw, t, "float32"), toks, [150, 1])
    assert_close(got, oracle.forward(raw, t, toks), "float32")


def test_split_key_ranges_in_decoding():
    """A few requests with long contexts: decode attention in several key ranges."""
    raw = cases.CASES["large"]
    t = cases.tensors(raw, 6)
    toks = prompt(900, raw["vocab"], 6)
    rp = make_replay(raw, t, "bfloat16", batch=1024)
    assert rp.engine._attn_split(1, 56)[1] > 1
    got = portions(rp, toks, [880, 1])
    assert_close(got, oracle.forward(raw, t, toks), "bfloat16")


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 0.1)])
def test_residual_stream_after_every_layer(dtype, tol):
    raw, t, toks, _ = wanted("mixed", 1, 230)
    toks, stream = toks[:70], []
    oracle.forward(raw, t, toks, residuals=stream)
    cfg = cases.engine_config(raw, dtype=dtype)
    cfg.engine.tap_residual = True
    eng = family("zubedra").engine(cfg, zubedra.weights_from_tensors(cfg.model, t.__getitem__, "cuda"))
    TraceReplay(eng, 64, 4).step([{"id": 0, "tokens": toks, "want": [0]}])
    for r, want in enumerate(stream):
        e = (eng.taps[r, :70, :raw["width"]].double().cpu() - want).abs().amax(-1) / want.pow(2).mean().sqrt()
        assert float(e.max() if dtype == "float32" else e.median()) < tol


def serve(raw, t, prompts, n_out, dtype, executor, *, batch=64, pages=40, requests=3, guards=False):
    cfg = cases.engine_config(raw, dtype=dtype, batch=batch, requests=requests, pages=pages)
    cfg.engine.debug_guards = guards
    eng = family("zubedra").engine(cfg, zubedra.weights_from_tensors(cfg.model, t.__getitem__, "cuda"), executor=executor)
    rm = RequestManager(vocab_size=raw["vocab"])
    for p in prompts:
        rm.add_request(len(p), n_out, 0.0, prompt=p)
    rm.finalize_stats()
    m = eng.model
    pool, state = DistKVPool(m.run_layers, 1, m.head_dim, pages, 16, 1), StateSlotPool(eng.num_slots)
    sch = Scheduler(pool, rm.avaliable_request_queue, global_batch_size=batch, max_batch_size=requests,
                    average_prefill_length=rm.average_prefill_length, average_decode_length=n_out, group_size=1,
                    state_pool=state, kv_window=m.kv_window)
    st = ServingLoop(eng, sch, rm, est_cycle_time=1.0).run()
    eng.check_status()
    eng.finalize()
    assert len(st.retired) == len(prompts) and pool.num_free_pages == pages and state.num_free == eng.num_slots
    return {r.req_idx: r.output for r in st.retired}


_generated = {}


@pytest.mark.parametrize("executor", ["python", "native", "graph"])
@pytest.mark.parametrize("name", ["mixed", "recurrent_first"])
def test_greedy_generation_through_the_serving_loop(executor, name):
    """Token feedback on the device, chunked prompts beside decoding, more requests than slots: in 32-bit exactly the
    oracle's tokens."""
    raw = cases.CASES[name]
    t = cases.tensors(raw, 5)
    prompts = [prompt(n, raw["vocab"], 10 + n) for n in (3, 141, 17, 1, 58)]
    out = serve(raw, t, prompts, 12, "float32", executor)
    for i, p in enumerate(prompts):
        if (name, i) not in _generated:
            _generated[name, i] = oracle.generate(raw, t, p.tolist(), 12)
        assert out[i] == _generated[name, i]


def test_greedy_generation_in_bf16_stays_near_the_oracle_arg_max():
    raw = cases.CASES["mixed"]
    t = cases.tensors(raw, 5)
    prompts = [prompt(n, raw["vocab"], 10 + n) for n in (3, 141, 17, 1, 58)]
    out = serve(raw, t, prompts, 12, "bfloat16", "native", guards=True)
    for i, p in enumerate(prompts):
        logits = oracle.forward(raw, t, p.tolist() + out[i][:-1])[len(p) - 1:]
        gap = logits.max(-1).values - logits[torch.arange(12), torch.tensor(out[i])]
        assert float(gap.max()) < 0.25 * float(logits.std())
