"""Kernels of the Taduzen family against fp32 PyTorch: dynamic-tanh passes and GEMM epilogues, fp32 GEMM, latent
attention in both forms with windows, table-routed experts."""
import pytest
import torch

import taduzen_oracle as oracle
from lightllm_b200 import ops
from lightllm_b200.ops import mla, moe
from lightllm_b200.ops import reference as ref

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def _norm(dev, W, seed, alpha):
    g = torch.Generator().manual_seed(seed)
    return ops.DytNorm((1 + 0.2 * torch.randn(W, generator=g)).to(dev), (0.3 * torch.randn(W, generator=g)).to(dev), alpha)


def _rel(got, want):
    return (got.float() - want.float()).norm().item() / max(want.float().norm().item(), 1e-12)


@pytest.mark.parametrize("dtype,tol", [(BF, 4e-3), (F32, 2e-6)])
@pytest.mark.parametrize("T,W", [(1, 64), (37, 320), (300, 2048)])
def test_dyt_row_passes(dev, dtype, tol, T, W):
    torch.manual_seed(T)
    a, b = _norm(dev, W, 1, 0.7), _norm(dev, W, 2, 1.3)
    table = torch.randn(91, W, device=dev).to(dtype)
    ids = torch.randint(0, 91, (T,), device=dev)
    x, h = ops.embedding_dyt(ids, table, a)
    assert torch.equal(x, table[ids].float()) and h.dtype == dtype
    assert _rel(h, oracle.dyt(x, a.w, a.b, a.alpha)) < tol
    assert _rel(ops.dyt(x, b, dtype), oracle.dyt(x, b.w, b.b, b.alpha)) < tol
    y = torch.randn(T, W, device=dev)
    want_x = x + oracle.dyt(y, a.w, a.b, a.alpha)
    h = ops.add_dyt_(x, y, a, b, dtype)
    assert _rel(x, want_x) < 1e-6 and _rel(h, oracle.dyt(want_x, b.w, b.b, b.alpha)) < tol


# row counts on both sides of the skinny / one-CTA / CTA-pair schedules, ragged rows, columns and K
@pytest.mark.parametrize("M,N,K", [(1, 192, 64), (5, 128, 72), (130, 256, 320), (64, 2048, 2048), (200, 1024, 1024),
                                   (33, 7168, 2048), (1500, 2048, 1024), (700, 448, 200)])
def test_gemm_epilogues(dev, M, N, K):
    torch.manual_seed(M + N)
    a = (torch.randn(M, K, device=dev) / K ** 0.5).to(BF)
    w = torch.randn(N, K, device=dev).to(BF)
    acc = a.float() @ w.float().t()
    assert _rel(ops.gemm(a, w, epi="relu2"), torch.relu(acc) ** 2) < 4e-3
    assert _rel(ops.gemm(a, w, epi="f32", out_scale=0.37), acc * 0.37) < 1e-5
    n1, n2 = _norm(dev, N, 3, 0.9), _norm(dev, N, 4, 0.6)
    x = torch.randn(M, N, device=dev)
    want = x + oracle.dyt(acc, n1.w, n1.b, n1.alpha)
    h = ops.gemm(a, w, epi="dyt", x=x, dyt=(n1, n2))
    assert _rel(x, want) < 1e-5 and _rel(h, oracle.dyt(want, n2.w, n2.b, n2.alpha)) < 4e-3
    assert int(ops.gemm_status(dev).item()) == 0


@pytest.mark.parametrize("M,N,K", [(1, 64, 40), (70, 192, 100), (129, 256, 512)])
def test_gemm_fp32(dev, M, N, K):
    torch.manual_seed(N)
    a, w = torch.randn(M, K, device=dev), torch.randn(N, K, device=dev)
    acc = (a.double() @ w.double().t()).float()
    assert _rel(ops.gemm(a, w), acc) < 1e-6
    assert _rel(ops.gemm(a, w, epi="f32", out_scale=1.7), acc * 1.7) < 1e-6
    assert _rel(ops.gemm(a, w, epi="relu2"), torch.relu(acc) ** 2) < 1e-6
    assert _rel(ops.gemm(a, w, epi="gated_silu"), ref.gated_act_interleaved(acc, "silu")) < 1e-6
    r = torch.randn(M, N, device=dev)
    assert _rel(ops.gemm(a, w, epi="residual", residual=r), acc + r) < 1e-6
    n1, n2 = _norm(dev, N, 3, 0.1), _norm(dev, N, 4, 0.6)
    x = torch.randn(M, N, device=dev)
    want = x + oracle.dyt(acc, n1.w, n1.b, n1.alpha)
    h = ops.gemm(a, w, epi="dyt", x=x, dyt=(n1, n2))
    assert _rel(x, want) < 1e-6 and _rel(h, oracle.dyt(want, n2.w, n2.b, n2.alpha)) < 2e-6
    a3, w3 = torch.randn(M, 3, K, device=dev), torch.randn(3, N, K, device=dev)
    assert _rel(mla.gemm_batched(a3, w3), torch.einsum("thk,hnk->thn", a3.double(), w3.double())) < 1e-6


def _paged(dev, ready, new, rank, row, dtype, seed, spare=13):
    """Latents of several requests in a shuffled pool, and the index tensors of a pass over their new tokens."""
    g = torch.Generator().manual_seed(seed)
    lens = [r + n for r, n in zip(ready, new)]
    total = sum(lens)
    pool = torch.full((total + spare, 1, row), 7.0)
    perm = torch.randperm(total + spare, generator=g)[:total].to(torch.int32)
    r2t = torch.zeros(len(lens) + 2, max(lens) + 3, dtype=torch.int32)
    cs, off = [], 0
    rows = torch.randperm(len(lens) + 2, generator=g)[: len(lens)].to(torch.int32)
    for i, L in enumerate(lens):
        c = torch.randn(L, rank, generator=g).to(dtype)
        r2t[rows[i], :L] = perm[off:off + L]
        pool[perm[off:off + L].long(), 0, :rank] = c.float()
        pool[perm[off:off + L].long(), 0, rank:] = 0
        cs.append(c)
        off += L
    pos = torch.cat([torch.arange(r, r + n) for r, n in zip(ready, new)]).to(torch.int32)
    bof = torch.repeat_interleave(torch.arange(len(new)), torch.tensor(new)).to(torch.int32)
    return pool.to(dev, dtype), r2t.to(dev), rows.to(dev), pos.to(dev), bof.to(dev), cs


@pytest.mark.parametrize("dtype,tol", [(BF, 6e-3), (F32, 2e-6)])
@pytest.mark.parametrize("rank,row", [(40, 48), (88, 112), (512, 512)])
def test_latent_norm_scatter(dev, dtype, tol, rank, row):
    torch.manual_seed(rank)
    T = 19
    wide = torch.randn(T, 64 + row, device=dev).to(dtype)
    src = wide[:, 64:]
    w = 1 + 0.3 * torch.randn(rank, device=dev)
    pool = torch.full((40, 1, row), 5.0, device=dev, dtype=dtype)
    slot = torch.randperm(40, device=dev)[:T].to(torch.int32)
    mla.latent_norm_scatter_(src, pool, w, slot, rank, 1e-3)
    got = pool[slot.long(), 0]
    assert _rel(got[:, :rank], oracle.rms(src[:, :rank].float(), w, 1e-3)) < tol
    assert (got[:, rank:] == 0).all()
    untouched = torch.ones(40, dtype=torch.bool, device=dev)
    untouched[slot.long()] = False
    assert (pool[untouched] == 5).all()


def _absorbed_want(q, cs, ready, new, scale, window):
    out, off = [], 0
    for c, r, n in zip(cs, ready, new):
        m = oracle.visible(n, r + n, r, window or 1 << 30)
        s = torch.einsum("nhd,md->hnm", q[off:off + n].double().cpu(), c.double()) * scale
        p = torch.softmax(s.masked_fill(~m[None], float("-inf")), -1)
        out.append(torch.einsum("hnm,md->nhd", p, c.double()))
        off += n
    return torch.cat(out)


CASES = [([0, 5, 64, 300], [1, 1, 1, 1]), ([0, 63, 200], [130, 2, 70])]


@pytest.mark.parametrize("ready,new", CASES)
@pytest.mark.parametrize("H,rank", [(4, 48), (16, 128), (20, 208), (3, 384), (8, 512)])
@pytest.mark.parametrize("window", [0, 1, 33, 100])
def test_absorbed_attention(dev, ready, new, H, rank, window):
    row = rank + 16
    pool, r2t, rows, pos, bof, cs = _paged(dev, ready, new, rank, row, BF, rank + window)
    T = sum(new)
    q = torch.randn(T, H, rank, device=dev).to(BF)
    want = _absorbed_want(q, cs, ready, new, 0.11, window)
    b = None if max(new) == 1 else bof
    for kw in ({"generic": True}, {"num_splits": 1}, {"num_splits": 3}, {"max_keys": 400}):
        got = mla.latent_attention(q, pool, r2t, rows, pos, b, 0.11, window, **kw)
        assert _rel(got.cpu(), want) < 5e-3, kw
    if rank <= 128:
        q32, p32 = q.float(), pool.float()
        got = mla.latent_attention(q32, p32, r2t, rows, pos, b, 0.11, window)
        assert _rel(got.cpu(), want) < 2e-6


def test_absorbed_attention_keeps_the_weights_in_32_bit(dev):
    """600 keys of almost equal weight and latents of alternating sign: the sum cancels, so weights rounded to bf16
    would show."""
    rank, n = 64, 600
    pool, r2t, rows, pos, bof, _ = _paged(dev, [n - 1], [1], rank, rank, BF, 5)
    sign = torch.where(torch.arange(n) % 2 == 0, 1.0, -1.0)
    c = torch.full((n, rank), 1.0) * sign[:, None]
    c[:, 0] = torch.linspace(-2, 2, n)
    c = c.to(BF)
    pool[r2t[rows[0], :n].long(), 0] = c.to(dev)
    q = torch.zeros(1, 2, rank, device=dev, dtype=BF)
    q[:, :, 0] = 0.5
    want = _absorbed_want(q, [c], [n - 1], [1], 1.0, 0)
    for kw in ({"num_splits": 1}, {"num_splits": 4}, {"generic": True}):
        got = mla.latent_attention(q, pool, r2t, rows, pos, None, 1.0, 0, **kw)
        assert (got.cpu().double() - want)[..., 1:].abs().max() < 1e-5, kw


@pytest.mark.parametrize("ready,new", [([0], [300]), ([0, 130, 7], [129, 2, 64]), ([500, 0, 64, 1], [1, 1, 200, 128])])
@pytest.mark.parametrize("H,dk,dv", [(3, 64, 64), (2, 128, 64), (2, 64, 128), (1, 128, 128)])
@pytest.mark.parametrize("window", [0, 1, 64, 129, 200])
def test_expanded_attention(dev, ready, new, H, dk, dv, window):
    rank = 48
    pool, r2t, rows, pos, bof, cs = _paged(dev, ready, new, rank, rank, BF, dk + window)
    kr = mla.KeyRange(torch.tensor(ready), torch.tensor(new), window, dev)
    c = mla.latent_gather(pool, r2t, rows, kr)
    start = kr.kv_start.tolist()
    assert torch.equal(c.cpu(), torch.cat([x[s:] for x, s in zip(cs, start)]))
    wkv = (torch.randn(H * (dk + dv), rank, device=dev) / rank ** 0.5).to(BF)
    kv = ops.gemm(c, wkv)
    T = sum(new)
    q = torch.randn(T, H * dk + 32, device=dev).to(BF)
    cu = torch.tensor([0] + list(torch.tensor(new).cumsum(0)), dtype=torch.int32, device=dev)
    got = mla.window_prefill(q[:, : H * dk], kv, H, dk, dv, cu, torch.tensor(ready, dtype=torch.int32, device=dev), kr,
                             max(new), 0.13)
    want, off, roff = [], 0, 0
    for r, n, s in zip(ready, new, start):
        m = r + n - s
        k = kv[roff:roff + m, : H * dk].double().view(m, H, dk)
        v = kv[roff:roff + m, H * dk:].double().view(m, H, dv)
        sc = torch.einsum("nhd,mhd->hnm", q[off:off + n, : H * dk].double().view(n, H, dk), k) * 0.13
        mask = oracle.visible(n, r + n, r, window or 1 << 30)[:, s:].to(dev)
        p = torch.softmax(sc.masked_fill(~mask[None], float("-inf")), -1)
        want.append(torch.einsum("hnm,mhd->nhd", p, v).reshape(n, -1))
        off, roff = off + n, roff + m
    assert _rel(got, torch.cat(want)) < 4e-3
    from lightllm_b200.ops._native import kernels
    assert kernels().llb_window_tc_status() == 0


@pytest.mark.parametrize("dtype,tol", [(BF, 6e-3), (F32, 2e-6)])
@pytest.mark.parametrize("T,E,k,I,Is", [(1, 3, 1, 64, 64), (50, 5, 3, 128, 192), (300, 8, 2, 64, 0)])
def test_table_routed_experts(dev, dtype, tol, T, E, k, I, Is):
    torch.manual_seed(T)
    W, V = 128, 77
    tables = [torch.rand(V, n, device=dev).topk(kk, -1)[1].to(torch.int32) for n, kk in ((4, 2), (E, k))]
    routing = moe.TableRouting([(tables[0], 0, 4), (tables[1], 0, E)])
    tok = torch.randint(0, V, (T,), device=dev)
    lays = routing.layouts(tok)
    for lay, t in zip(lays, tables):
        pair = lay.sorted_pair[lay.pair_row.long()]
        assert torch.equal(pair, torch.arange(T * t.shape[1], device=dev, dtype=torch.int32))
        assert torch.equal(lay.mblock_expert[(lay.pair_row // 128).long()], t[tok].reshape(-1))
    g, u = (torch.randn(E, I, W, device=dev) / W ** 0.5 for _ in range(2))
    d = torch.randn(E, W, I, device=dev) / I ** 0.5
    g, u, d = g.to(dtype), u.to(dtype), d.to(dtype)
    h = torch.randn(T, W, device=dev).to(dtype)
    gate_w = torch.randn(W, device=dev) / W ** 0.5 if Is else None
    shared = torch.randn(T, W, device=dev).to(dtype) if Is else None
    want = torch.zeros(T, W, device=dev, dtype=torch.float64)
    for n in range(T):
        for e in tables[1][tok[n]].tolist():
            want[n] += oracle.gated_mlp(h[n:n + 1].double(), g[e].double(), u[e].double(), d[e].double())[0] / k
    if Is:
        want += torch.sigmoid(h.double() @ gate_w.double())[:, None] * shared.double()
    n1, n2 = _norm(dev, W, 6, 0.8), _norm(dev, W, 7, 1.1)
    x = torch.randn(T, W, device=dev)
    wx = x + oracle.dyt(want, n1.w, n1.b, n1.alpha)
    w13 = ref.interleave_gate_up(g, u)
    y = moe.uniform_experts_dyt_(h, lays[1], w13, d, "silu", shared, gate_w, None, None, None)
    assert _rel(y, want) < tol
    hn = moe.uniform_experts_dyt_(h, lays[1], w13, d, "silu", shared, gate_w, x, n1, n2)
    assert _rel(x, wx) < tol and _rel(hn, oracle.dyt(wx, n2.w, n2.b, n2.alpha)) < tol


def test_tanh_error(dev):
    """The branch-free tanh of the bf16 passes, read back in fp32 through the stream: absolute error below 5e-7, relative
    error below 2e-6, over small, middle and large arguments."""
    W = 4096
    v = torch.cat([torch.linspace(-30, 30, W), torch.linspace(-0.3, 0.3, W), torch.logspace(-9, 2, W), -torch.logspace(-9, 2, W)])
    y = v.view(4, W).to(dev)
    unit = ops.DytNorm(torch.ones(W, device=dev), torch.zeros(W, device=dev), 1.0)
    x = torch.zeros(4, W, device=dev)
    ops.add_dyt_(x, y, unit, unit, BF)
    want = torch.tanh(y.double())
    err = (x.double() - want).abs()
    assert err.max() < 5e-7 and (err / want.abs().clamp_min(1e-30)).max() < 2e-6
