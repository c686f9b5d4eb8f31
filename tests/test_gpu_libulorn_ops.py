"""Kernels of the Libulorn family against the plain restatement in fp64: decayed matrix states (chunked and token by token),
windowed attention with its own value size, query / key norms with rotation, stream passes, clamped-gate GEMMs and experts."""
import pytest
import torch

import libulorn_plain as plain
from lightllm_b200 import ops
from lightllm_b200.common.infer_state import InferState
from lightllm_b200.ops import moe
from lightllm_b200.ops import reference as ref
from lightllm_b200.ops._native import kernels
from lightllm_b200.ops.linear_attn import ChunkPlan, DecayedState

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return (got - want).norm().item() / max(want.norm().item(), 1e-30)


def up(n, m):
    return -(-n // m) * m


def heads(x, padded):
    """[T, H, n] -> [T, H * padded], zero-padded."""
    T, H, n = x.shape
    return torch.nn.functional.pad(x, (0, padded - n)).reshape(T, H * padded)


def recurrence_case(dev, kind, dtype, new, ready, H, dim, vdim, rank=12, tau=16.0, cap=9.0, zscale=1.0, seed=0, decode=False,
                    scan=False, gate_shift=0.0):
    """Runs a pass over `new` tokens per request on top of `ready` cached ones; returns (output error, state errors)."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*s, scale=1.0):
        return (torch.randn(*s, generator=g) * scale).to(dtype).double()

    T, B = sum(new), len(new)
    dk, dv = up(dim, 16), up(vdim, 16)
    q, k, v, gate = rnd(T, H, dim), rnd(T, H, dim), rnd(T, H, vdim), rnd(T, H, vdim)
    a1, a2 = rnd(T, rank), rnd(H * dim, rank, scale=zscale / rank ** 0.5)
    bias = rnd(H * dim, scale=zscale) - gate_shift
    zi, zf = (torch.randn(T, H, generator=g) * 4).float(), (torch.randn(T, H, generator=g) * 4 + 2).float()
    w = 1 + 0.3 * torch.randn(vdim if kind == "gla" else H * vdim, generator=g)
    eps, out_scale = 1e-4, 0.7
    slots = torch.randperm(B + 3, generator=g)[:B].to(torch.int32)
    n_state = DecayedState.state_elems(kind, H, dk, dv)
    state = torch.full((B + 3, up(n_state, 4) + 32), 7.0)
    S0 = torch.randn(B, H, dim, vdim, generator=g)
    n0, m0 = torch.randn(B, H, dim, generator=g), torch.rand(B, H, generator=g) * 3
    S0p = torch.nn.functional.pad(S0, (0, dv - vdim, 0, dk - dim))
    for b in range(B):
        parts = [S0p[b].reshape(-1)]
        if kind == "mlstm":
            parts += [torch.nn.functional.pad(n0[b], (0, dk - dim)).reshape(-1), m0[b]]
        state[slots[b], :n_state] = torch.cat(parts)
    # plain
    want, ends, off = [], [], 0
    wv = w.double().view(-1, vdim)
    for b, n in enumerate(new):
        sl = slice(off, off + n)
        qs = q[sl] * dim ** -0.5
        fresh = ready[b] == 0
        if kind == "gla":
            z = a1[sl] @ a2.t() + bias
            decay = torch.sigmoid(z).pow(1 / tau).view(n, H, dim)
            o, S = plain.gated_linear_recurrence(qs, k[sl], v[sl], decay, None if fresh else S0[b].double())
            act = gate[sl] * torch.sigmoid(gate[sl])
            ends.append((S,))
        else:
            li, lf = plain.mlstm_gates(zi[sl].double(), zf[sl].double(), cap)
            st = None if fresh else (S0[b].double(), n0[b].double(), m0[b].double())
            o, st = plain.mlstm_recurrence(qs, k[sl], v[sl], li, lf, st)
            act = torch.sigmoid(gate[sl])
            ends.append(st)
        want.append(plain.rms(o, eps) * wv * act * out_scale)
        off += n
    want = torch.cat(want)
    # kernels: all projections are columns of one matrix
    r8 = up(rank, 8)
    cols = [heads(q, dk), heads(k, dk), heads(v, dv), heads(gate, dv), torch.nn.functional.pad(a1, (0, r8 - rank))]
    m = torch.cat(cols, 1).to(dev, dtype)
    pq, pk, pv, pg, pa = torch.split(m, [c.shape[1] for c in cols], 1)
    weight = torch.nn.functional.pad(w.view(-1, vdim), (0, dv - vdim)).reshape(-1).float().to(dev)
    kw = {}
    if kind == "gla":
        a2p = torch.nn.functional.pad(a2.view(H, dim, rank), (0, r8 - rank, 0, dk - dim)).reshape(H * dk, r8)
        kw = dict(tau=tau, a2=a2p.to(dev, dtype), a2_bias=torch.nn.functional.pad(bias.view(H, dim), (0, dk - dim)).reshape(-1)
                  .float().to(dev))
    else:
        kw = dict(cap=cap)
    rec = DecayedState(kind, H, dk, dv, dim, vdim, eps, weight, out_scale=out_scale, **kw)
    i32 = dict(dtype=torch.int32, device=dev)
    cu = torch.tensor([0] + list(torch.tensor(new).cumsum(0)), **i32)
    rdy = torch.tensor(ready, **i32)
    st = InferState(is_prefill=not decode, batch_size=B, num_tokens=T, max_kv_len=0, max_q_len=max(new),
                    b_req_idx=slots.to(dev), b_seq_len=rdy + 1, mem_index=None, cu_q=cu, b_ready_cache_len=rdy)
    st.seq_pos = rdy
    dev_state = state.to(dev)
    zz = torch.zeros(T, up(2 * H, 8))
    zz[:, :H], zz[:, H:2 * H] = zi, zf
    zz = zz.to(dev)
    wide = torch.full((T, 16 + H * dv), 3.0, device=dev, dtype=dtype)
    rec(pq, pk, pv, pg, dev_state[:, :n_state], st, a1=pa if kind == "gla" else None, zi=zz[:, :H], zf=zz[:, H:2 * H],
        out=wide[:, 16:], plan=ChunkPlan(torch.tensor(new), dev), token_by_token=scan)
    torch.cuda.synchronize()
    assert (wide[:, :16] == 3).all()
    got = wide[:, 16:].view(T, H, dv)
    assert (got[..., vdim:] == 0).all() and torch.isfinite(got).all()
    errs = []
    for b, e in enumerate(ends):
        row = dev_state[slots[b].long()].cpu()
        assert (row[n_state:] == 7).all()
        errs.append(rel(row[: H * dk * dv].view(H, dk, dv)[:, :dim, :vdim], e[0]))
        if kind == "mlstm":
            errs.append(rel(row[H * dk * dv: H * dk * (dv + 1)].view(H, dk)[:, :dim], e[1]))
            errs.append(rel(row[H * dk * (dv + 1): n_state], e[2]))
    others = torch.ones(B + 3, dtype=torch.bool)
    others[slots.long()] = False
    assert (dev_state.cpu()[others] == 7).all()
    return rel(got[..., :vdim], want), max(errs)


SHAPES = [(3, 24, 40), (2, 128, 128), (1, 16, 16), (2, 72, 200), (2, 256, 64), (1, 64, 320)]


@pytest.mark.parametrize("kind", ["gla", "mlstm"])
@pytest.mark.parametrize("H,dim,vdim", SHAPES)
def test_chunked_recurrence(dev, kind, H, dim, vdim):
    for i, (new, ready) in enumerate([([64], [0]), ([1, 2, 63, 65, 130], [0, 5, 0, 64, 7]), ([300, 17], [0, 100])]):
        out, state = recurrence_case(dev, kind, BF, new, ready, H, dim, vdim, seed=i)
        assert out < 4e-3 and state < 3e-5, (new, out, state)


@pytest.mark.parametrize("tau,zscale,shift", [(1.0, 1.0, 0.0), (1.0, 3.0, 6.0), (0.5, 1.0, 3.0), (40.0, 1.0, -6.0)])
def test_chunked_recurrence_any_decay(dev, tau, zscale, shift):
    """From decays that leave nothing of a token after the next one to decays of almost one."""
    out, state = recurrence_case(dev, "gla", BF, [200, 70], [0, 3], 2, 40, 48, rank=20, tau=tau, zscale=zscale,
                                 gate_shift=shift)
    assert out < 4e-3 and state < 3e-5, (out, state)


@pytest.mark.parametrize("kind", ["gla", "mlstm"])
@pytest.mark.parametrize("dtype,tol", [(BF, 4e-3), (F32, 8e-6)])
@pytest.mark.parametrize("H,dim,vdim", SHAPES + [(1, 300, 600)])
def test_recurrence_token_by_token(dev, kind, dtype, tol, H, dim, vdim):
    out, state = recurrence_case(dev, kind, dtype, [1] * 7, [0, 1, 2, 3, 64, 65, 0], H, dim, vdim, decode=True)
    assert out < tol and state < 5e-6, ("decode", out, state)
    out, state = recurrence_case(dev, kind, dtype, [1, 9, 30], [0, 3, 0], H, dim, vdim, scan=True)
    assert out < tol and state < 5e-6, ("prompt", out, state)


def test_chunked_and_token_by_token_agree_over_a_long_prompt(dev):
    for kind in ("gla", "mlstm"):
        out, state = recurrence_case(dev, kind, BF, [1500], [0], 2, 32, 32, seed=3)
        assert out < 4e-3 and state < 5e-5, (kind, out, state)


# ------------------------------------------------------------------------------------------------ attention
def paged(dev, dtype, new, ready, Hkv, D, DV, seed, spare=11):
    """Keys and values of several requests in a shuffled pool, and the state of a pass over their new tokens."""
    g = torch.Generator().manual_seed(seed)
    lens = [r + n for r, n in zip(ready, new)]
    B, total = len(new), sum(lens)
    pool = torch.randn(total + spare, Hkv * (D + DV), generator=g)
    perm = torch.randperm(total + spare, generator=g)[:total].to(torch.int32)
    r2t = torch.zeros(B + 2, max(lens) + 5, dtype=torch.int32)
    rows = torch.randperm(B + 2, generator=g)[:B].to(torch.int32)
    ks, off = [], 0
    for b, L in enumerate(lens):
        r2t[rows[b], :L] = perm[off:off + L]
        ks.append(perm[off:off + L].long())
        off += L
    pos = torch.cat([torch.arange(r, r + n) for r, n in zip(ready, new)]).to(torch.int32)
    bof = torch.repeat_interleave(torch.arange(B), torch.tensor(new)).to(torch.int32)
    cu = torch.tensor([0] + list(torch.tensor(new).cumsum(0)), dtype=torch.int32)
    st = InferState(is_prefill=True, batch_size=B, num_tokens=sum(new), max_kv_len=max(lens), max_q_len=max(new),
                    b_req_idx=rows.to(dev), b_seq_len=torch.tensor(lens, dtype=torch.int32, device=dev), mem_index=None,
                    position_ids=pos.to(dev), seq_pos=pos.to(dev), cu_q=cu.to(dev),
                    b_ready_cache_len=torch.tensor(ready, dtype=torch.int32, device=dev), batch_of_token=bof.to(dev))
    return pool.to(dtype), r2t.to(dev), st, ks


def attention_case(dev, dtype, new, ready, Hq, Hkv, D, DV, window, seed=0, decode=False, gated=True, sharp=1.0):
    pool, r2t, st, slots = paged(dev, dtype, new, ready, Hkv, D, DV, seed)
    st.is_prefill = not decode
    T = sum(new)
    g = torch.Generator().manual_seed(seed + 1)
    q = (torch.randn(T, Hq * D, generator=g) * sharp).to(dtype)
    gate = torch.randn(T, Hq, generator=g).to(dtype)
    scale = D ** -0.5
    want, off = [], 0
    for b, (n, r) in enumerate(zip(new, ready)):
        rows = pool[slots[b]].double()
        k, v = rows[:, : Hkv * D].view(-1, Hkv, D), rows[:, Hkv * D:].reshape(-1, Hkv, DV)
        qf = torch.zeros(r + n, Hq, D, dtype=F64)
        qf[r:] = q[off:off + n].double().view(n, Hq, D)
        want.append(plain.window_attention_fast(qf, k, v, scale, window or 1 << 30)[r:])
        off += n
    want = torch.cat(want)
    if gated:
        want = want * torch.sigmoid(gate.double()).unsqueeze(-1) * 1.3
    wide = torch.full((T, 8 + Hq * DV), 3.0, device=dev, dtype=dtype)
    qw = torch.cat([q, torch.zeros(T, 24, dtype=dtype)], 1).to(dev)
    gw = torch.cat([gate, torch.zeros(T, 8, dtype=dtype)], 1).to(dev)
    ops.window_attention(qw[:, : Hq * D], pool.to(dev), r2t, st, Hq, Hkv, D, DV, scale, window,
                         gw[:, :Hq] if gated else None, 1.3 if gated else 1.0, wide[:, 8:])
    torch.cuda.synchronize()
    assert kernels().llb_attn_tc_status() == 0
    assert (wide[:, :8] == 3).all()
    return rel(wide[:, 8:], want.reshape(T, -1))


ATT_SHAPES = [(6, 2, 64, 64), (4, 4, 64, 128), (4, 1, 128, 64), (8, 2, 128, 128), (3, 1, 128, 256), (2, 2, 192, 128),
              (2, 1, 256, 256), (4, 2, 256, 192), (2, 1, 64, 320)]


@pytest.mark.parametrize("dtype,tol", [(BF, 3e-3), (F32, 2e-6)])
@pytest.mark.parametrize("Hq,Hkv,D,DV", ATT_SHAPES)
def test_window_attention(dev, dtype, tol, Hq, Hkv, D, DV):
    new, ready = [1, 7, 130, 300], [0, 200, 0, 77]
    for window in (1, 2, 50, 128, 129, 0):
        assert attention_case(dev, dtype, new, ready, Hq, Hkv, D, DV, window, seed=window) < tol, ("prompt", window)
        assert attention_case(dev, dtype, [1] * 5, [0, 1, 63, 200, 500], Hq, Hkv, D, DV, window, decode=True) < tol, window
    assert attention_case(dev, dtype, new, ready, Hq, Hkv, D, DV, 40, gated=False, sharp=4.0) < tol


def test_window_attention_long_decode(dev):
    for window in (1000, 1500, 0):
        assert attention_case(dev, BF, [1, 1], [4000, 1499], 4, 2, 128, 128, window, decode=True) < 3e-3


@pytest.mark.parametrize("dtype,tol", [(BF, 3e-3), (F32, 1e-6)])
@pytest.mark.parametrize("Hq,Hkv,D,dim,DV,rot", [(6, 2, 64, 40, 128, 40), (3, 1, 128, 128, 256, 32), (2, 2, 64, 64, 64, 64),
                                                 (5, 5, 192, 150, 64, 6), (4, 2, 256, 256, 128, 0)])
def test_qk_norm_rope_scatter(dev, dtype, tol, Hq, Hkv, D, dim, DV, rot):
    g = torch.Generator().manual_seed(D + rot)
    T, n = 37, (Hq + Hkv) * D + Hkv * DV
    mask = (torch.arange(D) < dim).float()
    x = torch.randn(T, n + 8, generator=g)
    x[:, : (Hq + Hkv) * D] *= mask.repeat(Hq + Hkv)
    x = x.to(dtype)
    qw, kw = (mask * (1 + 0.3 * torch.randn(D, generator=g)) for _ in range(2))
    rcfg = {"dims": rot, "base": 500.0}
    cos, sin = ref.build_rope_cache(200, rot, 500.0, None)
    pos = torch.randint(0, 200, (T,), generator=g).to(torch.int32)
    slot = torch.randperm(60, generator=g)[:T].to(torch.int32)
    pool = torch.full((60, Hkv * (D + DV)), 5.0, dtype=dtype, device=dev)
    y = x.to(dev)
    ops.qk_norm_rope_scatter_(y[:, :n], pool, cos.to(dev), sin.to(dev), pos.to(dev), slot.to(dev), qw.to(dev), kw.to(dev), 1e-3,
                              Hq, Hkv, D, dim, DV, rot)
    xd = x.double()

    def want(lo, heads_, w):
        h = plain.rms(xd[:, lo:lo + heads_ * D].view(T, heads_, D)[..., :dim], 1e-3) * w[:dim].double()
        h = torch.stack([plain.rotate(h[t:t + 1], rcfg, int(pos[t]))[0] for t in range(T)]) if rot else h
        return torch.nn.functional.pad(h, (0, D - dim)).reshape(T, -1)

    assert rel(y[:, : Hq * D], want(0, Hq, qw)) < tol
    got = pool[slot.long().to(dev)]
    assert rel(got[:, : Hkv * D], want(Hq * D, Hkv, kw)) < tol
    assert torch.equal(got[:, Hkv * D:].cpu(), x[:, (Hq + Hkv) * D: n]) and torch.equal(y[:, n:].cpu(), x[:, n:])
    rest = torch.ones(60, dtype=torch.bool)
    rest[slot.long()] = False
    assert (pool.cpu()[rest] == 5).all()


# ------------------------------------------------------------------------------------------------ stream passes, experts
@pytest.mark.parametrize("ydt", [BF, F32])
@pytest.mark.parametrize("dtype,tol", [(BF, 3e-3), (F32, 1e-6)])
@pytest.mark.parametrize("T,width,W", [(1, 40, 64), (37, 320, 320), (50, 2048, 2048), (9, 5000, 5056), (3, 12000, 12032)])
def test_add_rms(dev, dtype, tol, ydt, T, width, W):
    g = torch.Generator().manual_seed(W)
    mask = (torch.arange(W) < width).float()
    x, y = torch.randn(T, W, generator=g) * mask, (torch.randn(T, W, generator=g) * mask).to(ydt)
    w, nw = ((1 + 0.3 * torch.randn(W, generator=g)) * mask for _ in range(2))
    want = x.double().clone()
    want[:, :width] += plain.rms(y.double()[:, :width], 1e-3) * w.double()[:width]
    xd = x.to(dev)
    h = ops.add_rms_(xd, y.to(dev), w.to(dev), width, 1e-3, dtype)
    assert rel(xd, want) < 1e-6 and rel(h, want) < tol and h.dtype == dtype
    xd = x.to(dev)
    h = ops.add_rms_(xd, y.to(dev), w.to(dev), width, 1e-3, dtype, nw.to(dev))
    assert rel(xd, want) < 1e-6 and rel(h[:, :width], plain.rms(want[:, :width], 1e-3) * nw.double()[:width]) < tol
    assert (h[:, width:] == 0).all()


@pytest.mark.parametrize("dtype", [BF, F32])
def test_embedding_pair(dev, dtype):
    g = torch.Generator().manual_seed(0)
    V, W, buckets = 50, 64, 23
    table, second = torch.randn(V, W, generator=g).to(dtype), torch.randn(buckets + 1, W, generator=g).to(dtype)
    big = ops.BigramTable(second.to(dev), buckets, 31, 7)
    big.slot_token = torch.full((40,), -1, dtype=torch.int32, device=dev)
    toks = {0: torch.randint(0, V, (9,), generator=g), 1: torch.randint(0, V, (4,), generator=g)}
    slots = torch.randperm(40, generator=g).to(torch.int32)
    r2t = torch.zeros(3, 16, dtype=torch.int32)
    r2t[2, :9], r2t[0, :4] = slots[:9], slots[9:13]
    r2t = r2t.to(dev)
    w = {"embed": table, "bigram": second}
    cfg = {"embedding": {"bigram": dict(buckets=buckets, mul_prev=31, mul_cur=7)}}
    want = {b: plain.embed(w, t.tolist(), cfg) for b, t in toks.items()}
    at = {0: 0, 1: 0}
    for step in ([(0, 3), (1, 1)], [(0, 1), (1, 1)], [(1, 2), (0, 5)]):
        ids = torch.cat([toks[b][at[b]:at[b] + n] for b, n in step])
        pos = torch.cat([torch.arange(at[b], at[b] + n) for b, n in step]).to(torch.int32)
        bof = torch.cat([torch.full((n,), i) for i, (b, n) in enumerate(step)]).to(torch.int32)
        req = torch.tensor([{0: 2, 1: 0}[b] for b, _ in step], dtype=torch.int32)
        mem = torch.cat([r2t.cpu()[{0: 2, 1: 0}[b], at[b]:at[b] + n] for b, n in step])
        decode = all(n == 1 for _, n in step)
        x, h = ops.embedding_pair(ids.to(dev), table.to(dev), big, r2t, req.to(dev), pos.to(dev), None if decode else bof.to(dev),
                                  mem.to(dev))
        exp = torch.cat([want[b][at[b]:at[b] + n] for b, n in step])
        assert rel(x, exp) < 1e-6 and rel(h, exp) < (3e-3 if dtype == BF else 1e-6)
        for b, n in step:
            at[b] += n


@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (5, 256, 72), (130, 512, 320), (64, 2048, 2048), (200, 3072, 1024),
                                   (1500, 2048, 1024), (3000, 5632, 512)])
def test_gemm_gated_clamp(dev, M, N, K):
    g = torch.Generator().manual_seed(M + N)
    a, w = (torch.randn(M, K, generator=g) * 2).to(BF), (torch.randn(N, K, generator=g) / K ** 0.5).to(BF)
    acc = a.double() @ w.double().t()
    v = acc.view(M, -1, 2, 32)
    gt, u = v[:, :, 0].clamp(max=1.1), v[:, :, 1].clamp(-1.1, 1.1)
    want = (gt * torch.sigmoid(1.5 * gt) * (u + 1)).reshape(M, N // 2)
    assert rel(ops.gemm(a.to(dev), w.to(dev), epi="gated_clamp", clamp=(1.5, 1.1)), want) < 4e-3
    assert int(ops.gemm_status(dev).item()) == 0
    if M * N * K < 1 << 28:
        assert rel(ops.gemm(a.float().to(dev), w.float().to(dev), epi="gated_clamp", clamp=(1.5, 1.1)), want) < 1e-6


@pytest.mark.parametrize("dtype,tol", [(BF, 5e-3), (F32, 2e-6)])
@pytest.mark.parametrize("T,E,k,ff,shared", [(1, 5, 2, 64, True), (40, 24, 3, 64, True), (300, 40, 6, 128, False)])
def test_routed_experts(dev, dtype, tol, T, E, k, ff, shared):
    g = torch.Generator().manual_seed(T)
    W = 192
    t = {"m.router": torch.randn(E, W, generator=g) / W ** 0.5}
    for e in [f"e{i}" for i in range(E)] + ["shared"]:
        t.update({f"m.{e}.gate": torch.randn(ff, W, generator=g) / 14, f"m.{e}.up": torch.randn(ff, W, generator=g) / 14,
                  f"m.{e}.down": torch.randn(W, ff, generator=g) / ff ** 0.5})
    t = {n: v.to(dtype) for n, v in t.items()}
    h, x = (torch.randn(T, W, generator=g) * 2).to(dtype), torch.randn(T, W, generator=g)
    cfg = {"router": {"experts": E, "top": k}, "expert": {"limit": 1.3}, "shared": {"limit": 0.9} if shared else None}
    y = plain.moe(t, "m.", h.double(), cfg)
    nw = 1 + 0.2 * torch.randn(W, generator=g)
    want = x.double() + plain.rms(y, 1e-5) * nw.double()
    d = {n: v.to(dev) for n, v in t.items()}
    w13 = torch.stack([ref.interleave_gate_up(d[f"m.e{e}.gate"], d[f"m.e{e}.up"]) for e in range(E)])
    w2 = torch.stack([d[f"m.e{e}.down"] for e in range(E)])
    hd, xd = h.to(dev), x.to(dev)
    router = torch.nn.functional.pad(d["m.router"], (0, 0, 0, -E % 8))
    ids, wts = moe.topk_softmax(ops.gemm(hd, router, epi="f32")[:, :E], k, renorm=False)
    want_ids, want_w = plain.route(t, "m.", h.double(), cfg["router"])
    assert torch.equal(ids.cpu().long().sort(-1)[0], want_ids.sort(-1)[0]) and rel(wts, want_w) < 1e-4
    sh = None
    if shared:
        gu = ref.interleave_gate_up(d["m.shared.gate"], d["m.shared.up"])
        sh = ops.gemm(ops.gemm(hd, gu, epi="gated_clamp", clamp=(1.702, 0.9)), d["m.shared.down"])
    out = moe.routed_experts_rms_(hd, ids, wts, w13, w2, (1.702, 1.3), sh, xd, nw.to(dev), W, 1e-5)
    assert rel(xd, want) < tol and rel(out, want) < tol
    total = moe.routed_experts_rms_(hd, ids, wts, w13, w2, (1.702, 1.3), sh, None, None, W, 1e-5)
    assert total.dtype == F32 and rel(total, y) < tol
