"""Kernels of the Katarax family against the plain restatement in fp64: latents with a rotated part in both forms of the attention,
kept first positions and biases by distance, rotations, output gates, grouped routing, stream passes, soft-capped logits."""
import pytest
import torch

import katarax_plain as plain
from lightllm_b200 import ops
from lightllm_b200.common.infer_state import InferState
from lightllm_b200.models.latent import LatentHeads
from lightllm_b200.ops import mla, moe
from lightllm_b200.ops import reference as ref
from lightllm_b200.ops._native import kernels

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return (got - want).norm().item() / max(want.norm().item(), 1e-30)


def rows_rel(got, want):
    """Largest relative error of a row."""
    got, want = got.double().cpu().flatten(1), want.double().cpu().flatten(1)
    return ((got - want).norm(dim=1) / want.norm(dim=1).clamp_min(1e-30)).max().item()


def paged(dev, dtype, new, ready, row, seed, spare=11):
    """Rows of several requests in a shuffled pool, and the state of a pass over their new tokens."""
    g = torch.Generator().manual_seed(seed)
    lens = [r + n for r, n in zip(ready, new)]
    B, total = len(new), sum(lens)
    pool = torch.randn(total + spare, row, generator=g)
    perm = torch.randperm(total + spare, generator=g)[:total].to(torch.int32)
    r2t = torch.zeros(B + 2, max(lens) + 5, dtype=torch.int32)
    rows = torch.randperm(B + 2, generator=g)[:B].to(torch.int32)
    slots, off = [], 0
    for b, L in enumerate(lens):
        r2t[rows[b], :L] = perm[off:off + L]
        slots.append(perm[off:off + L].long())
        off += L
    pos = torch.cat([torch.arange(r, r + n) for r, n in zip(ready, new)]).to(torch.int32)
    bof = torch.repeat_interleave(torch.arange(B), torch.tensor(new)).to(torch.int32)
    cu = torch.tensor([0] + list(torch.tensor(new).cumsum(0)), dtype=torch.int32)
    rd = torch.tensor(ready, dtype=torch.int32)
    st = InferState(is_prefill=True, batch_size=B, num_tokens=sum(new), max_kv_len=max(lens), max_q_len=max(new),
                    b_req_idx=rows.to(dev), b_seq_len=torch.tensor(lens, dtype=torch.int32, device=dev), mem_index=None,
                    position_ids=pos.to(dev), seq_pos=pos.to(dev), cu_q=cu.to(dev), b_ready_cache_len=rd.to(dev),
                    batch_of_token=bof.to(dev))
    st.extra["q_len_cpu"], st.extra["ready_cpu"] = torch.tensor(new, dtype=torch.int32), rd
    return pool.to(dtype), r2t.to(dev), st, slots


# ------------------------------------------------------------------------------------------------ kept positions, biases
def attention_case(dev, dtype, new, ready, Hq, Hkv, D, DV, window, keep, table=None, far=0, seed=0, decode=False, scale=None,
                   shape_kv=None):
    pool, r2t, st, slots = paged(dev, dtype, new, ready, Hkv * (D + DV), seed)
    st.is_prefill = not decode
    T = sum(new)
    q = torch.randn(T, Hq * D, generator=torch.Generator().manual_seed(seed + 1)).to(dtype)
    if shape_kv is not None:
        shape_kv(q.view(T, Hq, D), pool, slots)
    scale = D ** -0.5 if scale is None else scale
    want, off = [], 0
    for b, (n, r) in enumerate(zip(new, ready)):
        rows, L = pool[slots[b]].double(), r + n
        k, v = rows[:, : Hkv * D].view(-1, Hkv, D), rows[:, Hkv * D:].reshape(-1, Hkv, DV)
        qf = torch.zeros(L, Hq, D, dtype=F64)
        qf[r:] = q[off:off + n].double().view(n, Hq, D)
        bias = None if table is None else plain.distance_bias(table, L, far)
        want.append(plain.attend(qf, k, v, scale, plain.visible(L, window or None, keep), bias)[r:])
        off += n
    wide = torch.full((T, 8 + Hq * DV), 3.0, device=dev, dtype=dtype)
    qw = torch.cat([q, torch.zeros(T, 24, dtype=dtype)], 1).to(dev)
    bias = None if table is None else ops.DistanceBias(table.to(dev), far)
    ops.window_attention(qw[:, : Hq * D], pool.to(dev), r2t, st, Hq, Hkv, D, DV, scale, window, out=wide[:, 8:], keep=keep, bias=bias)
    torch.cuda.synchronize()
    assert kernels().llb_attn_tc_status() == 0 and (wide[:, :8] == 3).all()
    return rows_rel(wide[:, 8:], torch.cat(want).reshape(T, -1))


ATT_SHAPES = [(6, 2, 64, 64), (4, 1, 128, 64), (8, 2, 128, 128), (2, 2, 192, 128), (4, 2, 256, 192), (34, 1, 64, 128)]
RULES = [(0, 0, True), (1, 1, True), (50, 20, True), (128, 3, False), (129, 64, True), (40, 300, False), (64, 128, True)]


@pytest.mark.parametrize("dtype,tol", [(BF, 8e-3), (F32, 5e-6)])
@pytest.mark.parametrize("Hq,Hkv,D,DV", ATT_SHAPES)
def test_kept_positions_and_biases(dev, dtype, tol, Hq, Hkv, D, DV):
    g = torch.Generator().manual_seed(D)
    for window, keep, biased in RULES:
        rows, far = ((16, 100), (6, 33), (32, 500))[window % 3]
        table = torch.randn(rows, Hq, generator=g).to(BF) if biased else None
        kw = dict(table=table, far=far, seed=window)
        assert attention_case(dev, dtype, [1, 7, 130, 300], [0, 200, 0, 177], Hq, Hkv, D, DV, window, keep, **kw) < tol, (window, keep)
        assert attention_case(dev, dtype, [1] * 6, [0, 1, 63, 200, 500, 64], Hq, Hkv, D, DV, window, keep, decode=True, **kw) < tol


def test_long_decode_over_splits(dev):
    for window, keep, far in ((1000, 300, 2000), (1500, 5, 64), (0, 0, 128)):
        table = torch.randn(32, 4, generator=torch.Generator().manual_seed(far)).to(BF)
        assert attention_case(dev, BF, [1, 1], [4000, 1499], 4, 2, 128, 128, window, keep, table, far, decode=True) < 8e-3


@pytest.mark.parametrize("dtype,tol", [(BF, 8e-3), (F32, 5e-6)])
@pytest.mark.parametrize("decode", [False, True])
def test_kept_key_that_stands_out(dev, dtype, tol, decode):
    """One key outside the window takes nearly all the weight while it is a kept one; one place later it takes none."""
    for at in (0, 6, 7):
        def point(q, pool, slots):
            q[-1, :, 3] = 12.0
            pool[slots[0][at], 3] = 12.0
        new, ready = ([1], [600]) if decode else ([150], [451])
        assert attention_case(dev, dtype, new, ready, 4, 1, 64, 64, 100, 7, decode=decode, scale=0.2, shape_kv=point) < tol, at


# ------------------------------------------------------------------------------------------------ latents
@pytest.mark.parametrize("dtype,tol", [(BF, 5e-3), (F32, 2e-6)])
@pytest.mark.parametrize("rank,cols,n,row,q_rank,q_cols", [(40, 48, 16, 80, 56, 64), (512, 512, 64, 576, 1536, 1536),
                                                           (129, 144, 6, 152, 8, 16), (24, 32, 0, 32, 24, 24)])
def test_latent_rows(dev, dtype, tol, rank, cols, n, row, q_rank, q_cols):
    g = torch.Generator().manual_seed(rank)
    T = 37
    src = torch.randn(T, q_cols + cols + n + 24, generator=g)
    pad = -src.shape[1] % 8
    src = torch.nn.functional.pad(src, (0, pad)).to(dtype)
    w, qw = torch.rand(cols, generator=g) + 0.5, torch.rand(q_cols, generator=g) + 0.5
    for neighbours, fn in ((True, plain.rotate_neighbours), (False, plain.rotate_halves)):
        cos, sin = ref.build_rope_cache(300, max(n, 2), 900.0)
        rope = mla.LatentRope(cos.to(dev), sin.to(dev), n, neighbours) if n else None
        pos = torch.randint(0, 300, (T,), generator=g).to(torch.int32)
        pool = torch.full((60, row), 5.0, dtype=dtype, device=dev)
        slot = torch.randperm(60, generator=g)[:T].to(torch.int32)
        d = src.to(dev)
        out = mla.latent_prepare_(d[:, q_cols:], pool, w.to(dev), slot.to(dev), rank, cols, 1e-3, rope, pos.to(dev), d[:, :q_cols],
                                  qw.to(dev), q_rank)
        got = pool[slot.long().to(dev)].cpu()
        s = src.double()
        assert rel(got[:, :rank], plain.rms(s[:, q_cols:q_cols + rank], 1e-3) * w[:rank]) < tol
        assert (got[:, rank:cols] == 0).all() and (got[:, cols + n:] == 0).all()
        if n:
            x = s[:, None, q_cols + cols:q_cols + cols + n]
            want = torch.cat([fn(x[i:i + 1], dict(base=900.0, dims=n), int(pos[i]))[0] for i in range(T)])
            assert rel(got[:, cols:cols + n], want) < tol
        assert rel(out[:, :q_rank], plain.rms(s[:, :q_rank], 1e-3) * qw[:q_rank]) < tol and (out[:, q_rank:] == 0).all()
        free = torch.ones(60, dtype=torch.bool)
        free[slot.long()] = False
        assert (pool.cpu()[free] == 5).all()


@pytest.mark.parametrize("dtype,tol", [(BF, 4e-3), (F32, 1e-6)])
@pytest.mark.parametrize("H,pitch,off,n", [(3, 64, 24, 16), (16, 192, 128, 64), (1, 64, 5, 6), (5, 128, 0, 128)])
def test_rope_heads(dev, dtype, tol, H, pitch, off, n):
    g = torch.Generator().manual_seed(H)
    T = 29
    x = torch.randn(T, H * pitch + 16, generator=g).to(dtype)
    cos, sin = ref.build_rope_cache(500, n, 1e4)
    pos = torch.randint(0, 500, (T,), generator=g).to(torch.int32)
    for neighbours, fn in ((True, plain.rotate_neighbours), (False, plain.rotate_halves)):
        y = x.to(dev)
        ops.rope_heads_(y, cos.to(dev), sin.to(dev), pos.to(dev), H, pitch, off, n, neighbours)
        want = x.double().clone()
        v = want[:, : H * pitch].view(T, H, pitch)
        for i in range(T):
            v[i, :, off:off + n] = fn(v[i:i + 1, :, off:off + n], dict(base=1e4, dims=n), int(pos[i]))[0]
        assert rel(y, want) < tol
        got = y[:, : H * pitch].view(T, H, pitch).cpu()
        assert torch.equal(got[..., :off], x[:, : H * pitch].view(T, H, pitch)[..., :off])
        assert torch.equal(got[..., off + n:], x[:, : H * pitch].view(T, H, pitch)[..., off + n:])
        assert torch.equal(y[:, H * pitch:].cpu(), x[:, H * pitch:])


class _Bag:
    pass


def latent_case(dev, dtype, new, ready, H, dim, rot, vdim, rank, window, form, gated, seed=0):
    """The attention over latents in one form: error of the worst row."""
    g = torch.Generator().manual_seed(seed)
    lat, lw = LatentHeads(H, dim, rot, vdim, rank, 0.09, window), _Bag()
    uk = (torch.randn(H, dim, rank, generator=g) / rank ** 0.5).to(dtype)
    uv = (torch.randn(H, vdim, rank, generator=g) / rank ** 0.5).to(dtype)
    lat.load(lw, lambda t: t.to(dev, dtype).contiguous(), uk, uv)
    pool, r2t, st, slots = paged(dev, dtype, new, ready, lat.keys, seed)
    pool[:, rank:lat.rp] = 0
    pool[:, lat.rp + rot:] = 0
    st.is_prefill = form != "decode"
    T = sum(new)
    q = torch.randn(T, H, dim + rot, generator=g).to(dtype)
    gate = torch.randn(T, H, vdim, generator=g).to(dtype)
    want, off = [], 0
    for b, (n, r) in enumerate(zip(new, ready)):
        rows, L = pool[slots[b]].double(), r + n
        c = rows[:, :rank]
        k = torch.cat([torch.einsum("lr,hdr->lhd", c, uk.double()), rows[:, None, lat.rp:lat.rp + rot].expand(L, H, rot)], -1)
        v = torch.einsum("lr,hdr->lhd", c, uv.double())
        qf = torch.zeros(L, H, dim + rot, dtype=F64)
        qf[r:] = q[off:off + n].double()
        want.append(plain.attend(qf, k, v, 0.09, plain.visible(L, window or None))[r:])
        off += n
    want = torch.cat(want)
    if gated:
        want = want * torch.sigmoid(gate.double())
    qp = torch.nn.functional.pad(q, (0, lat.dp - dim - rot)).reshape(T, -1).to(dev)
    gp = torch.cat([torch.zeros(T, 16, dtype=dtype), torch.nn.functional.pad(gate, (0, lat.vp - vdim)).reshape(T, -1)], 1).to(dev)
    expanded = lat._expanded_range(qp, st) if form != "decode" else None
    if form == "expanded":
        kr = mla.KeyRange(torch.tensor(ready), torch.tensor(new), window, dev)
        lat._expanded_range = lambda *a: kr
    elif form == "absorbed":
        lat._expanded_range = lambda *a: None
    out = lat.attend(lw, qp, pool.to(dev), r2t, st, gp[:, 16:] if gated else None).view(T, H, lat.vp)
    torch.cuda.synchronize()
    assert kernels().llb_window_tc_status() == 0 and int(ops.gemm_status(dev).item()) == 0
    assert (out[..., vdim:] == 0).all()
    return rows_rel(out[..., :vdim], want), expanded


LATENTS = [(4, 24, 16, 40, 40), (16, 128, 64, 128, 512), (3, 40, 24, 72, 130), (20, 64, 64, 64, 200), (2, 160, 96, 128, 384)]


@pytest.mark.parametrize("H,dim,rot,vdim,rank", LATENTS)
@pytest.mark.parametrize("form", ["expanded", "absorbed"])
def test_latent_prompt(dev, form, H, dim, rot, vdim, rank):
    for window in (0, 1, 33, 64, 129, 200):
        for new, ready in (([300], [0]), ([129, 2, 64], [0, 130, 7]), ([1, 200, 128], [500, 64, 1])):
            err, _ = latent_case(dev, BF, new, ready, H, dim, rot, vdim, rank, window, form, window % 2 == 0, seed=window)
            assert err < 2e-2, (window, new, err)


@pytest.mark.parametrize("H,dim,rot,vdim,rank", LATENTS + [(2, 16, 8, 200, 24), (1, 32, 64, 64, 560)])
@pytest.mark.parametrize("dtype,tol", [(BF, 2e-2), (F32, 1e-5)])
def test_latent_decode(dev, dtype, tol, H, dim, rot, vdim, rank):
    for window in (0, 1, 64, 300):
        err, _ = latent_case(dev, dtype, [1] * 6, [0, 1, 63, 64, 300, 900], H, dim, rot, vdim, rank, window, "decode", True, seed=window)
        assert err < tol, (window, err)


def test_latent_form_follows_the_pass(dev):
    """Long prompts run the expanded form, short portions behind a long cache the absorbed one."""
    assert latent_case(dev, BF, [600], [0], 16, 128, 64, 128, 512, 0, "own", True)[1] is not None
    err, kr = latent_case(dev, BF, [2], [900], 16, 128, 64, 128, 512, 0, "own", True)
    assert kr is None and err < 2e-2


# ------------------------------------------------------------------------------------------------ rows, routing, logits
@pytest.mark.parametrize("dtype,tol", [(BF, 4e-3), (F32, 1e-6)])
@pytest.mark.parametrize("T,N", [(1, 8), (33, 200), (300, 2048)])
def test_sigmoid_mul(dev, dtype, tol, T, N):
    x, g = torch.randn(T, N + 8).to(dtype), (torch.randn(T, N + 24) * 4).to(dtype)
    y = x.to(dev)
    ops.sigmoid_mul_(y[:, :N], g.to(dev)[:, 8:N + 8])
    assert rel(y[:, :N], x[:, :N].double() * torch.sigmoid(g[:, 8:N + 8].double())) < tol
    assert torch.equal(y[:, N:].cpu(), x[:, N:])


@pytest.mark.parametrize("dtype,tol", [(BF, 4e-3), (F32, 1e-6)])
@pytest.mark.parametrize("Hq,Hkv,D,dim,DV,n", [(6, 2, 64, 40, 128, 24), (4, 0, 128, 128, 64, 128), (3, 3, 192, 150, 64, 6)])
def test_unit_heads(dev, dtype, tol, Hq, Hkv, D, dim, DV, n):
    """Rotation, then unit heads: queries in place, keys and values to the pool."""
    g = torch.Generator().manual_seed(D)
    T, N = 31, (Hq + Hkv) * D + Hkv * DV
    x = torch.randn(T, N, generator=g)
    x[:, : (Hq + Hkv) * D] *= (torch.arange(D) < dim).float().repeat(Hq + Hkv)
    x = x.to(dtype)
    cos, sin = ref.build_rope_cache(200, n, 700.0)
    pos, slot = torch.randint(0, 200, (T,), generator=g).to(torch.int32), torch.randperm(50, generator=g)[:T].to(torch.int32)
    pool, y = torch.full((50, max(Hkv, 1) * (D + DV)), 5.0, dtype=dtype, device=dev), x.to(dev)
    ops.qk_norm_rope_scatter_(y, pool, cos.to(dev), sin.to(dev), pos.to(dev), slot.to(dev), None, None, 1e-3, Hq, Hkv, D, dim, DV, n)
    heads = x[:, : (Hq + Hkv) * D].double().view(T, -1, D)[..., :dim]
    want = torch.cat([plain.rms(plain.rotate_halves(heads[i:i + 1], dict(base=700.0, dims=n), int(pos[i])), 1e-3) for i in range(T)])
    assert rel(y[:, : Hq * D].view(T, Hq, D)[..., :dim], want[:, :Hq]) < tol
    got = pool.cpu()[slot.long()]
    if Hkv:
        assert rel(got[:, : Hkv * D].view(T, Hkv, D)[..., :dim], want[:, Hq:]) < tol
        assert torch.equal(got[:, Hkv * D:], x[:, (Hq + Hkv) * D:])
    else:
        assert (got == 5).all()


@pytest.mark.parametrize("dtype,tol", [(BF, 4e-3), (F32, 1e-6)])
@pytest.mark.parametrize("T,width,W", [(1, 40, 64), (37, 320, 320), (9, 5000, 5056)])
def test_stream_passes(dev, dtype, tol, T, width, W):
    g = torch.Generator().manual_seed(W)
    mask = (torch.arange(W) < width).float()
    table, w = (torch.randn(50, W, generator=g) * mask).to(dtype), torch.rand(W, generator=g) * mask
    ids = torch.randint(0, 50, (T,), generator=g)
    none = torch.zeros((1, 1), dtype=torch.int32, device=dev)
    x, h = ops.embedding_pair(ids.to(dev), table.to(dev), None, none, None, None, None, None, norm=(w.to(dev), width, 1e-3))
    want = table[ids].double()
    assert torch.equal(x.cpu(), table[ids].float()) and rel(h[:, :width], plain.rms(want[:, :width], 1e-3) * w[:width]) < tol
    y = (torch.randn(T, W, generator=g) * mask).to(dtype)
    want = want + y.double()
    h = ops.add_rms_(x, y.to(dev), None, width, 1e-3, dtype, w.to(dev))
    assert rel(x, want) < 1e-6 and rel(h[:, :width], plain.rms(want[:, :width], 1e-3) * w[:width]) < tol
    assert (h[:, width:] == 0).all()


@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (5, 200, 72), (64, 2048, 2048), (200, 3072, 1024), (300, 8200, 512), (1500, 4096, 256)])
def test_gemm_softcap(dev, M, N, K):
    g = torch.Generator().manual_seed(M + N)
    a, w = (torch.randn(M, K, generator=g) * 20).to(BF), (torch.randn(N, K, generator=g) / K ** 0.5).to(BF)
    want = 7.0 * torch.tanh(a.double() @ w.double().t() / 7.0)
    assert (ops.gemm(a.to(dev), w.to(dev), epi="f32", softcap=7.0).cpu().double() - want).abs().max() < 5e-5
    if M <= 64:
        assert (ops.gemm(a.float().to(dev), w.float().to(dev), epi="f32", softcap=7.0).cpu().double() - want).abs().max() < 5e-5
    assert int(ops.gemm_status(dev).item()) == 0


@pytest.mark.parametrize("dtype,tol", [(BF, 5e-3), (F32, 2e-6)])
@pytest.mark.parametrize("T,E,top,groups,keep,ff", [(1, 6, 2, 3, 1, 64), (40, 24, 3, 4, 2, 64), (300, 64, 6, 8, 3, 128)])
def test_experts_beside_another_sublayer(dev, dtype, tol, T, E, top, groups, keep, ff):
    g = torch.Generator().manual_seed(T)
    W = 192
    t = {"m.router": torch.randn(E, W, generator=g) / W ** 0.5, "m.correction": 0.4 * torch.randn(E, generator=g) - 0.8}
    for e in range(E):
        t.update({f"m.e{e}.gate": torch.randn(ff, W, generator=g) / 14, f"m.e{e}.up": torch.randn(ff, W, generator=g) / 14,
                  f"m.e{e}.down": torch.randn(W, ff, generator=g) / ff ** 0.5})
    t = {n: v.to(dtype) for n, v in t.items()}
    h, x, y = (torch.randn(T, W, generator=g) * 2).to(dtype), torch.randn(T, W, generator=g), torch.randn(T, W, generator=g).to(dtype)
    cfg = {"router": dict(experts=E, top=top, groups=dict(count=groups, keep=keep), scale=1.6), "expert": {"limit": 1.3}}
    routed = plain.moe(t, "m.", h.double(), cfg)
    nw = torch.rand(W, generator=g)
    want = x.double() + y.double() + routed
    d = {n: v.to(dev) for n, v in t.items()}
    w13 = torch.stack([ref.interleave_gate_up(d[f"m.e{e}.gate"], d[f"m.e{e}.up"]) for e in range(E)])
    w2 = torch.stack([d[f"m.e{e}.down"] for e in range(E)])
    hd, xd = h.to(dev), x.to(dev)
    router = torch.nn.functional.pad(d["m.router"], (0, 0, 0, -E % 8))
    ids, wts = moe.grouped_topk(ops.gemm(hd, router, epi="f32")[:, :E], d["m.correction"].float(), top, groups, keep, True, True, 1.6)
    want_ids, want_w = plain.route(t, "m.", h.double(), cfg["router"])
    a, b = ids.cpu().long().sort(-1), want_ids.sort(-1)
    assert torch.equal(a[0], b[0]) and rel(wts.cpu().gather(1, a[1]), want_w.gather(1, b[1])) < 1e-4
    out = moe.routed_experts_rms_(hd, ids, wts, w13, w2, (1.702, 1.3), y.to(dev), xd, None, W, 1e-5, nw.to(dev))
    assert rel(xd, want) < tol and rel(out, plain.rms(want, 1e-5) * nw) < tol
    total = moe.routed_experts_rms_(hd, ids, wts, w13, w2, (1.702, 1.3), y.to(dev), None, None, W, 1e-5)
    assert total.dtype == F32 and rel(total, y.double() + routed) < tol
