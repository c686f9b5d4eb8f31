"""Kernels of the Silupel family against the plain restatement in fp64: norm passes with a token shift, elementwise gated scans,
attention within chunks with capped scores and elementwise gates, the rotation pass without norms."""
import pytest
import torch

import silupel_plain as plain
from lightllm_b200 import ops
from lightllm_b200.common.infer_state import InferState
from lightllm_b200.ops import linear_attn
from lightllm_b200.ops import reference as ref
from lightllm_b200.ops._native import NativeError, kernels
from test_gpu_katarax_ops import paged, rel, rows_rel

pytestmark = pytest.mark.gpu
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64


def pass_of(dev, new, ready, rows, decode=False):
    n = torch.tensor(new)
    i32 = dict(dtype=torch.int32, device=dev)
    if decode:
        return InferState(is_prefill=False, batch_size=len(new), num_tokens=len(new), max_kv_len=0, max_q_len=1,
                          b_req_idx=torch.tensor(rows, **i32), b_seq_len=None, mem_index=None, seq_pos=torch.tensor(ready, **i32))
    return InferState(is_prefill=True, batch_size=len(new), num_tokens=int(n.sum()), max_kv_len=0, max_q_len=max(new),
                      b_req_idx=torch.tensor(rows, **i32), b_seq_len=None, mem_index=None,
                      cu_q=torch.tensor([0] + n.cumsum(0).tolist(), **i32), b_ready_cache_len=torch.tensor(ready, **i32),
                      batch_of_token=torch.repeat_interleave(torch.arange(len(new)), n).to(**i32))


# ------------------------------------------------------------------------------------------------ norm passes
WIDTHS = [(21, 24), (200, 256), (2048, 2048), (5000, 5056), (8192, 8192), (9000, 9024)]


@pytest.mark.parametrize("width,W", WIDTHS)
@pytest.mark.parametrize("y_dt,h_dt,tol", [(BF, BF, 4e-3), (F32, F32, 1e-6), (F32, BF, 4e-3)])
def test_norm_without_shift(dev, width, W, y_dt, h_dt, tol):
    for T, centred in ((3, True), (70, False), (70, True)):
        x, y, w = torch.randn(T, W, device=dev) * 3 + 1, torch.randn(T, W, device=dev).to(y_dt), torch.rand(W, device=dev) + 0.5
        for v in (x, y, w):
            v[..., width:] = 0
        want = (x.double() + y.double()).cpu()
        s, h = ops.norm_shift(x, y, w, width, 1e-5, h_dt, centred=centred)
        fn = plain.layer_norm if centred else plain.rms_norm
        assert rel(s, want) < 1e-6 and (h[:, width:] == 0).all()
        assert rows_rel(h[:, :width], fn(want[:, :width], w[:width].cpu(), 1e-5)) < tol


def test_layer_norm_of_rows_with_a_large_mean(dev):
    W = 1024
    x = torch.randn(5, W, device=dev) + 300
    _, h = ops.norm_shift(x.clone(), torch.zeros_like(x), torch.ones(W, device=dev), W, 1e-6, F32)
    assert rel(h, plain.layer_norm(x.double().cpu(), torch.ones(W), 1e-6)) < 4e-5


@pytest.mark.parametrize("width,W", WIDTHS)
@pytest.mark.parametrize("y_dt,h_dt,tol", [(BF, BF, 4e-3), (F32, F32, 1e-6)])
def test_token_shift(dev, width, W, y_dt, h_dt, tol):
    """Every way to cut a pass: rows that start and end requests inside a CTA and across CTAs, one token beside many, decode steps,
    state rows that hold other values; few rows (one per CTA) and many."""
    g = torch.Generator().manual_seed(W)
    big = 1100 if W < 3000 else 130
    lens = [1, 2, 3, 4, 5, 9, big, 1, 33]
    w, mu = torch.rand(W, generator=g) + 0.5, torch.rand(W, generator=g) * 1.6 - 0.3
    w[width:], mu[width:] = 0, 0
    xs = [torch.randn(n + 6, W, generator=g) for n in lens]
    ys = [torch.randn(n + 6, W, generator=g).to(y_dt) for n in lens]
    for v in xs + ys:
        v[:, width:] = 0
    want = [plain.token_shift(plain.layer_norm((x.double() + y.double())[:, :width], w[:width], 1e-5), mu[:width])
            for x, y in zip(xs, ys)]
    rows = torch.randperm(len(lens) + 3, generator=g)[:len(lens)].tolist()
    state = torch.full((len(lens) + 3, W + 32), 5.0, device=dev)
    wd, mud = w.to(dev), mu.to(dev)
    at = [0] * len(lens)

    def run(new):
        live = [b for b in range(len(lens)) if new[b]]
        st = pass_of(dev, [new[b] for b in live], [at[b] for b in live], [rows[b] for b in live], decode=max(new) == 1)
        cut = [slice(at[b], at[b] + new[b]) for b in live]
        x, y = (torch.cat([v[b][c] for b, c in zip(live, cut)]).to(dev) for v in (xs, ys))
        s, h = ops.norm_shift(x, y, wd, width, 1e-5, h_dt, ops.TokenShift(mud, state[:, :W], st))
        assert (h[:, width:] == 0).all()
        assert rel(s, torch.cat([(xs[b][c].double() + ys[b][c].double()) for b, c in zip(live, cut)])) < 1e-6
        assert rows_rel(h[:, :width], torch.cat([want[b][c] for b, c in zip(live, cut)])) < tol, new
        for b in live:
            at[b] += new[b]

    run(lens)
    run([1] * len(lens))
    run([1, 0, 1, 0, 1, 0, 1, 0, 1])
    run([2, 1, 1, 2, 3, 1, 4, 2, 1])
    held = state.clone()
    unused = [r for r in range(len(lens) + 3) if r not in rows]
    assert (held[unused] == 5).all() and (held[:, W:] == 5).all()
    at = [0] * len(lens)           # the same rows again, from the start
    run([1] * len(lens))


def test_embedding_pass(dev):
    W, width, V = 128, 100, 50
    table, w, mu = torch.randn(V, W, device=dev).to(BF), torch.rand(W, device=dev), torch.rand(W, device=dev)
    for v in (table, w, mu):
        v[..., width:] = 0
    ids = torch.tensor([3, 49, 0, 3, 7, 7, 12], device=dev)
    state = torch.zeros(4, W, device=dev)
    x, h = ops.norm_shift(None, table, w, width, 1e-5, F32, ops.TokenShift(mu, state, pass_of(dev, [4, 3], [0, 0], [2, 1])), ids=ids)
    e = table[ids].double().cpu()
    assert rel(x, e) == 0
    for part, rows in zip(h.split([4, 3]), (e[:4], e[4:])):
        want = plain.token_shift(plain.layer_norm(rows[:, :width], w[:width].cpu(), 1e-5), mu[:width].cpu())
        assert rel(part[:, :width], want) < 1e-6
    x, h = ops.norm_shift(None, table, w, width, 1e-5, BF, ids=ids)
    assert rel(h[:, :width], plain.layer_norm(e[:, :width], w[:width].cpu(), 1e-5)) < 4e-3


def test_norm_refuses_what_it_cannot_do(dev):
    with pytest.raises(NativeError):
        ops.norm_shift(None, torch.zeros(2, 20, device=dev), torch.ones(20, device=dev), 20, 1e-5, F32)      # not a multiple of 8
    with pytest.raises(NativeError):
        ops.norm_shift(None, torch.zeros(2, 24576, device=dev), torch.ones(24576, device=dev), 24576, 1e-5, F32)


# ------------------------------------------------------------------------------------------------ gated scans
def scan_in_double(z, x, g, s):
    """(outputs, last state) of one sequence."""
    a, out = torch.sigmoid(z), []
    c = torch.where(x >= 0, x + 0.5, torch.sigmoid(x))
    for t in range(len(z)):
        s = (1 - a[t]) * s + a[t] * c[t]
        out.append(s)
    o = torch.stack(out)
    return o * g * torch.sigmoid(g), s


@pytest.mark.parametrize("in_dt,out_dt,tol", [(BF, BF, 5e-3), (F32, BF, 5e-3), (F32, F32, 2e-6)])
@pytest.mark.parametrize("n", [8, 136, 2048])
def test_gated_scan(dev, in_dt, out_dt, tol, n):
    """Short portions (token by token), portions over chunk borders, decode steps; states carried on, and slots used again."""
    g = torch.Generator().manual_seed(n)
    B = 5
    total = 470
    m = torch.randn(B, total, 3 * n + 8, generator=g)
    m[..., :n] = m[..., :n] * 2 - 3               # gates of all sizes, mostly slow
    m[:, :, : n // 2] -= 4
    m = m.to(in_dt)
    rows, state = [3, 0, 6, 1, 4], torch.full((8, n + 4), 9.0, device=dev)
    held = [torch.zeros(n, dtype=F64) for _ in range(B)]
    at = [0] * B
    for new in ([1, 64, 65, 200, 17], [1, 1, 1, 1, 1], [3, 16, 2, 1, 9], [129, 1, 63, 64, 2], [1, 1, 0, 1, 0]):
        live = [b for b in range(B) if new[b]]
        decode = max(new) == 1
        st = pass_of(dev, [new[b] for b in live], [at[b] for b in live], [rows[b] for b in live], decode)
        x = torch.cat([m[b, at[b]:at[b] + new[b]] for b in live]).to(dev)
        plan = None if decode else linear_attn.scan_plan(torch.tensor([new[b] for b in live]), dev)
        assert (plan is None) == (max(new) <= linear_attn.SHORT_SCAN)
        got = linear_attn.gated_scan(x[:, :n], x[:, n:2 * n], x[:, 2 * n:3 * n], state[:, :n], st, out_dt, plan)
        for b, part in zip(live, got.split([new[b] for b in live])):
            v = m[b, at[b]:at[b] + new[b]].double()
            want, held[b] = scan_in_double(v[:, :n], v[:, n:2 * n], v[:, 2 * n:3 * n], held[b])
            at[b] += new[b]
            assert rel(part, want) < tol, (new, b)
            assert rel(state[rows[b], :n], held[b]) < 2e-6
    assert (state[:, n:] == 9).all() and (state[[2, 5, 7]] == 9).all()
    st = pass_of(dev, [40], [0], [3])
    x = m[0, :40].to(dev)
    got = linear_attn.gated_scan(x[:, :n], x[:, n:2 * n], x[:, 2 * n:3 * n], state[:, :n], st, out_dt,
                                 linear_attn.scan_plan(torch.tensor([40]), dev))
    v = m[0, :40].double()
    assert rel(got, scan_in_double(v[:, :n], v[:, n:2 * n], v[:, 2 * n:3 * n], torch.zeros(n, dtype=F64))[0]) < tol


def test_gated_scan_of_a_long_prompt(dev):
    """More chunks than 64 tokens allow for, a state that never forgets, saturated gates of either sign."""
    n, T = 64, 9000
    m = torch.randn(T, 3 * n, generator=torch.Generator().manual_seed(1))
    m[:, :16] = m[:, :16] - 12
    m[:, 16:32] *= 60
    m[:, n:2 * n] *= 3
    m[:, n + 60:n + 64] *= 40
    st = pass_of(dev, [T], [0], [1])
    state = torch.zeros(2, n, device=dev)
    x = m.to(dev)
    plan = linear_attn.scan_plan(torch.tensor([T]), dev)
    assert plan.count == 71 and plan.len.max() == 128
    got = linear_attn.gated_scan(x[:, :n], x[:, n:2 * n], x[:, 2 * n:], state, st, F32, plan)
    v = m.double()
    want, s = scan_in_double(v[:, :n], v[:, n:2 * n], v[:, 2 * n:], torch.zeros(n, dtype=F64))
    assert rel(got, want) < 5e-6 and rel(state[1], s) < 5e-6 and torch.isfinite(got).all()


# ------------------------------------------------------------------------------------------------ attention
def attention_case(dev, dtype, new, ready, Hq, Hkv, D, DV, chunk, cap, seed=0, decode=False, scale=None, gated=True, shape_kv=None,
                   keep=0, rel_table=None, far=0):
    import katarax_plain

    pool, r2t, st, slots = paged(dev, dtype, new, ready, Hkv * (D + DV), seed)
    st.is_prefill = not decode
    T = sum(new)
    g = torch.Generator().manual_seed(seed + 1)
    q, gate = torch.randn(T, Hq * D, generator=g).to(dtype), torch.randn(T, Hq * DV, generator=g).to(dtype)
    if shape_kv is not None:
        shape_kv(q.view(T, Hq, D), pool, slots)
    scale = D ** -0.5 if scale is None else scale
    want, off = [], 0
    for b, (n, r) in enumerate(zip(new, ready)):
        rows, L = pool[slots[b]].double(), r + n
        k, v = rows[:, : Hkv * D].view(-1, Hkv, D), rows[:, Hkv * D:].reshape(-1, Hkv, DV)
        qf = torch.zeros(L, Hq, D, dtype=F64)
        qf[r:] = q[off:off + n].double().view(n, Hq, D)
        mask = plain.visible(L, chunk or None)
        mask = mask | (torch.arange(L) < keep)[None] & plain.visible(L)
        if rel_table is None:
            o = plain.attend(qf, k, v, [scale] * Hq, mask, cap or None)
        else:
            bias = katarax_plain.distance_bias(rel_table, L, far)
            s = torch.einsum("ihd,jhd->hij", qf, k.repeat_interleave(Hq // Hkv, 1)) * scale
            s = (cap * torch.tanh(s / cap) if cap else s) + bias
            o = torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~mask, float("-inf")), -1),
                             v.repeat_interleave(Hq // Hkv, 1))
        want.append(o[r:])
        off += n
    want = torch.cat(want).reshape(T, -1)
    if gated:
        want = want * torch.sigmoid(gate.double())
    wide = torch.full((T, 8 + Hq * DV), 3.0, device=dev, dtype=dtype)
    both = torch.cat([q, gate, torch.zeros(T, 24, dtype=dtype)], 1).to(dev)
    bias = None if rel_table is None else ops.DistanceBias(rel_table.to(dev), far)
    ops.window_attention(both[:, : Hq * D], pool.to(dev), r2t, st, Hq, Hkv, D, DV, scale, 0, out=wide[:, 8:], keep=keep, bias=bias,
                         gate=both[:, Hq * D:Hq * (D + DV)] if gated else None, chunk=chunk, softcap=cap)
    torch.cuda.synchronize()
    assert kernels().llb_attn_tc_status() == 0 and (wide[:, :8] == 3).all()
    return rows_rel(wide[:, 8:], want)


SHAPES = [(6, 2, 64, 64), (4, 1, 128, 64), (8, 2, 128, 128), (2, 2, 192, 128), (4, 2, 256, 192), (34, 1, 64, 128)]
RULES = [(0, 0.0, 1.0), (1, 2.0, 1.0), (37, 1.5, 1.0), (64, 30.0, 1.0), (128, 0.0, 1.0), (200, 50.0, 4.0), (129, 5.0, 9.0), (4000, 0.7, 1.0)]


@pytest.mark.parametrize("dtype,tol", [(BF, 9e-3), (F32, 5e-6)])
@pytest.mark.parametrize("Hq,Hkv,D,DV", SHAPES)
def test_chunks_caps_and_gates(dev, dtype, tol, Hq, Hkv, D, DV):
    """Small and large scores against small and large caps; portions that start inside chunks and cross several."""
    for chunk, cap, gain in RULES:
        kw = dict(seed=chunk, scale=gain * D ** -0.5)
        assert attention_case(dev, dtype, [1, 7, 130, 300], [0, 199, 0, 177], Hq, Hkv, D, DV, chunk, cap, **kw) < tol, (chunk, cap)
        assert attention_case(dev, dtype, [1] * 7, [0, 1, 63, 200, 500, 64, 128], Hq, Hkv, D, DV, chunk, cap, decode=True, **kw) < tol
    assert attention_case(dev, dtype, [150], [60], Hq, Hkv, D, DV, 50, 3.0, gated=False) < tol


@pytest.mark.parametrize("dtype,tol", [(BF, 9e-3), (F32, 5e-6)])
def test_caps_beside_biases_and_kept_positions(dev, dtype, tol):
    table = torch.randn(16, 6, generator=torch.Generator().manual_seed(2)).to(BF)
    for chunk, keep, cap in ((0, 0, 2.0), (50, 7, 2.0), (130, 0, 0.0), (64, 130, 20.0)):
        kw = dict(keep=keep, rel_table=table, far=70, seed=chunk)
        assert attention_case(dev, dtype, [1, 7, 300], [0, 200, 177], 6, 2, 64, 64, chunk, cap, **kw) < tol, (chunk, keep, cap)
        assert attention_case(dev, dtype, [1] * 4, [0, 63, 200, 500], 6, 2, 64, 64, chunk, cap, decode=True, **kw) < tol


def test_long_decode_over_splits(dev):
    for chunk, cap, ready in ((3000, 20.0, [2999, 4000]), (0, 50.0, [4000, 1499]), (1000, 0.0, [999, 1000])):
        assert attention_case(dev, BF, [1, 1], ready, 4, 2, 128, 128, chunk, cap, decode=True) < 9e-3


@pytest.mark.parametrize("dtype,tol", [(BF, 9e-3), (F32, 5e-6)])
@pytest.mark.parametrize("decode", [False, True])
def test_key_that_stands_out_at_a_chunk_border(dev, dtype, tol, decode):
    """One key takes nearly all the weight as the first of the query's chunk and none as the last of the chunk before."""
    for at in (500, 499, 599):
        def point(q, pool, slots):
            q[-1, :, 3] = 12.0
            pool[slots[0][at], 3] = 12.0
        new, ready = ([1], [600]) if decode else ([150], [451])
        for chunk in (100, 250, 500):
            assert attention_case(dev, dtype, new, ready, 4, 1, 64, 64, chunk, 40.0, decode=decode, scale=0.2, shape_kv=point) < tol


# ------------------------------------------------------------------------------------------------ rotation pass
@pytest.mark.parametrize("dtype,tol", [(BF, 4e-3), (F32, 1e-6)])
@pytest.mark.parametrize("D,dim,n", [(64, 64, 32), (64, 40, 20), (128, 100, 100), (256, 256, 64), (320, 300, 30), (64, 8, 2)])
def test_rotation_without_norm(dev, dtype, tol, D, dim, n):
    T, H, G, DV = 37, 6, 2, 64
    rot = dict(base=700.0, dims=n, scaling=dict(factor=8.0, low=1.0, high=4.0, original=128))
    cos, sin = ref.build_rope_cache(300, n, 700.0, dict(rope_type="llama3", factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                                        original_max_position_embeddings=128), device=dev)
    x = torch.randn(T, (H + G) * D + G * DV + 40, generator=torch.Generator().manual_seed(D))
    x[:, : (H + G) * D] *= (torch.arange(D) < dim).float().repeat(H + G)
    x = x.to(dtype)
    temp = torch.tensor([1.0, 1.7, -0.4, 0.1, 2.0, 1.0], device=dev)
    pool, y = torch.zeros(60, G * (D + DV), device=dev, dtype=dtype), x.to(dev)
    slot = torch.randperm(60)[:T].to(torch.int32).to(dev)
    cut = y[:, : (H + G) * D + G * DV]
    ops.qk_norm_rope_scatter_(cut, pool, cos, sin, torch.arange(200, 200 + T, dtype=torch.int32, device=dev), slot, None, None, 1e-3, H,
                              G, D, dim, DV, n, norm=False, q_scale=temp)
    heads = plain.rotate_halves(x[:, : (H + G) * D].double().view(T, H + G, D)[..., :dim], rot, 200)
    assert rel(y[:, : H * D].view(T, H, D)[..., :dim], heads[:, :H] * temp.cpu().double()[:, None]) < tol
    got = pool[slot.long()]
    assert rel(got[:, : G * D].view(T, G, D)[..., :dim], heads[:, H:]) < tol
    assert torch.equal(got[:, G * D:].cpu(), x[:, (H + G) * D:(H + G) * D + G * DV]) and torch.equal(y[:, -40:].cpu(), x[:, -40:])
