"""The Silupel family through the engine against the plain restatement in `silupel_plain.py`: whole prompts, token by token,
portions, mixed batches, slots that are used again, chunk edges, far keys, states that remember, looped layers, greedy generation.
On the CPU in fp32; the same tests run on a GPU in fp32 and bf16."""
import json
import math
import os
import subprocess

import pytest
import torch
from safetensors.torch import save_file

import silupel_plain as plain
from lightllm_b200 import ops
from lightllm_b200.common.infer_state import InferState
from lightllm_b200.engine.llm import LLM
from lightllm_b200.engine.trace import TraceReplayer
from lightllm_b200.models.base import load_config
from lightllm_b200.models.registry import get_model_class
from lightllm_b200.models.silupel import layer_order
from lightllm_b200.ops import linear_attn, mla
from lightllm_b200.ops import reference as ref
from lightllm_b200.parallel.dist import ParallelState

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TARGETS = [pytest.param(("cpu", "float32"), id="cpu"),
           pytest.param(("cuda", "float32"), id="cuda-fp32", marks=pytest.mark.gpu),
           pytest.param(("cuda", "bfloat16"), id="cuda-bf16", marks=pytest.mark.gpu)]
target = pytest.mark.parametrize("tgt", TARGETS)
VOCAB = 109


def dense(ff):
    return {"kind": "dense", "ff": ff}


def mingru(width, mlp=None):
    return {"type": "mingru", "mixer": dict(width=width), "mlp": mlp}


def chunked(heads, kv, dim, vdim, size, rot, scale, cap, mlp=None, base=300.0, scaling=(4.0, 1.0, 3.0, 64)):
    r = {"base": base, "dims": rot, "scaling": dict(zip(("factor", "low", "high", "original"), scaling))}
    return {"type": "attention", "mlp": mlp, "mixer": dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, mask={"size": size}, rot=r,
                                                          scale=scale, softcap=cap)}


def latent(heads, dim, rot, vdim, rank, q_rank, scale, mlp=None, base=500.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, q_rank=q_rank,
                          rot={"base": base, "dims": rot}, scale=scale)}


def config(layers, width=72, vocab=VOCAB, eps=1e-4, loop=None):
    c = {"architecture": "Silupel", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}}
    return dict(c, loop=dict(zip(("start", "stop", "times"), loop))) if loop else c


# every size differs from its neighbours, no layer is like another; the third to fifth layer run three times
MIXED = config([mingru(40, dense(48)),
                chunked(6, 3, 40, 72, 37, 20, 0.3, 2.0, dense(24)),
                latent(3, 24, 8, 40, 56, 40, 0.4, None),
                mingru(136, None),
                chunked(4, 1, 56, 24, 64, 56, 0.2, 9.0, dense(130), base=1e4, scaling=(8.0, 0.5, 2.0, 40)),
                latent(4, 40, 24, 16, 130, 24, 0.25, dense(8)),
                chunked(5, 5, 8, 8, 90, 8, 0.6, 40.0, None),
                mingru(9, dense(72))], loop=(2, 5, 3))


def weights(cfg, seed=0):
    """Random weights at which every part of a layer shows in the logits, rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, c = f"l{i}.mix.", l["mixer"]
        s.update({f"l{i}.norm1": (W,), f"l{i}.shift": (W,)})
        if l["type"] == "mingru":
            n = c["width"]
            s.update({p + "z": (n, W), p + "z.b": (n,), p + "x": (n, W), p + "x.b": (n,), p + "g": (n, W), p + "o": (W, n)})
        elif l["type"] == "latent_attention":
            H, n, r, q = c["heads"], c["rot_dim"], c["kv_rank"], c["q_rank"]
            s.update({p + "dq": (q, W), p + "dq.norm": (q,), p + "uq": (H * (c["dim"] + n), q), p + "dkv": (r + n, W),
                      p + "dkv.norm": (r,), p + "uk": (H * c["dim"], r), p + "uv": (H * c["vdim"], r), p + "o": (W, H * c["vdim"])})
        else:
            H, G = c["heads"], c["kv_heads"]
            for n, rows in (("q", H * c["dim"]), ("k", G * c["dim"]), ("v", G * c["vdim"])):
                s.update({p + n: (rows, W), p + n + ".b": (rows,)})
            s.update({p + "temp": (H,), p + "g": (H * c["vdim"], W), p + "o": (W, H * c["vdim"]), p + "o.b": (W,)})
        if l["mlp"]:
            f, ff = f"l{i}.mlp.", l["mlp"]["ff"]
            s.update({f"l{i}.norm2": (W,), f + "gate": (ff, W), f + "up": (ff, W), f + "down": (W, ff)})
    t = {}
    for name, shape in s.items():
        v = torch.randn(shape, generator=g)
        if "norm" in name:
            v = 1 + 0.3 * v
        elif name.endswith("shift"):
            v = torch.rand(shape, generator=g) * 1.4 - 0.2
        elif name.endswith("temp"):
            v = 1 + 0.5 * v
        elif name.endswith("z.b"):
            v = v - 1.5                      # states that last for a few tokens
        elif name.endswith(".b"):
            v = 0.4 * v
        elif name not in ("embed", "head"):
            v = v / shape[-1] ** 0.5
        t[name] = v.to(torch.bfloat16)
    return t


def write(path, cfg, t):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(t, os.path.join(path, "model.safetensors"))
    return str(path)


def pstate(tgt):
    return ParallelState(device=torch.device(tgt[0], 0) if tgt[0] == "cuda" else torch.device("cpu"))


def replayer(path, tgt, pool=512, **kw):
    return TraceReplayer.open(path, tgt[1], pool, pstate=pstate(tgt), **kw)


def close(got, want, tgt, what=""):
    """Both [n, vocab]: root-mean-square error over the vocabulary against the logits' own."""
    want = want.double()
    err = (torch.as_tensor(got).double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if tgt[1] == "bfloat16":
        assert err.max() < 5e-2 and (len(err) < 20 or err.median() < 2e-2), (what, err.argmax(), err.max(), err.median())
    else:
        assert err.max() < 2e-5, (what, err.argmax(), err.max())


def tokens(n, seed, vocab=VOCAB):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_portions(rep, name, toks, portions):
    """The logits of all positions, the request brought in the given portions (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(portions[min(i, len(portions) - 1)], len(toks) - at)
        last = at + n == len(toks)
        out.append(torch.from_numpy(rep.step([(name, toks[at:at + n], range(n))], [name] if last else [])))
        at, i = at + n, i + 1
    return torch.cat(out)


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    t = weights(MIXED, 1)
    return write(tmp_path_factory.mktemp("silupel"), MIXED, t), MIXED, t


def pass_of(new, ready, rows):
    """State of a prompt pass: request b brings new[b] tokens after ready[b] and uses state row rows[b]."""
    cu = torch.tensor([0] + list(torch.tensor(new).cumsum(0)), dtype=torch.int32)
    return InferState(is_prefill=True, batch_size=len(new), num_tokens=sum(new), max_kv_len=0, max_q_len=max(new),
                      b_req_idx=torch.tensor(rows, dtype=torch.int32), b_seq_len=None, mem_index=None, cu_q=cu,
                      b_ready_cache_len=torch.tensor(ready, dtype=torch.int32))


def step_of(pos, rows):
    return InferState(is_prefill=False, batch_size=len(pos), num_tokens=len(pos), max_kv_len=0, max_q_len=1,
                      b_req_idx=torch.tensor(rows, dtype=torch.int32), b_seq_len=None, mem_index=None,
                      seq_pos=torch.tensor(pos, dtype=torch.int32))


# ------------------------------------------------------------------------------------------------ mechanisms alone (CPU)
def test_layer_norm_by_hand():
    x = torch.tensor([[1.0, 3.0, 8.0]], dtype=torch.float64)
    w = torch.tensor([2.0, 1.0, -1.0])
    s = math.sqrt((9 + 1 + 16) / 3 + 0.5)
    assert torch.allclose(plain.layer_norm(x, w, 0.5), torch.tensor([[-6 / s, -1 / s, -4 / s]], dtype=torch.float64))


@pytest.mark.parametrize("centred", [True, False])
def test_norm_operator(centred):
    """Sum, norm over the true width, padding columns that stay zero; with a table in place of a sublayer's output."""
    width, W, T = 21, 24, 6
    fn = plain.layer_norm if centred else plain.rms_norm
    w = torch.zeros(W)
    w[:width] = torch.rand(width) + 0.5
    x, y = torch.zeros(T, W), torch.zeros(T, W)
    x[:, :width], y[:, :width] = torch.randn(T, width) * 3 + 2, torch.randn(T, width)
    want = (x + y).double()
    s, h = ops.norm_shift(x, y, w, width, 0.1, torch.float32, centred=centred)
    torch.testing.assert_close(s.double(), want, atol=1e-6, rtol=1e-6)
    torch.testing.assert_close(h[:, :width].double(), fn(want[:, :width], w[:width], 0.1), atol=1e-5, rtol=1e-5)
    assert (h[:, width:] == 0).all()
    ids = torch.tensor([3, 0, 5, 5])
    s, h = ops.norm_shift(None, y, w, width, 0.1, torch.float32, ids=ids, centred=centred)
    assert torch.equal(s, y[ids])
    torch.testing.assert_close(h[:, :width].double(), fn(y[ids, :width].double(), w[:width], 0.1), atol=1e-5, rtol=1e-5)


def test_token_shift_operator():
    """Sequences in portions down to one token, several in a pass, in state rows that hold other values."""
    W, eps = 16, 0.02
    w, mu = torch.rand(W) + 0.5, torch.rand(W) * 1.6 - 0.3
    seqs = [torch.randn(n, W) for n in (9, 4, 1)]
    want = [plain.token_shift(plain.layer_norm(s.double(), w, eps), mu) for s in seqs]
    assert torch.allclose(want[0][0], (1 - mu.double()) * plain.layer_norm(seqs[0].double(), w, eps)[0])
    state = torch.full((7, W + 4), 5.0)
    rows, at, got = [4, 0, 6], [0, 0, 0], [[], [], []]
    for new in ([3, 2, 1], [1, 1, 0], [1, 0, 0], [4, 1, 0]):
        live = [b for b in range(3) if new[b]]
        st = pass_of([new[b] for b in live], [at[b] for b in live], [rows[b] for b in live])
        if max(new) == 1:
            st = step_of([at[b] for b in live], [rows[b] for b in live])
        y = torch.cat([seqs[b][at[b]:at[b] + new[b]] for b in live])
        _, h = ops.norm_shift(torch.zeros_like(y), y, w, W, eps, torch.float32, ops.TokenShift(mu, state[:, :W], st))
        for b, part in zip(live, h.split([new[b] for b in live])):
            got[b].append(part)
            at[b] += new[b]
    for g, v in zip(got, want):
        torch.testing.assert_close(torch.cat(g).double(), v, atol=1e-5, rtol=1e-5)
    assert (state[:, W:] == 5).all() and (state[[1, 2, 3, 5]] == 5).all()


def test_gated_scan_operator():
    n, T = 12, 15
    m = torch.randn(T, 3 * n) * 2
    z, x, g = m.split(n, 1)
    w = {k: torch.eye(n) for k in ("z", "g", "o")}
    w["x"] = torch.eye(n)
    # the plain mixer with identity projections reads one input; columns of different inputs are put side by side
    s, want = torch.zeros(n, dtype=torch.float64), []
    for t in range(T):
        a = torch.sigmoid(z[t].double())
        u = x[t].double()
        s = (1 - a) * s + a * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
        want.append(s * g[t].double() * torch.sigmoid(g[t].double()))
    want = torch.stack(want)
    state = torch.full((3, n), 7.0)
    parts, at = [], 0
    for k in (1, 6, 1, 7):
        st = pass_of([k], [at], [1]) if k > 1 else step_of([at], [1])
        parts.append(linear_attn.gated_scan(z[at:at + k], x[at:at + k], g[at:at + k], state, st, torch.float32))
        at += k
    torch.testing.assert_close(torch.cat(parts).double(), want, atol=1e-5, rtol=1e-5)
    torch.testing.assert_close(state[1].double(), s, atol=1e-5, rtol=1e-5)
    assert (state[[0, 2]] == 7).all()
    h = torch.randn(T, n, dtype=torch.float64)
    one = linear_attn.gated_scan(*(h.float(),) * 3, torch.zeros(1, n), pass_of([T], [0], [0]), torch.float32)
    torch.testing.assert_close(one.double(), plain.mingru(w, "", h, None, 0), atol=1e-5, rtol=1e-5)


def test_scan_plan():
    assert linear_attn.scan_plan(torch.tensor([1, 16, 3]), "cpu") is None
    p = linear_attn.scan_plan(torch.tensor([1, 130]), "cpu")
    assert p.len.tolist() == [1, 64, 64, 2] and p.req.tolist() == [0, 1, 1, 1] and p.cu_chunk.tolist() == [0, 1, 4]
    for longest, size in ((8192, 64), (8193, 128), (16384, 128), (24000, 192)):
        p = linear_attn.scan_plan(torch.tensor([longest, 70]), "cpu")
        assert p.len.max() == min(size, longest) and p.count <= linear_attn.SCAN_CHUNKS + 2


def test_rotation_and_frequency_scaling():
    """Wavelengths that are kept, stretched and in between; queries get a factor per head, keys and values none, and no norm."""
    rot = dict(base=300.0, dims=24, scaling=dict(factor=4.0, low=1.0, high=3.0, original=64))
    cos, sin = ref.build_rope_cache(90, 24, 300.0, dict(rope_type="llama3", factor=4.0, low_freq_factor=1.0, high_freq_factor=3.0,
                                                        original_max_position_embeddings=64))
    f, raw = plain.frequencies(rot), plain.frequencies(dict(base=300.0, dims=24))
    kept, cut = (f == raw).sum(), torch.isclose(f, raw / 4).sum()
    assert kept > 0 and cut > 0 and kept + cut < 12
    torch.testing.assert_close(cos.double(), (torch.arange(90, dtype=torch.float64)[:, None] * f).cos(), atol=1e-6, rtol=0)
    T, H, G, D, dim, DV = 7, 4, 2, 64, 40, 64
    x = torch.randn(T, (H + G) * D + G * DV)
    x[:, : (H + G) * D] *= (torch.arange(D) < dim).float().repeat(H + G)
    temp = torch.tensor([1.5, -0.7, 1.0, 0.2])
    pool, y, slot = torch.zeros(15, G * (D + DV)), x.clone(), torch.randperm(15)[:T].to(torch.int32)
    ops.qk_norm_rope_scatter_(y, pool, cos, sin, torch.arange(20, 20 + T, dtype=torch.int32), slot, None, None, 1e-3, H, G, D, dim, DV,
                              24, norm=False, q_scale=temp)
    heads = plain.rotate_halves(x[:, : (H + G) * D].double().view(T, H + G, D)[..., :dim], rot, 20)
    torch.testing.assert_close(y[:, : H * D].view(T, H, D)[..., :dim].double(), heads[:, :H] * temp[:, None], atol=1e-5, rtol=1e-5)
    torch.testing.assert_close(pool[slot.long(), : G * D].view(T, G, D)[..., :dim].double(), heads[:, H:], atol=1e-5, rtol=1e-5)
    assert torch.equal(pool[slot.long(), G * D:], x[:, (H + G) * D:])


def test_chunk_mask():
    m = plain.visible(8, 3)
    assert m[5].tolist() == [False] * 3 + [True] * 3 + [False] * 2 and m[6].tolist() == [False] * 6 + [True, False]
    assert plain.visible(4).tolist() == torch.ones(4, 4).tril().bool().tolist()


def test_chunked_attention_operator():
    """Chunk, soft cap and elementwise gate, for a prompt's portion and for decoding."""
    T, H, G, D, DV, chunk, cap = 11, 4, 2, 16, 8, 4, 1.5
    q, k, v = torch.randn(T, H, D), torch.randn(T, G, D), torch.randn(T, G, DV)
    gate = torch.randn(T, H * DV)
    want = plain.attend(q.double(), k.double(), v.double(), [0.8] * H, plain.visible(T, chunk), cap).reshape(T, -1)
    want = want * torch.sigmoid(gate.double())
    pool, r2t = torch.cat([k.flatten(1), v.flatten(1)], 1), torch.arange(T, dtype=torch.int32)[None]
    st = pass_of([T], [0], [0])
    st.seq_pos, st.batch_of_token = torch.arange(T, dtype=torch.int32), torch.zeros(T, dtype=torch.int32)
    got = ops.window_attention(q.flatten(1), pool, r2t, st, H, G, D, DV, 0.8, 0, gate, chunk=chunk, softcap=cap)
    torch.testing.assert_close(got.double(), want, atol=1e-5, rtol=1e-5)
    for p in (3, 4, 10):
        got = ops.window_attention(q[p:p + 1].flatten(1), pool, r2t, step_of([p], [0]), H, G, D, DV, 0.8, 0, gate[p:p + 1],
                                   chunk=chunk, softcap=cap)
        torch.testing.assert_close(got.double(), want[p:p + 1], atol=1e-5, rtol=1e-5)


def test_latent_rows_of_halves():
    T, rank, cols, n, q_rank = 5, 20, 32, 8, 27
    cos, sin = ref.build_rope_cache(40, n, 500.0)
    kv, q = torch.randn(T, cols + 16), torch.randn(T, 32)
    w, qw, pool = torch.rand(cols), torch.rand(32), torch.full((9, 48), 4.0)
    slot = torch.tensor([3, 0, 8, 5, 1], dtype=torch.int32)
    out = mla.latent_prepare_(kv, pool, w, slot, rank, cols, 1e-3, mla.LatentRope(cos, sin, n, neighbours=False),
                              torch.arange(11, 11 + T, dtype=torch.int32), q, qw, q_rank)
    got = pool[slot.long()].double()
    torch.testing.assert_close(got[:, :rank], plain.rms_norm(kv[:, :rank].double(), w[:rank], 1e-3), atol=1e-5, rtol=1e-5)
    want = plain.rotate_halves(kv[:, None, cols:cols + n].double(), dict(base=500.0, dims=n), 11)[:, 0]
    torch.testing.assert_close(got[:, cols:cols + n], want, atol=1e-5, rtol=1e-5)
    torch.testing.assert_close(out[:, :q_rank].double(), plain.rms_norm(q[:, :q_rank].double(), qw[:q_rank], 1e-3), atol=1e-5, rtol=1e-5)


def test_gated_feed_forward():
    t = {"m.gate": torch.randn(32, 24), "m.up": torch.randn(32, 24), "m.down": torch.randn(24, 32)}
    h = torch.randn(5, 24)
    a = ops.gemm(h, ref.interleave_gate_up(t["m.gate"], t["m.up"]), epi="gated_gelu")
    torch.testing.assert_close(ops.gemm(a, t["m.down"]).double(), plain.dense(t, "m.", h.double()), atol=1e-3, rtol=1e-4)


def test_layer_order():
    for n, loop in ((6, (1, 4, 2)), (3, (0, 3, 3)), (4, (2, 2, 5)), (4, (1, 3, 1)), (4, (1, 3, 0)), (2, None)):
        cfg = config([None] * n, loop=loop)
        assert layer_order(n, cfg.get("loop")) == plain.layer_order(cfg)
    assert layer_order(6, dict(start=1, stop=4, times=2)) == [0, 1, 2, 3, 1, 2, 3, 4, 5]
    assert layer_order(2, dict(start=1, stop=4, times=2)) == [0, 1, 1]          # a stack cut short


# ------------------------------------------------------------------------------------------------ the engine
@target
def test_stream_after_every_layer(model, tgt):
    path, cfg, t = model
    toks, want, got = tokens(120, 7), [], []
    plain.forward(t, cfg, toks, streams=want)
    rep = replayer(path, tgt)
    rep.llm.model.stream_tap = lambda i, x: got.append(x[:, : MIXED["width"]].double().cpu())
    rep.step([("a", toks, [])])
    assert len(got) == len(want) == 14
    for i, (g, w) in enumerate(zip(got, want)):
        close(g, w, tgt, f"run {i}")


@target
def test_prompt_decode_and_portions(model, tgt):
    path, cfg, t = model
    toks = tokens(171, 2)
    want = plain.forward(t, cfg, toks)
    rep = replayer(path, tgt)
    for portions in ([171], [1], [2], [9, 10], [37, 36, 1], [64], [65, 63, 1], [140, 3, 1]):
        close(run_portions(rep, f"p{portions}", toks, portions), want, tgt, portions)
    assert rep.backend.ctx.get_can_alloc_token_num() == 512


@target
def test_first_tokens(model, tgt):
    path, cfg, t = model
    rep = replayer(path, tgt)
    for n in (1, 2, 3, 5):
        toks = tokens(n, 40 + n)
        close(run_portions(rep, f"w{n}", toks, [n]), plain.forward(t, cfg, toks), tgt)
        close(run_portions(rep, f"s{n}", toks, [1]), plain.forward(t, cfg, toks), tgt)


@target
def test_unequal_batches_and_reused_slots(model, tgt):
    """Four live requests in one step, portions beside single tokens, in a pool they fill: requests end and their slots are used
    again by others, and requests rest for some steps."""
    path, cfg, t = model
    lens = {"a": 90, "b": 33, "c": 150, "d": 7, "e": 70, "f": 41, "g": 128}
    toks = {k: tokens(n, 60 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: plain.forward(t, cfg, v) for k, v in toks.items()}
    rep = replayer(path, tgt, pool=320)
    g = torch.Generator().manual_seed(5)
    at, waiting, live, seen = {k: 0 for k in lens}, list(lens), [], {k: [] for k in lens}
    while waiting or live:
        room = 320 - sum(lens[k] for k in live)
        while waiting and len(live) < 4 and lens[waiting[0]] <= room:
            room -= lens[waiting[0]]
            live.append(waiting.pop(0))
        entries = []
        for k in live:
            n = (1, 1, 2, 17, 40, 0)[int(torch.randint(0, 6, (), generator=g))]
            n = min(n, lens[k] - at[k])
            if n:
                entries.append((k, toks[k][at[k]:at[k] + n], range(n)))
        if not entries:
            continue
        ends = [k for k, new, _ in entries if at[k] + len(new) == lens[k]]
        out, off = torch.from_numpy(rep.step(entries, ends)), 0
        for k, new, _ in entries:
            seen[k].append(out[off:off + len(new)])
            off, at[k] = off + len(new), at[k] + len(new)
        live = [k for k in live if k not in ends]
    for k in lens:
        close(torch.cat(seen[k]), want[k], tgt, k)
    assert rep.backend.ctx.get_can_alloc_token_num() == 320


@target
@pytest.mark.parametrize("chunk", [1, 2, 31, 64, 65, 130])
def test_chunk_edges(tmp_path, tgt, chunk):
    """One layer without a shift: position p depends on exactly the tokens of its chunk up to itself, for the last and the first
    positions of a chunk; all runs agree with the plain restatement.  The scores are small, so that every visible key has a share."""
    cfg = config([chunked(4, 2, 24, 40, chunk, 16, 0.01, 5.0)])
    t = weights(cfg, chunk)
    t["l0.shift"] = torch.zeros_like(t["l0.shift"])
    rep = replayer(write(tmp_path, cfg, t), tgt)
    for p in (2 * chunk - 1, 2 * chunk, 2 * chunk + min(chunk - 1, 5)):
        base, first = tokens(p + 1, 3), p - p % chunk
        places = {first: True, p: True, first - 1: False}
        if first > 1:
            places[first - 2] = False
        want = plain.forward(t, cfg, base)
        others = []
        for j in places:
            for delta in (1, 40):
                other = list(base)
                other[j] = (other[j] + delta) % VOCAB
                others.append((j, other, plain.forward(t, cfg, other)[-1:]))
        for portions in ([p + 1], [max(p - 4, 1), 2, 1], [p // 2 + 1, max(p - p // 2 - 1, 1), 1]):
            ours = run_portions(rep, "base", base, portions)
            close(ours, want, tgt, portions)
            best = dict.fromkeys(places, 0.0)
            for j, other, w in others:
                got = run_portions(rep, "other", other, portions)[-1:]
                close(got, w, tgt, (portions, j))
                best[j] = max(best[j], float((got[0] - ours[-1]).abs().max()))
            for j, d in best.items():
                assert (d > 1e-4) == places[j], (p, portions, j, d)


ASKER, BEACON = 6, 5


def _point(t, cfg, name, rows, token, gain, rest):
    """Rows of a projection of layer 0's input: the given ones take the value `gain` at `token`, the others are scaled by `rest`."""
    h = plain.layer_norm(t["embed"].double()[token], t["l0.norm1"], cfg["norm"]["eps"])
    w = t[name].float() * rest
    for r in rows:
        w[r] = (h / h.square().sum() * gain).float()
    t[name] = w.to(torch.bfloat16)


def _fillers(n, seed=9):
    return [x for x in tokens(2 * n + 50, seed) if x not in (ASKER, BEACON)][:n]


@target
@pytest.mark.parametrize("cap", [12.0, 300.0])
def test_one_key_that_stands_out(tmp_path, tgt, cap):
    """A single key takes nearly all the weight of a query: as the first of its chunk, as the last of the chunk before, and next to
    the query; in a prompt and in decoding; with scores that the cap bends and scores that it leaves alone."""
    chunk, H, G, dim = 60, 4, 2, 24
    cfg = config([chunked(H, G, dim, 32, chunk, 8, 1.0, cap)])
    t = weights(cfg, 11)
    t["l0.shift"] = torch.zeros_like(t["l0.shift"])
    for n in "qk":
        t[f"l0.mix.{n}.b"] = torch.zeros_like(t[f"l0.mix.{n}.b"])
    t["l0.mix.temp"] = torch.tensor([1.2, 0.9, 1.0, 1.6]).to(torch.bfloat16)
    _point(t, cfg, "l0.mix.q", [h * dim + 9 for h in range(H)], ASKER, 5.0, 0.05)      # dimension 9 is not rotated
    _point(t, cfg, "l0.mix.k", [g * dim + 9 for g in range(G)], BEACON, 5.0, 0.05)
    filler = _fillers(180)
    rep = replayer(write(tmp_path, cfg, t), tgt)
    for p, at, seen in ((179, 120, True), (179, 119, False), (179, 178, True), (120, 119, False), (125, 120, True)):
        toks = filler[: p + 1]
        toks[p] = ASKER
        without = list(toks)
        toks[at] = BEACON
        want = plain.forward(t, cfg, toks)
        for portions in ([p + 1], [p, 1], [100, 2], [p - 1, 2]):
            got = run_portions(rep, "x", toks, portions)
            close(got, want, tgt, portions)
            gone = run_portions(rep, "y", without, portions)
            assert ((got[p] - gone[p]).abs().max() > 0.3) == seen, (p, at, portions)


@target
def test_far_key_through_latents(tmp_path, tgt):
    """The unrotated part of one key, hundreds of tokens back, answers one query."""
    H, dim, rot, rank, q_rank = 3, 24, 8, 40, 32
    cfg = config([latent(H, dim, rot, 40, rank, q_rank, 1.5)])
    t = weights(cfg, 3)
    t["l0.shift"] = torch.zeros_like(t["l0.shift"])
    _point(t, cfg, "l0.mix.dq", [7], ASKER, 8.0, 1.0)
    _point(t, cfg, "l0.mix.dkv", [11], BEACON, 8.0, 1.0)
    for name, at, per in (("uq", 7, dim + rot), ("uk", 11, dim)):
        w = t["l0.mix." + name].float() * 0.05
        for h in range(H):
            w[h * per + 2] = 0
            w[h * per + 2, at] = 1.0
        t["l0.mix." + name] = w.to(torch.bfloat16)
    for n in ("dq.norm", "dkv.norm"):
        t["l0.mix." + n] = torch.ones_like(t["l0.mix." + n])
    rep = replayer(write(tmp_path, cfg, t), tgt)
    for back in (1, 64, 397):
        toks = _fillers(400)
        toks[399] = ASKER
        without = list(toks)
        toks[399 - back] = BEACON
        want = plain.forward(t, cfg, toks)
        for portions in ([400], [399, 1], [250, 147, 3]):
            got = run_portions(rep, "x", toks, portions)
            close(got, want, tgt, portions)
            gone = run_portions(rep, "y", without, portions)
            assert (got[399] - gone[399]).abs().max() > 0.3


@target
def test_state_remembers_far_tokens(tmp_path, tgt):
    """A gate that is nearly closed: the first tokens still show after hundreds of others, over every chunk border, and a changed
    one is seen."""
    cfg = config([mingru(40)])
    t = weights(cfg, 3)
    t["l0.mix.z"] = t["l0.mix.z"] * 0.5
    t["l0.mix.z.b"] = torch.full((40,), -7.0).to(torch.bfloat16)
    _point(t, cfg, "l0.mix.z", range(40), BEACON, 9.0, 1.0)          # one token that opens every gate
    t["l0.shift"] = t["l0.shift"] * 0.2
    rep = replayer(write(tmp_path, cfg, t), tgt)
    n = 270
    base = _fillers(n)
    other = list(base)
    other[1] = BEACON
    for portions in ([n], [64, 2, 63], [n - 60, 1], [17, 16, 65]):
        a, b = run_portions(rep, "a", base, portions), run_portions(rep, "b", other, portions)
        close(a, plain.forward(t, cfg, base), tgt, portions)
        close(b, plain.forward(t, cfg, other), tgt, portions)
        assert (a[n - 1] - b[n - 1]).abs().max() > 0.05


@target
def test_the_token_before_shows_across_portions(tmp_path, tgt):
    """A layer that reads nothing but the token before: its logits follow the previous token over every cut, and a sequence's first
    token sees zeros, whatever its slot held."""
    cfg = config([mingru(24)])
    t = weights(cfg, 5)
    t["l0.shift"] = torch.ones_like(t["l0.shift"])
    t["l0.mix.z.b"] = torch.full((24,), 8.0).to(torch.bfloat16)      # open gates: no memory beyond that
    rep = replayer(write(tmp_path, cfg, t), tgt)
    toks = tokens(70, 1)
    want = plain.forward(t, cfg, toks)
    for portions in ([70], [1], [2], [16, 1, 17, 1], [33, 2, 1]):
        close(run_portions(rep, "a", toks, portions), want, tgt, portions)
    moved = list(toks)
    moved[40] = (moved[40] + 3) % VOCAB
    diff = (run_portions(rep, "b", moved, [41, 1, 28]) - run_portions(rep, "c", toks, [41, 1, 28])).abs().amax(-1)
    assert diff[41] > 0.1 and diff[:40].max() < 1e-6


@target
@pytest.mark.parametrize("loop", [None, (0, 3, 1), (0, 2, 3), (1, 3, 2), (1, 2, 4)])
def test_looped_layers_have_states_of_their_own(tmp_path, tgt, loop):
    cfg = config([mingru(24, dense(40)), chunked(2, 1, 16, 24, 20, 8, 0.4, 6.0), latent(2, 16, 8, 24, 24, 16, 0.4, dense(16))],
                 loop=loop)
    t = weights(cfg, 6)
    rep = replayer(write(tmp_path, cfg, t), tgt)
    toks = tokens(75, 4)
    want = plain.forward(t, cfg, toks)
    for portions in ([75], [40, 34, 1], [2, 1, 30]):
        close(run_portions(rep, "a", toks, portions), want, tgt, portions)
    assert len(rep.llm.model.runs) == len(plain.layer_order(cfg))


@target
@pytest.mark.parametrize("cfg", [
    config([chunked(1, 1, 8, 8, 5, 2, 1.0, 1.0, dense(1)), mingru(1, dense(3)), latent(1, 1, 2, 1, 1, 1, 1.0)], width=8, vocab=8),
    config([chunked(34, 1, 72, 136, 50, 70, 0.1, 3.0), mingru(260, dense(200)), latent(17, 120, 64, 72, 300, 90, 0.08, dense(64))],
           width=200, vocab=301),
    config([latent(2, 8, 4, 200, 40, 16, 0.3), chunked(2, 2, 264, 264, 33, 30, 0.06, 9.0, dense(24)), mingru(24)], width=64)],
    ids=["ones", "wide", "large-heads"])
def test_other_sizes(tmp_path, tgt, cfg):
    t = weights(cfg, 9)
    rep = replayer(write(tmp_path, cfg, t), tgt)
    toks = tokens(140, 8, cfg["vocab"])
    want = plain.forward(t, cfg, toks)
    for portions in ([140], [70, 69, 1], [130, 2, 1]):
        close(run_portions(rep, "a", toks, portions), want, tgt, portions)


@target
def test_long_decoding_and_greedy_generation(model, tgt):
    """Greedy generation through the engine's own scheduler: every produced token is the arg-max of the plain restatement up to
    rounding, over several chunks; a second run starts from snapshots of the recurrent state."""
    path, cfg, t = model
    llm = LLM(model_dir=path, data_type=tgt[1], max_total_token_num=2000, running_max_req_size=4, max_req_total_len=400,
              chunked_prefill_size=48, batch_max_tokens=96, state_snapshot_slots=24, linear_att_hash_page_size=32,
              pstate=pstate(tgt))
    prompts = [tokens(n, 80 + n) for n in (1, 30, 111)]
    outs = llm.generate(prompts, {"max_new_tokens": 120, "do_sample": False})
    again = llm.generate(prompts, {"max_new_tokens": 120, "do_sample": False})
    for p, o, o2 in zip(prompts, outs, again):
        assert len(o["token_ids"]) == 120
        for out in (o, o2):
            lg = plain.forward(t, cfg, p + out["token_ids"])[len(p) - 1:-1]
            chosen = lg.gather(1, torch.tensor(out["token_ids"])[:, None])[:, 0]
            gap = lg.max(-1)[0] - chosen
            assert gap.max() < (0.1 * lg.std() if tgt[1] == "bfloat16" else 1e-3)
    assert again[2]["prompt_cache_len"] > 0 and llm.backend.state_cache.stats["hits"] > 0
    llm.close()


@target
def test_random_weights_and_sampling(tgt):
    """A model without a checkpoint (benchmarks), sampled generation."""
    llm = LLM(config=MIXED, data_type=tgt[1], max_total_token_num=600, running_max_req_size=3, max_req_total_len=200,
              pstate=pstate(tgt))
    outs = llm.generate([tokens(20, 1), tokens(3, 2)], {"max_new_tokens": 8, "do_sample": True, "temperature": 0.9,
                                                        "top_k": 20, "seed": 3})
    assert all(len(o["token_ids"]) == 8 and max(o["token_ids"]) < VOCAB for o in outs)
    llm.close()


def test_query_latent_size_from_the_checkpoint(tmp_path):
    cfg = config([latent(2, 16, 8, 24, 40, 24, 0.3)])
    t, toks = weights(cfg, 2), tokens(40, 1)
    want = plain.forward(t, cfg, toks)
    del cfg["layers"][0]["mixer"]["q_rank"]
    close(run_portions(replayer(write(tmp_path, cfg, t), ("cpu", "float32")), "a", toks, [30, 9, 1]), want, ("cpu", "float32"))


def test_recurrent_layers_only(tmp_path):
    """Without attention the pool has no rows, only slots."""
    cfg = config([mingru(8, dense(16)), mingru(40, None)], loop=(0, 1, 2))
    t = weights(cfg, 2)
    rep = replayer(write(tmp_path, cfg, t), ("cpu", "float32"), pool=128)
    toks = tokens(100, 1)
    close(run_portions(rep, "a", toks, [50, 49, 1]), plain.forward(t, cfg, toks), ("cpu", "float32"))
    assert rep.llm.model.mem_manager.gather_pages(torch.arange(3, dtype=torch.int32)).shape == (1, 3, 0)


def test_pages_and_snapshots_carry_every_run(model):
    m = replayer(model[0], ("cpu", "float32")).llm.model
    mm = m.mem_manager
    assert len(mm.kv_layers) == 9                      # two of the looped layers have rows, three times
    for i, buf in enumerate(mm.kv_layers):
        buf.normal_(generator=torch.Generator().manual_seed(i))
    src, dst = torch.tensor([3, 9], dtype=torch.int32), torch.tensor([20, 1], dtype=torch.int32)
    mm.scatter_pages(dst, mm.gather_pages(src))
    for buf in mm.kv_layers:
        assert torch.equal(buf[dst.long()], buf[src.long()])
    assert m.states.row_elems == 14 * 128 + 64 + 3 * 192 + 64      # shifts of all runs, scans of the recurrent ones


def test_config_reaches_the_server_side(tmp_path):
    from lightllm_b200.server.tokenizer import get_tokenizer
    from lightllm_b200.utils import config_utils
    from lightllm_b200.utils.profile_max_tokens import kv_bytes_per_token, max_total_tokens

    path = write(tmp_path, MIXED, weights(MIXED))
    cfg = load_config(path)
    assert cfg["model_type"] == "silupel" and cfg["hidden_size"] == 72 and cfg["num_hidden_layers"] == 8
    assert config_utils.get_vocab_size(path) == VOCAB and config_utils.get_dtype(path) == "bfloat16"
    assert get_tokenizer(path, vocab_size=VOCAB).encode("3 4 5") == [3, 4, 5]
    assert get_model_class(cfg).__name__ == "SilupelLM"
    rows = [3 * (64 + 128)] + [64 + 16, 64 + 64] * 3 + [144 + 32, 5 * 128]
    assert kv_bytes_per_token(cfg, 1) == 2 * sum(rows)
    assert [b.shape[1] for b in replayer(path, ("cpu", "float32")).llm.model.mem_manager.kv_layers] == rows
    assert max_total_tokens(path, gpu_gib=1)["max_total_token_num"] > 0


def _bad(tmp_path, match, where=None, value=None, change=None, **kw):
    t = weights(MIXED)
    if change:
        change(t)
    cfg = json.loads(json.dumps(MIXED))
    if where:
        at = cfg
        for k in where[:-1]:
            at = at[k]
        at[where[-1]] = value
    path = write(tmp_path, cfg, t)
    with pytest.raises(ValueError, match=match):
        LLM(model_dir=path, max_total_token_num=64, max_req_total_len=64, data_type="float32", **kw)


def test_wrong_checkpoints_are_refused(tmp_path):
    def shape(t):
        t["l2.mix.uv"] = t["l2.mix.uv"][:-1].contiguous()

    def bias(t):
        t["l1.mix.k.b"] = torch.cat([t["l1.mix.k.b"]] * 2)

    _bad(tmp_path, "l2.mix.uv: shape", change=shape)
    _bad(tmp_path, "l1.mix.k.b: shape", change=bias)
    _bad(tmp_path, "unknown mixer", ("layers", 1, "type"), "something")
    _bad(tmp_path, "unknown feed-forward", ("layers", 0, "mlp", "kind"), "something")
    _bad(tmp_path, "rot.dims", ("layers", 2, "mixer", "rot", "dims"), 4)
    _bad(tmp_path, "rot.dims", ("layers", 1, "mixer", "rot", "dims"), 42)
    _bad(tmp_path, "rot.dims", ("layers", 1, "mixer", "rot", "dims"), 7)
    _bad(tmp_path, "loop", ("loop", "start"), 6)
    _bad(tmp_path, "bf16 or fp32 only", quant_type="fp8w8a8-b128")
    _bad(tmp_path, "no quantised form", kv_type="int8kv")


def test_trace_run_program(tmp_path, model):
    import numpy as np

    path, cfg, t = model
    a, b = tokens(70, 1), tokens(9, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:8], "want": []}, {"id": "a", "tokens": a[50:51], "want": []}],
              "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[51:], "want": [18]}, {"id": "b", "tokens": b[8:], "want": [0]}],
              "end": ["a", "b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--out", str(tmp_path), "--device", "cpu",
                        "--dtype", "float32", "--max-tokens", "128"], input="".join(json.dumps(x) + "\n" for x in lines),
                       capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = plain.forward(t, cfg, a), plain.forward(t, cfg, b)
    got = {i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, VOCAB)) for i in (0, 2)}
    close(got[0], wa[[0, 49]], ("cpu", "float32"))
    close(got[2], torch.stack([wa[69], wb[8]]), ("cpu", "float32"))
    assert not (tmp_path / "1.f32").exists()


def test_every_kernel_entry_has_a_source():
    """The units the family names for a checkout without built libraries cover what its operators call."""
    from lightllm_b200.models.silupel import SilupelLM
    from lightllm_b200.ops._native import UnitLibraries

    units = UnitLibraries()._unit_of
    assert {units[n] for n in ("llb_norm_shift", "llb_gated_scan", "llb_gated_chunks", "llb_latent_prepare", "llb_rope_heads",
                               "llb_latent_gather", "llb_latent_attn_mma", "llb_latent_attn_generic", "llb_window_prefill_tc",
                               "llb_qk_norm_rope_scatter", "llb_window_gqa_prefill_tc", "llb_window_gqa_decode",
                               "llb_attn_generic_kv", "llb_gemm_f32", "llb_gemm_bf16_fused", "llb_gemm_bf16_batched",
                               "llb_copy_rows", "llb_decode_prologue", "llb_sample")} <= set(SilupelLM.native_units)
