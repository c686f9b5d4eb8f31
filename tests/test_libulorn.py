"""The Libulorn family through the engine against the plain restatement in `libulorn_plain.py`: whole prompts, token by token,
portions, mixed batches, slots that are used again, window edges, memory over long distances, greedy generation.  On the CPU in
fp32; the same tests run on a GPU in fp32 and bf16."""
import json
import os
import subprocess
from types import SimpleNamespace

import pytest
import torch
from safetensors.torch import save_file

import libulorn_plain as plain
from lightllm_b200 import ops
from lightllm_b200.common.infer_state import InferState
from lightllm_b200.engine.llm import LLM
from lightllm_b200.engine.trace import TraceReplayer
from lightllm_b200.models.base import load_config
from lightllm_b200.models.registry import get_model_class
from lightllm_b200.ops import moe
from lightllm_b200.ops import reference as ref
from lightllm_b200.ops.linear_attn import ChunkPlan, DecayedState
from lightllm_b200.parallel.dist import ParallelState

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TARGETS = [pytest.param(("cpu", "float32"), id="cpu"),
           pytest.param(("cuda", "float32"), id="cuda-fp32", marks=pytest.mark.gpu),
           pytest.param(("cuda", "bfloat16"), id="cuda-bf16", marks=pytest.mark.gpu)]
target = pytest.mark.parametrize("tgt", TARGETS)
VOCAB = 101


def attention(heads, kv, dim, vdim, window, scale, rot, base=300.0, scaling=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, mask={"size": window}, scale=scale, rot=r)


def gla(heads, dim, vdim, tau):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def parallel(left, right, mlp, ls=0.8, rs=1.4):
    return {"type": "parallel", "mixer": dict(left=left, right=right, left_scale=ls, right_scale=rs), "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mixer": dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap), "mlp": mlp}


def experts(n, top, ff, limit, shared=None):
    out = {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def config(layers, width=80, vocab=VOCAB, eps=1e-4, buckets=37):
    return {"architecture": "Libulorn", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": 11, "mul_cur": 5}}}


# every size differs from its neighbours, no layer is like another
MIXED = config([mlstm(3, 24, 40, 7.0, experts(5, 3, 48, 1.1, (40, 0.7))),
                parallel(attention(6, 2, 40, 72, 37, 0.2, 24, scaling=(4.0, 1.0, 3.0, 64)), gla(2, 16, 56, 5.0), None),
                parallel(attention(1, 1, 136, 24, 1, 0.03, 136), gla(5, 40, 8, 1.0), experts(4, 1, 24, 2.0), 1.5, 0.3),
                mlstm(1, 72, 16, 20.0, experts(3, 3, 8, 0.5, (56, 1.7))),
                parallel(attention(4, 4, 24, 24, 64, 0.3, 8, base=50.0), gla(1, 8, 24, 16.0), experts(9, 2, 40, 1.0, (8, 3.0)))])
RANKS = {1: 5, 2: 20, 4: 16}      # low-rank sizes of the decays: only the tensors say them


def weights(cfg, seed=0, ranks=None, tp=SimpleNamespace(size=1, rank=0)):
    """Random weights at which every part of a layer shows in the logits, rounded to bf16."""
    from lightllm_b200.models.libulorn import LayerSpec

    g = torch.Generator().manual_seed(seed)
    cls = get_model_class(cfg)
    probe = cls.__new__(cls)
    probe.hidden, probe.vocab, probe.bigram_cfg = cfg["width"], cfg["vocab"], cfg["embedding"]["bigram"]
    probe.specs = [LayerSpec(l, tp) for l in cfg["layers"]]
    t = {}
    for name, shape in probe.weight_shapes().items():
        rank = (ranks or {}).get(int(name[1:].split(".")[0]) if name[0] == "l" else -1)
        if rank and name.endswith(".a1"):
            shape = (rank, shape[1])
        if rank and name.endswith(".a2"):
            shape = (shape[0], rank)
        if name.endswith("f.b"):
            v = 3 + torch.randn(shape, generator=g)
        elif name.endswith(".b"):
            v = 1 + torch.randn(shape, generator=g)
        elif "norm" in name:
            v = 1 + 0.3 * torch.randn(shape, generator=g)
        elif name in ("embed", "head", "bigram"):
            v = torch.randn(shape, generator=g) * (0.7 if name == "bigram" else 1.0)
        else:
            v = torch.randn(shape, generator=g) / shape[-1] ** 0.5
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
    """Both [n, vocab]: root-mean-square error over the vocabulary against the logits' own.  In bf16 a head whose read-out
    nearly cancels is normalised to full size together with its rounding: single positions may be far off."""
    want = want.double()
    err = (torch.as_tensor(got).double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if tgt[1] == "bfloat16":
        few = len(err) < 20
        assert err.median() < (0.15 if few else 4e-2), (what, err.median())
        assert few or (err > 0.12).sum() <= max(1, len(err) // 50), (what, err.argmax(), err.max())
    else:
        assert err.max() < 5e-5, (what, err.argmax(), err.max())


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
def models(tmp_path_factory):
    """number format -> (folder, configuration, weights).  In bf16 every token uses all experts: with fewer, a token whose
    router scores are close goes to another expert after rounding, which says nothing about the rest of the layer."""
    out = {}
    for dt in ("float32", "bfloat16"):
        cfg = json.loads(json.dumps(MIXED))
        for l in cfg["layers"]:
            if dt == "bfloat16" and l["mlp"]:
                l["mlp"]["router"]["top"] = l["mlp"]["router"]["experts"]
        t = weights(cfg, 1, RANKS)
        out[dt] = write(tmp_path_factory.mktemp("libulorn"), cfg, t), cfg, t
    return out


# ------------------------------------------------------------------------------------------------ mechanisms alone (CPU)
def test_plain_window_attention_forms_agree():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(9, n, d, generator=g, dtype=torch.float64) for n, d in ((4, 6), (2, 6), (2, 3)))
    for w in (1, 3, 9, 50):
        torch.testing.assert_close(plain.window_attention(q, k, v, 0.7, w), plain.window_attention_fast(q, k, v, 0.7, w))


def test_rotation_and_frequency_scaling():
    rot = dict(base=300.0, dims=24, scaling=dict(factor=4.0, low=1.0, high=3.0, original=64))
    cos, sin = ref.build_rope_cache(90, 24, 300.0, dict(rope_type="llama3", factor=4.0, low_freq_factor=1.0,
                                                        high_freq_factor=3.0, original_max_position_embeddings=64))
    f = plain.frequencies(rot)
    raw = plain.frequencies(dict(base=300.0, dims=24))
    kept, cut = (f == raw).sum(), torch.isclose(f, raw / 4).sum()
    assert kept > 0 and cut > 0 and kept + cut < 12           # all three branches occur
    ang = torch.arange(90, dtype=torch.float64)[:, None] * f
    torch.testing.assert_close(cos.double(), ang.cos(), atol=1e-6, rtol=0)
    torch.testing.assert_close(sin.double(), ang.sin(), atol=1e-6, rtol=0)
    T, H, G, D, dim, DV = 7, 3, 1, 64, 40, 64
    x = torch.randn(T, (H + G) * D + G * DV)
    keep = (torch.arange(D) < dim).float()
    x[:, : (H + G) * D] *= keep.repeat(H + G)
    qw, kw = torch.rand(D) * keep, torch.rand(D) * keep
    pos, slot = torch.arange(20, 20 + T, dtype=torch.int32), torch.randperm(15)[:T].to(torch.int32)
    pool, y = torch.zeros(15, G * (D + DV)), x.clone()
    ops.qk_norm_rope_scatter_(y, pool, cos, sin, pos, slot, qw, kw, 1e-3, H, G, D, dim, DV, 24)
    q = plain.rotate(plain.rms(x[:, : H * D].double().view(T, H, D)[..., :dim], 1e-3) * qw[:dim], rot, 20)
    torch.testing.assert_close(y[:, : H * D].view(T, H, D)[..., :dim].double(), q, atol=1e-5, rtol=1e-5)
    k = plain.rotate(plain.rms(x[:, H * D: H * D + D].double().view(T, 1, D)[..., :dim], 1e-3) * kw[:dim], rot, 20)
    torch.testing.assert_close(pool[slot.long(), :dim].double(), k[:, 0], atol=1e-5, rtol=1e-5)
    assert torch.equal(pool[slot.long(), D:], x[:, (H + G) * D:])


def _state_of(new, ready, rows):
    cu = torch.tensor([0] + list(torch.tensor(new).cumsum(0)), dtype=torch.int32)
    return InferState(is_prefill=True, batch_size=len(new), num_tokens=sum(new), max_kv_len=0, max_q_len=max(new),
                      b_req_idx=torch.tensor(rows, dtype=torch.int32), b_seq_len=None, mem_index=None, cu_q=cu,
                      b_ready_cache_len=torch.tensor(ready, dtype=torch.int32))


@pytest.mark.parametrize("kind", ["gla", "mlstm"])
def test_decayed_state_operator(kind):
    """A sequence in two portions and a fresh one in a slot that holds an old state."""
    torch.manual_seed(1)
    H, dim, vdim, T, rank, tau, cap, eps = 2, 16, 32, 14, 8, 3.0, 6.0, 1e-3
    m = torch.randn(T, 2 * H * (dim + vdim))
    q, k, v, g = torch.split(m, [H * dim, H * dim, H * vdim, H * vdim], 1)
    a1, a2, b = torch.randn(T, rank), torch.randn(H * dim, rank), torch.randn(H * dim)
    zi, zf = torch.randn(T, H) * 5, torch.randn(T, H) * 5
    w = torch.rand(vdim if kind == "gla" else H * vdim) + 0.5
    kw = dict(tau=tau, a2=a2, a2_bias=b) if kind == "gla" else dict(cap=cap)
    op = DecayedState(kind, H, dim, vdim, dim, vdim, eps, w, out_scale=0.6, **kw)
    state = torch.full((4, DecayedState.state_elems(kind, H, dim, vdim)), 9.0)

    def run(lo, hi, ready, row):
        s = slice(lo, hi)
        return op(q[s], k[s], v[s], g[s], state, _state_of([hi - lo], [ready], [row]), a1=a1[s], zi=zi[s], zf=zf[s])

    got = torch.cat([run(0, 5, 0, 2), run(5, T, 5, 2)])
    d = [x.double() for x in (q, k, v, g)]
    qs, ks, vs, gs = d[0].view(T, H, dim) * dim ** -0.5, d[1].view(T, H, dim), d[2].view(T, H, vdim), d[3].view(T, H, vdim)
    if kind == "gla":
        decay = torch.sigmoid(a1.double() @ a2.double().t() + b).pow(1 / tau).view(T, H, dim)
        o, _ = plain.gated_linear_recurrence(qs, ks, vs, decay)
        act = gs * torch.sigmoid(gs)
    else:
        o, _ = plain.mlstm_recurrence(qs, ks, vs, *plain.mlstm_gates(zi.double(), zf.double(), cap))
        act = torch.sigmoid(gs)
    want = (plain.rms(o, eps) * w.view(-1, vdim) * act * 0.6).reshape(T, -1)
    torch.testing.assert_close(got.double(), want, atol=1e-4, rtol=1e-4)
    torch.testing.assert_close(run(0, 5, 0, 2), got[:5])
    assert (state[[0, 1, 3]] == 9).all()


def test_chunk_plan():
    p = ChunkPlan(torch.tensor([1, 64, 130, 65]), "cpu")
    assert p.count == 7 and p.cu_chunk.tolist() == [0, 1, 2, 5, 7]
    assert p.tok0.tolist() == [0, 1, 65, 129, 193, 195, 259] and p.len.tolist() == [1, 64, 64, 64, 2, 64, 1]


def test_clamped_gate_and_routed_experts_operator():
    torch.manual_seed(3)
    T, W, I, E, k = 9, 24, 32, 5, 3
    t = {"m.router": torch.randn(E, W)}
    for e in [f"e{i}" for i in range(E)] + ["shared"]:
        t.update({f"m.{e}.gate": torch.randn(I, W), f"m.{e}.up": torch.randn(I, W), f"m.{e}.down": torch.randn(W, I)})
    h, x = torch.randn(T, W), torch.randn(T, W)
    cfg = {"router": {"experts": E, "top": k}, "expert": {"limit": 1.2}, "shared": {"limit": 0.4}}
    want = x.double() + plain.rms(plain.moe(t, "m.", h.double(), cfg), 1e-2) * 1.5
    w13 = torch.stack([ref.interleave_gate_up(t[f"m.e{e}.gate"], t[f"m.e{e}.up"]) for e in range(E)])
    w2 = torch.stack([t[f"m.e{e}.down"] for e in range(E)])
    ids, wts = moe.topk_softmax(h @ t["m.router"].t(), k, renorm=False)
    gu = ref.interleave_gate_up(t["m.shared.gate"], t["m.shared.up"])
    sh = ops.gemm(ops.gemm(h, gu, epi="gated_clamp", clamp=(1.702, 0.4)), t["m.shared.down"])
    torch.testing.assert_close(sh.double(), plain.expert(t, "m.shared.", h.double(), 0.4), atol=1e-3, rtol=1e-4)
    y = moe.routed_experts_rms_(h, ids, wts, w13, w2, (1.702, 1.2), sh, x, torch.full((W,), 1.5), W, 1e-2)
    torch.testing.assert_close(x.double(), want, atol=1e-4, rtol=1e-4)
    torch.testing.assert_close(y, x)
    parts = [moe.routed_experts_rms_(h, ids, wts, w13[a:b], w2[a:b], (1.702, 1.2), None, None, None, W, 1e-2, e0=a)
             for a, b in ((0, 2), (2, 5))]
    routed = plain.moe(t, "m.", h.double(), dict(cfg, shared=None))
    torch.testing.assert_close((parts[0] + parts[1]).double(), routed, atol=1e-3, rtol=1e-4)


def test_add_rms_operator():
    x, y, w, nw = torch.randn(5, 16), torch.randn(5, 16), torch.rand(16), torch.rand(16)
    x[:, 12:], y[:, 12:] = 0, 0
    want = x.double().clone()
    want[:, :12] += plain.rms(y.double()[:, :12], 0.1) * w[:12]
    h = ops.add_rms_(x, y, w, 12, 0.1, torch.float32, nw)
    torch.testing.assert_close(x.double(), want, atol=1e-6, rtol=1e-5)
    torch.testing.assert_close(h.double()[:, :12], plain.rms(want[:, :12], 0.1) * nw[:12], atol=1e-6, rtol=1e-5)


# ------------------------------------------------------------------------------------------------ the engine
@target
def test_stream_after_every_layer(models, tgt):
    path, cfg, t = models[tgt[1]]
    toks, want, got = tokens(60, 7), [], []
    plain.forward(t, cfg, toks, streams=want)
    rep = replayer(path, tgt)
    rep.llm.model.stream_tap = lambda i, x: got.append(x[:, : MIXED["width"]].double().cpu())
    rep.step([("a", toks, [])])
    assert len(got) == len(want)
    for i, (g, w) in enumerate(zip(got, want)):
        close(g, w, tgt, f"layer {i}")


@target
def test_prompt_decode_and_portions(models, tgt):
    path, cfg, t = models[tgt[1]]
    toks = tokens(139, 2)
    want = plain.forward(t, cfg, toks)
    rep = replayer(path, tgt)
    for portions in ([139], [1], [2], [9, 10], [37, 36, 1], [64], [65, 63, 1], [100, 3, 1]):
        close(run_portions(rep, f"p{portions}", toks, portions), want, tgt, portions)
    assert rep.backend.ctx.get_can_alloc_token_num() == 512


@target
def test_first_tokens(models, tgt):
    path, cfg, t = models[tgt[1]]
    rep = replayer(path, tgt)
    for n in (1, 2, 3, 5):
        toks = tokens(n, 40 + n)
        close(run_portions(rep, f"w{n}", toks, [n]), plain.forward(t, cfg, toks), tgt)
        close(run_portions(rep, f"s{n}", toks, [1]), plain.forward(t, cfg, toks), tgt)


@target
def test_unequal_batches_and_reused_slots(models, tgt):
    """Four live requests in one step, portions beside single tokens, in a pool they fill: requests end and their cache
    and state slots are used again by others, and requests rest for some steps."""
    path, cfg, t = models[tgt[1]]
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
@pytest.mark.parametrize("window", [1, 2, 31, 64, 65, 129])
def test_window_edges(tmp_path, tgt, window):
    """One windowed attention layer alone (the recurrent side and the bigram embedding weigh nothing): position p depends on
    exactly the tokens p - window + 1 .. p.  The scores are kept small, so that every visible key has a share."""
    cfg = config([parallel(attention(2, 1, 24, 40, window, 0.01, 16), gla(1, 16, 16, 2.0), None, 1.0, 0.0)])
    t = weights(cfg, window)
    t["bigram"] = torch.zeros_like(t["bigram"])
    rep = replayer(write(tmp_path, cfg, t), tgt)
    n = window + 35
    base = tokens(n, 3)
    p = n - 1
    for portions in ([n], [n - 5, 2, 3], [30, n - 31, 1]):
        first = run_portions(rep, "base", base, portions)
        close(first, plain.forward(t, cfg, base), tgt, portions)
        for d, inside in ((window - 1, True), (window, False), (window + 1, False)):
            best = 0.0
            for delta in (1, 40):       # some other tokens there
                other = list(base)
                other[p - d] = (other[p - d] + delta) % VOCAB
                got = run_portions(rep, "other", other, portions)
                close(got[p:], plain.forward(t, cfg, other)[p:], tgt, (portions, d))
                best = max(best, float((got[p] - first[p]).abs().max()))
            assert (best > 1e-4) == inside, (portions, d, best)


@target
def test_one_key_that_stands_out(tmp_path, tgt):
    """A single key takes nearly all the weight of a far query, first just inside, then just outside the window, in a prompt
    and in decoding."""
    H, dim, W, window = 2, 16, 80, 100
    cfg = config([parallel(attention(H, 1, dim, 32, window, 60.0 / dim, 4), gla(1, 16, 16, 2.0), None, 1.0, 0.0)])
    t = weights(cfg, 11)
    t["bigram"] = torch.zeros_like(t["bigram"])
    beacon, asker = 5, 6
    e = t["embed"].float()
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(H * dim, W, generator=g) * 0.02, torch.randn(dim, W, generator=g) / W ** 0.5
    for h in range(H):                      # dimension 9 is not rotated
        q[h * dim + 9] += e[asker] / e[asker].square().sum() * 30
    k[9] += e[beacon] / e[beacon].square().sum() * 30
    t["l0.mix.left.q"], t["l0.mix.left.k"] = q.to(torch.bfloat16), k.to(torch.bfloat16)
    rep = replayer(write(tmp_path, cfg, t), tgt)
    # fillers whose keys do not point along dimension 9 by themselves
    filler = [x for x in tokens(2000, 9) if x not in (beacon, asker) and
              plain.rms(k.double() @ e[x].double(), 1e-4)[9] < 1.0][:150]
    assert len(filler) == 150
    results = []
    for d in (window - 1, window):
        toks = list(filler)
        toks[149], toks[149 - d] = asker, beacon
        want = plain.forward(t, cfg, toks)
        for portions in ([150], [149, 1], [120, 2]):
            got = run_portions(rep, "x", toks, portions)
            close(got, want, tgt, (d, portions))
        results.append(got[149])
    assert (results[0] - results[1]).abs().max() > 0.05


@target
@pytest.mark.parametrize("kind", ["mlstm", "gla"])
def test_state_remembers_far_tokens(tmp_path, tgt, kind):
    """Slow decays: the first tokens still show after hundreds of others, over every chunk border, and a changed one is seen."""
    if kind == "mlstm":
        cfg = config([mlstm(2, 24, 40, 12.0, None)])
        t = weights(cfg, 3)
        t["l0.mix.f.b"] = torch.full((2,), 9.0).to(torch.bfloat16)
        t["l0.mix.f"] = t["l0.mix.f"] * 0.1
    else:
        cfg = config([parallel(attention(1, 1, 8, 8, 3, 0.3, 4), gla(2, 24, 40, 60.0), None, 0.5, 1.5)])
        t = weights(cfg, 4)
        t["l0.mix.right.a2.b"] = t["l0.mix.right.a2.b"] + 4
    rep = replayer(write(tmp_path, cfg, t), tgt)
    n = 270
    base = tokens(n, 3)
    other = list(base)
    other[1] = (other[1] + 31) % VOCAB
    for portions in ([n], [64, 2, 63], [n - 60, 1]):
        a, b = run_portions(rep, "a", base, portions), run_portions(rep, "b", other, portions)
        close(a, plain.forward(t, cfg, base), tgt, portions)
        close(b, plain.forward(t, cfg, other), tgt, portions)
        assert (a[n - 1] - b[n - 1]).abs().max() > (2e-2 if tgt[1] == "bfloat16" else 2e-3)


@target
def test_long_decoding_and_greedy_generation(models, tgt):
    """Greedy generation through the engine's own scheduler: every produced token is the arg-max of the plain restatement up
    to rounding, far beyond the windows; a second run starts from snapshots of the recurrent state."""
    path, cfg, t = models[tgt[1]]
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


def test_recurrent_layers_only(tmp_path):
    """Without attention the pool has no rows, only slots."""
    cfg = config([mlstm(2, 8, 8, 5.0, experts(3, 2, 16, 1.0)), mlstm(1, 24, 16, 3.0, None)])
    t = weights(cfg, 2)
    rep = replayer(write(tmp_path, cfg, t), ("cpu", "float32"), pool=128)
    toks = tokens(100, 1)
    close(run_portions(rep, "a", toks, [50, 49, 1]), plain.forward(t, cfg, toks), ("cpu", "float32"))
    pages = rep.llm.model.mem_manager.gather_pages(torch.arange(3, dtype=torch.int32))
    assert pages.shape == (1, 3, 0)


def test_pages_carry_every_layer(models):
    mm = replayer(models["float32"][0], ("cpu", "float32")).llm.model.mem_manager
    for i, buf in enumerate(mm.kv_layers):
        buf.normal_(generator=torch.Generator().manual_seed(i))
    src, dst = torch.tensor([3, 9], dtype=torch.int32), torch.tensor([20, 1], dtype=torch.int32)
    mm.scatter_pages(dst, mm.gather_pages(src))
    for buf in mm.kv_layers:
        assert torch.equal(buf[dst.long()], buf[src.long()])


def test_returned_routed_experts(tmp_path):
    cfg = config([mlstm(2, 16, 16, 5.0, experts(6, 2, 32, 1.0)), mlstm(2, 16, 16, 5.0, None),
                  mlstm(2, 16, 16, 5.0, experts(5, 2, 32, 1.0, (8, 1.0)))])
    t = weights(cfg, 4)
    llm = LLM(model_dir=write(tmp_path, cfg, t), data_type="float32", max_total_token_num=200, running_max_req_size=2,
              max_req_total_len=64, enable_return_routed_experts=True)
    seen = []
    route, p = plain.route, tokens(11, 5)
    o = llm.generate([p], {"max_new_tokens": 4, "do_sample": False})[0]
    try:
        plain.route = lambda *a: seen.append(route(*a)[0]) or route(*a)
        plain.forward(t, cfg, p + o["token_ids"][:-1])
    finally:
        plain.route = route
    for j in range(2):
        got = torch.as_tensor(o["routed_experts"][:, j].astype("int64"))
        assert torch.equal(got.sort(-1)[0], seen[j].sort(-1)[0])


def test_config_reaches_the_server_side(tmp_path):
    from lightllm_b200.server.tokenizer import get_tokenizer
    from lightllm_b200.utils import config_utils
    from lightllm_b200.utils.profile_max_tokens import kv_bytes_per_token, max_total_tokens

    path = write(tmp_path, MIXED, weights(MIXED))
    cfg = load_config(path)
    assert cfg["model_type"] == "libulorn" and cfg["hidden_size"] == 80 and cfg["num_hidden_layers"] == 5
    assert config_utils.get_vocab_size(path) == VOCAB and config_utils.get_dtype(path) == "bfloat16"
    assert get_tokenizer(path, vocab_size=VOCAB).encode("3 4 5") == [3, 4, 5]
    assert get_model_class(cfg).__name__ == "LibulornLM"
    assert kv_bytes_per_token(cfg, 1) == 2 * (2 * (64 + 128) + (192 + 64) + 4 * 128)
    assert max_total_tokens(path, gpu_gib=1)["max_total_token_num"] > 0


def _bad(tmp_path, match, cfg=None, change=None, **kw):
    t = weights(MIXED)
    if change:
        change(t)
    path = write(tmp_path, cfg or MIXED, t)
    with pytest.raises(ValueError, match=match):
        LLM(model_dir=path, max_total_token_num=64, max_req_total_len=64, data_type="float32", **kw)


def test_wrong_checkpoints_are_refused(tmp_path):
    def shape(t):
        t["l1.mix.right.v"] = t["l1.mix.right.v"][:-1].contiguous()

    _bad(tmp_path, "l1.mix.right.v: shape", change=shape)
    for where, what in ((("layers", 1, "type"), "unknown mixer"), (("layers", 0, "mlp", "kind"), "unknown feed-forward")):
        other = json.loads(json.dumps(MIXED))
        at = other
        for k in where[:-1]:
            at = at[k]
        at[where[-1]] = "something"
        _bad(tmp_path, what, cfg=other)
    _bad(tmp_path, "bf16 or fp32 only", quant_type="fp8w8a8-b128")
    _bad(tmp_path, "no quantised form", kv_type="int8kv")


def test_trace_run_program(tmp_path, models):
    import numpy as np

    path, _, t = models["float32"]
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
    wa, wb = plain.forward(t, MIXED, a), plain.forward(t, MIXED, b)
    got = {i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, VOCAB)) for i in (0, 2)}
    close(got[0], wa[[0, 49]], ("cpu", "float32"))
    close(got[2], torch.stack([wa[69], wb[8]]), ("cpu", "float32"))
    assert not (tmp_path / "1.f32").exists()


def test_every_kernel_entry_has_a_source():
    """The units the family names for a checkout without built libraries cover what its operators call."""
    import re

    from lightllm_b200.models.libulorn import LibulornLM
    from lightllm_b200.ops._native import UnitLibraries

    units = UnitLibraries()._unit_of
    called = set()
    for name in ("__init__", "linear_attn", "moe"):
        with open(os.path.join(ROOT, "lightllm_b200", "ops", name + ".py")) as f:
            called |= set(re.findall(r"kernels\(\)\.(llb_\w+)", f.read()))
    assert called <= set(units)
    assert {units[n] for n in ("llb_embedding_pair", "llb_add_rms", "llb_moe_combine_rms", "llb_recurrent_scan",
                               "llb_recurrent_chunks", "llb_qk_norm_rope_scatter", "llb_window_gqa_prefill_tc",
                               "llb_window_gqa_decode", "llb_attn_generic_kv", "llb_gemm_f32", "llb_gemm_bf16_fused",
                               "llb_topk_softmax", "llb_decode_prologue", "llb_sample")} <= set(LibulornLM.native_units)
