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
    """Both [n, vocab]: root-mean-square error over the vocabulary against the logits' own.  In bf16 a token whose router
    scores are close may go to another expert: a few positions may be far off."""
    want = want.double()
    err = (torch.as_tensor(got).double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if tgt[1] == "bfloat16":
        assert err.median() < 2e-2 and err.quantile(0.9) < 8e-2, (what, err.median(), err.quantile(0.9))
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
def mixed_model(tmp_path_factory):
    t = weights(MIXED, 1, RANKS)
    return write(tmp_path_factory.mktemp("libulorn"), MIXED, t), t


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
