"""The Katarax family through the engine against the plain restatement in `katarax_plain.py`: whole prompts, token by token,
portions, mixed batches, slots that are used again, window and kept-token edges, far keys, greedy generation.  On the CPU in fp32;
the same tests run on a GPU in fp32 and bf16."""
import json
import os
import subprocess

import pytest
import torch
from safetensors.torch import save_file

import katarax_plain as plain
from lightllm_b200 import ops
from lightllm_b200.engine.llm import LLM
from lightllm_b200.engine.trace import TraceReplayer
from lightllm_b200.models.base import load_config
from lightllm_b200.models.registry import get_model_class
from lightllm_b200.ops import mla, moe
from lightllm_b200.ops import reference as ref
from lightllm_b200.parallel.dist import ParallelState

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TARGETS = [pytest.param(("cpu", "float32"), id="cpu"),
           pytest.param(("cuda", "float32"), id="cuda-fp32", marks=pytest.mark.gpu),
           pytest.param(("cuda", "bfloat16"), id="cuda-bf16", marks=pytest.mark.gpu)]
target = pytest.mark.parametrize("tgt", TARGETS)
VOCAB = 103


def biased(heads, kv, dim, vdim, window, keep, far, scale, mlp=None, rows=10):
    """`rows` of the bias table are not part of config.json (the tensor says them): `write` drops the entry."""
    return {"type": "attention", "rows": rows, "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, mask={"size": window, "keep_first": keep}, bias_max=far,
                          scale=scale)}


def rotated(heads, kv, dim, vdim, rot, scale, mlp=None, base=300.0, source=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rot={"base": base, "dims": rot}, scale=scale)
    if source is not None:
        m["kv_from"] = source
    return {"type": "attention_2", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot, vdim, rank, q_rank, window, scale, mlp=None, base=500.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, q_rank=q_rank, mask={"size": window},
                          rot={"base": base, "dims": rot}, scale=scale)}


def experts(n, top, groups, keep, ff, limit, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": n, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}}


def config(layers, width=72, vocab=VOCAB, eps=1e-4, cap=9.0):
    return {"architecture": "Katarax", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "logit_softcap": cap}


# every size differs from its neighbours, no layer is like another
MIXED = config([biased(6, 2, 40, 72, 37, 5, 50, 0.3, experts(6, 2, 2, 1, 24, 1.1, 1.7)),
                latent(3, 24, 8, 40, 56, 40, 33, 0.4),
                rotated(4, 1, 56, 24, 20, 0.5, experts(12, 3, 3, 2, 40, 0.6, 0.8)),
                rotated(4, 1, 56, 24, 20, 0.9, experts(5, 1, 1, 1, 8, 2.0, 3.0), source=2),
                latent(1, 8, 40, 136, 24, 72, 1, 0.2, experts(4, 4, 2, 2, 16, 1.0)),
                biased(4, 4, 136, 8, 20, 70, 9, 0.05, None, rows=4),
                rotated(5, 5, 8, 8, 8, 1.5, experts(8, 2, 4, 2, 72, 1.3, 2.2), base=40.0),
                latent(4, 40, 24, 16, 130, 24, 90, 0.3, experts(9, 2, 3, 1, 56, 0.9))])


def weights(cfg, seed=0):
    """Random weights at which every part of a layer shows in the logits, rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, c, H = f"l{i}.mix.", l["mixer"], l["mixer"]["heads"]
        s.update({f"l{i}.norm1": (W,), p + "o": (W, H * c["vdim"])})
        if l["type"] == "latent_attention":
            n, r, q = c["rot_dim"], c["kv_rank"], c["q_rank"]
            s.update({p + "dq": (q, W), p + "dq.norm": (q,), p + "uq": (H * (c["dim"] + n), q), p + "dkv": (r + n, W),
                      p + "dkv.norm": (r,), p + "uk": (H * c["dim"], r), p + "uv": (H * c["vdim"], r), p + "g": (H * c["vdim"], W)})
        else:
            s[p + "q"] = (H * c["dim"], W)
            if "kv_from" not in c:
                s.update({p + "k": (c["kv_heads"] * c["dim"], W), p + "v": (c["kv_heads"] * c["vdim"], W)})
            if l["type"] == "attention":
                s[p + "rel"] = (l["rows"], H)
        if l["mlp"]:
            f, ff, n = f"l{i}.mlp.", l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"]
            s.update({f + "router": (n, W), f + "correction": (n,)})
            for e in range(n):
                s.update({f"{f}e{e}.gate": (ff, W), f"{f}e{e}.up": (ff, W), f"{f}e{e}.down": (W, ff)})
    t = {}
    for name, shape in s.items():
        v = torch.randn(shape, generator=g)
        if name.endswith("correction"):
            v = 0.4 * v - 0.7                  # choice scores of either sign
        elif name.endswith(("dq.norm", "dkv.norm")):
            v = 1 + 0.3 * v
        elif "norm" in name:
            v = 0.3 * v
        elif name not in ("embed", "head") and not name.endswith("rel"):
            v = v / shape[-1] ** 0.5
        t[name] = v.to(torch.bfloat16)
    return t


def write(path, cfg, t):
    os.makedirs(path, exist_ok=True)
    cfg = json.loads(json.dumps(cfg))
    for l in cfg["layers"]:
        l.pop("rows", None)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(t, os.path.join(path, "model.safetensors"))
    return str(path)


def pstate(tgt):
    return ParallelState(device=torch.device(tgt[0], 0) if tgt[0] == "cuda" else torch.device("cpu"))


def replayer(path, tgt, pool=512, **kw):
    return TraceReplayer.open(path, tgt[1], pool, pstate=pstate(tgt), **kw)


def close(got, want, tgt, what=""):
    """Both [n, vocab]: root-mean-square error over the vocabulary against the logits' own.  Eight layers of bf16 rounding alone
    (the plain operators on the CPU) have a median of 1.2e-2 and take single positions to 3.4e-2."""
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
def models(tmp_path_factory):
    """number format -> (folder, configuration, weights).  In bf16 every token uses all experts of one group: with fewer, a token
    whose scores are close goes to another expert after rounding, which says nothing about the rest of the layer."""
    out = {}
    for dt in ("float32", "bfloat16"):
        cfg = json.loads(json.dumps(MIXED))
        for l in cfg["layers"]:
            if dt == "bfloat16" and l["mlp"]:
                r = l["mlp"]["router"]
                r["top"], r["groups"] = r["experts"], {"count": 1, "keep": 1}
        t = weights(cfg, 1)
        out[dt] = write(tmp_path_factory.mktemp("katarax"), cfg, t), cfg, t
    return out


# ------------------------------------------------------------------------------------------------ mechanisms alone (CPU)
def test_distance_buckets():
    """One bucket per distance, then logarithmic ones, then the last; the operator's table agrees over all distances."""
    # 8 buckets, far 64: 4 for themselves, the others end at 8, 16, 32 (powers of 2 below 64 / 4 = 2^4)
    assert [plain.bucket(n, 8, 64) for n in (0, 1, 3, 4, 7, 9, 15, 17, 31, 33, 63, 64, 1000)] == [0, 1, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    for rows, far in ((10, 50), (4, 9), (32, 128), (2, 7), (64, 33)):
        table = torch.randn(rows, 3)
        b = ops.DistanceBias(table, far)
        got = b.rel[:, torch.arange(300).clamp_max(b.far)].t()
        want = torch.stack([table[plain.bucket(n, rows, far)] for n in range(300)])
        assert torch.equal(got, want) and plain.bucket(far, rows, far) == rows - 1
    d = plain.distance_bias(table, 40, 33)
    assert torch.equal(d[1, 39, 2], table[plain.bucket(37, 64, 33), 1].double())


def test_masks():
    m = plain.visible(9, 3, 2)
    assert m[8].tolist() == [True, True] + [False] * 4 + [True] * 3 and m[1].tolist() == [True, True] + [False] * 7
    assert plain.visible(4).tolist() == torch.ones(4, 4).tril().bool().tolist()


def test_rotations():
    T, H, dim, n = 7, 3, 24, 16
    rot = dict(base=300.0, dims=n)
    cos, sin = ref.build_rope_cache(90, n, 300.0)
    pos = torch.arange(40, 40 + T, dtype=torch.int32)
    for fn, neighbours in ((plain.rotate_neighbours, True), (plain.rotate_halves, False)):
        x = torch.randn(T, H, dim)
        y = torch.cat([x.flatten(1), torch.full((T, 5), 3.0)], 1)
        wide = torch.zeros(T, H, 32)
        wide[..., 8:] = x                                    # the rotated columns start at 8 inside heads of 32
        wide = wide.flatten(1)
        ops.rope_heads_(wide, cos, sin, pos, H, 32, 8, n, neighbours)
        torch.testing.assert_close(wide.view(T, H, 32)[..., 8:].double(), fn(x.double(), rot, 40), atol=1e-5, rtol=1e-5)
        ops.rope_heads_(y, cos, sin, pos, H, dim, 0, n, neighbours)
        torch.testing.assert_close(y[:, : H * dim].view(T, H, dim).double(), fn(x.double(), rot, 40), atol=1e-5, rtol=1e-5)
        assert (y[:, H * dim:] == 3).all()
    # length is kept, so a norm without a weight may come before or after
    x = torch.randn(T, H, dim, dtype=torch.float64)
    torch.testing.assert_close(plain.rms(plain.rotate_halves(x, rot), 1e-3), plain.rotate_halves(plain.rms(x, 1e-3), rot))


@pytest.mark.parametrize("Hkv", [2, 0])
def test_unit_heads_operator(Hkv):
    T, H, D, dim, DV, n = 6, 4, 64, 40, 64, 12
    rot = dict(base=70.0, dims=n)
    cos, sin = ref.build_rope_cache(60, n, 70.0)
    x = torch.randn(T, (H + Hkv) * D + Hkv * DV)
    x[:, : (H + Hkv) * D] *= (torch.arange(D) < dim).float().repeat(H + Hkv)
    pool, y = torch.zeros(15, max(Hkv, 1) * (D + DV)), x.clone()
    slot = torch.randperm(15)[:T].to(torch.int32)
    ops.qk_norm_rope_scatter_(y, pool, cos, sin, torch.arange(9, 9 + T, dtype=torch.int32), slot, None, None, 1e-3, H, Hkv, D, dim,
                              DV, n)
    heads = x[:, : (H + Hkv) * D].view(T, -1, D)[..., :dim].double()
    want = plain.rms(plain.rotate_halves(heads, rot, 9), 1e-3)
    torch.testing.assert_close(y[:, : H * D].view(T, H, D)[..., :dim].double(), want[:, :H], atol=1e-5, rtol=1e-5)
    if Hkv:
        got = pool[slot.long()]
        torch.testing.assert_close(got[:, : Hkv * D].view(T, Hkv, D)[..., :dim].double(), want[:, H:], atol=1e-5, rtol=1e-5)
        assert torch.equal(got[:, Hkv * D:], x[:, (H + Hkv) * D:])
    else:
        assert (pool == 0).all()


def test_latent_rows_operator():
    T, rank, cols, n, q_rank = 5, 20, 32, 8, 27
    cos, sin = ref.build_rope_cache(40, n, 500.0)
    rope = mla.LatentRope(cos, sin, n)
    kv, q = torch.randn(T, cols + 16), torch.randn(T, 32)
    w, qw = torch.rand(cols), torch.rand(32)
    pool, slot = torch.full((9, 56), 4.0), torch.tensor([3, 0, 8, 5, 1], dtype=torch.int32)
    out = mla.latent_prepare_(kv, pool, w, slot, rank, cols, 1e-3, rope, torch.arange(11, 11 + T, dtype=torch.int32), q, qw, q_rank)
    got = pool[slot.long()].double()
    torch.testing.assert_close(got[:, :rank], plain.rms(kv[:, :rank].double(), 1e-3) * w[:rank], atol=1e-5, rtol=1e-5)
    want = plain.rotate_neighbours(kv[:, None, cols:cols + n].double(), dict(base=500.0, dims=n), 11)[:, 0]
    torch.testing.assert_close(got[:, cols:cols + n], want, atol=1e-5, rtol=1e-5)
    assert (got[:, rank:cols] == 0).all() and (got[:, cols + n:] == 0).all() and (pool[[2, 4, 6, 7]] == 4).all()
    torch.testing.assert_close(out[:, :q_rank].double(), plain.rms(q[:, :q_rank].double(), 1e-3) * qw[:q_rank], atol=1e-5, rtol=1e-5)
    assert (out[:, q_rank:] == 0).all()


def _router(E, W, seed=0):
    g = torch.Generator().manual_seed(seed)
    return {"m.router": torch.randn(E, W, generator=g) / W ** 0.5, "m.correction": 0.4 * torch.randn(E, generator=g) - 0.8}


@pytest.mark.parametrize("E,top,groups,keep", [(12, 3, 3, 2), (16, 4, 8, 3), (6, 2, 1, 1), (8, 8, 2, 2), (10, 5, 5, 3)])
def test_grouped_router(E, top, groups, keep):
    """Choice scores of either sign (a closed group's count as minus infinity, not 0), weights without the correction."""
    t, h = _router(E, 24, E), torch.randn(50, 24, generator=torch.Generator().manual_seed(E)) * 2
    c = dict(experts=E, top=top, groups=dict(count=groups, keep=keep), scale=1.9)
    ids, val = plain.route(t, "m.", h.double(), c)
    got, w = moe.grouped_topk(h @ t["m.router"].t(), t["m.correction"], top, groups, keep, True, True, 1.9)
    order, o2 = ids.sort(-1), got.long().sort(-1)
    assert torch.equal(order[0], o2[0])
    torch.testing.assert_close(w.gather(1, o2[1]).double(), val.gather(1, order[1]), atol=1e-5, rtol=1e-5)
    choice = torch.sigmoid(h.double() @ t["m.router"].double().t()) + t["m.correction"]
    assert (choice.gather(1, ids) < 0).any()
    for r in range(len(h)):      # by hand, one token at a time
        sums = [sum(sorted(choice[r, a * (E // groups):(a + 1) * (E // groups)].tolist())[-2:]) for a in range(groups)]
        best = sorted(range(groups), key=lambda a: -sums[a])[:keep]
        allowed = [e for e in range(E) if e // (E // groups) in best]
        assert set(ids[r].tolist()) == set(sorted(allowed, key=lambda e: -choice[r, e])[:top])


def test_experts_beside_another_sublayer():
    torch.manual_seed(3)
    T, W, I, E = 9, 24, 32, 6
    t = _router(E, W)
    for e in range(E):
        t.update({f"m.e{e}.gate": torch.randn(I, W), f"m.e{e}.up": torch.randn(I, W), f"m.e{e}.down": torch.randn(W, I)})
    h, x, y, nw = torch.randn(T, W), torch.randn(T, W), torch.randn(T, W), torch.rand(W)
    cfg = {"router": dict(experts=E, top=2, groups=dict(count=2, keep=1), scale=1.4), "expert": {"limit": 1.2}}
    routed = plain.moe(t, "m.", h.double(), cfg)
    want = x.double() + y.double() + routed
    w13 = torch.stack([ref.interleave_gate_up(t[f"m.e{e}.gate"], t[f"m.e{e}.up"]) for e in range(E)])
    w2 = torch.stack([t[f"m.e{e}.down"] for e in range(E)])
    ids, wts = moe.grouped_topk(h @ t["m.router"].t(), t["m.correction"], 2, 2, 1, True, True, 1.4)
    out = moe.routed_experts_rms_(h, ids, wts, w13, w2, (1.702, 1.2), y, x, None, W, 1e-2, nw)
    torch.testing.assert_close(x.double(), want, atol=1e-3, rtol=1e-4)
    torch.testing.assert_close(out.double(), plain.rms(want, 1e-2) * nw, atol=1e-4, rtol=1e-4)
    parts = [moe.routed_experts_rms_(h, ids, wts, w13[a:b], w2[a:b], (1.702, 1.2), None, None, None, W, 1e-2, e0=a)
             for a, b in ((0, 2), (2, 6))]
    torch.testing.assert_close((parts[0] + parts[1]).double(), routed, atol=1e-3, rtol=1e-4)


def test_stream_passes_and_head():
    table, ids, w = torch.randn(20, 16), torch.tensor([3, 0, 19]), torch.rand(16)
    table[:, 12:], w[12:] = 0, 0
    x, h = ops.embedding_pair(ids, table, None, None, None, None, None, None, norm=(w, 12, 0.1))
    assert torch.equal(x, table[ids])
    torch.testing.assert_close(h.double()[:, :12], plain.rms(table[ids, :12].double(), 0.1) * w[:12], atol=1e-6, rtol=1e-5)
    x, y = torch.randn(5, 16), torch.randn(5, 16)
    x[:, 12:], y[:, 12:] = 0, 0
    want = x.double() + y.double()
    h = ops.add_rms_(x, y, None, 12, 0.1, torch.float32, w)
    torch.testing.assert_close(x.double(), want, atol=1e-6, rtol=1e-5)
    torch.testing.assert_close(h.double()[:, :12], plain.rms(want[:, :12], 0.1) * w[:12], atol=1e-6, rtol=1e-5)
    a, b = torch.randn(4, 8) * 4, torch.randn(6, 8)
    z = a.double() @ b.double().t()
    torch.testing.assert_close(ops.gemm(a, b, epi="f32", softcap=5.0).double(), 5 * torch.tanh(z / 5), atol=1e-5, rtol=1e-5)
    g = torch.randn(4, 8)
    want = a.double() * torch.sigmoid(g.double())
    torch.testing.assert_close(ops.sigmoid_mul_(a, g).double(), want, atol=1e-6, rtol=1e-5)


# ------------------------------------------------------------------------------------------------ the engine
@target
def test_stream_after_every_layer(models, tgt):
    path, cfg, t = models[tgt[1]]
    toks, want, got = tokens(120, 7), [], []
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
    toks = tokens(171, 2)
    want = plain.forward(t, cfg, toks)
    rep = replayer(path, tgt)
    for portions in ([171], [1], [2], [9, 10], [37, 36, 1], [64], [65, 63, 1], [140, 3, 1]):
        close(run_portions(rep, f"p{portions}", toks, portions), want, tgt, portions)
    assert rep.backend.ctx.get_can_alloc_token_num() == 512


@target
def test_first_tokens(models, tgt):
    path, cfg, t = models[tgt[1]]
    rep = replayer(path, tgt)
    for n in (1, 2, 3, 5, 6):
        toks = tokens(n, 40 + n)
        close(run_portions(rep, f"w{n}", toks, [n]), plain.forward(t, cfg, toks), tgt)
        close(run_portions(rep, f"s{n}", toks, [1]), plain.forward(t, cfg, toks), tgt)


@target
def test_unequal_batches_and_reused_slots(models, tgt):
    """Four live requests in one step, portions beside single tokens, in a pool they fill: requests end and their slots are used
    again by others, and requests rest for some steps."""
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


def _dependence(tmp_path, tgt, cfg, seed, n, places, portion_sets):
    """The last position's logits change with the token at place j exactly for the places said to be seen; all runs agree with
    the plain restatement.  The scores are small, so that every visible key has a share."""
    t = weights(cfg, seed)
    rep = replayer(write(tmp_path, cfg, t), tgt)
    base = tokens(n, 3)
    want = plain.forward(t, cfg, base)
    plan = []
    for j, inside in places:
        for delta in (1, 40):       # some other tokens there
            other = list(base)
            other[j] = (other[j] + delta) % VOCAB
            plan.append((j, inside, other, plain.forward(t, cfg, other)[-1:]))
    for portions in portion_sets:
        first = run_portions(rep, "base", base, portions)
        close(first, want, tgt, portions)
        best = {}
        for j, inside, other, w in plan:
            got = run_portions(rep, "other", other, portions)[-1:]
            close(got, w, tgt, (portions, j))
            best[j, inside] = max(best.get((j, inside), 0.0), float((got[0] - first[-1]).abs().max()))
        for (j, inside), d in best.items():
            assert (d > 1e-4) == inside, (portions, j, d)


@target
@pytest.mark.parametrize("window,keep", [(1, 0), (2, 3), (31, 1), (64, 64), (65, 7), (129, 20)])
def test_window_and_kept_token_edges(tmp_path, tgt, window, keep):
    """One layer: position p depends on exactly the tokens p - window + 1 .. p and the first `keep`."""
    n = window + keep + 35
    p = n - 1
    places = [(p - window + 1, True), (p - window, False), (p - window - 1, False), (keep, False)]
    if keep:
        places += [(0, True), (keep - 1, True)]
    _dependence(tmp_path, tgt, config([biased(4, 2, 24, 40, window, keep, 30, 0.01)]), window, n, places,
                ([n], [n - 5, 2, 3], [30, n - 31, 1]))


@target
@pytest.mark.parametrize("window", [1, 2, 31, 64, 65, 129])
def test_latent_window_edges(tmp_path, tgt, window):
    n = window + 35
    p = n - 1
    _dependence(tmp_path, tgt, config([latent(4, 24, 16, 40, 40, 32, window, 0.01)]), window, n,
                [(p - window + 1, True), (p - window, False), (p - window - 1, False)], ([n], [n - 5, 2, 3], [30, n - 31, 1]))


ASKER, BEACON = 6, 5


def _point(t, cfg, name, rows, token, gain, rest):
    """Rows of a projection of layer 0's input: the given ones take the value `gain` at `token`, the others are scaled by `rest`."""
    h = plain.centred_norm(t, "l0.norm1", t["embed"].double(), cfg["norm"]["eps"])[token]
    w = t[name].float() * rest
    for r in rows:
        w[r] = (h / h.square().sum() * gain).float()
    t[name] = w.to(torch.bfloat16)


def _fillers(n, seed=9):
    return [x for x in tokens(2 * n + 50, seed) if x not in (ASKER, BEACON)][:n]


@target
@pytest.mark.parametrize("distance,kept", [(99, False), (100, False), (140, True), (140, False)])
def test_one_key_that_stands_out(tmp_path, tgt, distance, kept):
    """A single key takes nearly all the weight of a far query: just inside and just outside the window, and far away as the last
    of the kept first tokens and as the next one; in a prompt and in decoding."""
    window, H, G, dim = 100, 4, 2, 24
    keep = 10 if kept else 9
    cfg = config([biased(H, G, dim, 32, window, keep, 60, 1.0)])
    t = weights(cfg, 11)
    _point(t, cfg, "l0.mix.q", [h * dim + 9 for h in range(H)], ASKER, 5.0, 0.05)
    _point(t, cfg, "l0.mix.k", [g * dim + 9 for g in range(G)], BEACON, 5.0, 0.05)
    filler = _fillers(150)
    toks = list(filler)
    toks[149], toks[149 - distance] = ASKER, BEACON
    without = list(toks)
    without[149 - distance] = filler[149 - distance]
    rep = replayer(write(tmp_path, cfg, t), tgt)
    want = plain.forward(t, cfg, toks)
    for portions in ([150], [149, 1], [120, 2], [148, 2]):
        got = run_portions(rep, "x", toks, portions)
        close(got, want, tgt, portions)
        gone = run_portions(rep, "y", without, portions)
        assert ((got[149] - gone[149]).abs().max() > 0.3) == (distance < window or kept)


@target
def test_latent_key_that_stands_out(tmp_path, tgt):
    """The same through latents: the unrotated part of one key answers one query, just inside and just outside the window."""
    H, dim, rot, rank, q_rank, window = 3, 24, 8, 40, 32, 80
    cfg = config([latent(H, dim, rot, 40, rank, q_rank, window, 1.5)])
    t = weights(cfg, 3)
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
    filler = _fillers(150)
    rep = replayer(write(tmp_path, cfg, t), tgt)
    for distance, seen in ((window - 1, True), (window, False)):
        toks = list(filler)
        toks[149] = ASKER
        without = list(toks)
        toks[149 - distance] = BEACON
        want = plain.forward(t, cfg, toks)
        for portions in ([150], [149, 1], [60, 88, 2]):
            got = run_portions(rep, "x", toks, portions)
            close(got, want, tgt, portions)
            gone = run_portions(rep, "y", without, portions)
            assert ((got[149] - gone[149]).abs().max() > 0.3) == seen


@target
def test_far_key_through_another_layers_cache(tmp_path, tgt):
    """A layer without keys of its own finds a key hundreds of tokens back in the other layer's cache."""
    H, G, dim = 4, 2, 24
    cfg = config([rotated(H, G, dim, 32, 6, 0.0), rotated(H, G, dim, 32, 6, 1.5, source=0)])
    t = weights(cfg, 4)
    t["l0.mix.o"] = torch.zeros_like(t["l0.mix.o"])          # layer 0 adds nothing: layer 1 reads the same rows
    t["l1.norm1"] = t["l0.norm1"].clone()
    _point(t, cfg, "l1.mix.q", [h * dim + 20 for h in range(H)], ASKER, 8.0, 0.05)     # dimension 20 is not rotated
    _point(t, cfg, "l0.mix.k", [g * dim + 20 for g in range(G)], BEACON, 8.0, 1.0)
    filler = _fillers(400)
    toks = list(filler)
    toks[399], toks[3] = ASKER, BEACON
    rep = replayer(write(tmp_path, cfg, t), tgt)
    want = plain.forward(t, cfg, toks)
    gone = plain.forward(t, cfg, filler[:399] + [ASKER])
    assert (want[399] - gone[399]).abs().max() > 0.3
    for portions in ([400], [399, 1], [250, 147, 3]):
        close(run_portions(rep, "x", toks, portions), want, tgt, portions)


@target
def test_far_distances_share_the_last_bias(tmp_path, tgt):
    """A bias table whose last rows dominate: distances from `far` on, and those just below it, take nearly all the weight."""
    cfg = config([biased(2, 1, 16, 24, 400, 0, 40, 0.01, rows=8)])
    t = weights(cfg, 8)
    rel = torch.zeros(8, 2)
    rel[7] = 8.0
    rel[6, 1] = 11.0
    t["l0.mix.rel"] = rel.to(torch.bfloat16)
    rep = replayer(write(tmp_path, cfg, t), tgt)
    toks = tokens(300, 2)
    want = plain.forward(t, cfg, toks)
    for portions in ([300], [39, 1, 1, 1, 258], [290, 1]):
        close(run_portions(rep, "x", toks, portions), want, tgt, portions)


@target
def test_long_decoding_and_greedy_generation(models, tgt):
    """Greedy generation through the engine's own scheduler: every produced token is the arg-max of the plain restatement up to
    rounding, far beyond the windows; a second run finds its prompt in the prefix cache."""
    path, cfg, t = models[tgt[1]]
    llm = LLM(model_dir=path, data_type=tgt[1], max_total_token_num=2000, running_max_req_size=4, max_req_total_len=400,
              chunked_prefill_size=48, batch_max_tokens=96, pstate=pstate(tgt))
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
    assert again[2]["prompt_cache_len"] > 0
    llm.close()


@target
def test_random_weights_and_sampling(tgt):
    """A model without a checkpoint (benchmarks), sampled generation."""
    cfg = json.loads(json.dumps(MIXED))
    cfg["layers"][0]["mixer"]["bias_max"] = cfg["layers"][5]["mixer"]["bias_max"] = 60     # random tables have 16 rows
    llm = LLM(config=cfg, data_type=tgt[1], max_total_token_num=600, running_max_req_size=3, max_req_total_len=200,
              pstate=pstate(tgt))
    outs = llm.generate([tokens(20, 1), tokens(3, 2)], {"max_new_tokens": 8, "do_sample": True, "temperature": 0.9,
                                                        "top_k": 20, "seed": 3})
    assert all(len(o["token_ids"]) == 8 and max(o["token_ids"]) < VOCAB for o in outs)
    llm.close()


def test_pages_carry_every_layer(models):
    mm = replayer(models["float32"][0], ("cpu", "float32")).llm.model.mem_manager
    assert len(mm.kv_layers) == 7                      # one layer reads another's rows
    for i, buf in enumerate(mm.kv_layers):
        buf.normal_(generator=torch.Generator().manual_seed(i))
    src, dst = torch.tensor([3, 9], dtype=torch.int32), torch.tensor([20, 1], dtype=torch.int32)
    mm.scatter_pages(dst, mm.gather_pages(src))
    for buf in mm.kv_layers:
        assert torch.equal(buf[dst.long()], buf[src.long()])


def test_returned_routed_experts(tmp_path):
    cfg = config([rotated(2, 1, 16, 16, 8, 0.3, experts(6, 2, 2, 1, 32, 1.0)), rotated(2, 2, 16, 16, 8, 0.3),
                  latent(2, 16, 8, 16, 24, 16, 9, 0.3, experts(8, 2, 4, 3, 32, 1.0))])
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
    assert cfg["model_type"] == "katarax" and cfg["hidden_size"] == 72 and cfg["num_hidden_layers"] == 8
    assert config_utils.get_vocab_size(path) == VOCAB and config_utils.get_dtype(path) == "bfloat16"
    assert get_tokenizer(path, vocab_size=VOCAB).encode("3 4 5") == [3, 4, 5]
    assert get_model_class(cfg).__name__ == "KataraxLM"
    rows = [2 * (64 + 128), 64 + 16, 64 + 64, 32 + 48, 4 * (192 + 64), 5 * 128, 144 + 32]
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
        t["l1.mix.uv"] = t["l1.mix.uv"][:-1].contiguous()

    _bad(tmp_path, "l1.mix.uv: shape", change=shape)
    _bad(tmp_path, "unknown mixer", ("layers", 1, "type"), "something")
    _bad(tmp_path, "unknown feed-forward", ("layers", 0, "mlp", "kind"), "something")
    for j in (3, 4, 0, 5, -1):
        _bad(tmp_path, "kv_from", ("layers", 3, "mixer", "kv_from"), j)
    _bad(tmp_path, "kv_from", ("layers", 3, "mixer", "vdim"), 32)
    _bad(tmp_path, "equal groups", ("layers", 2, "mlp", "router", "groups", "count"), 5)
    _bad(tmp_path, "at least `top`", ("layers", 2, "mlp", "router", "top"), 9)
    _bad(tmp_path, "rot.dims", ("layers", 1, "mixer", "rot", "dims"), 4)
    _bad(tmp_path, "bf16 or fp32 only", quant_type="fp8w8a8-b128")
    _bad(tmp_path, "no quantised form", kv_type="int8kv")


def test_trace_run_program(tmp_path, models):
    import numpy as np

    path, cfg, t = models["float32"]
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
    from lightllm_b200.models.katarax import KataraxLM
    from lightllm_b200.ops._native import UnitLibraries

    units = UnitLibraries()._unit_of
    assert {units[n] for n in ("llb_embedding_pair", "llb_add_rms", "llb_moe_combine_rms", "llb_latent_prepare", "llb_rope_heads",
                               "llb_latent_gather", "llb_latent_attn_mma", "llb_latent_attn_generic", "llb_window_prefill_tc",
                               "llb_sigmoid_mul", "llb_qk_norm_rope_scatter", "llb_window_gqa_prefill_tc", "llb_window_gqa_decode",
                               "llb_attn_generic_kv", "llb_gemm_f32", "llb_gemm_bf16_fused", "llb_gemm_bf16_batched",
                               "llb_grouped_topk", "llb_copy_rows", "llb_decode_prologue", "llb_sample")} <= \
        set(KataraxLM.native_units)
