"""The Taduzen family through the engine against the plain restatement in `taduzen_oracle.py`: whole prompts, token by
token, portions, mixed batches, pool reuse, window edges, long decoding, greedy generation.  On the CPU in fp32; the same
tests run on a GPU in fp32 and bf16."""
import json
import os
import subprocess

import pytest
import torch
from safetensors.torch import save_file

import taduzen_oracle as oracle
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


def mixer(heads, dim, vdim, rank, window, scale):
    return dict(heads=heads, dim=dim, vdim=vdim, kv_rank=rank, mask={"size": window} if window else None, scale=scale)


def layer(m, mlp):
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff, shared=None):
    out = {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def config(layers, width=80, vocab=101, eps=1e-4, logit_scale=0.7):
    return {"architecture": "Taduzen", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "logit_scale": logit_scale}


# every size differs from its neighbours, no layer is like another
MIXED = config([layer(mixer(3, 24, 40, 56, 37, 0.21), experts(5, 3, 48, 40)),
                layer(mixer(1, 72, 8, 24, 9, 0.1), None),
                layer(mixer(2, 130, 144, 72, 21, 0.08), experts(4, 1, 24)),
                layer(mixer(6, 16, 100, 40, 1, 0.3), dense(120)),
                layer(mixer(4, 40, 24, 104, 64, 0.15), experts(3, 2, 8, 56))])


def weights(cfg, seed=0, gain=1.0):
    """Random weights at which every part of a layer shows in the logits, rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    cls = get_model_class(cfg)
    probe = cls.__new__(cls)
    from lightllm_b200.models.taduzen import LayerSpec

    probe.hidden, probe.vocab, probe.specs = cfg["width"], cfg["vocab"], [LayerSpec(l) for l in cfg["layers"]]
    t = {}
    for name, shape in probe.weight_shapes().items():
        if name.endswith(".table"):
            n = probe.specs[int(name[1:].split(".")[0])].experts
            t[name] = torch.rand(shape[0], n, generator=g).topk(shape[1], -1)[1].to(torch.int32)
            continue
        if name.endswith(".alpha"):
            v = 0.5 + torch.rand((), generator=g)
        elif name.endswith(".b"):
            v = 0.2 * torch.randn(shape, generator=g)
        elif "norm" in name:
            v = 1 + 0.3 * torch.randn(shape, generator=g)
        elif name in ("embed", "head"):
            v = torch.randn(shape, generator=g)
        else:
            v = torch.randn(shape, generator=g) / shape[-1] ** 0.5
            if name.endswith(("mix.q", "mix.uk")):
                v = v * gain
            if name.endswith(".sg"):
                v = v * 3
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
    want = want.to(torch.float64)
    err = (torch.as_tensor(got).to(torch.float64) - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    limit = 3e-2 if tgt[1] == "bfloat16" else 2e-5
    assert err.max() < limit, (what, err.argmax(), err.max())


def tokens(n, seed, vocab=101):
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
    t = weights(MIXED, 1, gain=2.0)
    return write(tmp_path_factory.mktemp("taduzen"), MIXED, t), t


# ------------------------------------------------------------------------------------------------ mechanisms alone (CPU)
def test_dyt_operators():
    torch.manual_seed(0)
    n1 = ops.DytNorm(torch.randn(24), torch.randn(24), 0.7)
    n2 = ops.DytNorm(torch.randn(24), torch.randn(24), 1.6)
    table, ids = torch.randn(9, 24), torch.tensor([3, 3, 8, 0])
    x, h = ops.embedding_dyt(ids, table, n1)
    assert torch.equal(x, table[ids])
    torch.testing.assert_close(h, oracle.dyt(x, n1.w, n1.b, 0.7))
    y, x0 = torch.randn(4, 24), x.clone()
    h = ops.add_dyt_(x, y, n1, n2, torch.float32)
    torch.testing.assert_close(x, x0 + oracle.dyt(y, n1.w, n1.b, 0.7))
    torch.testing.assert_close(h, oracle.dyt(x, n2.w, n2.b, 1.6))
    a, w, x1 = torch.randn(4, 16), torch.randn(24, 16), x.clone()
    h = ops.gemm(a, w, epi="dyt", x=x, dyt=(n2, n1))
    torch.testing.assert_close(x, x1 + oracle.dyt(a @ w.t(), n2.w, n2.b, 1.6))
    torch.testing.assert_close(h, oracle.dyt(x, n1.w, n1.b, 0.7))
    up, down = torch.randn(24, 16), torch.randn(16, 24)
    torch.testing.assert_close(ops.gemm(ops.gemm(a, up, epi="relu2"), down), oracle.relu_squared_mlp(a, up, down))


@pytest.mark.parametrize("window", [1, 5, 0])
def test_latent_attention_operator(window):
    torch.manual_seed(window)
    H, dim, vdim, rank, n = 3, 10, 6, 12, 17
    h = torch.randn(n, 20)
    w_q, w_dkv, w_norm = torch.randn(H * dim, 20), torch.randn(rank, 20), torch.randn(rank)
    w_uk, w_uv = torch.randn(H * dim, rank), torch.randn(H * vdim, rank)
    pool = torch.zeros(40, 1, 16)
    slots = torch.randperm(40)[:n].to(torch.int32)
    mla.latent_norm_scatter_(torch.nn.functional.pad(h @ w_dkv.t(), (0, 4)), pool, w_norm, slots, rank, 1e-2)
    c = oracle.latent_of(h, w_dkv, w_norm, 1e-2)
    torch.testing.assert_close(pool[slots.long(), 0, :rank], c)
    assert (pool[slots.long(), 0, rank:] == 0).all()
    r2t = slots[None].clone()
    q = (h @ w_q.t()).view(n, H, dim)
    q_lat = mla.gemm_batched(q, torch.nn.functional.pad(w_uk.view(H, dim, rank), (0, 4)).transpose(1, 2).contiguous())
    o_lat = mla.latent_attention(q_lat, pool, r2t, torch.zeros(1, dtype=torch.int32), torch.arange(n, dtype=torch.int32),
                                 torch.zeros(n, dtype=torch.int32), 0.2, window)
    o = mla.gemm_batched(o_lat[..., :rank], w_uv.view(H, vdim, rank)).reshape(n, -1)
    want = oracle.latent_attention_core(q.reshape(n, -1), c, w_uk, w_uv, H, 0.2,
                                        oracle.visible(n, n, 0, window or 1 << 30))
    torch.testing.assert_close(o, want, atol=1e-4, rtol=1e-4)


def test_key_range():
    kr = mla.KeyRange(torch.tensor([0, 10, 3]), torch.tensor([4, 2, 1]), 6, "cpu")
    assert kr.kv_start.tolist() == [0, 5, 0] and kr.cu_kv.tolist() == [0, 4, 11, 15] and kr.rows == 15
    assert mla.KeyRange(torch.tensor([7]), torch.tensor([2]), 0, "cpu").kv_start.tolist() == [0]


@pytest.mark.parametrize("shared", [True, False])
def test_table_routed_experts_operator(shared):
    torch.manual_seed(3)
    T, W, I, E, k, V = 7, 12, 32, 4, 3, 20
    table = torch.rand(V, E).topk(k, -1)[1].to(torch.int32)
    tok = torch.randint(0, V, (T,))
    t = {"m.table": table, "m.shared.sg": torch.randn(1, W)}
    for e in [f"e{i}" for i in range(E)] + ["shared"]:
        t.update({f"m.{e}.gate": torch.randn(I, W), f"m.{e}.up": torch.randn(I, W), f"m.{e}.down": torch.randn(W, I)})
    h = torch.randn(T, W)
    cfg = {"router": {"experts": E, "top": k}, "shared": {"ff": I} if shared else None}
    want = oracle.moe(t, "m.", h, tok, cfg)
    w13 = torch.stack([ref.interleave_gate_up(t[f"m.e{e}.gate"], t[f"m.e{e}.up"]) for e in range(E)])
    w2 = torch.stack([t[f"m.e{e}.down"] for e in range(E)])
    lay = moe.TableRouting([(table, 0, E)]).layouts(tok)[0]
    sh = oracle.gated_mlp(h, t["m.shared.gate"], t["m.shared.up"], t["m.shared.down"]) if shared else None
    got = moe.uniform_experts_dyt_(h, lay, w13, w2, "silu", sh, t["m.shared.sg"][0] if shared else None, None, None, None)
    torch.testing.assert_close(got, want, atol=1e-4, rtol=1e-4)
    # two ranks with half of the experts each add up
    parts = [moe.uniform_experts_dyt_(h, lay, w13[e:e + 2], w2[e:e + 2], "silu", None, None, None, None, None, e0=e)
             for e in (0, 2)]
    routed = oracle.moe(t, "m.", h, tok, dict(cfg, shared=None))
    torch.testing.assert_close(parts[0] + parts[1], routed, atol=1e-4, rtol=1e-4)


# ------------------------------------------------------------------------------------------------ the engine
@target
def test_stream_after_every_layer(mixed_model, tgt):
    path, t = mixed_model
    toks, want, got = tokens(60, 7), [], []
    oracle.forward(t, MIXED, toks, stream=want)
    rep = replayer(path, tgt)
    rep.llm.model.stream_tap = lambda i, x: got.append(x[:, : MIXED["width"]].double().cpu())
    rep.step([("a", toks, [])])
    assert len(got) == len(want)
    for i, (g, w) in enumerate(zip(got, want)):
        close(g, w, tgt, f"layer {i}")


@target
def test_prompt_decode_and_portions(mixed_model, tgt):
    path, t = mixed_model
    toks = tokens(171, 2)
    want = oracle.forward(t, MIXED, toks)
    rep = replayer(path, tgt)
    for portions in ([171], [1], [2], [3], [9, 10], [37, 36, 1], [64], [65, 63, 1], [100, 2, 1]):
        close(run_portions(rep, f"p{portions}", toks, portions), want, tgt, portions)
    assert rep.backend.ctx.get_can_alloc_token_num() == 512


@target
def test_first_tokens(mixed_model, tgt):
    path, t = mixed_model
    rep = replayer(path, tgt)
    for n in (1, 2, 3, 5):
        toks = tokens(n, 40 + n)
        close(run_portions(rep, f"w{n}", toks, [n]), oracle.forward(t, MIXED, toks), tgt)
        close(run_portions(rep, f"s{n}", toks, [1]), oracle.forward(t, MIXED, toks), tgt)


@target
def test_unequal_batches_and_pool_reuse(mixed_model, tgt):
    """Four live requests in one step, portions beside single tokens, in a pool they fill: requests end and their slots
    are used again by others, and one request rests for some steps."""
    path, t = mixed_model
    lens = {"a": 90, "b": 33, "c": 150, "d": 7, "e": 70, "f": 41, "g": 128}
    toks = {k: tokens(n, 60 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: oracle.forward(t, MIXED, v) for k, v in toks.items()}
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
@pytest.mark.parametrize("window", [1, 2, 31, 64, 65, 150])
def test_window_edges(tmp_path, tgt, window):
    """One attention layer: position p depends on exactly the tokens p - window + 1 .. p.  The scores are kept
    small, so that every visible key has a share of the weight."""
    cfg = config([layer(mixer(2, 24, 40, 32, window, 0.05), None)])
    t = weights(cfg, window)
    path = write(tmp_path, cfg, t)
    rep = replayer(path, tgt)
    n = 190
    base = tokens(n, 3)
    p = n - 1
    for portions in ([n], [n - 1, 1], [n - 5, 2, 3], [64, 64, 1]):
        ref_logits = run_portions(rep, "base", base, portions)
        close(ref_logits, oracle.forward(t, cfg, base), tgt, portions)
        for d, inside in ((window - 1, True), (window, False), (window + 1, False), (0, True)):
            if d > p:
                continue
            best = 0.0
            for delta in (1, 17, 40):       # some other tokens there
                other = list(base)
                other[p - d] = (other[p - d] + delta) % cfg["vocab"]
                got = run_portions(rep, "other", other, portions)
                close(got[p:], oracle.forward(t, cfg, other)[p:], tgt, (portions, d))
                best = max(best, float((got[p] - ref_logits[p]).abs().max()))
            assert (best > 1e-4) == inside, (portions, d, best)


@target
def test_one_key_that_stands_out(tmp_path, tgt):
    """A single key takes all the weight of a far query (score 40 above the others), first just inside, then just outside
    the window, in a prompt and in decoding."""
    H, dim, rank, W, V, window = 2, 16, 24, 80, 101, 100
    cfg = config([layer(mixer(H, dim, 32, rank, window, 1.0), None)], eps=1e-5)
    t = weights(cfg, 11)
    beacon, asker = 5, 6
    n1 = {k: t["l0.norm1" + k].float() for k in ("", ".b", ".alpha")}
    hid = oracle.dyt(t["embed"].float(), n1[""], n1[".b"], n1[".alpha"])
    c = oracle.latent_of(hid, t["l0.mix.dkv"].float(), t["l0.mix.dkv.norm"].float(), 1e-5)
    q = torch.zeros(H * dim, W)
    uk = torch.zeros(H * dim, rank)
    for h in range(H):                      # score of (asker, key) = 40 * cosine of the key's latent with the beacon's
        q[h * dim] = hid[asker] / hid[asker].square().sum() * 40
        uk[h * dim] = c[beacon] / c[beacon].square().sum()
    t["l0.mix.q"], t["l0.mix.uk"] = q.to(torch.bfloat16), uk.to(torch.bfloat16)
    path = write(tmp_path, cfg, t)
    rep = replayer(path, tgt)
    filler = [x for x in tokens(400, 9) if x not in (beacon, asker)][:250]
    results = []
    for d in (window - 1, window):
        toks = list(filler)
        toks[249], toks[249 - d] = asker, beacon
        want = oracle.forward(t, cfg, toks)
        for portions in ([250], [249, 1], [200, 2]):
            got = run_portions(rep, "x", toks, portions)
            close(got, want, tgt, (d, portions))
        results.append(got[249])
    assert (results[0] - results[1]).abs().max() > 0.05


@target
def test_long_decoding_and_greedy_generation(mixed_model, tgt):
    """Greedy generation through the engine's own scheduler with the prefix cache on: every produced token is the arg-max
    of the oracle up to rounding, far beyond the windows."""
    path, t = mixed_model
    llm = LLM(model_dir=path, data_type=tgt[1], max_total_token_num=2000, running_max_req_size=4, max_req_total_len=400,
              chunked_prefill_size=48, batch_max_tokens=96, pstate=pstate(tgt))
    prompts = [tokens(n, 80 + n) for n in (1, 30, 111)]
    outs = llm.generate(prompts, {"max_new_tokens": 120, "do_sample": False})
    again = llm.generate(prompts, {"max_new_tokens": 120, "do_sample": False})
    slack = 0.15 if tgt[1] == "bfloat16" else 1e-3
    for p, o, o2 in zip(prompts, outs, again):
        assert len(o["token_ids"]) == 120
        for out in (o, o2):
            lg = oracle.forward(t, MIXED, p + out["token_ids"])[len(p) - 1:-1]
            chosen = lg.gather(1, torch.tensor(out["token_ids"])[:, None])[:, 0]
            assert (lg.max(-1)[0] - chosen).max() < slack
    assert again[2]["prompt_cache_len"] > 0
    llm.close()


@target
def test_random_weights_and_sampling(tgt):
    """A model without a checkpoint (benchmarks), sampled generation."""
    llm = LLM(config=MIXED, data_type=tgt[1], max_total_token_num=600, running_max_req_size=3, max_req_total_len=200,
              pstate=pstate(tgt))
    outs = llm.generate([tokens(20, 1), tokens(3, 2)], {"max_new_tokens": 8, "do_sample": True, "temperature": 0.9,
                                                        "top_k": 20, "seed": 3})
    assert all(len(o["token_ids"]) == 8 and max(o["token_ids"]) < 101 for o in outs)
    llm.close()


def test_returned_routed_experts(tmp_path):
    cfg = config([layer(mixer(2, 24, 40, 32, 8, 0.3), experts(5, 2, 32)), layer(mixer(2, 24, 40, 32, 8, 0.3), dense(40)),
                  layer(mixer(2, 24, 40, 32, 8, 0.3), experts(4, 2, 32, 8))])
    t = weights(cfg, 4)
    llm = LLM(model_dir=write(tmp_path, cfg, t), data_type="float32", max_total_token_num=200, running_max_req_size=2,
              max_req_total_len=64, enable_return_routed_experts=True)
    p = tokens(11, 5)
    o = llm.generate([p], {"max_new_tokens": 4, "do_sample": False})[0]
    ids = torch.tensor(p + o["token_ids"][:-1])
    for j, l in enumerate((0, 2)):
        assert torch.equal(torch.as_tensor(o["routed_experts"][:, j].astype("int64")), t[f"l{l}.mlp.table"][ids].long())


def test_config_reaches_the_server_side(tmp_path):
    from lightllm_b200.server.tokenizer import get_tokenizer
    from lightllm_b200.utils import config_utils

    path = write(tmp_path, MIXED, weights(MIXED))
    cfg = load_config(path)
    assert cfg["model_type"] == "taduzen" and cfg["hidden_size"] == 80 and cfg["num_hidden_layers"] == 5
    assert config_utils.get_vocab_size(path) == 101 and config_utils.get_dtype(path) == "bfloat16"
    assert get_tokenizer(path, vocab_size=101).encode("3 4 5") == [3, 4, 5]
    assert get_model_class(cfg).__name__ == "TaduzenLM"
    with pytest.raises(ValueError, match="unsupported architecture"):
        get_model_class({"architecture": "Nothing"})


def _bad(tmp_path, match, cfg=None, change=None, **kw):
    t = weights(MIXED)
    if change:
        change(t)
    path = write(tmp_path, cfg or MIXED, t)
    with pytest.raises(ValueError, match=match):
        LLM(model_dir=path, max_total_token_num=64, max_req_total_len=64, data_type="float32", **kw)


def test_wrong_checkpoints_are_refused(tmp_path):
    def table(t):
        t["l0.mlp.table"][7, 0] = 5

    def shape(t):
        t["l1.mix.uv"] = t["l1.mix.uv"][:, :-1].contiguous()

    _bad(tmp_path, "names an expert outside", change=table)
    _bad(tmp_path, "l1.mix.uv: shape", change=shape)
    other = json.loads(json.dumps(MIXED))
    other["layers"][1]["type"] = "something"
    _bad(tmp_path, "unknown mixer", cfg=other)
    _bad(tmp_path, "bf16 or fp32 only", quant_type="fp8w8a8-b128")
    _bad(tmp_path, "no quantised form", kv_type="int8kv")


def _trace(path, lines, out, *extra):
    return subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--out", str(out), "--device", "cpu",
                           *extra], input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True,
                          timeout=240)


def test_trace_run_program(tmp_path, mixed_model):
    import numpy as np

    path, t = mixed_model
    a, b = tokens(70, 1), tokens(9, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:8], "want": []}, {"id": "a", "tokens": a[50:51], "want": []}],
              "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[51:], "want": [18]}, {"id": "b", "tokens": b[8:], "want": [0]}],
              "end": ["a", "b"]}]
    r = _trace(path, lines, tmp_path, "--dtype", "float32", "--max-tokens", "128")
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = oracle.forward(t, MIXED, a), oracle.forward(t, MIXED, b)
    got = {i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, 101)) for i in (0, 2)}
    close(got[0], wa[[0, 49]], ("cpu", "float32"))
    close(got[2], torch.stack([wa[69], wb[8]]), ("cpu", "float32"))
    assert not (tmp_path / "1.f32").exists()


def test_every_kernel_entry_has_a_source():
    """Without built libraries entry points are looked up in the sources; the units a family names cover what its
    operators call."""
    import re

    from lightllm_b200.models.taduzen import TaduzenLM
    from lightllm_b200.ops._native import UnitLibraries

    units = UnitLibraries()._unit_of
    called = set()
    for name in ("__init__", "mla", "moe"):
        with open(os.path.join(ROOT, "lightllm_b200", "ops", name + ".py")) as f:
            called |= set(re.findall(r"kernels\(\)\.(llb_\w+)", f.read()))
    assert called <= set(units)
    assert UnitLibraries()._needs["attention"] == ["attention_tc"]
    assert not any(UnitLibraries()._needs[u] for u in TaduzenLM.native_units)
    assert {units[n] for n in ("llb_dyt", "llb_gemm_f32", "llb_gemm_bf16_fused", "llb_latent_attn_mma", "llb_moe_table_align",
                               "llb_window_prefill_tc", "llb_decode_prologue", "llb_sample")} <= set(TaduzenLM.native_units)


def test_capacity_estimate(tmp_path):
    from lightllm_b200.utils.profile_max_tokens import kv_bytes_per_token, max_total_tokens

    path = write(tmp_path, MIXED, weights(MIXED))
    assert kv_bytes_per_token(load_config(path), 1) == 5 * 112 * 2      # five layers, the widest latent padded to 112
    assert max_total_tokens(path, gpu_gib=1)["max_total_token_num"] > 0
