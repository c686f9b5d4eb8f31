"""Libulorn beside the framework's closest model (Qwen3-Next: linear attention with matrix states, gated softmax attention,
routed and shared experts) at equal sizes: configurations and kernels for `design_bench`.

Four layers each: two recurrent ones and two with attention.  A "parallel" layer of Libulorn has a recurrence next to its
attention, so it has two recurrences more than the other model.  Kernels: time and fraction of the roofline (the slower of
bytes / measured copy bandwidth and operations / measured bf16 rate), the numbers of either model's own work."""
from __future__ import annotations

import json

import torch

LAYERS, DIM, VOCAB = 4, 128, 32768
# width, attention heads and kv heads, recurrent heads (key and value size 128 as well), experts, experts per token, expert
# size, shared size, window
SIZES = {
    "small": dict(width=1024, heads=8, kv=2, rec=8, experts=32, top=4, ff=512, shared=512, window=1024),
    "base": dict(width=2048, heads=16, kv=4, rec=16, experts=64, top=6, ff=768, shared=768, window=4096),
    "wide": dict(width=4096, heads=32, kv=8, rec=32, experts=64, top=6, ff=1408, shared=1408, window=4096),
}


def config(z, layers=LAYERS):
    left = dict(heads=z["heads"], kv_heads=z["kv"], dim=DIM, vdim=DIM, mask={"size": z["window"]}, scale=DIM ** -0.5,
                rot={"base": 1e4, "dims": DIM // 4,
                     "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}})
    rec = dict(heads=z["rec"], dim=DIM, vdim=DIM)
    moe = dict(kind="moe", router={"experts": z["experts"], "top": z["top"]}, expert={"ff": z["ff"], "limit": 7.0},
               shared={"ff": z["shared"], "limit": 7.0})
    mixers = [("mlstm", dict(rec, gate_cap=15.0)),
              ("parallel", dict(left=left, right=dict(rec, tau=16.0), left_scale=1.0, right_scale=1.0))]
    return {"architecture": "Libulorn", "width": z["width"], "vocab": VOCAB, "norm": {"eps": 1e-5},
            "embedding": {"bigram": {"buckets": VOCAB - 1, "mul_prev": 1009, "mul_cur": 31}},
            "layers": [dict(zip(("type", "mixer"), mixers[2 * i // layers]), mlp=moe) for i in range(layers)]}


def closest_config(z, layers=LAYERS):
    return dict(model_type="qwen3_next", hidden_size=z["width"], num_hidden_layers=layers, vocab_size=VOCAB,
                num_attention_heads=z["heads"], num_key_value_heads=z["kv"], head_dim=DIM, partial_rotary_factor=0.25,
                layer_types=["linear_attention" if 2 * i < layers else "full_attention" for i in range(layers)],
                linear_num_key_heads=z["rec"], linear_num_value_heads=z["rec"], linear_key_head_dim=DIM,
                linear_value_head_dim=DIM, linear_conv_kernel_dim=4, num_experts=z["experts"],
                num_experts_per_tok=z["top"], moe_intermediate_size=z["ff"], norm_topk_prob=True,
                shared_expert_intermediate_size=z["shared"], intermediate_size=z["ff"], rms_norm_eps=1e-5, rope_theta=1e4,
                decoder_sparse_step=1, mlp_only_layers=[])


def kernels(size: str, T: int = 8192, B: int = 64, ctx: int = 4096):
    from .. import ops
    from ..common.infer_state import InferState
    from ..ops import linear_attn as la
    from ..ops import moe
    from ..ops import reference as ref
    from .design_bench import peaks
    from .kernel_bench import timeit

    z = SIZES[size]
    W, H, G, R, E, k, ff, win = (z[n] for n in ("width", "heads", "kv", "rec", "experts", "top", "ff", "window"))
    hbm, tf = peaks()
    dev, BF = torch.device("cuda"), torch.bfloat16
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)

    def rnd(*s, dtype=BF):
        return torch.randn(*s, device=dev).mul_(0.05).to(dtype)

    def measure(fn, bytes_, flops):
        t = timeit(fn, flush, reps=1)
        return t * 1e6, max(bytes_ / hbm, flops / tf) / t

    def pair(what, ours, like):
        (u1, f1), (u2, f2) = measure(*ours), measure(*like)
        print(json.dumps({"kernel": what, "size": size, "us": round(u1, 1), "roofline": round(f1, 3),
                          "qwen3_next_us": round(u2, 1), "qwen3_next_roofline": round(f2, 3),
                          "ratio": round(f1 / f2, 2)}), flush=True)

    def i32(*a):
        return torch.tensor(a, dtype=torch.int32, device=dev)

    ones, nw = torch.ones(W, device=dev), torch.ones(W, device=dev, dtype=BF)
    hn, hn16 = torch.ones(DIM, device=dev), torch.ones(DIM, device=dev, dtype=BF)
    slots = torch.randperm(B * (ctx + 1), device=dev).to(torch.int32)
    r2t = slots.view(B, ctx + 1)
    pool = rnd(B * (ctx + 1), 2 * G, DIM)
    flat = pool.view(-1, 2 * G * DIM)
    cos, sin = ref.build_rope_cache(ctx + T, DIM // 4, 1e4, None, device=dev)
    req, bseq = torch.arange(B, device=dev, dtype=torch.int32), torch.full((B,), ctx + 1, device=dev, dtype=torch.int32)

    # ---- rows around the stream ----
    ow = rnd(W, (H + R) * DIM)
    for t in (T, B):
        a, x, res = rnd(t, (H + R) * DIM), rnd(t, W, dtype=torch.float32), rnd(t, W)
        fl, wb = 2.0 * t * W * (H + R) * DIM, (W + t) * (H + R) * DIM * 2

        def ours():
            ops.add_rms_(x, ops.gemm(a, ow), ones, W, 1e-5, BF)

        def like():
            ops.gemm(a, ow, epi="residual", residual=res, out=res)
            ops.rmsnorm(res, nw, 1e-5)

        pair(f"output projection + norm, {t} rows", (ours, wb + t * W * 14, fl), (like, wb + t * W * 8, fl))
    table, second, ids = rnd(VOCAB, W), rnd(VOCAB, W), torch.randint(0, VOCAB, (T,), device=dev)
    big = ops.BigramTable(second, VOCAB - 1, 1009, 31)
    big.slot_token = torch.zeros(B * (ctx + 1), dtype=torch.int32, device=dev)
    pos_t = torch.arange(T, device=dev, dtype=torch.int32) % ctx
    bof = torch.arange(T, device=dev, dtype=torch.int32) // ctx
    pair(f"embedding, {T} rows",
         (lambda: ops.embedding_pair(ids, table, big, r2t, req, pos_t, bof, slots[:T]), T * W * 10, 0),
         (lambda: ops.rmsnorm(ops.embedding(ids, table), nw, 1e-5), T * W * 8, 0))
    for t in (T, B):
        qkv = rnd(t, (H + 2 * G) * DIM)
        n = t * (H + 2 * G) * DIM * 4
        p = pos_t[:t]
        pair(f"query / key norm, rotation, scatter, {t} rows",
             (lambda: ops.qk_norm_rope_scatter_(qkv, flat, cos, sin, p, slots[:t], hn, hn, 1e-5, H, G, DIM, DIM, DIM,
                                                DIM // 4), n, 0),
             (lambda: ops.rope_kv_scatter_(qkv, pool, cos, sin, p, slots[:t], H, G, DIM, DIM // 4, hn16, hn16, 1e-5), n, 0))

    # ---- attention ----
    q, gate = rnd(B, H * DIM), rnd(B, H)
    st = InferState(is_prefill=False, batch_size=B, num_tokens=B, max_kv_len=ctx + 1, max_q_len=1, b_req_idx=req,
                    b_seq_len=bseq, mem_index=None, seq_pos=bseq - 1)
    keys = min(win, ctx + 1)
    pair(f"decode attention, {B} requests at {ctx} (window {win})",
         (lambda: ops.window_attention(q, flat, r2t, st, H, G, DIM, DIM, 0.1, win, gate),
          B * (keys * 2 * G + 2 * H) * DIM * 2, 0),
         (lambda: ops.gqa_decode(q, pool, r2t, req, bseq, H, G, DIM, ctx + 1, 0.1),
          B * ((ctx + 1) * 2 * G + 2 * H) * DIM * 2, 0))
    n = T // 4
    q, gate = rnd(T, H * DIM), rnd(T, H)
    cu, zero = torch.arange(0, T + 1, n, device=dev, dtype=torch.int32), torch.zeros(4, device=dev, dtype=torch.int32)
    r2p = slots[:T].view(4, n).contiguous()
    pst = InferState(is_prefill=True, batch_size=4, num_tokens=T, max_kv_len=n, max_q_len=n, b_req_idx=req[:4],
                     b_seq_len=None, mem_index=None, cu_q=cu, b_ready_cache_len=zero)
    pairs = 4 * sum(min(i + 1, win) for i in range(n))
    byt = (2 * H + 2 * G) * T * DIM * 2
    pair(f"prompt attention, 4 x {n} (window {win})",
         (lambda: ops.window_attention(q, flat, r2p, pst, H, G, DIM, DIM, 0.1, win, gate), byt, pairs * H * 4.0 * DIM),
         (lambda: ops.gqa_prefill(q, pool, r2p, req[:4], cu, zero, H, G, DIM, n, 0.1), byt,
          4 * n * (n + 1) / 2 * H * 4.0 * DIM))

    # ---- recurrences ----
    rank = 16
    a2, a2b, w = rnd(R * DIM, rank), torch.zeros(R * DIM, device=dev), torch.ones(DIM, device=dev)
    recs = {"gla": la.DecayedState("gla", R, DIM, DIM, DIM, DIM, 1e-5, w, tau=16.0, a2=a2, a2_bias=a2b),
            "mlstm": la.DecayedState("mlstm", R, DIM, DIM, DIM, DIM, 1e-5, w.repeat(R), cap=15.0)}
    for t in (B, 4 * B):
        m = rnd(t, 4 * R * DIM + rank)
        parts = torch.split(m, [R * DIM] * 4 + [rank], 1)
        zif = torch.randn(t, 2 * R, device=dev)
        dst = InferState(is_prefill=False, batch_size=t, num_tokens=t, max_kv_len=ctx, max_q_len=1,
                         b_req_idx=torch.arange(t, device=dev, dtype=torch.int32), b_seq_len=None, mem_index=None,
                         seq_pos=torch.full((t,), ctx, device=dev, dtype=torch.int32))
        mixed, cw = rnd(t, 3 * R * DIM, dtype=torch.float32), rnd(3 * R * DIM, 4, dtype=torch.float32)
        cs, ss = rnd(t, 3 * R * DIM, 3), rnd(t, R, DIM, DIM, dtype=torch.float32)
        g, beta, zz = -torch.rand(t, R, device=dev), torch.rand(t, R, device=dev), rnd(t, R, DIM)
        sb = 2 * t * R * DIM * DIM * 4

        def like_step():
            la.rmsnorm_gated(la.conv_and_delta_step(mixed, cs, cw, ss, dst.b_req_idx, g, beta, R, R, DIM, DIM), zz, w, 1e-5)

        for kind, rec in recs.items():
            state = rnd(t, la.DecayedState.state_elems(kind, R, DIM, DIM), dtype=torch.float32)
            pair(f"{kind} step + output step, {t} requests",
                 (lambda: rec(*parts[:4], state, dst, a1=parts[4] if kind == "gla" else None, zi=zif[:, :R], zf=zif[:, R:]),
                  sb + t * R * DIM * 10, 0),
                 (like_step, sb + t * R * DIM * (3 * 4 + 3 * 12 + 4), 0))
    m = rnd(T, 4 * R * DIM + rank)
    parts = torch.split(m, [R * DIM] * 4 + [rank], 1)
    zif = torch.randn(T, 2 * R, device=dev)
    plan = la.ChunkPlan(torch.full((4,), n), dev)
    qf, kf, vf = (rnd(n, R, DIM, dtype=torch.float32) for _ in range(3))
    gf, bf = -torch.rand(n, R, device=dev), torch.rand(n, R, device=dev)
    S0, zz = torch.zeros(R, DIM, DIM, device=dev), rnd(T, R, DIM)

    def like_prompt():
        o = torch.cat([la.gated_delta_chunked(qf, kf, vf, gf, bf, S0)[0] for _ in range(4)])
        la.rmsnorm_gated(o, zz, w, 1e-5)

    # inside a chunk of 64: scores and their product with the values (half of the square), the state's read-out and update
    fl = T * R * (2.0 * 32 * 2 * DIM + 4.0 * DIM * DIM)
    for kind, rec in recs.items():
        state = torch.zeros(4, la.DecayedState.state_elems(kind, R, DIM, DIM), device=dev)
        pair(f"{kind} prompt + output step, 4 x {n}",
             (lambda: rec(*parts[:4], state, pst, a1=parts[4] if kind == "gla" else None, zi=zif[:, :R], zf=zif[:, R:],
                          plan=plan), T * R * DIM * 10, fl),
             (like_prompt, T * R * DIM * (12 + 6), fl))

    # ---- experts ----
    w13, w2 = rnd(E, 2 * ff, W), rnd(E, W, ff)
    sg, sd = rnd(2 * z["shared"], W), rnd(W, z["shared"])
    for t in (T, B):
        h, x, sh, res = rnd(t, W), rnd(t, W, dtype=torch.float32), rnd(t, W), rnd(t, W)
        idl = torch.rand(t, E, device=dev).topk(k, -1)[1].to(torch.int32)
        wts = torch.full((t, k), 1.0 / k, device=dev)
        fl = 2.0 * t * k * 3 * ff * W
        byt = min(E, t * k) * 3 * ff * W * 2 + t * k * (W * 8 + ff * 4)

        def like_experts():
            out = sh.clone()
            moe.fused_experts(h, w13, w2, idl, wts, out=out, accumulate=True)
            ops.add_rmsnorm_(res, out, nw, 1e-5)

        pair(f"experts + norm, {t} rows",
             (lambda: moe.routed_experts_rms_(h, idl, wts, w13, w2, (1.702, 7.0), sh, x, ones, W, 1e-5), byt + t * W * 12, fl),
             (like_experts, byt + t * W * 10, fl))
        s = z["shared"]
        pair(f"shared expert, {t} rows",
             (lambda: ops.gemm(ops.gemm(h, sg, epi="gated_clamp", clamp=(1.702, 7.0)), sd),
              (3 * s * W + t * (2 * W + 2 * s)) * 2, 6.0 * t * s * W),
             (lambda: ops.gemm(ops.gemm(h, sg, epi="gated_silu"), sd), (3 * s * W + t * (2 * W + 2 * s)) * 2,
              6.0 * t * s * W))
