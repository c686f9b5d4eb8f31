"""Silupel beside the framework's closest models at equal sizes, for `design_bench`: Qwen2 (grouped-query attention with biases,
dense feed-forwards) and DeepSeek-V2 with dense feed-forwards (latent attention with query latents and a rotated part); the
recurrence beside Libulorn's gated linear attention.

Four layers each; Silupel has minGRU, chunked attention, latent attention, chunked attention.  Kernels: time and fraction of the
roofline (the slower of bytes / measured copy bandwidth and operations / measured bf16 rate), the numbers of either model's own
work."""
from __future__ import annotations

import json

import torch

LAYERS, DIM, ROT, RANK, VOCAB = 4, 128, 64, 512, 32768
CAP = 50.0
# width, heads, key / value heads, query latent, feed-forward size, chunk
SIZES = {
    "small": dict(width=1024, heads=8, kv=2, q_rank=768, ff=4096, chunk=1536),
    "base": dict(width=2048, heads=16, kv=4, q_rank=1536, ff=8192, chunk=8192),
    "wide": dict(width=4096, heads=32, kv=8, q_rank=1536, ff=14336, chunk=8192),
}


def config(z):
    gqa = dict(heads=z["heads"], kv_heads=z["kv"], dim=DIM, vdim=DIM, scale=DIM ** -0.5, mask={"size": z["chunk"]}, softcap=CAP,
               rot={"base": 1e4, "dims": DIM, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}})
    lat = dict(heads=z["heads"], dim=DIM, rot_dim=ROT, vdim=DIM, kv_rank=RANK, q_rank=z["q_rank"], rot={"base": 1e4, "dims": ROT},
               scale=(DIM + ROT) ** -0.5)
    mixers = [("mingru", dict(width=z["width"])), ("attention", gqa), ("latent_attention", lat), ("attention", gqa)]
    return {"architecture": "Silupel", "width": z["width"], "vocab": VOCAB, "norm": {"eps": 1e-5},
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": z["ff"]}} for t, m in mixers]}


def qwen_config(z):
    return dict(model_type="qwen2", hidden_size=z["width"], num_hidden_layers=LAYERS, vocab_size=VOCAB,
                num_attention_heads=z["heads"], num_key_value_heads=z["kv"], head_dim=DIM, intermediate_size=z["ff"],
                rms_norm_eps=1e-6, rope_theta=1e4)


def deepseek_config(z):
    return dict(model_type="deepseek_v2", hidden_size=z["width"], num_hidden_layers=LAYERS, vocab_size=VOCAB,
                num_attention_heads=z["heads"], num_key_value_heads=z["heads"], q_lora_rank=z["q_rank"], kv_lora_rank=RANK,
                qk_nope_head_dim=DIM, qk_rope_head_dim=ROT, v_head_dim=DIM, intermediate_size=z["ff"],
                moe_intermediate_size=z["ff"], n_routed_experts=2, n_shared_experts=1, num_experts_per_tok=1,
                first_k_dense_replace=LAYERS, norm_topk_prob=False, scoring_func="softmax", topk_method="greedy", n_group=1,
                topk_group=1, rms_norm_eps=1e-5, rope_theta=1e4)


CLOSEST = {"qwen2": qwen_config, "deepseek_v2": deepseek_config}


def kernels(size: str, T: int = 8192, B: int = 64, ctx: int = 4096):
    from .. import ops
    from ..common.infer_state import InferState
    from ..models.latent import LatentHeads
    from ..ops import linear_attn as la
    from ..ops import mla
    from ..ops import reference as ref
    from .design_bench import peaks
    from .kernel_bench import timeit

    z = SIZES[size]
    W, H, G, Q, ff, chunk = (z[n] for n in ("width", "heads", "kv", "q_rank", "ff", "chunk"))
    hbm, tf = peaks()
    dev, BF = torch.device("cuda"), torch.bfloat16
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)

    def rnd(*s, dtype=BF):
        return torch.randn(*s, device=dev).mul_(0.05).to(dtype)

    def measure(fn, bytes_, flops):
        t = timeit(fn, flush, reps=1)
        return t * 1e6, max(bytes_ / hbm, flops / tf) / t

    def pair(what, like_name, ours, like):
        (u1, f1), (u2, f2) = measure(*ours), measure(*like)
        print(json.dumps({"kernel": what, "size": size, "us": round(u1, 1), "roofline": round(f1, 3), "like": like_name,
                          "like_us": round(u2, 1), "like_roofline": round(f2, 3), "ratio": round(f1 / f2, 2)}), flush=True)

    QW, DS, LB = "qwen2", "deepseek_v2", "libulorn"
    ones, mu, nw = torch.ones(W, device=dev), torch.full((W,), 0.5, device=dev), torch.ones(W, device=dev, dtype=BF)
    slots = torch.randperm(B * (ctx + 1), device=dev).to(torch.int32)
    r2t = slots.view(B, ctx + 1)
    pool = rnd(B * (ctx + 1), 2 * G, DIM)
    flat = pool.view(-1, 2 * G * DIM)
    cos, sin = ref.build_rope_cache(ctx + T, ROT, 1e4, None, device=dev)
    cos2, sin2 = ref.build_rope_cache(ctx + T, DIM, 1e4, None, device=dev)
    pos_t = torch.arange(T, device=dev, dtype=torch.int32) % ctx
    req = torch.arange(4 * B, device=dev, dtype=torch.int32)
    bseq = torch.full((B,), ctx + 1, device=dev, dtype=torch.int32)

    def prompts(b):
        n = T // b
        return InferState(is_prefill=True, batch_size=b, num_tokens=T, max_kv_len=n, max_q_len=n, b_req_idx=req[:b], b_seq_len=None,
                          mem_index=None, cu_q=torch.arange(0, T + 1, n, device=dev, dtype=torch.int32),
                          b_ready_cache_len=torch.zeros(b, device=dev, dtype=torch.int32),
                          batch_of_token=torch.repeat_interleave(torch.arange(b, device=dev, dtype=torch.int32), n))

    def step(t):
        return InferState(is_prefill=False, batch_size=t, num_tokens=t, max_kv_len=ctx + 1, max_q_len=1, b_req_idx=req[:t],
                          b_seq_len=bseq[:t], mem_index=None, seq_pos=torch.full((t,), ctx, device=dev, dtype=torch.int32))

    n, pst = T // 4, prompts(4)
    cu, zero = pst.cu_q, pst.b_ready_cache_len

    # ---- rows around the stream ----
    state = torch.zeros(4 * B, W, device=dev)
    for t, st in ((T, pst), (B, step(B))):
        x, y, res = rnd(t, W, dtype=torch.float32), rnd(t, W), rnd(t, W)
        shift = ops.TokenShift(mu, state, st)
        like = (lambda: ops.add_rmsnorm_(res, y, nw, 1e-5), t * W * 8, 0)
        pair(f"sum + layer norm, {t} rows", QW, (lambda: ops.norm_shift(x, y, ones, W, 1e-5, BF), t * W * 12, 0), like)
        sb = 8 * W * (4 if t == T else B)
        pair(f"sum + layer norm + token shift, {t} rows", QW,
             (lambda: ops.norm_shift(x, y, ones, W, 1e-5, BF, shift), t * W * 12 + sb, 0), like)
    table, ids = rnd(VOCAB, W), torch.randint(0, VOCAB, (T,), device=dev)
    shift = ops.TokenShift(mu, state, pst)
    pair(f"embedding + first norm + token shift, {T} rows", QW,
         (lambda: ops.norm_shift(None, table, ones, W, 1e-5, BF, shift, ids), T * W * 8, 0),
         (lambda: ops.rmsnorm(ops.embedding(ids, table), nw, 1e-5), T * W * 8, 0))

    # ---- projections and feed-forward ----
    cols = (2 * H + 2 * G) * DIM
    wi, wl, bi, bl = rnd(cols, W), rnd((H + 2 * G) * DIM, W), rnd(cols), rnd((H + 2 * G) * DIM)
    gu, dn = rnd(2 * ff, W), rnd(W, ff)
    for t in (T, B):
        h, a = rnd(t, W), rnd(t, ff)

        def mat(rows, c):
            return (c * W + rows * (W + c)) * 2, 2.0 * rows * W * c

        pair(f"query, key, value, gate projection + biases, {t} rows", QW, (lambda: ops.gemm(h, wi, bias=bi), *mat(t, cols)),
             (lambda: ops.gemm(h, wl, bias=bl), *mat(t, (H + 2 * G) * DIM)))
        byt, fl = (2 * ff * W + t * (W + ff)) * 2, 4.0 * t * W * ff
        pair(f"gate and up + activation, {t} rows", QW, (lambda: ops.gemm(h, gu, epi="gated_gelu"), byt, fl),
             (lambda: ops.gemm(h, gu, epi="gated_silu"), byt, fl))
        res = rnd(t, W)
        pair(f"down, {t} rows", QW, (lambda: ops.gemm(a, dn), (ff * W + t * (W + ff)) * 2, 2.0 * t * W * ff),
             (lambda: ops.gemm(a, dn, epi="residual", residual=res, out=res), (ff * W + t * (2 * W + ff)) * 2, 2.0 * t * W * ff))

    # ---- new keys, values, latents ----
    lat = LatentHeads(H, DIM, ROT, DIM, RANK, 0.07, 0)
    lpool, rope = rnd(B * (ctx + 1), lat.keys), mla.LatentRope(cos, sin, ROT, neighbours=False)
    kn, qn, kn16, qn16 = (torch.ones(m, device=dev, dtype=d) for m, d in ((RANK, torch.float32), (Q, torch.float32), (RANK, BF), (Q, BF)))
    temp = torch.ones(H, device=dev)
    for t in (T, B):
        p, sl, qkv = pos_t[:t], slots[:t], rnd(t, (H + 2 * G) * DIM)
        byt = t * (H + 2 * G) * DIM * 4
        pair(f"rotation, temperatures, scatter, {t} rows", QW,
             (lambda: ops.qk_norm_rope_scatter_(qkv, flat, cos2, sin2, p, sl, None, None, 1e-5, H, G, DIM, DIM, DIM, DIM, norm=False,
                                                q_scale=temp), byt, 0),
             (lambda: ops.rope_kv_scatter_(qkv, pool, cos2, sin2, p, sl, H, G, DIM), byt, 0))
        proj, q3 = rnd(t, Q + lat.keys), rnd(t, H, DIM + ROT)
        q2 = q3.view(t, -1)
        byt = t * (Q * 4 + lat.keys * 4 + H * ROT * 4)

        def ours():
            mla.latent_prepare_(proj[:, Q:], lpool, kn, sl, RANK, RANK, 1e-5, rope, p, proj[:, :Q], qn, Q)
            ops.rope_heads_(q2, cos, sin, p, H, DIM + ROT, DIM, ROT, False)

        def like():
            ops.rmsnorm(proj[:, :Q], qn16, 1e-5)
            ops.mla_rope_kv_scatter_(q3, proj[:, Q:], lpool, kn16, cos, sin, p, sl, DIM, ROT, RANK, 1e-5)

        pair(f"latent norms, rotation, scatter, {t} rows", DS, (ours, byt, 0), (like, byt, 0))

    # ---- decode attention ----
    st, cu1 = step(B), torch.arange(B + 1, dtype=torch.int32, device=dev)
    q, gate = rnd(B, H * DIM), rnd(B, H * DIM)
    seen = ctx % chunk + 1
    pair(f"chunked decode attention, {B} requests at {ctx} (chunk {chunk}: {seen} keys)", QW,
         (lambda: ops.window_attention(q, flat, r2t, st, H, G, DIM, DIM, 0.1, 0, gate, chunk=chunk, softcap=CAP),
          B * (seen * 2 * G + 3 * H) * DIM * 2, 0),
         (lambda: ops.gqa_decode(q, pool, r2t, req[:B], bseq, H, G, DIM, ctx + 1, 0.1), B * ((ctx + 1) * 2 * G + 2 * H) * DIM * 2, 0))
    ql, dql, dqp = rnd(B, H, lat.keys), rnd(B, H, RANK), rnd(B, H, DIM + ROT)[:, :, DIM:]
    byt, fl = B * ((ctx + 1) * lat.keys + H * (lat.keys + RANK)) * 2, B * H * (ctx + 1) * 2.0 * (lat.keys + RANK)
    pair(f"latent decode attention, {B} requests at {ctx}", DS,
         (lambda: mla.latent_attention(ql, lpool, r2t, req[:B], st.seq_pos, None, 0.07, 0, ctx + 1, rank=RANK), byt, fl),
         (lambda: mla.mla_attention(dql, dqp, lpool, r2t, req[:B], bseq, cu1, st.seq_pos, RANK, 0.07, False, 1, ctx + 1), byt, fl))

    # ---- prompt attention: 4 prompts of T / 4 ----
    r2p = slots[:T].view(4, n).contiguous()
    full = 4 * n * (n + 1) / 2
    q, gate = rnd(T, H * DIM), rnd(T, H * DIM)
    like = (lambda: ops.gqa_prefill(q, pool, r2p, req[:4], cu, zero, H, G, DIM, n, 0.1), (2 * H + 2 * G) * T * DIM * 2, full * H * 4.0 * DIM)
    big = q.float().mul(6000).to(BF)         # scores of either side of the cap
    for c in (chunk, 512):
        pairs = 4 * sum(i % c + 1 for i in range(n))
        for what, qq in (("", q), (", scores at the cap", big)):
            pair(f"chunked prompt attention, 4 x {n} (chunk {c}{what})", QW,
                 (lambda: ops.window_attention(qq, flat, r2p, pst, H, G, DIM, DIM, 0.1, 0, gate, chunk=c, softcap=CAP),
                  (3 * H + 2 * G) * T * DIM * 2, pairs * H * 4.0 * DIM), like)
    kr = mla.KeyRange(torch.zeros(4), torch.full((4,), n), 0, dev)
    q, kv = rnd(T, H * lat.dp), rnd(T, H * (lat.dp + lat.vp))
    dql, dqp = rnd(T, H, RANK), rnd(T, H, DIM + ROT)[:, :, DIM:]
    seqp = torch.full((4,), n, device=dev, dtype=torch.int32)
    pair(f"latent prompt attention, 4 x {n}", DS,
         (lambda: mla.window_prefill(q, kv, H, lat.dp, lat.vp, cu, zero, kr, n, 0.07), T * H * (2 * lat.dp + 2 * DIM) * 2,
          full * H * 2.0 * (DIM + ROT + DIM)),
         (lambda: mla.mla_attention(dql, dqp, lpool, r2p, req[:4], seqp, cu, zero, RANK, 0.07, True, n, n,
                                    batch_of=pst.batch_of_token), T * (lat.keys + H * (lat.keys + RANK)) * 2,
          full * H * 2.0 * (lat.keys + RANK)))

    # ---- recurrence: minGRU over `width` channels | gated linear attention of the same value width ----
    R, rank = W // DIM, 16
    a2, a2b, w1 = rnd(R * DIM, rank), torch.zeros(R * DIM, device=dev), torch.ones(DIM, device=dev)
    rec = la.DecayedState("gla", R, DIM, DIM, DIM, DIM, 1e-5, w1, tau=16.0, a2=a2, a2_bias=a2b)
    parts, gp = rnd(T, 3 * W).split(W, 1), torch.split(rnd(T, 4 * R * DIM + rank), [R * DIM] * 4 + [rank], 1)
    for b in (4, 1):
        ps, lens = prompts(b), torch.full((b,), T // b)
        plan, gplan = la.scan_plan(lens, dev), la.ChunkPlan(lens, dev)
        gstate = torch.zeros(b, la.DecayedState.state_elems("gla", R, DIM, DIM), device=dev)
        pair(f"minGRU prompt, {b} x {T // b}", LB, (lambda: la.gated_scan(*parts, state, ps, BF, plan), T * W * 8, 0),
             (lambda: rec(*gp[:4], gstate, ps, a1=gp[4], plan=gplan), T * W * 10, T * R * (2.0 * 32 * 2 * DIM + 4.0 * DIM * DIM)))
    for t in (B, 4 * B):
        parts, gp = rnd(t, 3 * W).split(W, 1), torch.split(rnd(t, 4 * R * DIM + rank), [R * DIM] * 4 + [rank], 1)
        gstate, dst = rnd(t, la.DecayedState.state_elems("gla", R, DIM, DIM), dtype=torch.float32), step(t)
        pair(f"minGRU step, {t} requests", LB, (lambda: la.gated_scan(*parts, state, dst, BF), t * W * 16, 0),
             (lambda: rec(*gp[:4], gstate, dst, a1=gp[4]), 2 * t * R * DIM * DIM * 4 + t * W * 10, 0))
