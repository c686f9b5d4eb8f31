"""Katarax beside the framework's closest models at equal sizes, for `design_bench`: DeepSeek-V3 (latent attention with query
latents and a rotated part, grouped sigmoid routing) and Qwen3-MoE (grouped-query attention with query / key norms, routed experts).

Four layers each; Katarax has one of every kind (latent with a window, biased with a window and kept tokens, rotated, rotated on
the cache of the layer before).  Kernels: time and fraction of the roofline (the slower of bytes / measured copy bandwidth and
operations / measured bf16 rate), the numbers of either model's own work."""
from __future__ import annotations

import json

import torch

LAYERS, DIM, ROT, RANK, VOCAB = 4, 128, 64, 512, 32768
KEEP, FAR, BUCKETS = 64, 128, 16
# width, heads, key / value heads, query latent, experts, experts per token, groups and kept ones, expert size, window
SIZES = {
    "small": dict(width=1024, heads=8, kv=2, q_rank=768, experts=32, top=4, groups=(4, 2), ff=512, window=1024),
    "base": dict(width=2048, heads=16, kv=4, q_rank=1536, experts=64, top=6, groups=(8, 3), ff=1408, window=4096),
    "wide": dict(width=4096, heads=32, kv=8, q_rank=1536, experts=64, top=6, groups=(8, 3), ff=1408, window=4096),
}


def config(z):
    rot = {"base": 1e4, "dims": DIM}
    gqa = dict(heads=z["heads"], kv_heads=z["kv"], dim=DIM, vdim=DIM, scale=DIM ** -0.5)
    mixers = [("latent_attention", dict(heads=z["heads"], dim=DIM, rot_dim=ROT, vdim=DIM, kv_rank=RANK, q_rank=z["q_rank"],
                                        mask={"size": z["window"]}, rot={"base": 1e4, "dims": ROT}, scale=(DIM + ROT) ** -0.5)),
              ("attention", dict(gqa, mask={"size": z["window"], "keep_first": KEEP}, bias_max=FAR)),
              ("attention_2", dict(gqa, rot=rot)), ("attention_2", dict(gqa, rot=rot, kv_from=2))]
    moe = dict(kind="moe", expert={"ff": z["ff"], "limit": 7.0},
               router={"experts": z["experts"], "top": z["top"], "scale": 2.5,
                       "groups": dict(zip(("count", "keep"), z["groups"]))})
    return {"architecture": "Katarax", "width": z["width"], "vocab": VOCAB, "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
            "layers": [{"type": t, "mixer": m, "mlp": moe} for t, m in mixers]}


def deepseek_config(z):
    return dict(model_type="deepseek_v3", hidden_size=z["width"], num_hidden_layers=LAYERS, vocab_size=VOCAB,
                num_attention_heads=z["heads"], num_key_value_heads=z["heads"], q_lora_rank=z["q_rank"], kv_lora_rank=RANK,
                qk_nope_head_dim=DIM, qk_rope_head_dim=ROT, v_head_dim=DIM, intermediate_size=z["ff"],
                moe_intermediate_size=z["ff"], n_routed_experts=z["experts"], n_shared_experts=0,
                num_experts_per_tok=z["top"], first_k_dense_replace=0, norm_topk_prob=True, routed_scaling_factor=2.5,
                n_group=z["groups"][0], topk_group=z["groups"][1], rms_norm_eps=1e-5, rope_theta=1e4)


def qwen_config(z):
    return dict(model_type="qwen3_moe", hidden_size=z["width"], num_hidden_layers=LAYERS, vocab_size=VOCAB,
                num_attention_heads=z["heads"], num_key_value_heads=z["kv"], head_dim=DIM, intermediate_size=z["ff"],
                moe_intermediate_size=z["ff"], num_experts=z["experts"], num_experts_per_tok=z["top"], norm_topk_prob=True,
                rms_norm_eps=1e-6, rope_theta=1e4, decoder_sparse_step=1, mlp_only_layers=[])


CLOSEST = {"deepseek_v3": deepseek_config, "qwen3_moe": qwen_config}


def kernels(size: str, T: int = 8192, B: int = 64, ctx: int = 4096):
    from .. import ops
    from ..common.infer_state import InferState
    from ..models.latent import LatentHeads
    from ..ops import mla, moe
    from ..ops import reference as ref
    from .design_bench import peaks
    from .kernel_bench import timeit

    z = SIZES[size]
    W, H, G, Q, E, k, ff, win = (z[n] for n in ("width", "heads", "kv", "q_rank", "experts", "top", "ff", "window"))
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

    DS, QW = "deepseek_v3", "qwen3_moe"
    ones, nw, hn16 = torch.ones(W, device=dev), torch.ones(W, device=dev, dtype=BF), torch.ones(DIM, device=dev, dtype=BF)
    lat = LatentHeads(H, DIM, ROT, DIM, RANK, 0.07, win)
    slots = torch.randperm(B * (ctx + 1), device=dev).to(torch.int32)
    r2t = slots.view(B, ctx + 1)
    lpool, pool = rnd(B * (ctx + 1), lat.keys), rnd(B * (ctx + 1), 2 * G, DIM)
    flat = pool.view(-1, 2 * G * DIM)
    cos, sin = ref.build_rope_cache(ctx + T, ROT, 1e4, None, device=dev)
    cos2, sin2 = ref.build_rope_cache(ctx + T, DIM, 1e4, None, device=dev)
    rope = mla.LatentRope(cos, sin, ROT)
    pos_t = torch.arange(T, device=dev, dtype=torch.int32) % ctx
    req = torch.arange(B, device=dev, dtype=torch.int32)
    bseq = torch.full((B,), ctx + 1, device=dev, dtype=torch.int32)
    bias = ops.DistanceBias(rnd(BUCKETS, H), FAR)

    # ---- rows around the stream ----
    ow = rnd(W, H * DIM)
    for t in (T, B):
        a, res = rnd(t, H * DIM), rnd(t, W)
        fl, wb = 2.0 * t * W * H * DIM, (W + t) * H * DIM * 2

        def like():
            ops.gemm(a, ow, epi="residual", residual=res, out=res)
            ops.rmsnorm(res, nw, 1e-5)

        pair(f"output projection (its sum and norm come with the experts), {t} rows", DS,
             (lambda: ops.gemm(a, ow), wb + t * W * 2, fl), (like, wb + t * W * 8, fl))
    table, ids = rnd(VOCAB, W), torch.randint(0, VOCAB, (T,), device=dev)
    pair(f"embedding + first norm, {T} rows", DS,
         (lambda: ops.embedding_pair(ids, table, None, r2t, req, pos_t, None, slots[:T], norm=(ones, W, 1e-5)), T * W * 8, 0),
         (lambda: ops.rmsnorm(ops.embedding(ids, table), nw, 1e-5), T * W * 8, 0))
    head = rnd(VOCAB, W)
    for t in (B, 512):
        a = rnd(t, W)
        byt, fl = (VOCAB + t) * W * 2 + t * VOCAB * 4, 2.0 * t * VOCAB * W
        pair(f"logits, {t} rows", DS, (lambda: ops.gemm(a, head, epi="f32", softcap=30.0), byt, fl),
             (lambda: ops.gemm(a, head, epi="f32"), byt, fl))

    # ---- new keys, values, latents ----
    kn, qn, kn16, qn16 = (torch.ones(n, device=dev, dtype=d) for n, d in ((RANK, torch.float32), (Q, torch.float32), (RANK, BF), (Q, BF)))
    for t in (T, B):
        proj, q3 = rnd(t, Q + lat.keys + H * DIM), rnd(t, H, DIM + ROT)
        q2, p, sl = q3.view(t, -1), pos_t[:t], slots[:t]
        byt = t * (Q * 4 + lat.keys * 4 + H * ROT * 4)

        def ours():
            mla.latent_prepare_(proj[:, Q:Q + lat.keys], lpool, kn, sl, RANK, RANK, 1e-5, rope, p, proj[:, :Q], qn, Q)
            ops.rope_heads_(q2, cos, sin, p, H, DIM + ROT, DIM, ROT)

        def like():
            ops.rmsnorm(proj[:, :Q], qn16, 1e-5)
            ops.mla_rope_kv_scatter_(q3, proj[:, Q:Q + lat.keys], lpool, kn16, cos, sin, p, sl, DIM, ROT, RANK, 1e-5)

        pair(f"latent norms, rotation, scatter, {t} rows", DS, (ours, byt, 0), (like, byt, 0))
        qkv = rnd(t, (H + 2 * G) * DIM)
        byt = t * (H + 2 * G) * DIM * 4
        like = (lambda: ops.rope_kv_scatter_(qkv, pool, cos2, sin2, p, sl, H, G, DIM, DIM, hn16, hn16, 1e-5), byt, 0)
        pair(f"rotation, unit heads, scatter, {t} rows", QW,
             (lambda: ops.qk_norm_rope_scatter_(qkv, flat, cos2, sin2, p, sl, None, None, 1e-5, H, G, DIM, DIM, DIM, DIM), byt, 0), like)
        pair(f"rotation, unit queries (shared cache), {t} rows", QW,
             (lambda: ops.qk_norm_rope_scatter_(qkv, flat, cos2, sin2, p, sl, None, None, 1e-5, H, 0, DIM, DIM, DIM, DIM),
              t * H * DIM * 4, 0), like)
        pair(f"key / value scatter, {t} rows", QW,
             (lambda: ops.copy_rows(flat, qkv[:, H * DIM:], sl, None, t), t * 2 * G * DIM * 4, 0), like)

    # ---- decode attention ----
    st = InferState(is_prefill=False, batch_size=B, num_tokens=B, max_kv_len=ctx + 1, max_q_len=1, b_req_idx=req,
                    b_seq_len=bseq, mem_index=None, seq_pos=bseq - 1)
    keys, cu1, pos_b = min(win, ctx + 1), torch.arange(B + 1, dtype=torch.int32, device=dev), bseq - 1
    ql, dql, dqp = rnd(B, H, lat.keys), rnd(B, H, RANK), rnd(B, H, DIM + ROT)[:, :, DIM:]
    pair(f"latent decode attention, {B} requests at {ctx} (window {win})", DS,
         (lambda: mla.latent_attention(ql, lpool, r2t, req, pos_b, None, 0.07, win, keys, rank=RANK),
          B * (keys * lat.keys + H * (lat.keys + RANK)) * 2, B * H * keys * 2.0 * (lat.keys + RANK)),
         (lambda: mla.mla_attention(dql, dqp, lpool, r2t, req, bseq, cu1, pos_b, RANK, 0.07, False, 1, ctx + 1),
          B * ((ctx + 1) * lat.keys + H * (lat.keys + RANK)) * 2, B * H * (ctx + 1) * 2.0 * (lat.keys + RANK)))
    o, gate = rnd(B, H * DIM), rnd(B, H * DIM)
    wuv, ol = rnd(H, DIM, RANK), rnd(B, H, RANK)
    byt = (H * DIM * RANK + B * H * (RANK + DIM)) * 2
    pair(f"latent values out, {B} rows | gated", DS,
         (lambda: ops.sigmoid_mul_(mla.gemm_batched(ol, wuv).view(B, -1), gate), byt + B * H * DIM * 6, 0),
         (lambda: mla.gemm_batched(ol, wuv), byt, 0))
    q = rnd(B, H * DIM)
    seen = min(win + KEEP, ctx + 1)
    like = (lambda: ops.gqa_decode(q, pool, r2t, req, bseq, H, G, DIM, ctx + 1, 0.1), B * ((ctx + 1) * 2 * G + 2 * H) * DIM * 2, 0)
    pair(f"biased decode attention, {B} requests at {ctx} (window {win} + {KEEP})", QW,
         (lambda: ops.window_attention(q, flat, r2t, st, H, G, DIM, DIM, 0.1, win, keep=KEEP, bias=bias),
          B * (seen * 2 * G + 2 * H) * DIM * 2, 0), like)
    pair(f"rotated decode attention, {B} requests at {ctx}", QW,
         (lambda: ops.window_attention(q, flat, r2t, st, H, G, DIM, DIM, 0.1, 0), B * ((ctx + 1) * 2 * G + 2 * H) * DIM * 2, 0), like)

    # ---- prompt attention: 4 prompts of T / 4 ----
    n = T // 4
    cu, zero = torch.arange(0, T + 1, n, device=dev, dtype=torch.int32), torch.zeros(4, device=dev, dtype=torch.int32)
    r2p = slots[:T].view(4, n).contiguous()
    pst = InferState(is_prefill=True, batch_size=4, num_tokens=T, max_kv_len=n, max_q_len=n, b_req_idx=req[:4],
                     b_seq_len=None, mem_index=None, cu_q=cu, b_ready_cache_len=zero)
    kr = mla.KeyRange(torch.zeros(4), torch.full((4,), n), win, dev)
    pairs, full = 4 * sum(min(i + 1, win) for i in range(n)), 4 * n * (n + 1) / 2
    q, kv, gate = rnd(T, H * lat.dp), rnd(T, H * (lat.dp + lat.vp)), rnd(T, H * DIM)
    dql, dqp = rnd(T, H, RANK), rnd(T, H, DIM + ROT)[:, :, DIM:]
    bof = torch.repeat_interleave(torch.arange(4, device=dev, dtype=torch.int32), n)
    seqp = torch.full((4,), n, device=dev, dtype=torch.int32)
    pair(f"latent prompt attention, 4 x {n} (window {win})", DS,
         (lambda: mla.window_prefill(q, kv, H, lat.dp, lat.vp, cu, zero, kr, n, 0.07, gate), T * H * (2 * lat.dp + 3 * DIM) * 2,
          pairs * H * 2.0 * (DIM + ROT + DIM)),
         (lambda: mla.mla_attention(dql, dqp, lpool, r2p, req[:4], seqp, cu, zero, RANK, 0.07, True, n, n, batch_of=bof),
          T * (lat.keys + H * (lat.keys + RANK)) * 2, full * H * 2.0 * (lat.keys + RANK)))
    wkv, uk, qn3 = rnd(H * (lat.dp + lat.vp), lat.keys), rnd(H, RANK, DIM), rnd(T, H, DIM)
    pair(f"rows of {T} keys, expanded | queries taken into the latent space", DS,
         (lambda: ops.gemm(mla.latent_gather(lpool, r2p, req[:4], kr), wkv),
          ((T + wkv.shape[0]) * lat.keys + T * wkv.shape[0] + 2 * T * lat.keys) * 2, 2.0 * T * RANK * 2 * H * DIM),
         (lambda: mla.gemm_batched(qn3, uk), (H * RANK * DIM + T * H * (DIM + RANK)) * 2, 2.0 * T * H * RANK * DIM))
    q = rnd(T, H * DIM)
    byt = (2 * H + 2 * G) * T * DIM * 2
    like = (lambda: ops.gqa_prefill(q, pool, r2p, req[:4], cu, zero, H, G, DIM, n, 0.1), byt, full * H * 4.0 * DIM)
    for w in sorted({win, 512}):
        wp = 4 * sum(min(i + 1, w + min(KEEP, max(i + 1 - w, 0))) for i in range(n))
        pair(f"biased prompt attention, 4 x {n} (window {w} + {KEEP})", QW,
             (lambda: ops.window_attention(q, flat, r2p, pst, H, G, DIM, DIM, 0.1, w, keep=KEEP, bias=bias), byt, wp * H * 4.0 * DIM),
             like)
    pair(f"rotated prompt attention, 4 x {n}", QW,
         (lambda: ops.window_attention(q, flat, r2p, pst, H, G, DIM, DIM, 0.1, 0), byt, full * H * 4.0 * DIM), like)

    # ---- experts ----
    w13, w2, router, corr = rnd(E, 2 * ff, W), rnd(E, W, ff), rnd(E, W), torch.zeros(E, device=dev)
    for t in (T, B):
        h, x, y, res = rnd(t, W), rnd(t, W, dtype=torch.float32), rnd(t, W), rnd(t, W)
        idl = torch.rand(t, E, device=dev).topk(k, -1)[1].to(torch.int32)
        wts = torch.full((t, k), 1.0 / k, device=dev)
        fl = 2.0 * t * k * 3 * ff * W
        byt = min(E, t * k) * 3 * ff * W * 2 + t * k * (W * 8 + ff * 4)

        def route(bias_):
            return moe.grouped_topk(ops.gemm(h, router, epi="f32"), bias_, k, *z["groups"], True, True, 2.5)

        rb = (E + t) * W * 2 + t * k * 8
        pair(f"router, {t} rows", DS, (lambda: route(corr), rb, 0), (lambda: route(corr), rb, 0))

        def like_experts():
            out = torch.empty_like(h)
            moe.fused_experts(h, w13, w2, idl, wts, out=out)
            ops.add_rmsnorm_(res, out, nw, 1e-5)

        pair(f"experts + both sublayers' sum + norm, {t} rows", DS,
             (lambda: moe.routed_experts_rms_(h, idl, wts, w13, w2, (1.702, 7.0), y, x, None, W, 1e-5, ones), byt + t * W * 12, fl),
             (like_experts, byt + t * W * 8, fl))
