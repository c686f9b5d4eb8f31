"""The kernels of the Taduzen family beside the like kernels of DeepSeek-V2 at equal sizes: time and fraction of the
roofline (the slower of bytes / measured copy bandwidth and operations / measured bf16 rate).  Used by `design_bench`."""
from __future__ import annotations

import json

import torch

from .design_bench import DIM, SIZES, VOCAB, peaks
from .kernel_bench import timeit

BF = torch.bfloat16


def kernels(size: str, T: int = 8192, B: int = 64, ctx: int = 4096):
    from .. import ops
    from ..ops import mla, moe
    from ..ops import reference as ref

    z = SIZES[size]
    W, H, R, E, k, ff, win = z["width"], z["heads"], z["rank"], z["experts"], z["top"], z["ff"], z["window"]
    hbm, tf = peaks()
    dev = torch.device("cuda")
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)

    def rnd(*s, dtype=BF):
        return torch.randn(*s, device=dev).mul_(0.05).to(dtype)

    def measure(fn, bytes_, flops):
        t = timeit(fn, flush, reps=1)
        return t * 1e6, max(bytes_ / hbm, flops / tf) / t

    def pair(what, ours, like):
        (u1, f1), (u2, f2) = measure(*ours), measure(*like)
        print(json.dumps({"kernel": what, "size": size, "us": round(u1, 1), "roofline": round(f1, 3),
                          "deepseek_v2_us": round(u2, 1), "deepseek_v2_roofline": round(f2, 3),
                          "ratio": round(f1 / f2, 2)}), flush=True)

    n1 = ops.DytNorm(torch.ones(W, device=dev), torch.zeros(W, device=dev), 0.5)
    nw = torch.ones(W, device=dev, dtype=BF)

    # ---- projections into the stream: GEMM with both norms in the epilogue | GEMM with residual, then RMSNorm ----
    ow = rnd(W, H * DIM)
    for t in (T, B):
        a, x, res = rnd(t, H * DIM), rnd(t, W, dtype=torch.float32), rnd(t, W)
        fl, wb = 2.0 * t * W * H * DIM, W * H * DIM * 2 + t * H * DIM * 2

        def like():
            ops.gemm(a, ow, epi="residual", residual=res, out=res)
            ops.rmsnorm(res, nw, 1e-5)

        pair(f"output projection + norms, {t} rows",
             (lambda: ops.gemm(a, ow, epi="dyt", x=x, dyt=(n1, n1)), wb + t * W * 10, fl),
             (like, wb + t * W * 8, fl))

    # ---- first row pass ----
    table, ids = rnd(VOCAB, W), torch.randint(0, VOCAB, (T,), device=dev)
    pair(f"embedding + first norm, {T} rows", (lambda: ops.embedding_dyt(ids, table, n1), T * W * 8, 0),
         (lambda: ops.rmsnorm(ops.embedding(ids, table), nw, 1e-5), T * W * 8, 0))

    # ---- latents into the pool ----
    slots = torch.randperm(B * (ctx + 1), device=dev).to(torch.int32)
    pool = rnd(B * (ctx + 1), 1, R)
    dpool = rnd(B * (ctx + 1), 1, 576)
    src, dsrc, q3 = rnd(T, H * DIM + R), rnd(T, 576), rnd(T, H, 192)
    kn, dkn = torch.ones(R, device=dev), torch.ones(512, device=dev, dtype=BF)
    cos, sin = ref.build_rope_cache(ctx + T, 64, 1e4, None, device=dev)
    pos_t = torch.arange(T, device=dev, dtype=torch.int32)
    pair(f"latent norm + scatter, {T} rows",
         (lambda: mla.latent_norm_scatter_(src[:, H * DIM:], pool, kn, slots[:T], R, 1e-5), T * R * 4, 0),
         (lambda: ops.mla_rope_kv_scatter_(q3, dsrc, dpool, dkn, cos, sin, pos_t, slots[:T], 128, 64, 512, 1e-5),
          T * (576 * 4 + H * 64 * 4), 0))

    # ---- decode attention ----
    r2t = slots.view(B, ctx + 1)
    req = torch.arange(B, device=dev, dtype=torch.int32)
    seq = torch.full((B,), ctx + 1, device=dev, dtype=torch.int32)
    cu = torch.arange(B + 1, device=dev, dtype=torch.int32)
    ql, dql, dqp = rnd(B, H, R), rnd(B, H, 512), rnd(B, H, 192)[:, :, 128:]
    keys = min(win, ctx + 1)
    pos_b = seq - 1
    pair(f"decode attention, {B} requests at {ctx} (window {win})",
         (lambda: mla.latent_attention(ql, pool, r2t, req, pos_b, None, 0.1, win, keys), B * (keys * R + 2 * H * R) * 2,
          B * H * keys * 4.0 * R),
         (lambda: mla.mla_attention(dql, dqp, dpool, r2t, req, seq, cu, pos_b, 512, 0.1, False, 1, ctx + 1),
          B * ((ctx + 1) * 576 + H * 1088) * 2, B * H * (ctx + 1) * 2.0 * 1088))

    # ---- prompt attention: 4 prompts of T / 4 ----
    n = T // 4
    r2p = slots[:T].view(4, n).contiguous()
    cup = torch.arange(0, T + 1, n, device=dev, dtype=torch.int32)
    zero = torch.zeros(4, device=dev, dtype=torch.int32)
    kr = mla.KeyRange(torch.zeros(4), torch.full((4,), n), win, dev)
    wkv = rnd(2 * H * DIM, R)
    q, kv = rnd(T, H * DIM), rnd(T, 2 * H * DIM)
    pairs = 4 * sum(min(i + 1, win) for i in range(n))
    dql, dqp = rnd(T, H, 512), rnd(T, H, 192)[:, :, 128:]
    bof = torch.repeat_interleave(torch.arange(4, device=dev, dtype=torch.int32), n)
    seqp = torch.full((4,), n, device=dev, dtype=torch.int32)
    fl, dfl = pairs * H * 4.0 * DIM, 4 * n * (n + 1) / 2 * H * 2.0 * 1088
    byt = T * H * DIM * 2 * 4
    like = (lambda: mla.mla_attention(dql, dqp, dpool, r2p, req[:4], seqp, cup, zero, 512, 0.1, True, n, n, batch_of=bof),
            T * (576 + H * 1088) * 2, dfl)
    pair(f"prompt attention, 4 x {n} (window {win})",
         (lambda: mla.window_prefill(q, kv, H, DIM, DIM, cup, zero, kr, n, 0.1), byt, fl), like)
    up = 2.0 * T * R * 2 * H * DIM
    ub, uk = (R * 2 * H * DIM + T * R + T * 2 * H * DIM) * 2, rnd(H, 512, DIM)
    pair(f"latents of {T} keys, expanded | queries taken into the latent space",
         (lambda: ops.gemm(mla.latent_gather(pool, r2p, req[:4], kr), wkv), ub + T * R * 4, up),
         (lambda: mla.gemm_batched(q.view(T, H, DIM), uk), (H * 512 * DIM + T * H * DIM + T * H * 512) * 2,
          2.0 * T * H * 512 * DIM))

    # ---- experts ----
    w13, w2 = rnd(E, 2 * ff, W), rnd(E, W, ff)
    tables = torch.rand(VOCAB, E, device=dev).topk(k, -1)[1].to(torch.int32)
    routing = moe.TableRouting([(tables, 0, E)])
    four = moe.TableRouting([(tables, 0, E)] * 4)
    gate = torch.ones(W, device=dev)
    for t in (T, B):
        h, x, sh, res = rnd(t, W), rnd(t, W, dtype=torch.float32), rnd(t, W), rnd(t, W)
        tok = torch.randint(0, VOCAB, (t,), device=dev)
        lay = routing.layouts(tok)[0]
        fl = 2.0 * t * k * 3 * ff * W
        used = min(E, t * k)
        byt = used * 3 * ff * W * 2 + t * k * (W * 8 + ff * 4)
        wts = torch.full((t, k), 1.0 / k, device=dev)
        idl = tables[tok].contiguous()

        def like_experts():
            out = sh.clone()
            moe.fused_experts(h, w13, w2, idl, wts, out=out, accumulate=True)
            ops.add_rmsnorm_(res, out, nw, 1e-5)

        pair(f"expert-sorted layouts of 4 layers, {t} rows", (lambda: four.layouts(tok), 4 * t * k * 12, 0),
             (lambda: [moe.moe_align(idl, E) for _ in range(4)], 4 * t * k * 12, 0))
        pair(f"experts + norms, {t} rows",
             (lambda: moe.uniform_experts_dyt_(h, lay, w13, w2, "silu", sh, gate, x, n1, n1), byt + t * W * 14, fl),
             (like_experts, byt + t * W * 10, fl))

    # ---- dense feed-forward ----
    dff = z["dense"]
    up_w, gu_w, dn_w = rnd(dff, W), rnd(2 * dff, W), rnd(W, dff)
    for t in (T, B):
        h = rnd(t, W)
        pair(f"dense up + activation, {t} rows",
             (lambda: ops.gemm(h, up_w, epi="relu2"), (dff * W + t * W + t * dff) * 2, 2.0 * t * dff * W),
             (lambda: ops.gemm(h, gu_w, epi="gated_silu"), (2 * dff * W + t * W + t * dff) * 2, 4.0 * t * dff * W))
        a, x, res = rnd(t, dff), rnd(t, W, dtype=torch.float32), rnd(t, W)

        def like_down():
            ops.gemm(a, dn_w, epi="residual", residual=res, out=res)
            ops.rmsnorm(res, nw, 1e-5)

        pair(f"dense down + norms, {t} rows",
             (lambda: ops.gemm(a, dn_w, epi="dyt", x=x, dyt=(n1, n1)), (dff * W + t * dff) * 2 + t * W * 10,
              2.0 * t * dff * W),
             (like_down, (dff * W + t * dff) * 2 + t * W * 8, 2.0 * t * dff * W))
