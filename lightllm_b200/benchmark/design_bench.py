"""Prefill and decode throughput of a model design beside the framework's closest model at equal sizes, and the kernels
of both with their roofline fractions.  Taduzen: DeepSeek-V2 (latent attention, routed and shared experts); Libulorn:
Qwen3-Next (`design_libulorn.py`); Katarax: DeepSeek-V3 and Qwen3-MoE (`design_katarax.py`); Silupel: Qwen2 and
DeepSeek-V2 with dense feed-forwards (`design_silupel.py`).

    python bench.py --design taduzen|libulorn|katarax|silupel [--design-size small|base|wide] [--design-kernels]

Random weights, random tokens, bf16.  Whole passes through the models' own forward (decode as CUDA graph), timed with CUDA
events after three warm-up passes; a pass reads far more weight bytes than L2 holds.  Kernels: median of 10 samples with L2
flushed before each.  One JSON object per line.
"""
from __future__ import annotations

import importlib
import json
import os

import torch

# width, heads, latent, experts, experts per token, expert size, shared size, dense size, window
SIZES = {
    "small": dict(width=1024, heads=8, rank=256, experts=32, top=4, ff=512, shared=1024, dense=4096, window=1024),
    "base": dict(width=2048, heads=16, rank=512, experts=64, top=6, ff=1408, shared=2816, dense=10944, window=4096),
    "wide": dict(width=4096, heads=32, rank=512, experts=64, top=6, ff=1408, shared=2816, dense=11008, window=4096),
}
LAYERS, DIM, VOCAB = 4, 128, 32768


def taduzen_config(z, layers=LAYERS):
    mixer = dict(heads=z["heads"], dim=DIM, vdim=DIM, kv_rank=z["rank"], scale=DIM ** -0.5, mask={"size": z["window"]})
    moe = dict(kind="moe", router={"experts": z["experts"], "top": z["top"]}, expert={"ff": z["ff"]},
               shared={"ff": z["shared"]})
    return {"architecture": "Taduzen", "width": z["width"], "vocab": VOCAB, "norm": {"eps": 1e-5}, "logit_scale": 0.5,
            "layers": [{"type": "latent_attention", "mixer": mixer,
                        "mlp": {"kind": "dense", "ff": z["dense"]} if i == 0 else moe} for i in range(layers)]}


def deepseek_config(z, layers=LAYERS):
    """Latent size and rotary size are fixed by its kernels (512, 64)."""
    return dict(model_type="deepseek_v2", hidden_size=z["width"], num_hidden_layers=layers, vocab_size=VOCAB,
                num_attention_heads=z["heads"], num_key_value_heads=z["heads"], q_lora_rank=None, kv_lora_rank=512,
                qk_nope_head_dim=DIM, qk_rope_head_dim=64, v_head_dim=DIM, intermediate_size=z["dense"],
                moe_intermediate_size=z["ff"], n_routed_experts=z["experts"], n_shared_experts=z["shared"] // z["ff"],
                num_experts_per_tok=z["top"], first_k_dense_replace=1, norm_topk_prob=False, scoring_func="softmax",
                topk_method="greedy", n_group=1, topk_group=1, rms_norm_eps=1e-5, rope_theta=1e4)


def _model(cfg, tokens, max_len, reqs):
    from ..models.registry import get_model
    from ..parallel.dist import ParallelState

    return get_model(cfg, pstate=ParallelState(device=torch.device("cuda", 0)), max_total_token_num=tokens,
                     max_req_num=reqs, max_seq_length=max_len + 8, batch_max_tokens=16384, graph_max_batch_size=reqs,
                     graph_max_len_in_batch=max_len + 8)


def _input(model, B, ready, new, prefill):
    from ..common.infer_state import ModelInput

    n = B * new
    g = torch.Generator().manual_seed(0)
    r2t = torch.randperm(B * (ready + new), generator=g).to(torch.int32).view(B, ready + new)
    model.req_manager.req_to_token_indexs[:B, : ready + new] = r2t.to(model.device)
    seq = torch.full((B,), ready + new, dtype=torch.int32)
    mi = ModelInput(batch_size=B, total_token_num=B * (ready + new), max_kv_len=ready + new, is_prefill=prefill,
                    b_req_idx=torch.arange(B, dtype=torch.int32), b_seq_len=seq,
                    mem_indexes=r2t[:, ready:].reshape(-1).clone(), max_q_len=new)
    if prefill:
        mi.input_ids = torch.randint(0, VOCAB, (n,), generator=g)
        mi.b_ready_cache_len = torch.full((B,), ready, dtype=torch.int32)
        mi.b_q_len = torch.full((B,), new, dtype=torch.int32)
    else:
        model.req_manager.req_to_next_token_ids[:B, 0] = torch.randint(0, VOCAB, (B,), generator=g).to(model.device)
    return mi


def _time_pass(model, mi, steps):
    for _ in range(3):
        model.forward(mi)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(steps):
        model.forward(mi)
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / steps


PREFILL = [(4, 0, 2048), (1, 0, 8192), (8, 4096, 512)]      # requests, cached tokens, new tokens
DECODE = [(16, 4096), (64, 4096), (256, 1024)]              # requests, context


def _design(name):
    """(sizes, configuration, {closest model: its configuration}, kernels)"""
    if name == "taduzen":
        from .design_kernels import kernels

        return SIZES, taduzen_config, {"deepseek_v2": deepseek_config}, kernels
    if name in ("katarax", "silupel"):
        d = importlib.import_module(f".design_{name}", __package__)
        return d.SIZES, d.config, d.CLOSEST, d.kernels
    from . import design_libulorn as d

    return d.SIZES, d.config, {"qwen3_next": d.closest_config}, d.kernels


def passes(design: str, size: str, steps: int):
    sizes, config, closest, _ = _design(design)
    z = sizes[size]
    res = {}
    for name, cfg in ((design, config(z)), *((n, make(z)) for n, make in closest.items())):
        tokens = max(max(b * (r + n) for b, r, n in PREFILL), max(b * (c + 1) for b, c in DECODE)) + 64
        model = _model(cfg, tokens, 8192, 256)
        for b, ready, new in PREFILL:
            ms = _time_pass(model, _input(model, b, ready, new, True), max(steps, 5))
            res[name, f"prefill {b}x{new}+{ready}"] = (ms, b * new)
        for b, ctx in DECODE:
            ms = _time_pass(model, _input(model, b, ctx, 1, False), 10 * max(steps, 5))
            res[name, f"decode {b} at {ctx}"] = (ms, b)
        model.flush_graphs()
        del model
        torch.cuda.empty_cache()
    for (name, what), (ms, n) in res.items():
        if name != design:
            continue
        line = {"design": design, "size": size, "pass": what, "ms": round(ms, 3), "tokens_per_s": round(n / ms * 1e3)}
        for c in closest:
            other = res[c, what][0]
            line.update({f"{c}_ms": round(other, 3), f"{c}_tokens_per_s": round(n / other * 1e3),
                         "speedup" if len(closest) == 1 else f"speedup_{c}": round(other / ms, 2)})
        print(json.dumps(dict(line, layers=LAYERS, dtype="bf16", data="synthetic")), flush=True)


def run(args):
    sizes, *_, kernels = _design(args.design)
    for s in [args.design_size] if args.design_size else list(sizes):
        passes(args.design, s, args.steps)
        if args.design_kernels:
            kernels(s)


def peaks():
    hbm, tf = 6.65e12, 1.59e15
    path = os.path.join(os.path.dirname(__file__), "..", "..", "MEASURED_PEAKS.json")
    if os.path.exists(path):
        p = json.load(open(path))
        hbm, tf = p.get("hbm_gbs", 6650) * 1e9, p.get("bf16_tflops", 1590) * 1e12
    return hbm, tf
