"""Multi-head latent attention (DeepSeek-V2/V3) over the latent KV pool.

The pool row of a token is `[c_kv (kv_lora_rank, already RMS-normalised) | k_pe (rope dim, rotated)]`,
one "head", shared by all query heads.  Attention runs in the absorbed form: the query is moved into
the latent space with W_UK (`q_lat = q_nope . W_UK`), scores are `q_lat . c_kv + q_pe . k_pe`, the
value read is the same `c_kv`, and W_UV brings the result back (`o = (P . c_kv) . W_UV^T`).

`mla_attention(...)` covers prefill (causal, cached-prefix aware) and decode; CUDA tensors use
`csrc/mla.cu`, CPU tensors the fp32 restatement below.

Reference: lightllm/models/deepseek2/layer_infer/transformer_layer_infer.py:75-214 and its MLA
Triton / FlashInfer back-ends.
"""
from __future__ import annotations

import math

import torch

from . import DTYPE_CODES, _count, gemm_f32
from ._native import c_int, check, f32, i64, kernels, ptr, stream


def ref_mla_attention(q_lat, q_pe, kv_layer, req_to_token, b_req_idx, b_seq_len, cu_q, b_ready_len, kv_lora, scale):
    """q_lat [T, h, kv_lora], q_pe [T, h, rope]; kv_layer [slots, 1, kv_lora + rope].
    Request b owns query rows cu_q[b]:cu_q[b+1] at positions ready_len[b] + i; returns o_lat [T, h, kv_lora]."""
    T, h, _ = q_lat.shape
    out = torch.zeros(T, h, kv_lora, dtype=q_lat.dtype, device=q_lat.device)
    B = b_req_idx.shape[0]
    for b in range(B):
        s0, s1 = int(cu_q[b]), int(cu_q[b + 1])
        n = s1 - s0
        if n == 0:
            continue
        ready = int(b_ready_len[b])
        L = ready + n
        slots = req_to_token[int(b_req_idx[b]), :L].long()
        kv = kv_layer[slots, 0].float()
        c, kpe = kv[:, :kv_lora], kv[:, kv_lora:]
        s = torch.einsum("nhd,ld->hnl", q_lat[s0:s1].float(), c) + torch.einsum("nhr,lr->hnl", q_pe[s0:s1].float(), kpe)
        s = s * scale
        qpos = torch.arange(n, device=q_lat.device) + ready
        mask = torch.arange(L, device=q_lat.device)[None, :] <= qpos[:, None]
        s = s.masked_fill(~mask[None], float("-inf"))
        p = torch.softmax(s, dim=-1)
        out[s0:s1] = torch.einsum("hnl,ld->nhd", p, c).to(q_lat.dtype)
    return out


def mla_attention(q_lat, q_pe, kv_layer, req_to_token, b_req_idx, b_seq_len, cu_q, b_ready_len, kv_lora, scale,
                  is_prefill: bool, max_q_len: int = 1, max_kv_len: int = 0, batch_of=None):
    if not q_lat.is_cuda:
        return ref_mla_attention(q_lat, q_pe, kv_layer, req_to_token, b_req_idx, b_seq_len, cu_q, b_ready_len, kv_lora,
                                 scale)
    T, h, _ = q_lat.shape
    rope = q_pe.shape[-1]
    assert kv_lora == 512 and rope == 64, "the MLA kernel is specialised for kv_lora_rank 512 / rope 64"
    assert q_lat.is_contiguous() and q_pe.stride(-1) == 1
    out = torch.empty((T, h, kv_lora), dtype=q_lat.dtype, device=q_lat.device)
    B = b_req_idx.shape[0]
    check(kernels().llb_mla_attention(ptr(q_lat), ptr(q_pe), i64(q_pe.stride(0)), i64(q_pe.stride(1)), ptr(kv_layer),
                                      ptr(req_to_token), i64(req_to_token.stride(0)), ptr(b_req_idx), ptr(cu_q),
                                      ptr(b_ready_len), ptr(batch_of), ptr(out), c_int(B), c_int(T), c_int(h),
                                      c_int(max_q_len),
                                      f32(scale), stream()), "mla_attention")
    _count()
    return out


def gemm_batched(a, w, out=None):
    """Per-head GEMM: a [T, h, K] (any row / head strides, unit inner stride), w [h, N, K] -> out [T, h, N].
    Used for the W_UK / W_UV absorption steps of MLA."""
    T, h, K = a.shape
    N = w.shape[1]
    if not a.is_cuda:
        return torch.einsum("thk,hnk->thn", a.float(), w.float()).to(a.dtype)
    if a.dtype == torch.float32:
        return gemm_f32(a, w, out=out)
    from . import gemm_status

    assert a.stride(2) == 1 and w.is_contiguous()
    if out is None:
        out = torch.empty((T, h, N), dtype=a.dtype, device=a.device)
    check(kernels().llb_gemm_bf16_batched(ptr(a), i64(a.stride(0)), i64(a.stride(1)), ptr(w), ptr(out),
                                          i64(out.stride(0)), i64(out.stride(1)), c_int(T), c_int(N), c_int(K),
                                          c_int(h), ptr(gemm_status(a.device)), stream()), "gemm_batched")
    _count()
    return out


# ---------------------------------------------------------------------------------------------------------------------
# Latent attention with any latent size, optional rotary part, optional sliding window, bf16 or fp32.  The pool row is
# [latent, zero-padded to `rank` columns | rotated key part], zero-padded to the row pitch.  A query sees its own position and the window - 1 before it (window 0:
# all before it).
#   absorbed form   scores and values in the latent space, straight from the pool (decode, short portions)
#   expanded form   keys and values of every head are formed for the positions a prompt pass can see, then attention
#                   per head (fewer operations per key for long prompts)
# ---------------------------------------------------------------------------------------------------------------------
class LatentRope:
    """Rotation of the key part behind a latent: tables [positions, dims / 2] fp32, pairs of neighbours or of halves."""

    def __init__(self, cos, sin, dims: int, neighbours: bool = True):
        self.cos, self.sin, self.dims, self.neighbours = cos, sin, int(dims), neighbours


def latent_prepare_(kv_a, kv_layer, norm_w, slot, rank: int, cols: int, eps: float, rope=None, pos=None, q_a=None, q_w=None,
                    q_rank: int = 0):
    """kv_layer[slot[t]] = [RMSNorm(kv_a[t, :rank]) * norm_w (fp32), zero to `cols` columns | kv_a[t, cols : cols + rope.dims]
    rotated to position pos[t]], padding columns zero.  q_a [T, q_cols]: latents of the queries, q_rank values; returns their
    RMSNorm * q_w, zero-padded [T, q_cols] (else None)."""
    row, dims = kv_layer.shape[-1], rope.dims if rope is not None else 0
    T = kv_a.shape[0]
    if not kv_a.is_cuda:
        from . import reference as ref

        def norm(v, n, w, width):
            v = ref.rms_over(v[:, :n].float(), n, eps) * w[:n]
            return torch.nn.functional.pad(v, (0, width - n))

        out = torch.zeros(T, row)
        out[:, :cols] = norm(kv_a, rank, norm_w, cols)
        if dims:
            out[:, cols:cols + dims] = ref.rotate_pairs(kv_a[:, cols:cols + dims].float(), rope.cos, rope.sin, pos,
                                                        rope.neighbours)
        kv_layer.view(-1, row)[slot.long()] = out.to(kv_layer.dtype)
        return None if q_a is None else norm(q_a, q_rank, q_w, q_a.shape[1]).to(q_a.dtype)
    assert kv_a.stride(1) == 1 and kv_a.dtype == kv_layer.dtype and kv_layer.is_contiguous()
    assert norm_w.dtype == torch.float32 and slot.dtype == torch.int32
    q_out = None
    if q_a is not None:
        assert q_a.stride(1) == 1 and q_a.dtype == kv_a.dtype and q_w.dtype == torch.float32
        q_out = torch.empty(q_a.shape, dtype=q_a.dtype, device=q_a.device)
    r = rope if dims else None
    check(kernels().llb_latent_prepare(ptr(kv_a), c_int(DTYPE_CODES[kv_a.dtype]), i64(kv_a.stride(0)), ptr(kv_layer),
                                       c_int(row), ptr(norm_w), ptr(slot), c_int(T), c_int(rank), c_int(cols),
                                       ptr(r.cos if r else None), ptr(r.sin if r else None), ptr(pos), c_int(dims),
                                       c_int(1 if r is None or r.neighbours else 0), ptr(q_a),
                                       i64(q_a.stride(0) if q_a is not None else 0), ptr(q_out), c_int(q_rank),
                                       c_int(q_a.shape[1] if q_a is not None else 0), ptr(q_w), f32(eps), stream()),
          "latent_prepare")
    _count()
    return q_out


def latent_norm_scatter_(kv_a, kv_layer, norm_w, slot, rank: int, eps: float):
    """`latent_prepare_` of rows that are a latent alone."""
    latent_prepare_(kv_a, kv_layer, norm_w, slot, rank, kv_layer.shape[-1], eps)


def ref_latent_attention(q_lat, kv_layer, req_to_token, b_req_idx, pos, batch_of, scale, window: int = 0, rank: int = 0):
    T, H, keys = q_lat.shape
    rank = rank or keys
    flat = kv_layer.view(-1, kv_layer.shape[-1])
    out = torch.empty((T, H, rank), dtype=q_lat.dtype, device=q_lat.device)
    for t in range(T):
        b = int(batch_of[t]) if batch_of is not None else t
        p = int(pos[t])
        j0 = max(0, p - window + 1) if window else 0
        c = flat[req_to_token[int(b_req_idx[b]), j0:p + 1].long(), :keys].float()
        w = torch.softmax(q_lat[t].float() @ c.t() * scale, dim=-1)
        out[t] = (w @ c[:, :rank]).to(out.dtype)
    return out


def latent_num_splits(T: int, H: int, max_keys: int, sms: int = 148) -> int:
    """Shares the keys of a query are cut into so that the grid fills the GPU: modelled as waves x tiles per CTA plus
    the cost of merging."""
    tiles = max(1, -(-max_keys // 64))
    ctas = T * -(-H // 16)
    best, best_cost = 1, None
    for s in range(1, min(tiles, 64) + 1):
        cost = -(-ctas * s // sms) * (-(-tiles // s) + 2.0) + (0.0 if s == 1 else 2.0 + 0.02 * s)
        if best_cost is None or cost < best_cost:
            best, best_cost = s, cost
    return best


def latent_attention(q_lat, kv_layer, req_to_token, b_req_idx, pos, batch_of, scale, window: int = 0, max_keys: int = 0,
                     num_splits: int = 0, generic: bool = False, rank: int = 0):
    """Absorbed form.  q_lat [T, H, keys] (padding columns zero), of whose columns the first `rank` are latent (0: all);
    pos / batch_of: position and request of every query token (batch_of None: token i belongs to request i).  Returns
    [T, H, rank].
    `max_keys`: the most keys a query may see.  `generic`: the kernel without tensor cores (always used for fp32 and for
    rows above 576 values, 512 of them latent)."""
    if not q_lat.is_cuda:
        return ref_latent_attention(q_lat, kv_layer, req_to_token, b_req_idx, pos, batch_of, scale, window, rank)
    T, H, keys = q_lat.shape
    rank = rank or keys
    row = kv_layer.shape[-1]
    assert q_lat.is_contiguous() and kv_layer.is_contiguous() and q_lat.dtype == kv_layer.dtype
    assert pos.dtype == torch.int32 and b_req_idx.dtype == torch.int32
    out = torch.empty((T, H, rank), dtype=q_lat.dtype, device=q_lat.device)
    if generic or q_lat.dtype != torch.bfloat16 or rank > 512 or keys > 576 or rank % 8 or keys % 8:
        check(kernels().llb_latent_attn_generic(ptr(q_lat), c_int(DTYPE_CODES[q_lat.dtype]), ptr(kv_layer), c_int(row),
                                                ptr(req_to_token), i64(req_to_token.stride(0)), ptr(b_req_idx), ptr(pos),
                                                ptr(batch_of), ptr(out), c_int(T), c_int(H), c_int(keys), c_int(rank), f32(scale),
                                                c_int(window), stream()), "latent_attn_generic")
        _count()
        return out
    splits = num_splits or latent_num_splits(T, H, max_keys or 64)
    po = pl = None
    if splits > 1:
        n = splits * T * H
        po = torch.empty(n * rank, dtype=torch.float32, device=q_lat.device)
        pl = torch.empty(n * 2, dtype=torch.float32, device=q_lat.device)
    check(kernels().llb_latent_attn_mma(ptr(q_lat), ptr(kv_layer), c_int(row), ptr(req_to_token),
                                        i64(req_to_token.stride(0)), ptr(b_req_idx), ptr(pos), ptr(batch_of), ptr(out),
                                        ptr(po), ptr(pl), c_int(T), c_int(H), c_int(keys), c_int(rank), c_int(splits),
                                        f32(scale), c_int(window), stream()), "latent_attn_mma")
    _count(2 if splits > 1 else 1)
    return out


class KeyRange:
    """The cached positions a prompt pass can see through a window: request b contributes positions kv_start[b] ..
    (last new position), laid out back to back from row cu_kv[b] on."""

    def __init__(self, ready, q_len, window: int, device):
        ready, q_len = ready.to(torch.int64).cpu(), q_len.to(torch.int64).cpu()
        start = (ready - (window - 1)).clamp_min(0) if window else torch.zeros_like(ready)
        n = ready + q_len - start
        cu = torch.zeros(len(n) + 1, dtype=torch.int32)
        cu[1:] = torch.cumsum(n, 0)
        self.window, self.rows = window, int(cu[-1])
        self.kv_start = start.to(torch.int32).to(device, non_blocking=True)
        self.cu_kv = cu.to(device, non_blocking=True)


def latent_gather(kv_layer, req_to_token, b_req_idx, kr: KeyRange):
    """[rows, row pitch]: the latents of the range, in order."""
    row = kv_layer.shape[-1]
    out = torch.empty((kr.rows, row), dtype=kv_layer.dtype, device=kv_layer.device)
    check(kernels().llb_latent_gather(ptr(kv_layer), c_int(row * kv_layer.element_size()), ptr(req_to_token),
                                      i64(req_to_token.stride(0)), ptr(b_req_idx), ptr(kr.cu_kv), ptr(kr.kv_start),
                                      ptr(out), c_int(b_req_idx.shape[0]), c_int(kr.rows), stream()), "latent_gather")
    _count()
    return out


def window_prefill(q, kv, H: int, dk: int, dv: int, cu_q, b_ready_len, kr: KeyRange, max_q_len: int, scale, gate=None):
    """Expanded form on the tcgen05 tensor cores: q [T, >= H * dk] (row stride free), kv [rows, H * dk | H * dv], key sizes
    up to 256 and value sizes up to 128, multiples of 64; gate [T, H * dv] or None: the result times sigmoid(gate).  Returns
    [T, H * dv]."""
    assert q.dtype == torch.bfloat16 and kv.dtype == torch.bfloat16 and q.stride(1) == 1 and kv.is_contiguous()
    assert kv.shape == (kr.rows, H * (dk + dv)) and cu_q.dtype == torch.int32
    T, B = q.shape[0], cu_q.shape[0] - 1
    out = torch.empty((T, H * dv), dtype=q.dtype, device=q.device)
    check(kernels().llb_window_prefill_tc(ptr(q), i64(q.stride(0)), ptr(kv), i64(kv.stride(0)), c_int(kr.rows), ptr(cu_q),
                                          ptr(kr.cu_kv), ptr(kr.kv_start), ptr(b_ready_len), ptr(out),
                                          i64(out.stride(0)), c_int(B), c_int(T), c_int(max_q_len), c_int(H), c_int(dk),
                                          c_int(dv), f32(scale), c_int(kr.window), ptr(gate),
                                          i64(gate.stride(0) if gate is not None else 0), stream()), "window_prefill_tc")
    _count()
    return out
