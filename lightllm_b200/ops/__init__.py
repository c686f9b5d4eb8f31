"""Operator layer: every hot op as a hand-written sm_100a kernel (CUDA tensors) with a plain
PyTorch fp32 restatement (`ops.reference`) that serves CPU tensors and the numerics tests.

CUDA tensors always take the kernel path; if the native library is missing the call raises.
"""
from __future__ import annotations

import ctypes
import math
from typing import Optional

import torch

from . import kv_quant
from . import reference as ref
from ._native import NativeError, c_int, c_void_p, check, f32, i64, kernels, ptr, stream

EPI_CODES = {"store": 0, "residual": 1, "gated_silu": 2, "f32": 3, "gated_gelu": 4, "relu2": 5, "dyt": 6,
             "gated_clamp": 7}
DTYPE_CODES = {torch.float32: 0, torch.bfloat16: 1}   # kernels that exist in both number formats

import os as _os

_GEMM_DEBUG_TORCH = _os.environ.get("LLB_GEMM_DEBUG_TORCH", "0") == "1"

# launch counter: the number of kernels of this package launched (claimed in bench output)
_launches = 0


def launch_count() -> int:
    return _launches


def _count(n=1):
    global _launches
    _launches += n


def _is_cuda(t) -> bool:
    return t.is_cuda


def _req_bf16(*ts):
    for t in ts:
        if t is not None and t.dtype != torch.bfloat16:
            raise NativeError(f"CUDA kernels take bf16 tensors, got {t.dtype}")


# --------------------------------------------------------------------------------------
def rmsnorm(x, w, eps: float, w_offset: float = 0.0, out=None):
    if not _is_cuda(x):
        return ref.rmsnorm(x, w, eps, w_offset)
    _req_bf16(x, w)
    H = x.shape[-1]
    x2 = x.reshape(-1, H)
    if x2.stride(-1) != 1:
        x2 = x2.contiguous()
    T = x2.shape[0]
    if out is None:
        out = torch.empty((T, H), dtype=x.dtype, device=x.device)
    check(kernels().llb_rmsnorm(ptr(out), ptr(x2), ptr(w), c_int(T), c_int(H), f32(eps), f32(w_offset),
                                i64(x2.stride(0)), i64(out.stride(0)), stream()), "rmsnorm")
    _count()
    return out.view(*x.shape[:-1], H)


def add_rmsnorm_(residual, x, w, eps: float, w_offset: float = 0.0, out=None):
    """residual += x (in place); returns rmsnorm(residual)."""
    if not _is_cuda(x):
        return ref.add_rmsnorm_(residual, x, w, eps, w_offset)
    _req_bf16(residual, x, w)
    assert residual.is_contiguous() and x.is_contiguous()
    T, H = x.shape
    if out is None:
        out = torch.empty_like(x)
    check(kernels().llb_add_rmsnorm(ptr(out), ptr(residual), ptr(x), ptr(w), c_int(T), c_int(H), f32(eps),
                                    f32(w_offset), stream()), "add_rmsnorm")
    _count()
    return out


def gated_act(x, act: str = "silu", out=None):
    if not _is_cuda(x):
        return ref.gated_act(x, act)
    _req_bf16(x)
    assert x.is_contiguous()
    T, N = x.shape
    if out is None:
        out = torch.empty((T, N // 2), dtype=x.dtype, device=x.device)
    check(kernels().llb_gated_act(ptr(out), ptr(x), c_int(T), c_int(N // 2), c_int(0 if act == "silu" else 1),
                                  stream()), "gated_act")
    _count()
    return out


def rope_kv_scatter_(qkv, kv_layer, cos, sin, pos, slot, Hq, Hkv, D, rot_dim=None, q_norm_w=None, k_norm_w=None,
                     norm_eps=1e-6, norm_w_offset=0.0):
    """rot_dim None = full head; 0 = no rotation (ALiBi / learned positions: K and V are only scattered)."""
    rot_dim = D if rot_dim is None else rot_dim
    if isinstance(kv_layer, kv_quant.QuantKVLayer):
        return kv_quant.rope_kv_scatter_(qkv, kv_layer, cos, sin, pos, slot, Hq, Hkv, D, rot_dim, q_norm_w, k_norm_w,
                                         norm_eps, norm_w_offset)
    if not _is_cuda(qkv):
        return ref.rope_kv_scatter_(qkv, kv_layer, cos, sin, pos, slot, Hq, Hkv, D, rot_dim, q_norm_w, k_norm_w,
                                    norm_eps, norm_w_offset)
    _req_bf16(qkv, kv_layer, q_norm_w, k_norm_w)
    assert qkv.stride(-1) == 1 and kv_layer.is_contiguous()
    assert pos.dtype == torch.int32 and slot.dtype == torch.int32
    T = qkv.shape[0]
    if D not in (64, 128, 256) or rot_dim % 16 != 0:
        assert q_norm_w is None and k_norm_w is None, "q/k norm needs a head size of 64, 128 or 256"
        assert rot_dim == 0 or (cos.dtype == torch.float32 and cos.shape[-1] == rot_dim // 2)
        check(kernels().llb_rope_kv_scatter_generic(ptr(qkv), ptr(kv_layer), ptr(cos), ptr(sin), ptr(pos), ptr(slot),
                                                    c_int(T), c_int(Hq), c_int(Hkv), c_int(D), c_int(rot_dim),
                                                    i64(qkv.stride(0)), stream()), "rope_kv_scatter_generic")
        _count()
        return qkv
    assert rot_dim == 0 or (cos.dtype == torch.float32 and cos.shape[-1] == rot_dim // 2)
    check(kernels().llb_rope_kv_scatter(ptr(qkv), ptr(kv_layer), ptr(cos), ptr(sin), ptr(pos), ptr(slot),
                                        ptr(q_norm_w), ptr(k_norm_w), f32(norm_eps), f32(norm_w_offset), c_int(T),
                                        c_int(Hq), c_int(Hkv), c_int(D), c_int(rot_dim), i64(qkv.stride(0)),
                                        stream()), "rope_kv_scatter")
    _count()
    return qkv


def mla_rope_kv_scatter_(q3, kv_a, kv_layer, kv_norm_w, cos, sin, pos, slot, nope, rope, kv_lora, eps):
    """RoPE on the rope part of q (in place), RMSNorm of the kv latent, RoPE of k_pe, scatter of
    [c_kv | k_pe] into the latent pool -- one launch."""
    if not _is_cuda(q3):
        return ref.mla_rope_kv_scatter_(q3, kv_a, kv_layer, kv_norm_w, cos, sin, pos, slot, nope, rope, kv_lora, eps)
    _req_bf16(q3, kv_a, kv_layer, kv_norm_w)
    T, hq, qd = q3.shape
    assert q3.stride(2) == 1 and kv_a.stride(1) == 1 and kv_layer.is_contiguous()
    check(kernels().llb_mla_rope_kv_scatter(ptr(q3), i64(q3.stride(0)), i64(q3.stride(1)), ptr(kv_a),
                                            i64(kv_a.stride(0)), ptr(kv_layer), ptr(kv_norm_w), ptr(cos), ptr(sin),
                                            ptr(pos), ptr(slot), c_int(T), c_int(hq), c_int(nope), c_int(rope),
                                            c_int(kv_lora), f32(eps), stream()), "mla_rope_kv_scatter")
    _count()
    return q3


def embedding(ids, table, vocab_start: int = 0, vocab_end: Optional[int] = None):
    vocab_end = vocab_start + table.shape[0] if vocab_end is None else vocab_end
    if not _is_cuda(table):
        return ref.embedding(ids, table, vocab_start, vocab_end)
    _req_bf16(table)
    assert ids.dtype == torch.int64 and ids.is_contiguous()
    T, H = ids.shape[0], table.shape[1]
    out = torch.empty((T, H), dtype=table.dtype, device=table.device)
    check(kernels().llb_embedding(ptr(out), ptr(ids), ptr(table), c_int(T), c_int(H), c_int(vocab_start),
                                  c_int(vocab_end), stream()), "embedding")
    _count()
    return out


# --------------------------------------------------------------------------------------
_status_words = {}


def gemm_status(device) -> torch.Tensor:
    """Device int that receives a code if a bounded wait inside a GEMM ran out (0 = healthy)."""
    key = torch.device(device).index or 0
    if key not in _status_words:
        _status_words[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _status_words[key]


_sk_scratch = {}


def _stream_k_scratch(device):
    """fp32 partial-tile buffer and per-tile arrival counters for the stream-K schedule (per device;
    all GEMMs of a stream share them, which is safe because they run back to back on that stream)."""
    key = torch.device(device).index or 0
    cur = _sk_scratch.get(key)
    if cur is None:
        sms = torch.cuda.get_device_properties(device).multi_processor_count
        # counters: [0, 8192) stream-K tiles (self-resetting); [8192, 16384) arrival counters of the split-K kernel
        cur = (torch.empty(sms * 2 * 128 * 256, dtype=torch.float32, device=device),
               torch.zeros(16384, dtype=torch.int32, device=device))
        _sk_scratch[key] = cur
    return cur


class TiledWeight:
    """A [N, K] weight stored as [N/128][K/64][128][64]: every 128-row x 64-column tile (what one TMA box of
    the GEMM kernels fetches) is 16 contiguous KB, so that weight streaming reads whole DRAM pages instead of
    128-byte pieces 2K bytes apart."""

    def __init__(self, w: torch.Tensor, swizzle: bool = False):
        N, K = w.shape
        assert N % 128 == 0 and K % 64 == 0, "tiled weights need N % 128 == 0 and K % 64 == 0"
        self.N, self.K = N, K
        self.swizzled = swizzle
        t = w.view(N // 128, 128, K // 64, 64).permute(0, 2, 1, 3).contiguous()
        if swizzle:  # the 128B-swizzle shared-memory image: 16-byte chunk c of row r sits at chunk c ^ (r % 8)
            r = torch.arange(128, device=w.device).view(128, 1)
            c = torch.arange(8, device=w.device).view(1, 8)
            idx = (c ^ (r & 7)).view(1, 1, 128, 8, 1).expand(N // 128, K // 64, 128, 8, 8)
            t = t.view(N // 128, K // 64, 128, 8, 8).gather(3, idx).contiguous()
        self.data = t.view(-1, 64)
        self.shape = (N, K)
        self.dtype, self.device = w.dtype, w.device

    def dense(self) -> torch.Tensor:
        N, K = self.N, self.K
        assert not self.swizzled
        return self.data.view(N // 128, K // 64, 128, 64).permute(0, 2, 1, 3).reshape(N, K)


_autotuner = None


def _tuned_bn(M: int, N: int, K: int, epi: str) -> int:
    global _autotuner
    if _autotuner is None:
        from ..utils import autotuner as _autotuner_mod

        _autotuner = _autotuner_mod
    return _autotuner.gemm_lookup(M, N, K, epi)


def gemm(a, w, epi: str = "store", residual=None, bias=None, out=None, bn: int = 0, stream_k: int = 0,
         out_scale: float = 1.0, x=None, dyt=None, clamp=None, softcap: float = 0.0):
    """C = A . W^T on the tcgen05 tensor cores.  a [M, K], w [N, K] (checkpoint layout).  fp32 operands run on the
    CUDA cores in fp32 (`csrc/gemm_f32.cu`).

    epi: "store" | "residual" (C += residual) | "gated_silu"/"gated_gelu" (w rows interleaved with
    `reference.interleave_gate_up`, C is [M, N/2]) | "f32" (fp32 output, e.g. logits, times
    `out_scale`; with softcap > 0 then softcap * tanh(. / softcap)) |
    "relu2" (square of relu) | "dyt": with the fp32 residual stream x [M, N] and dyt = (post, next) `DytNorm`s,
    x += post(A . W^T) in place and C = next(x) | "gated_clamp": interleaved as the other gated forms, with
    clamp = (alpha, limit): g = min(g, limit), u = clamp(u, -limit, limit), C = (u + 1) g sigmoid(alpha g).
    stream_k: 0 whole tiles per CTA (default: fastest on every measured shape), 1 stream-K, -1 heuristic.
    """
    if type(w).__name__ == "Fp8Weight":  # block-scaled e4m3 weight: quantise the activations, fp8 tensor cores
        from . import fp8

        return fp8.gemm_fp8(a, w, epi, residual, bias, out)
    if type(w).__name__ == "Int8Weight":  # per-channel s8 weight, per-token s8 activations, s32 accumulation
        from . import int8

        return int8.gemm_int8(a, w, epi, residual, bias, out)
    if not _is_cuda(a):
        res = ref.gemm(a, w, epi, residual, bias, out_scale=out_scale, x=x, dyt=dyt, clamp=clamp, softcap=softcap)
        if out is not None:
            out.copy_(res)
            return out
        return res
    if a.dtype == torch.float32:
        return gemm_f32(a, w, epi, residual, bias, out, out_scale, x, dyt, clamp=clamp, softcap=softcap)
    _req_bf16(a, w, residual, bias)
    if epi in ("dyt", "gated_clamp") or out_scale != 1.0 or softcap > 0:
        return _gemm_fused(a, w, epi, bias, out, bn, out_scale, x, dyt, clamp, softcap)
    if _GEMM_DEBUG_TORCH:  # debugging aid only (LLB_GEMM_DEBUG_TORCH=1): bypasses the tcgen05 kernel
        res = ref.gemm(a, w, epi, residual, bias)
        if out is not None:
            out.copy_(res)
            return out
        return res
    M, K = a.shape
    N = w.shape[0]
    tiled = isinstance(w, TiledWeight)
    if bn == 0 and stream_k == 0 and M <= 256 and bias is None and not tiled:  # a tuned variant, if one is stored
        bn = _tuned_bn(M, N, K, epi)
    ldw = (-2 if w.swizzled else -1) if tiled else w.stride(0)
    if tiled:
        w = w.data
    else:
        assert w.shape[1] == K and w.stride(1) == 1
    assert a.stride(1) == 1
    n_out = N // 2 if epi.startswith("gated") else N
    if out is None:
        out = torch.empty((M, n_out), dtype=torch.float32 if epi == "f32" else a.dtype, device=a.device)
    if epi == "residual":
        assert residual.shape == out.shape and residual.stride(0) == out.stride(0)
    skp, skc = (None, None) if (stream_k == 0 and not 2000 <= bn < 3100) else _stream_k_scratch(a.device)
    check(kernels().llb_gemm_bf16(ptr(a), i64(a.stride(0)), ptr(w), i64(ldw), ptr(out), i64(out.stride(0)),
                                  ptr(residual), ptr(bias), c_int(M), c_int(N), c_int(K), c_int(EPI_CODES[epi]),
                                  c_int(bn), c_int(stream_k), ptr(skp), i64(skp.numel() if skp is not None else 0),
                                  ptr(skc), c_int(skc.numel() if skc is not None else 0),
                                  ptr(gemm_status(a.device)), stream()), "gemm_bf16")
    _count()
    return out


def _dyt_args(n):
    """(w, b, alpha) of a DytNorm, or nulls."""
    return (ptr(None), ptr(None), f32(1.0)) if n is None else (ptr(n.w), ptr(n.b), f32(n.alpha))


def _clamp_args(clamp):
    alpha, limit = clamp if clamp is not None else (1.0, float("inf"))
    return f32(alpha), f32(limit)


def _gemm_fused(a, w, epi, bias, out, bn, out_scale, x, dyt, clamp=None, softcap=0.0):
    M, K = a.shape
    N = w.shape[0]
    assert w.shape[1] == K and w.stride(1) == 1 and a.stride(1) == 1
    if out is None:
        out = torch.empty((M, N // 2 if epi.startswith("gated") else N),
                          dtype=torch.float32 if epi == "f32" else a.dtype, device=a.device)
    post, nxt = dyt if dyt is not None else (None, None)
    if epi == "dyt":
        assert x.dtype == torch.float32 and x.shape == (M, N) and x.stride(0) == out.stride(0) and x.stride(1) == 1
    check(kernels().llb_gemm_bf16_fused(ptr(a), i64(a.stride(0)), ptr(w), i64(w.stride(0)), ptr(out),
                                        i64(out.stride(0)), ptr(bias), c_int(M), c_int(N), c_int(K),
                                        c_int(EPI_CODES[epi]), c_int(bn), f32(out_scale), ptr(x), *_dyt_args(post),
                                        *_dyt_args(nxt), *_clamp_args(clamp), f32(softcap), ptr(gemm_status(a.device)),
                                        stream()), "gemm_bf16_fused")
    _count()
    return out


def gemm_f32(a, w, epi="store", residual=None, bias=None, out=None, out_scale=1.0, x=None, dyt=None,
             mblock_expert=None, clamp=None, softcap=0.0):
    """fp32 GEMM, same epilogues as `gemm`.  a [M, K] and w [N, K]; or a [M, batch, K] and w [batch, N, K] (per-head
    products, out [M, batch, N]); or grouped with w [E, N, K] and the expert of every 128-row block."""
    grouped = mblock_expert is not None
    batched = a.dim() == 3
    batch = a.shape[1] if batched else 1
    M, K = a.shape[0], a.shape[-1]
    N = w.shape[-2]
    assert w.dtype == torch.float32 and w.shape[-1] == K and a.stride(-1) == 1 and w.stride(-1) == 1
    assert w.dim() == (3 if grouped or batched else 2)
    n_out = N // 2 if epi.startswith("gated") else N
    if out is None:
        out = torch.empty((M, batch, n_out) if batched else (M, n_out), dtype=torch.float32, device=a.device)
    post, nxt = dyt if dyt is not None else (None, None)
    if epi == "residual":
        assert residual.shape == out.shape and residual.stride(0) == out.stride(0)
    if epi == "dyt":
        assert x.shape == (M, N) and x.stride(0) == out.stride(0)
    check(kernels().llb_gemm_f32(ptr(a), i64(a.stride(0)), i64(a.stride(1) if batched else 0), ptr(w),
                                 i64(w.stride(-2)), i64(w.stride(0) if batched else 0), ptr(out), i64(out.stride(0)),
                                 i64(out.stride(1) if batched else 0), ptr(residual), ptr(bias), ptr(x),
                                 *_dyt_args(post), *_dyt_args(nxt), ptr(mblock_expert), c_int(M), c_int(N), c_int(K),
                                 c_int(batch), c_int(EPI_CODES[epi]), f32(out_scale), *_clamp_args(clamp), f32(softcap),
                                 stream()), "gemm_f32")
    _count()
    return out


# --------------------------------------------------------------------------------------
_decode_scratch = {}


def _scratch(device, n_o: int, n_lse: int):
    key = torch.device(device).index or 0
    cur = _decode_scratch.get(key)
    if cur is None or cur[0].numel() < n_o or cur[1].numel() < n_lse:
        cur = (torch.empty(max(n_o, 1 << 20), dtype=torch.float32, device=device),
               torch.empty(max(n_lse, 1 << 14), dtype=torch.float32, device=device))
        _decode_scratch[key] = cur
    return cur


def gqa_decode_num_splits(B, Hq, Hkv, max_seq_len) -> int:
    return int(kernels().llb_gqa_decode_num_splits(c_int(B), c_int(Hq), c_int(Hkv), c_int(max_seq_len)))


def gqa_decode(q, kv_layer, req_to_token, b_req_idx, b_seq_len, Hq, Hkv, D, max_seq_len: int, sm_scale=None,
               out=None, num_splits: Optional[int] = None, scratch=None):
    """Paged GQA decode attention. q [B, Hq*D] or [B, Hq, D] (row stride arbitrary)."""
    if isinstance(kv_layer, kv_quant.QuantKVLayer):
        return kv_quant.gqa_decode(q, kv_layer, req_to_token, b_req_idx, b_seq_len, Hq, Hkv, D, max_seq_len, sm_scale,
                                   out, num_splits, scratch)
    if not _is_cuda(q):
        return ref.gqa_decode(q.reshape(q.shape[0], Hq, D), kv_layer, req_to_token, b_req_idx, b_seq_len, Hq, Hkv, D,
                              sm_scale)
    _req_bf16(q, kv_layer)
    B = q.shape[0]
    assert q.stride(-1) == 1 and kv_layer.is_contiguous()
    assert req_to_token.dtype == torch.int32 and b_req_idx.dtype == torch.int32 and b_seq_len.dtype == torch.int32
    scale = sm_scale if sm_scale is not None else 1.0 / math.sqrt(D)
    if out is None:
        out = torch.empty((B, Hq, D), dtype=q.dtype, device=q.device)
    if num_splits is None:
        num_splits = gqa_decode_num_splits(B, Hq, Hkv, max_seq_len)
    po = pl = None
    if num_splits > 1:
        po, pl = scratch if scratch is not None else _scratch(q.device, B * Hq * num_splits * D, B * Hq * num_splits)
    check(kernels().llb_gqa_decode(ptr(q), i64(q.stride(0)), ptr(kv_layer), ptr(req_to_token),
                                   i64(req_to_token.stride(0)), ptr(b_req_idx), ptr(b_seq_len), ptr(out),
                                   i64(out.stride(0)), ptr(po), ptr(pl), c_int(B), c_int(Hq), c_int(Hkv), c_int(D),
                                   c_int(num_splits), f32(scale), stream()), "gqa_decode")
    _count(2 if num_splits > 1 else 1)
    return out


def gqa_prefill(q, kv_layer, req_to_token, b_req_idx, cu_q, b_ready_len, Hq, Hkv, D, max_q_len: int, sm_scale=None,
                out=None):
    """Causal varlen prefill attention over (cached prefix + new tokens). q [T, Hq*D] or [T, Hq, D]."""
    if isinstance(kv_layer, kv_quant.QuantKVLayer):
        return kv_quant.gqa_prefill(q, kv_layer, req_to_token, b_req_idx, cu_q, b_ready_len, Hq, Hkv, D, max_q_len,
                                    sm_scale, out)
    if not _is_cuda(q):
        return ref.gqa_prefill(q.reshape(q.shape[0], Hq, D), kv_layer, req_to_token, b_req_idx, cu_q, b_ready_len, Hq,
                               Hkv, D, sm_scale)
    _req_bf16(q, kv_layer)
    T = q.shape[0]
    B = b_req_idx.shape[0]
    assert q.stride(-1) == 1 and kv_layer.is_contiguous()
    assert cu_q.dtype == torch.int32 and b_ready_len.dtype == torch.int32
    scale = sm_scale if sm_scale is not None else 1.0 / math.sqrt(D)
    if out is None:
        out = torch.empty((T, Hq, D), dtype=q.dtype, device=q.device)
    check(kernels().llb_gqa_prefill(ptr(q), i64(q.stride(0)), ptr(kv_layer), ptr(req_to_token),
                                    i64(req_to_token.stride(0)), ptr(b_req_idx), ptr(cu_q), ptr(b_ready_len),
                                    ptr(out), i64(out.stride(0)), c_int(B), c_int(max_q_len), c_int(Hq), c_int(Hkv),
                                    c_int(D), f32(scale), stream()), "gqa_prefill")
    _count()
    return out


# --------------------------------------------------------------------------------------
def decode_prologue(req_to_token, next_token, b_req_idx, b_seq_len, new_slot, ids_out=None, pos_out=None):
    """ids[b] = next_token[req]; pos[b] = seq_len-1; req_to_token[req, seq_len-1] = new_slot[b]."""
    B = b_req_idx.shape[0]
    dev = b_req_idx.device
    if ids_out is None:
        ids_out = torch.empty(B, dtype=torch.int64, device=dev)
    if pos_out is None:
        pos_out = torch.empty(B, dtype=torch.int32, device=dev)
    if not b_req_idx.is_cuda:
        r = b_req_idx.long()
        ids_out.copy_(next_token[r, 0] if next_token.dim() == 2 else next_token[r])
        pos_out.copy_(b_seq_len - 1)
        req_to_token[r, (b_seq_len - 1).long()] = new_slot
        return ids_out, pos_out
    nt_stride = next_token.stride(0)
    check(kernels().llb_decode_prologue(ptr(ids_out), ptr(pos_out), ptr(req_to_token), ptr(next_token),
                                        ptr(b_req_idx), ptr(b_seq_len), ptr(new_slot), c_int(B),
                                        i64(req_to_token.stride(0)), c_int(nt_stride), stream()), "decode_prologue")
    _count()
    return ids_out, pos_out


def prefill_prologue(req_to_token, b_req_idx, b_ready_len, cu_q, new_slot, total_tokens: int):
    """positions / batch index of every new token and the slot table update, one launch."""
    dev = b_req_idx.device
    pos = torch.empty(total_tokens, dtype=torch.int32, device=dev)
    batch_of = torch.empty(total_tokens, dtype=torch.int32, device=dev)
    B = b_req_idx.shape[0]
    if not b_req_idx.is_cuda:
        for b in range(B):
            s, e = int(cu_q[b]), int(cu_q[b + 1])
            r = int(b_ready_len[b])
            pos[s:e] = torch.arange(r, r + e - s, dtype=torch.int32)
            batch_of[s:e] = b
            req_to_token[int(b_req_idx[b]), r:r + e - s] = new_slot[s:e]
        return pos, batch_of
    check(kernels().llb_prefill_prologue(ptr(pos), ptr(batch_of), ptr(req_to_token), ptr(b_req_idx), ptr(b_ready_len),
                                         ptr(cu_q), ptr(new_slot), c_int(B), i64(req_to_token.stride(0)), stream()),
          "prefill_prologue")
    _count()
    return pos, batch_of


def scatter_next_token_(next_token, sampled, b_req_idx, has_out=None):
    if not sampled.is_cuda:
        r = b_req_idx.long()
        if has_out is not None:
            m = has_out.bool()
            r, sampled = r[m], sampled[m]
        if next_token.dim() == 2:
            next_token[r, 0] = sampled
        else:
            next_token[r] = sampled
        return next_token
    B = sampled.shape[0]
    check(kernels().llb_scatter_next_token(ptr(next_token), ptr(sampled), ptr(b_req_idx), ptr(has_out), c_int(B),
                                           c_int(next_token.stride(0)), stream()), "scatter_next_token")
    _count()
    return next_token


def copy_rows(dst, src, dst_idx=None, src_idx=None, n_rows: Optional[int] = None):
    """dst[dst_idx[i]] = src[src_idx[i]] over rows (first dim); pinned host tensors allowed on either side."""
    if n_rows is None:
        n_rows = (dst_idx if dst_idx is not None else src_idx if src_idx is not None else src).shape[0]
    on_gpu = dst.is_cuda or src.is_cuda
    if not on_gpu:
        di = dst_idx.long() if dst_idx is not None else torch.arange(n_rows)
        si = src_idx.long() if src_idx is not None else torch.arange(n_rows)
        dst[di] = src[si]
        return dst
    row_bytes = src[0].numel() * src.element_size()
    check(kernels().llb_copy_rows(ptr(dst), ptr(src), ptr(dst_idx), ptr(src_idx), c_int(n_rows), i64(row_bytes),
                                  i64(dst.stride(0) * dst.element_size()), i64(src.stride(0) * src.element_size()),
                                  stream()), "copy_rows")
    _count()
    return dst


# --------------------------------------------------------------------------------------
def apply_penalty_(logits, presence, frequency, repetition, cu, tok_ids, tok_cnt, mask_cu=None, mask_ids=None):
    if not logits.is_cuda:
        return ref.apply_penalty_(logits, presence, frequency, repetition, cu, tok_ids, tok_cnt, mask_cu, mask_ids)
    assert logits.dtype == torch.float32
    B, V = logits.shape
    check(kernels().llb_apply_penalty(ptr(logits), i64(logits.stride(0)), ptr(presence), ptr(frequency),
                                      ptr(repetition), ptr(cu), ptr(tok_ids), ptr(tok_cnt), ptr(mask_cu),
                                      ptr(mask_ids), c_int(B), c_int(V), stream()), "apply_penalty")
    _count()
    return logits


def greedy_partials(logits, idx_off: int = 0):
    """First pass of the all-greedy sampler over (a vocabulary shard of) the logits: [B, S, 3] fp32 rows of
    (max, arg-max as global token id bits, sum exp(x - max)).  S depends on B and the shard width only."""
    B, V = logits.shape
    splits = max(1, min(64, 2368 // max(B, 1), V // 2048))
    if not logits.is_cuda:
        return ref.greedy_partials(logits, idx_off, splits)
    dt = {torch.float32: 0, torch.bfloat16: 1}[logits.dtype]
    part = torch.empty((B, splits, 3), dtype=torch.float32, device=logits.device)
    check(kernels().llb_greedy_partial(ptr(logits), c_int(dt), i64(logits.stride(0)), c_int(B), c_int(V),
                                       c_int(idx_off), ptr(part), c_int(splits), stream()), "greedy_partial")
    _count()
    return part


def greedy_merge(parts):
    """parts [R, B, S, 3] (the partials of R vocabulary shards) -> (ids int64 [B], logprob fp32 [B])."""
    R, B, S, _ = parts.shape
    if not parts.is_cuda:
        return ref.greedy_merge(parts)
    parts = parts.contiguous()
    ids = torch.empty(B, dtype=torch.int64, device=parts.device)
    lp = torch.empty(B, dtype=torch.float32, device=parts.device)
    check(kernels().llb_greedy_merge(ptr(parts), c_int(B), c_int(S), c_int(R), ptr(ids), ptr(lp), stream()),
          "greedy_merge")
    _count()
    return ids, lp


def sample(logits, temperature=None, top_p=None, top_k=None, seeds=None, steps=None, want_logprob=True):
    """Returns (ids int64 [B], logprob fp32 [B]).  Rows with top_k == 1 (or top_k None) are greedy.
    `logits` may be vocabulary-parallel (`common.infer_state.ShardedLogits`): an all-greedy batch is then
    sampled from the shards (a few KB exchanged per step), anything else from the gathered matrix."""
    if hasattr(logits, "greedy"):
        if temperature is None and top_k is None and top_p is None:
            return logits.greedy()
        logits = logits.full()
    if not logits.is_cuda:
        return ref.sample(logits, temperature, top_p, top_k, seeds, steps)
    B, V = logits.shape
    dt = {torch.float32: 0, torch.bfloat16: 1}[logits.dtype]
    ids = torch.empty(B, dtype=torch.int64, device=logits.device)
    lp = torch.empty(B, dtype=torch.float32, device=logits.device) if want_logprob else None
    if temperature is None and top_k is None and top_p is None:  # every row greedy: many CTAs per row
        splits = max(1, min(64, 2368 // B, V // 2048))
        scratch = torch.empty(B * splits * 3, dtype=torch.float32, device=logits.device)
        check(kernels().llb_sample_greedy(ptr(logits), c_int(dt), i64(logits.stride(0)), c_int(B), c_int(V), ptr(scratch),
                                          c_int(splits), ptr(ids), ptr(lp), stream()), "sample_greedy")
        _count(2)
        return ids, lp
    if seeds is not None:
        assert seeds.dtype == torch.int64
    check(kernels().llb_sample(ptr(logits), c_int(dt), i64(logits.stride(0)), c_int(B), c_int(V), ptr(temperature),
                               ptr(top_p), ptr(top_k), ptr(seeds), ptr(steps), ptr(ids), ptr(lp), stream()), "sample")
    _count()
    return ids, lp


def token_logprob(logits, ids):
    if not logits.is_cuda:
        return ref.token_logprob(logits, ids)
    B, V = logits.shape
    dt = {torch.float32: 0, torch.bfloat16: 1}[logits.dtype]
    out = torch.empty(B, dtype=torch.float32, device=logits.device)
    check(kernels().llb_token_logprob(ptr(logits), c_int(dt), i64(logits.stride(0)), c_int(B), c_int(V), ptr(ids),
                                      ptr(out), stream()), "token_logprob")
    _count()
    return out


# --------------------------------------------------------------------------------------
def layernorm(x, w, b, eps: float, residual=None):
    """LayerNorm(x [+ residual]) * w + b; with `residual` the sum is written back into it (in place)."""
    if not _is_cuda(x):
        return ref.layernorm(x, w, b, eps, residual)
    _req_bf16(x, w)
    assert x.is_contiguous() and (residual is None or residual.is_contiguous())
    T, H = x.shape
    out = torch.empty_like(x)
    check(kernels().llb_layernorm(ptr(out), ptr(residual), ptr(x), ptr(w), ptr(b), c_int(T), c_int(H), f32(eps),
                                  stream()), "layernorm")
    _count()
    return out


def act_(x, kind: str, alpha: float = 1.0):
    """In-place activation (silu | gelu | gelu_tanh | relu) or scaling (kind "scale", factor alpha)."""
    if not _is_cuda(x):
        return ref.act_(x, kind, alpha)
    _req_bf16(x)
    assert x.is_contiguous()
    check(kernels().llb_act_(ptr(x), i64(x.numel()), c_int(ref.ACT_KINDS[kind]), f32(alpha), stream()), "act")
    _count()
    return x


def attention_generic(q, kv_layer, req_to_token, b_req_idx, pos, batch_of, Hq, Hkv, D, sm_scale, window: int = 0,
                      softcap: float = 0.0, alibi=None, sinks=None):
    """Causal paged attention for any head size <= 256 with sliding window / ALiBi / soft-cap / sinks.
    q [T, Hq*D] or [T, Hq, D]; returns [T, Hq, D]."""
    T = q.shape[0]
    if isinstance(kv_layer, kv_quant.QuantKVLayer):
        return kv_quant.attention_generic(q, kv_layer, req_to_token, b_req_idx, pos, batch_of, Hq, Hkv, D, sm_scale,
                                          window, softcap, alibi, sinks)
    if not _is_cuda(q):
        return ref.attention_generic(q.reshape(T, Hq, D), kv_layer, req_to_token, b_req_idx, pos, batch_of, Hq, Hkv, D,
                                     sm_scale, window, softcap, alibi, sinks)
    _req_bf16(q, kv_layer)
    assert q.stride(-1) == 1 and kv_layer.is_contiguous() and pos.dtype == torch.int32
    out = torch.empty((T, Hq, D), dtype=q.dtype, device=q.device)
    check(kernels().llb_attn_generic(ptr(q), i64(q.stride(0)), ptr(kv_layer), ptr(req_to_token),
                                     i64(req_to_token.stride(0)), ptr(b_req_idx), ptr(pos), ptr(batch_of), ptr(out),
                                     i64(out.stride(0)), c_int(T), c_int(Hq), c_int(Hkv), c_int(D), f32(sm_scale),
                                     c_int(window), f32(softcap), ptr(alibi), ptr(sinks), stream()), "attn_generic")
    _count()
    return out


# --------------------------------------------------------------------------------------
class DytNorm:
    """Dynamic-tanh norm: tanh(alpha * v) * w + b, elementwise, in fp32.  `alpha` is a host number."""

    __slots__ = ("w", "b", "alpha")

    def __init__(self, w: torch.Tensor, b: torch.Tensor, alpha: float):
        self.w, self.b, self.alpha = w.float().contiguous(), b.float().contiguous(), float(alpha)


def embedding_dyt(ids, table, norm: DytNorm):
    """(x, h): x = the table's rows as the fp32 residual stream, h = norm(x) in the table's number format."""
    if not _is_cuda(table):
        x = table[ids].float()
        return x, ref.dyt(x, norm).to(table.dtype)
    T, W = ids.shape[0], table.shape[1]
    x = torch.empty((T, W), dtype=torch.float32, device=table.device)
    h = torch.empty((T, W), dtype=table.dtype, device=table.device)
    assert ids.dtype == torch.int64 and ids.is_contiguous() and table.is_contiguous()
    check(kernels().llb_embedding_dyt(ptr(ids), ptr(table), c_int(DTYPE_CODES[table.dtype]), i64(table.shape[0]), ptr(x),
                                      ptr(h), c_int(T), c_int(W), *_dyt_args(norm), stream()), "embedding_dyt")
    _count()
    return x, h


def dyt(x, norm: DytNorm, dtype):
    """norm(x) of the fp32 stream x [T, W], in `dtype`."""
    if not _is_cuda(x):
        return ref.dyt(x, norm).to(dtype)
    assert x.dtype == torch.float32 and x.is_contiguous()
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    check(kernels().llb_dyt(ptr(x), ptr(h), c_int(DTYPE_CODES[dtype]), c_int(x.shape[0]), c_int(x.shape[1]),
                            *_dyt_args(norm), stream()), "dyt")
    _count()
    return h


def add_dyt_(x, y, post: DytNorm, nxt: DytNorm, dtype):
    """x += post(y) in place (fp32 stream); returns nxt(x) in `dtype`."""
    if not _is_cuda(x):
        x.add_(ref.dyt(y.float(), post))
        return ref.dyt(x, nxt).to(dtype)
    assert x.dtype == torch.float32 and x.is_contiguous() and y.is_contiguous() and x.shape == y.shape
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    check(kernels().llb_add_dyt(ptr(x), ptr(y), c_int(DTYPE_CODES[y.dtype]), ptr(h), c_int(DTYPE_CODES[dtype]),
                                c_int(x.shape[0]), c_int(x.shape[1]), *_dyt_args(post), *_dyt_args(nxt), stream()),
          "add_dyt")
    _count()
    return h


# --------------------------------------------------------------------------------------
class BigramTable:
    """Second embedding table, looked up by the pair (previous token, token): row (prev * mul_prev + token * mul_cur) mod
    buckets of `table` [buckets + 1, W], the last row for a sequence's first token.  `slot_token` (int32, one entry per
    pool slot) keeps the token id behind every cached position, so the previous token of a later pass is found through the
    request table like its keys."""

    def __init__(self, table: torch.Tensor, buckets: int, mul_prev: int, mul_cur: int):
        assert table.shape[0] == buckets + 1
        self.table, self.buckets, self.mul_prev, self.mul_cur = table, int(buckets), int(mul_prev), int(mul_cur)
        self.slot_token = None


def embedding_pair(ids, table, bigram, req_to_token, b_req_idx, pos, batch_of, mem_index, norm=None):
    """(x, h): x = the table's rows (+ the bigram table's) as the fp32 residual stream, h = x in the table's format, or
    rms(x) * w of the first `width` columns with norm = (w, width, eps).  batch_of None: row t is the one token of request t."""
    if not _is_cuda(table):
        x = table[ids].float()
        if bigram is not None:
            x = x + ref.bigram_rows(ids, bigram, req_to_token, b_req_idx, pos, batch_of, mem_index).float()
        return x, (x if norm is None else ref.rms_over(x, *norm[1:]) * norm[0]).to(table.dtype)
    T, W = ids.shape[0], table.shape[1]
    x = torch.empty((T, W), dtype=torch.float32, device=table.device)
    h = torch.empty((T, W), dtype=table.dtype, device=table.device)
    assert ids.dtype == torch.int64 and ids.is_contiguous() and table.is_contiguous()
    g = bigram
    nw, width, eps = norm if norm is not None else (None, W, 1.0)
    check(kernels().llb_embedding_pair(ptr(ids), ptr(table), c_int(DTYPE_CODES[table.dtype]), i64(table.shape[0]),
                                       ptr(g.table if g else None), i64(g.buckets if g else 1),
                                       i64(g.mul_prev if g else 0), i64(g.mul_cur if g else 0),
                                       ptr(g.slot_token if g else None), ptr(mem_index), ptr(pos), ptr(batch_of),
                                       ptr(b_req_idx), ptr(req_to_token), i64(req_to_token.stride(0)), ptr(x), ptr(h),
                                       c_int(T), c_int(W), ptr(nw), c_int(width), f32(eps), stream()), "embedding_pair")
    _count()
    return x, h


def add_rms_(x, y, w, width: int, eps: float, dtype, next_w=None):
    """x += rms(y) * w in place (fp32 stream, the mean taken over the first `width` columns; w None: x += y); returns x, or
    rms(x) * next_w, in `dtype`."""
    if not _is_cuda(x):
        return ref.add_rms_(x, y, w, width, eps, dtype, next_w)
    assert x.dtype == torch.float32 and x.is_contiguous() and y.is_contiguous() and x.shape == y.shape
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    check(kernels().llb_add_rms(ptr(y), c_int(DTYPE_CODES[y.dtype]), ptr(x), ptr(h), c_int(DTYPE_CODES[dtype]), ptr(w),
                                ptr(next_w), c_int(x.shape[0]), c_int(width), c_int(x.shape[1]), f32(eps), stream()),
          "add_rms")
    _count()
    return h


class TokenShift:
    """Shift of a norm's output towards the row of the token before (`norm_shift`): h = n + (n_before - n) * mu, element by element;
    mu fp32 [W]; state fp32 [slots, W] (any row pitch) keeps the n of every request's last token."""

    def __init__(self, mu, state, st):
        self.mu, self.state, self.st = mu, state, st


def norm_shift(x, y, w, width: int, eps: float, dtype, shift=None, ids=None, centred=True):
    """(x', h): x' = x + y (fp32 stream; x None: y; ids given: y is a table and row t is y[ids[t]]), h = norm(x') * w in `dtype`, the
    statistics taken over the first `width` columns (centred: layer norm without a bias, else RMS norm), moved by `shift`
    (`TokenShift` or None).  x may be changed in place."""
    if not _is_cuda(y):
        return ref.norm_shift(x, y, w, width, eps, dtype, shift, ids, centred)
    T = y.shape[0] if ids is None else ids.shape[0]
    W = y.shape[1]
    prompt = shift is not None and shift.st.is_prefill
    assert y.is_contiguous() and (x is None or x.is_contiguous() and x.dtype == torch.float32 and x.shape == (T, W))
    assert ids is None or ids.dtype == torch.int64 and ids.is_contiguous()
    out = x if x is not None and not prompt else torch.empty((T, W), dtype=torch.float32, device=y.device)
    h = torch.empty((T, W), dtype=dtype, device=y.device)
    mu = state = req = cu = first = batch = None
    if shift is not None:
        st, mu, state = shift.st, shift.mu, shift.state
        assert state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] == W
        req, first = st.b_req_idx, st.b_ready_cache_len if prompt else st.seq_pos
        cu, batch = (st.cu_q, st.batch_of_token) if prompt else (None, None)
    check(kernels().llb_norm_shift(ptr(y), c_int(DTYPE_CODES[y.dtype]), ptr(ids), i64(y.shape[0]), ptr(x), ptr(out), ptr(h),
                                   c_int(DTYPE_CODES[dtype]), ptr(w), c_int(T), c_int(width), c_int(W), c_int(int(centred)),
                                   f32(eps), ptr(mu), ptr(state), i64(state.stride(0) if state is not None else 0), ptr(req),
                                   ptr(cu), ptr(first), ptr(batch), stream()), "norm_shift")
    _count()
    return out, h


def qk_norm_rope_scatter_(qkv, kv_layer, cos, sin, pos, slot, q_w, k_w, eps, Hq, Hkv, D, dim, DV, rot_dim, norm=True, q_scale=None):
    """Rows [Hq * D | Hkv * D | Hkv * DV] of qkv: RMS norm of every q and k head over its first `dim` elements (weights
    q_w, k_w fp32 [D], None: ones), rotation of the first rot_dim, q in place, K and V to kv_layer[slot] ([slots, Hkv * (D + DV)]).
    Hkv = 0: queries only.  Without weights, norm and rotation may be read in either order.  norm False: no norm.  q_scale (fp32
    [Hq] or None): a factor per query head."""
    if not _is_cuda(qkv):
        return ref.qk_norm_rope_scatter_(qkv, kv_layer, cos, sin, pos, slot, q_w, k_w, eps, Hq, Hkv, D, dim, DV, rot_dim,
                                          norm, q_scale)
    assert qkv.stride(1) == 1 and (Hkv == 0 or kv_layer.is_contiguous() and qkv.dtype == kv_layer.dtype)
    check(kernels().llb_qk_norm_rope_scatter(ptr(qkv), c_int(DTYPE_CODES[qkv.dtype]), i64(qkv.stride(0)), ptr(kv_layer),
                                             ptr(cos), ptr(sin), ptr(pos), ptr(slot), ptr(q_w), ptr(k_w), f32(eps),
                                             c_int(int(norm)), ptr(q_scale), c_int(qkv.shape[0]), c_int(Hq), c_int(Hkv), c_int(D), c_int(dim), c_int(DV),
                                             c_int(rot_dim), stream()), "qk_norm_rope_scatter")
    _count()
    return qkv


def rope_heads_(x, cos, sin, pos, H, pitch, off, dims, neighbours=True):
    """Rotary positions on columns off .. off + dims of every head of x [T, >= H * pitch] (heads `pitch` apart), in place: pairs
    of neighbours (2 i, 2 i + 1), or of halves (i, i + dims / 2).  cos, sin [positions, dims / 2] fp32."""
    if dims == 0:
        return x
    if not _is_cuda(x):
        v = x[:, : H * pitch].reshape(-1, H, pitch)
        v[..., off:off + dims] = ref.rotate_pairs(v[..., off:off + dims].float(), cos, sin, pos, neighbours).to(x.dtype)
        x[:, : H * pitch] = v.reshape(-1, H * pitch)
        return x
    assert x.stride(1) == 1 and pos.dtype == torch.int32 and cos.shape[-1] == dims // 2
    check(kernels().llb_rope_heads(ptr(x), c_int(DTYPE_CODES[x.dtype]), i64(x.stride(0)), ptr(cos), ptr(sin), ptr(pos),
                                   c_int(x.shape[0]), c_int(H), c_int(pitch), c_int(off), c_int(dims),
                                   c_int(1 if neighbours else 0), stream()), "rope_heads")
    _count()
    return x


def sigmoid_mul_(x, gate):
    """x *= sigmoid(gate) element by element, both [T, N] with rows of any pitch."""
    if not _is_cuda(x):
        return x.copy_(x.float() * torch.sigmoid(gate.float()))
    assert x.stride(1) == 1 and gate.stride(1) == 1 and x.shape == gate.shape and x.dtype == gate.dtype
    check(kernels().llb_sigmoid_mul(ptr(x), c_int(DTYPE_CODES[x.dtype]), i64(x.stride(0)), ptr(gate), i64(gate.stride(0)),
                                    c_int(x.shape[0]), c_int(x.shape[1]), stream()), "sigmoid_mul")
    _count()
    return x


def window_decode_splits(T: int, Hq: int, Hkv: int, keys: int) -> int:
    """Shares the keys of a decode step are cut into: about two CTAs per SM (more measured slower), at least 256 keys each."""
    ctas = T * Hkv * -(-(Hq // Hkv) // 16)
    return max(1, min(296 // ctas, -(-keys // 256), 64))


_WINDOW_SIZES = (64, 128, 192, 256)   # head sizes of the tensor-core kernels


class DistanceBias:
    """Learned bias per head and bucket of the distance n between query and key.  With B rows in the table: bucket n for
    n < B / 2, beyond that B / 2 buckets spaced by logarithm up to the distance `far`, the last one for all from there on.
    Kept as `rel` [heads, far + 1] fp32: the bias of every distance up to `far`, rows that may be read PAD places further on
    either side."""

    PAD = 64

    def __init__(self, table: torch.Tensor, far: int):
        B, half = table.shape[0], table.shape[0] // 2
        assert half >= 1 and far > half, "distance bias: the far distance lies beyond half of the buckets"
        step = math.log(far / half)
        rows = [n if n < half else min(B - 1, half + math.floor(math.log(n / half) / step * (B - half)))
                for n in range(far + 1)]
        rows = [rows[0]] * self.PAD + rows + [rows[-1]] * self.PAD
        self.far = int(far)
        self.rel = table.float()[torch.tensor(rows, device=table.device)].t().contiguous()[:, self.PAD:self.PAD + far + 1]


def window_attention(q, kv_layer, req_to_token, st, Hq, Hkv, D, DV, sm_scale, window, gate=None, out_scale=1.0, out=None,
                     keep=0, bias=None, chunk=0, softcap=0.0):
    """Causal paged attention with key size D and value size DV through a sliding window (0: none) for the pass `st`
    (InferState); the first `keep` positions are seen through any window.  chunk > 0, instead of a window: only positions of the
    query's own chunk (of `chunk` positions, counted from 0).  q [T, >= Hq * D]; softcap > 0: scaled scores s become
    softcap * tanh(s / softcap); bias (`DistanceBias` or None) is added to them; gate [T, Hq] (or None): head h is multiplied by
    sigmoid(gate[:, h]), gate [T, Hq * DV]: element by element; all heads by out_scale.  Returns out [T, Hq * DV]."""
    assert not (window and chunk)
    T = q.shape[0]
    if out is None:
        out = torch.empty((T, Hq * DV), dtype=q.dtype, device=q.device)
    if not _is_cuda(q):
        return ref.window_attention(q, kv_layer, req_to_token, st.b_req_idx, st.seq_pos,
                                    st.batch_of_token if st.is_prefill else None, Hq, Hkv, D, DV, sm_scale, window, gate,
                                    out_scale, out, keep, bias, chunk, softcap)
    assert q.stride(1) == 1 and kv_layer.is_contiguous() and out.stride(1) == 1
    gs, elem = (0, 0) if gate is None else (gate.stride(0), int(gate.shape[1] != Hq))
    assert not elem or gate.shape[1] == Hq * DV
    rel, far, stride = (bias.rel, bias.far, bias.rel.stride(0)) if bias is not None else (None, 0, 0)
    tail = (f32(sm_scale), c_int(window), c_int(keep), ptr(rel), c_int(far), i64(stride), c_int(chunk), f32(softcap), ptr(gate),
            i64(gs), c_int(elem), f32(out_scale), stream())
    if q.dtype == torch.bfloat16 and D in _WINDOW_SIZES and DV % 64 == 0 and sm_scale > 0:
        common = (ptr(q), i64(q.stride(0)), ptr(kv_layer), ptr(req_to_token), i64(req_to_token.stride(0)),
                  ptr(st.b_req_idx))
        if st.is_prefill:
            check(kernels().llb_window_gqa_prefill_tc(*common, ptr(st.cu_q), ptr(st.b_ready_cache_len), ptr(out),
                                                      i64(out.stride(0)), c_int(st.batch_size), c_int(st.max_q_len),
                                                      c_int(Hq), c_int(Hkv), c_int(D), c_int(DV), *tail),
                  "window_gqa_prefill_tc")
            _count()
            return out
        if DV in _WINDOW_SIZES:
            reach = window or chunk
            keys = min(reach + keep, st.max_kv_len) if reach > 0 else st.max_kv_len
            n = window_decode_splits(T, Hq, Hkv, keys)
            po = pl = None
            if n > 1:
                po = torch.empty(T * Hq * n * DV, dtype=torch.float32, device=q.device)
                pl = torch.empty(T * Hq * n, dtype=torch.float32, device=q.device)
            check(kernels().llb_window_gqa_decode(*common, ptr(st.b_seq_len), ptr(out), i64(out.stride(0)), ptr(po), ptr(pl),
                                                  c_int(T), c_int(Hq), c_int(Hkv), c_int(D), c_int(DV), c_int(n), *tail),
                  "window_gqa_decode")
            _count(2 if n > 1 else 1)
            return out
    check(kernels().llb_attn_generic_kv(ptr(q), c_int(DTYPE_CODES[q.dtype]), i64(q.stride(0)), ptr(kv_layer),
                                        ptr(req_to_token), i64(req_to_token.stride(0)), ptr(st.b_req_idx),
                                        ptr(st.seq_pos), ptr(st.batch_of_token if st.is_prefill else None), ptr(out),
                                        i64(out.stride(0)), c_int(T), c_int(Hq), c_int(Hkv), c_int(D), c_int(DV), *tail),
          "attn_generic_kv")
    _count()
    return out
