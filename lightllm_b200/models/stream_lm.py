"""Base of the families whose residual stream is fp32 and whose layers have sizes of their own (`layers` in config.json): what
they share in loading weights, in the forward pass and in what they refuse.

Sizes that kernels cannot take are padded with zeros when the weights are loaded; `hidden_p` is the padded width."""
from __future__ import annotations

import torch

from .. import ops
from ..common.infer_state import InferState, ShardedLogits
from ..common.mem_manager import LayeredKVMemoryManager
from ..ops import reference as ref
from .base import TransformerLM
from .weights import get_shaped, tp_range
from .weights import pad_zeros as _pad
from .weights import round_up as _up

ACT_ALPHA = 1.702          # slope of the clamped gate of the experts


class StreamLM(TransformerLM):
    supports_float32 = True
    stream_tap = None          # fn(layer, stream): sees the residual stream after every layer (tests)
    logit_softcap = 0.0        # > 0: logits are softcap * tanh(logits / softcap)

    def _check_options(self):
        """Refuses what these families do not have.  Expects `self.specs` with `moe` and `top`."""
        name = self.model_type
        self.ep = bool(self.extra.get("enable_ep_moe", False))
        if self.quant_cfg.any_fp8:
            raise ValueError(f"{name}: weights run in bf16 or fp32 only (--quant_type none)")
        if self.ep and self.ps.dp_size > 1:
            raise ValueError(f"{name}: expert parallelism works inside a tensor-parallel group, not with --dp > 1")
        if self.extra.get("enable_return_routed_experts") and len({s.top for s in self.specs if s.moe}) > 1:
            raise ValueError(f"{name}: returned routed experts need the same number of experts in every layer")

    # ------------------------------------------------------------------ weights
    def _heads(self, src, name, heads, size, padded, h0, h1):
        """Rows of heads h0 .. h1 of a per-head projection, every head padded to `padded` rows: [n * padded, hidden_p]."""
        w = get_shaped(src, name, heads * size, self.hidden).view(heads, size, self.hidden)[h0:h1]
        return _pad(w, h1 - h0, padded, self.hidden_p).reshape(-1, self.hidden_p)

    def _out_heads(self, src, name, heads, size, padded, h0, h1):
        """Columns of heads h0 .. h1 of an output projection, every head padded: [hidden_p, n * padded]."""
        o = get_shaped(src, name, self.hidden, heads * size).view(self.hidden, heads, size)[:, h0:h1]
        return _pad(o, self.hidden_p, h1 - h0, padded).reshape(self.hidden_p, -1)

    def _narrow(self, w, rows, multiple=8):
        """Rows of a narrow projection, padded to a multiple of 8 rows."""
        return _pad(w, _up(rows, multiple), self.hidden_p)

    def _vec(self, t, *sizes):
        return self._dev(_pad(t.float(), *sizes), torch.float32)

    def _load_gated(self, src, p, ff, i0, i1):
        """(gate | up interleaved [2I, width], down [width, I]) of the columns i0 .. i1 of a feed-forward, padded."""
        W, P, I = self.hidden, self.hidden_p, _up(i1 - i0, 64)
        g, u = (_pad(get_shaped(src, p + n, ff, W)[i0:i1], I, P) for n in ("gate", "up"))
        return ref.interleave_gate_up(g, u), _pad(get_shaped(src, p + "down", W, ff)[:, i0:i1], P, I)

    def _load_experts(self, lw, src, p, experts, ff):
        """Experts stacked as in `models/moe.py`; returns the range of this rank's experts."""
        tp, r = self.tp.size, self.tp.rank
        if self.ep and tp > 1:
            (e0, e1), (i0, i1) = tp_range(experts, r, tp), (0, ff)
        else:
            (e0, e1), (i0, i1) = (0, experts), tp_range(ff, r, tp)
        mats = [self._load_gated(src, f"{p}e{e}.", ff, i0, i1) for e in range(e0, e1)]
        lw.w13 = self._dev(torch.stack([a for a, _ in mats]))
        lw.w2 = self._dev(torch.stack([b for _, b in mats]))
        lw.e0 = e0
        return e0, e1

    def _load_embed_and_head(self, src):
        W, P = self.hidden, self.hidden_p
        self.embed_w = self._dev(_pad(get_shaped(src, "embed", self.vocab, W), self.vocab, P))
        self.embed_range = (0, self.vocab)
        v0, v1 = tp_range(self.vocab, self.tp.rank, self.tp.size)
        self.lm_head_w = self._dev(_pad(get_shaped(src, "head", self.vocab, W)[v0:v1], _up(v1 - v0, 8), P))
        self.final_norm_w = None

    # ------------------------------------------------------------------ memory (families with rows per layer)
    def _kv_rows(self):
        raise NotImplementedError

    def kv_bytes_per_token(self):
        return LayeredKVMemoryManager.bytes_per_token(self.dtype, self._kv_rows())

    def _make_mem_manager(self, size):
        if self.extra.get("kv_type") not in (None, "none", "None"):
            raise ValueError("--llm_kv_type: the layers' caches have no quantised form here")
        return LayeredKVMemoryManager(size, self.dtype, self._kv_rows(), self.device)

    # ------------------------------------------------------------------ forward
    def _make_decode_state(self, B, b_req_idx, b_seq_len, mem_index, max_kv_len, num_splits=None):
        return InferState(is_prefill=False, batch_size=B, num_tokens=B, max_kv_len=max_kv_len, max_q_len=1,
                          b_req_idx=b_req_idx, b_seq_len=b_seq_len, mem_index=mem_index)

    def _graph_decode_splits(self, bucket):
        return 1        # per layer, from its window (ops.window_attention, ops.mla.latent_attention)

    def _reduced(self, a, w, bias=None):
        """a . w^T (+ bias, of one rank), summed over the tensor-parallel ranks."""
        if self.tp.size == 1:
            return ops.gemm(a, w, bias=bias)
        y = ops.gemm(a, w, epi="f32", bias=bias)
        self.tp.all_reduce_(y)
        return y

    def _lm_head(self, h, normed: bool = True):
        assert normed, "the layer stack returns normalised rows"
        v = self.vocab // self.tp.size
        logits = ops.gemm(h, self.lm_head_w, epi="f32", softcap=self.logit_softcap)[:, :v]
        if self.tp.size == 1:
            return logits
        return ShardedLogits(logits.contiguous(), self.tp, self.tp.rank * v, self.vocab)
