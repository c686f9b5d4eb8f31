"""Heads of latent attention over a pool of latents (`ops.mla`), in the form that a pass makes cheaper:

  absorbed   queries are taken into the latent space and read every pool row once for all heads (decode, short portions)
  expanded   keys and values of every head are formed for the positions a prompt pass can see (longer prompts, bf16)

A pool row is [latent, padded to rp | rotated key part] of `keys` values; a query head is [unrotated | rotated], padded to dp.
Both forms treat the rotated part as further latent columns: the up-projections copy it with an identity block."""
from __future__ import annotations

import torch

from .. import ops
from ..common.infer_state import InferState
from ..ops import mla as mla_ops
from .weights import pad_zeros, round_up


class LatentHeads:
    def __init__(self, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, scale: float, window: int):
        self.heads, self.dim, self.rot_dim, self.rank = heads, dim, rot_dim, rank
        self.scale, self.window = scale, window
        self.rp, self.dp, self.vp = round_up(rank, 16), round_up(dim + rot_dim, 64), round_up(vdim, 64)
        self.rot_pad = round_up(rot_dim, 16)
        self.keys = self.rp + self.rot_pad

    def load(self, lw, dev, uk, uv):
        """uk [heads, dim, rank], uv [heads, vdim, rank]: up-projections of the unrotated keys and of the values, in the forms that
        `attend` finds in the layer's weights lw; dev: moves a tensor to the model's device and number format."""
        n = self.heads
        k = pad_zeros(uk, n, self.dp, self.keys)
        if self.rot_dim:
            i = torch.arange(self.rot_dim)
            k[:, self.dim + i, self.rp + i] = 1
        v = pad_zeros(uv, n, self.vp, self.keys)
        lw.w_uk_t = dev(k.transpose(1, 2))                                                   # q -> q_lat
        lw.w_ukv = dev(torch.cat([k.reshape(n * self.dp, -1), v.reshape(n * self.vp, -1)]))  # pool row -> k | v
        lw.w_uv = dev(v[..., : self.rp])                                                     # o_lat -> o

    def attend(self, lw, q, kv_layer, r2t, st: InferState, gate=None):
        """q [T, heads * dp], rotated; gate [T, heads * vp] or None: the result times sigmoid(gate).  Returns [T, heads * vp]."""
        T, n = q.shape[0], self.heads
        kr = self._expanded_range(q, st) if st.is_prefill else None
        if kr is not None:
            c = mla_ops.latent_gather(kv_layer, r2t, st.b_req_idx, kr)
            kv = ops.gemm(c[:, : self.keys], lw.w_ukv)           # [rows, heads * dp | heads * vp]
            return mla_ops.window_prefill(q, kv, n, self.dp, self.vp, st.cu_q, st.b_ready_cache_len, kr, st.max_q_len,
                                          self.scale, gate)
        q_lat = mla_ops.gemm_batched(q.view(T, n, self.dp), lw.w_uk_t)
        o_lat = mla_ops.latent_attention(q_lat, kv_layer, r2t, st.b_req_idx, st.seq_pos,
                                         st.batch_of_token if st.is_prefill else None, self.scale, self.window,
                                         min(self.window or st.max_kv_len, st.max_kv_len), rank=self.rp)
        o = mla_ops.gemm_batched(o_lat, lw.w_uv).reshape(T, n * self.vp)
        return o if gate is None else ops.sigmoid_mul_(o, gate)

    def _expanded_range(self, q, st: InferState):
        """The positions to expand keys and values for when this prompt pass runs the expanded form, else None."""
        if not q.is_cuda or q.dtype != torch.bfloat16 or self.dp > 256 or self.vp > 128 or self.scale <= 0:
            return None
        cache = st.extra.setdefault("key_ranges", {})
        if self.window not in cache:
            q_len, ready = st.extra["q_len_cpu"].to(torch.int64), st.extra["ready_cpu"].to(torch.int64)
            seq = ready + q_len
            pairs = int((q_len * (seq.clamp_max(self.window) if self.window else seq)).sum())
            cache[self.window] = (mla_ops.KeyRange(ready, q_len, self.window, q.device), pairs)
        kr, pairs = cache[self.window]
        # multiply-adds per head; the absorbed kernel works on 16-row tiles of heads with mma.sync at about a quarter
        # of the tcgen05 rate
        expanded = kr.rows * self.keys * (self.dp + self.vp) + pairs * (self.dp + 2 * self.vp)
        absorbed = st.num_tokens * (self.keys * self.dp + self.rp * self.vp) + \
            4 * pairs * (self.keys + 2 * self.rp) * (round_up(self.heads, 16) / self.heads)
        return kr if expanded < absorbed else None
