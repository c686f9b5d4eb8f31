"""Katarax: three kinds of attention layers, each beside a mixture-of-experts feed-forward that reads the same input, around an
fp32 residual stream.

    stream = embed[token];  per layer: h = norm(stream), stream += mixer(h) + experts(h)   (a layer may have no experts)
    logits = cap * tanh(head . final(stream) / cap)

Mixers: "latent_attention" (queries and keys / values through latents, a rotated key part shared by the heads, sliding window,
output gate), "attention" (no rotation, a learned bias per distance, window with kept first tokens) and "attention_2" (rotation,
then unit query and key heads; may read another layer's keys and values).  Every layer has its own sizes and constants (`layers`
in config.json).  How it maps onto this package:

  * one GEMM gives every projection of a mixer; mixer and router read the same rows, and one pass adds the mixer's output and the
    weighted experts to the fp32 stream and writes the next layer's normalised input (`ops.moe.routed_experts_rms_`)
  * latents: `models/latent.py`; the pool row of a token is [latent | rotated key part]
  * other attention: paged keys and values with separate sizes; window, kept tokens and biases inside the attention kernels
    (`ops.window_attention`).  A norm without a weight commutes with a rotation: `ops.qk_norm_rope_scatter_` does both
  * a layer that reads another layer's cache projects queries only and has no pool rows of its own
  * experts: sigmoid scores, choice by corrected scores inside the best groups (`ops.moe.grouped_topk`), clamped gate

Sizes that kernels cannot take are padded with zeros when the weights are loaded (width, head sizes and feed-forward sizes to 64,
latents and the rotated part to 16, everything narrow to 8).
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..common.infer_state import InferState
from ..ops import mla as mla_ops
from ..ops import moe as moe_ops
from ..ops import reference as ref
from .base import LayerWeights
from .latent import LatentHeads
from .registry import register_config, register_model
from .stream_lm import ACT_ALPHA, StreamLM
from .weights import get_shaped, kv_head_range, tp_range
from .weights import pad_zeros as _pad
from .weights import round_up as _up

LATENT, BIASED, ROTATED = "latent_attention", "attention", "attention_2"


def _kv_row(kind: str, m: dict, kv_heads: int) -> int:
    """Elements of a layer's pool row (0: it reads another layer's)."""
    if kind == LATENT:
        return _up(m["kv_rank"], 16) + _up(m["rot_dim"], 16)
    return 0 if m.get("kv_from") is not None else kv_heads * (_up(m["dim"], 64) + _up(m["vdim"], 64))


@register_config("Katarax")
def normalize_katarax(cfg: dict) -> dict:
    """The keys the rest of the framework reads (HF spelling), next to the design's own."""
    layers = cfg["layers"]
    mix = [l["mixer"] for l in layers]
    moe = [l["mlp"]["router"] for l in layers if l.get("mlp")]
    out = dict(cfg, model_type="katarax", hidden_size=cfg["width"], vocab_size=cfg["vocab"], num_hidden_layers=len(layers),
               num_attention_heads=max(m["heads"] for m in mix),
               num_key_value_heads=max(m.get("kv_heads", 1) for m in mix),
               head_dim=max(m["dim"] + m.get("rot_dim", 0) for m in mix),
               kv_elems_per_token=sum(_kv_row(l["type"], l["mixer"], l["mixer"].get("kv_heads", 1)) for l in layers))
    if moe:
        out.update(num_experts=max(r["experts"] for r in moe), num_experts_per_tok=max(r["top"] for r in moe),
                   decoder_sparse_step=1, mlp_only_layers=[i for i, l in enumerate(layers) if not l.get("mlp")])
    return out


class LayerSpec:
    """Sizes and constants of one layer."""

    def __init__(self, c: dict, tp):
        self.type = c["type"]
        if self.type not in (LATENT, BIASED, ROTATED):
            raise ValueError(f"unknown mixer {self.type!r}")
        m = c["mixer"]
        self.heads, self.dim, self.vdim = m["heads"], m["dim"], m["vdim"]
        assert self.heads % tp.size == 0, "attention heads must divide by tp"
        self.scale = float(m["scale"])
        mask = m.get("mask") or {}
        self.window, self.keep = int(mask.get("size") or 0), int(mask.get("keep_first") or 0)
        self.rot = m.get("rot")
        self.kv_from = m.get("kv_from")
        self.hq = self.heads // tp.size
        self.vp = _up(self.vdim, 64)
        if self.type == LATENT:
            self.rank, self.rot_dim, self.q_rank = m["kv_rank"], m["rot_dim"], m.get("q_rank")
            self.kv_heads = 1
            if self.rot["dims"] != self.rot_dim:
                raise ValueError("latent attention: rot.dims must be rot_dim")
            if self.keep:
                raise ValueError("latent attention: no kept first tokens")
            self.dp = _up(self.dim + self.rot_dim, 64)
        else:
            self.kv_heads = m["kv_heads"]
            assert self.heads % self.kv_heads == 0, "attention heads must divide by the key / value heads"
            self.kv_range = kv_head_range(self.kv_heads, tp.rank, tp.size)
            self.hkv = self.kv_range[1] - self.kv_range[0]
            self.dp = _up(self.dim, 64)
            self.far = m.get("bias_max")
        self.kv_row = _kv_row(self.type, m, 1 if self.type == LATENT else self.hkv)
        f = c.get("mlp")
        self.moe = f is not None
        if f is None:
            return
        if f["kind"] != "moe":
            raise ValueError(f"unknown feed-forward {f['kind']!r}")
        r = f["router"]
        self.experts, self.top, self.router_scale = r["experts"], r["top"], float(r.get("scale") or 1.0)
        g = r.get("groups") or {"count": 1, "keep": 1}
        self.groups, self.kept_groups = g["count"], g["keep"]
        if self.experts % self.groups or self.top > self.experts // self.groups * self.kept_groups:
            raise ValueError("router: experts form equal groups, and the kept ones hold at least `top` experts")
        self.ff, self.clamp = f["expert"]["ff"], (ACT_ALPHA, float(f["expert"]["limit"]))


def _check_sources(specs):
    for i, s in enumerate(specs):
        if s.kv_from is None:
            continue
        j = s.kv_from
        o = specs[j] if 0 <= j < i else None
        if s.type == LATENT or o is None or o.type != s.type or o.kv_from is not None or \
                (o.kv_heads, o.dim, o.vdim) != (s.kv_heads, s.dim, s.vdim):
            raise ValueError(f"layer {i}: kv_from {j} names no earlier layer with keys and values of its own and equal sizes")


@register_model("katarax")
class KataraxLM(StreamLM):
    model_type = "katarax"
    native_units = ("attention", "attention_generic", "attention_tc", "gemm_f32", "gemm_tcgen05", "latent_attn", "moe",
                    "ops_basic", "rms_stream", "sampling", "window_prefill_tc")

    # ------------------------------------------------------------------ config
    def _read_config(self, c: dict):
        self.hidden, self.vocab = c["width"], c["vocab"]
        self.hidden_p = _up(self.hidden, 64)
        self.specs = [LayerSpec(l, self.tp) for l in c["layers"]]
        _check_sources(self.specs)
        self.num_layers = len(self.specs)
        self.eps = c["norm"]["eps"]
        self.logit_softcap = float(c.get("logit_softcap") or 0.0)
        self.tie_embeddings = False
        # what the engine reads of any model
        self.num_q_heads = max(s.heads for s in self.specs)
        self.num_kv_heads = self.hkv = max(s.kv_heads for s in self.specs)
        self.hq = max(s.hq for s in self.specs)
        self.head_dim = max(max(s.dp, s.vp) for s in self.specs)
        self.rot_dim = 0
        self.inter = None
        self._check_options()

    # ------------------------------------------------------------------ weights
    def weight_shapes(self) -> Dict[str, tuple]:
        W = self.hidden
        s = {"embed": (self.vocab, W), "head": (self.vocab, W), "final.norm": (W,)}
        for i, l in enumerate(self.specs):
            p, m = f"l{i}.", f"l{i}.mix."
            s[p + "norm1"] = (W,)
            s[m + "o"] = (W, l.heads * l.vdim)
            if l.type == LATENT:
                qr = l.q_rank or l.rank
                s.update({m + "dq": (qr, W), m + "dq.norm": (qr,), m + "uq": (l.heads * (l.dim + l.rot_dim), qr),
                          m + "dkv": (l.rank + l.rot_dim, W), m + "dkv.norm": (l.rank,),
                          m + "uk": (l.heads * l.dim, l.rank), m + "uv": (l.heads * l.vdim, l.rank),
                          m + "g": (l.heads * l.vdim, W)})
            else:
                s[m + "q"] = (l.heads * l.dim, W)
                if l.kv_from is None:
                    s.update({m + "k": (l.kv_heads * l.dim, W), m + "v": (l.kv_heads * l.vdim, W)})
                if l.type == BIASED:
                    s[m + "rel"] = (16, l.heads)
            if l.moe:
                f = p + "mlp."
                s.update({f + "router": (l.experts, W), f + "correction": (l.experts,)})
                for e in range(l.experts):
                    q = f"{f}e{e}."
                    s.update({q + "gate": (l.ff, W), q + "up": (l.ff, W), q + "down": (W, l.ff)})
        return s

    def weight_inits(self):
        """Random initialisation of what is not a matrix: norms of one, no corrections."""
        def fill(value):
            return lambda shape, gen, device: torch.full(shape, value, dtype=self.dtype, device=device)

        return {n: fill(1.0 if n.endswith(("dq.norm", "dkv.norm")) else 0.0) for n, shape in self.weight_shapes().items()
                if len(shape) == 1}

    def _load_norm(self, src, name):
        return self._vec(1.0 + get_shaped(src, name, self.hidden).float(), self.hidden_p)   # stored around zero

    def _load_weights(self, src):
        self._load_embed_and_head(src)
        self.final_norm = self._load_norm(src, "final.norm")
        self.layers = []
        for i, l in enumerate(self.specs[: self.num_layers]):
            lw = LayerWeights()
            p = f"l{i}."
            lw.spec = l
            lw.norm1 = self._load_norm(src, p + "norm1")
            (self._load_latent if l.type == LATENT else self._load_attention)(lw, src, p + "mix.", l)
            h0, h1 = tp_range(l.heads, self.tp.rank, self.tp.size)
            lw.o_w = self._dev(self._out_heads(src, p + "mix.o", l.heads, l.vdim, l.vp, h0, h1))
            if l.moe:
                f = p + "mlp."
                lw.router_w = self._dev(self._narrow(get_shaped(src, f + "router", l.experts, self.hidden), l.experts))
                lw.correction = self._vec(get_shaped(src, f + "correction", l.experts), l.experts)
                self._load_experts(lw, src, f, l.experts, l.ff)
            self.layers.append(lw)

    def _load_attention(self, lw, src, m, l: LayerSpec):
        h0, h1 = tp_range(l.heads, self.tp.rank, self.tp.size)
        rows = [self._heads(src, m + "q", l.heads, l.dim, l.dp, h0, h1)]
        if l.kv_from is None:
            rows += [self._heads(src, m + "k", l.kv_heads, l.dim, l.dp, *l.kv_range),
                     self._heads(src, m + "v", l.kv_heads, l.vdim, l.vp, *l.kv_range)]
        lw.in_w = self._dev(torch.cat(rows))
        if l.type == BIASED:
            table = get_shaped(src, m + "rel", src.shape(m + "rel")[0], l.heads)[:, h0:h1]
            lw.bias = ops.DistanceBias(table.to(self.device), l.far)

    def _load_latent(self, lw, src, m, l: LayerSpec):
        h0, h1 = tp_range(l.heads, self.tp.rank, self.tp.size)
        n, W = h1 - h0, self.hidden
        qr = l.q_rank or src.shape(m + "dq")[0]
        q16 = _up(qr, 16)
        lat = lw.latent = LatentHeads(n, l.dim, l.rot_dim, l.vdim, l.rank, l.scale, l.window)
        dkv = get_shaped(src, m + "dkv", l.rank + l.rot_dim, W)
        parts = [self._narrow(get_shaped(src, m + "dq", qr, W), qr, 16), self._narrow(dkv[: l.rank], l.rank, 16),
                 self._narrow(dkv[l.rank:], l.rot_dim, 16), self._heads(src, m + "g", l.heads, l.vdim, l.vp, h0, h1)]
        lw.in_w = self._dev(torch.cat(parts))
        lw.q_rank, lw.q_cols = qr, q16
        lw.q_norm = self._vec(get_shaped(src, m + "dq.norm", qr), q16)
        lw.kv_norm = self._vec(get_shaped(src, m + "dkv.norm", l.rank), lat.rp)
        per = l.dim + l.rot_dim
        uq = get_shaped(src, m + "uq", l.heads * per, qr).view(l.heads, per, qr)[h0:h1]
        lw.uq_w = self._dev(_pad(uq, n, l.dp, q16).reshape(n * l.dp, q16))
        uk = get_shaped(src, m + "uk", l.heads * l.dim, l.rank).view(l.heads, l.dim, l.rank)[h0:h1]
        uv = get_shaped(src, m + "uv", l.heads * l.vdim, l.rank).view(l.heads, l.vdim, l.rank)[h0:h1]
        lat.load(lw, self._dev, uk, uv)

    def _init_rope(self):
        """Rotary tables (layers with the same rotation share them)."""
        self.cos = self.sin = None
        n, tables = max(self.max_seq_length + 8, 16), {}
        for lw in self.layers:
            rot = lw.spec.rot
            if lw.spec.type == BIASED or not rot:
                continue
            key = (rot["base"], rot["dims"])
            if key not in tables:
                tables[key] = ref.build_rope_cache(n, rot["dims"], rot["base"], None, device=self.device)
            lw.rope = mla_ops.LatentRope(*tables[key], rot["dims"], neighbours=lw.spec.type == LATENT)

    # ------------------------------------------------------------------ memory
    def _kv_rows(self):
        return [s.kv_row for s in self.specs[: self.num_layers] if s.kv_row]

    def _init_mem(self, max_total_token_num, mem_fraction):
        kv = 0
        for lw in self.layers:
            if lw.spec.kv_from is not None:
                lw.kv_slot = self.layers[lw.spec.kv_from].kv_slot
            else:
                lw.kv_slot = kv
                kv += 1
        super()._init_mem(max_total_token_num, mem_fraction)

    # ------------------------------------------------------------------ forward
    def _embed(self, ids, st):
        x, st.extra["first_normed"] = ops.embedding_pair(ids, self.embed_w, None, self.req_manager.req_to_token_indexs,
                                                         st.b_req_idx, st.seq_pos, None, st.mem_index,
                                                         norm=(self.layers[0].norm1, self.hidden, self.eps))
        return x

    def _layers_forward(self, x, st: InferState):
        """x: the fp32 residual stream.  Returns the final norm's output."""
        h = st.extra.pop("first_normed")
        n = len(self.layers)
        for i, lw in enumerate(self.layers):
            after = self.layers[i + 1].norm1 if i + 1 < n else self.final_norm
            a = (self._latent_mixer if lw.spec.type == LATENT else self._attention_mixer)(lw, h, st)
            h = self._moe(i, lw, h, ops.gemm(a, lw.o_w), x, after, st) if lw.spec.moe else \
                ops.add_rms_(x, self._reduced(a, lw.o_w), None, self.hidden, self.eps, self.dtype, after)
            if self.stream_tap is not None:
                self.stream_tap(i, x)
        st.extra["normed"] = True
        return h

    def _latent_mixer(self, lw, h, st: InferState):
        l, lat = lw.spec, lw.latent
        proj = ops.gemm(h, lw.in_w)                              # [T, query latent | latent | rotated part | gate]
        kv_at, g_at = lw.q_cols, lw.q_cols + lat.keys
        kv_layer = self._kv_layer(lw.kv_slot)
        cq = mla_ops.latent_prepare_(proj[:, kv_at:g_at], kv_layer, lw.kv_norm, st.mem_index, l.rank, lat.rp, self.eps,
                                     lw.rope, st.position_ids, proj[:, :kv_at], lw.q_norm, lw.q_rank)
        q = ops.gemm(cq, lw.uq_w)
        ops.rope_heads_(q, lw.rope.cos, lw.rope.sin, st.position_ids, l.hq, l.dp, l.dim, lw.rope.dims, lw.rope.neighbours)
        return lat.attend(lw, q, kv_layer, self.req_manager.req_to_token_indexs, st, proj[:, g_at:])

    def _attention_mixer(self, lw, h, st: InferState):
        l = lw.spec
        proj = ops.gemm(h, lw.in_w)                              # [T, q heads | k heads | v heads]
        nq = l.hq * l.dp
        kv_layer = self._kv_layer(lw.kv_slot)
        if l.type == ROTATED:
            ops.qk_norm_rope_scatter_(proj, kv_layer, lw.rope.cos, lw.rope.sin, st.position_ids, st.mem_index, None, None,
                                      self.eps, l.hq, 0 if l.kv_from is not None else l.hkv, l.dp, l.dim, l.vp, lw.rope.dims)
        elif l.kv_from is None:
            ops.copy_rows(kv_layer, proj[:, nq:], st.mem_index, None, h.shape[0])
        return ops.window_attention(proj[:, :nq], kv_layer, self.req_manager.req_to_token_indexs, st, l.hq, l.hkv, l.dp, l.vp,
                                    l.scale, l.window, keep=l.keep, bias=lw.bias)

    def _moe(self, i, lw, h, y, x, after, st):
        """x += y + the experts' output for h; returns the next norm of x."""
        l = lw.spec
        logits = ops.gemm(h, lw.router_w, epi="f32")[:, : l.experts]
        ids, weights = moe_ops.grouped_topk(logits, lw.correction, l.top, l.groups, l.kept_groups, True, True, l.router_scale)
        if self.route_capture is not None:
            self.route_capture.capture(i, ids, st.mem_index)
        one = self.tp.size == 1
        out = moe_ops.routed_experts_rms_(h, ids, weights, lw.w13, lw.w2, l.clamp, y, x if one else None, None, self.hidden,
                                          self.eps, after if one else None, lw.e0)
        if one:
            return out
        self.tp.all_reduce_(out)
        return ops.add_rms_(x, out, None, self.hidden, self.eps, self.dtype, after)
