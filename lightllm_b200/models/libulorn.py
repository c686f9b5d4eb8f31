"""Libulorn: recurrent layers with a matrix memory (mLSTM) and layers that run windowed attention and gated linear attention
side by side, mixture-of-experts feed-forwards, and RMS norms on the sublayers' outputs only, around an fp32 residual stream
that starts as token embedding + bigram embedding.

    stream = embed[token] + bigram[(previous, token)];  per layer: stream += norm1(mixer(stream)), stream += norm2(ff(stream))
    logits = head . final(stream)

Every layer has its own sizes and constants (`layers` in config.json).  How it maps onto this package:

  * a sublayer reads the stream rounded to the format of its matrix products; the pass that normalises a sublayer's output
    and adds it to the fp32 stream writes that rounding too (`ops.add_rms_`, `ops.moe.routed_experts_rms_`)
  * one GEMM gives every projection of a mixer, one GEMM takes both sides of a "parallel" layer back to the stream: their
    outputs lie side by side, already gated and scaled.  Gate projections that a recurrence exponentiates keep fp32
  * attention: paged KV with separate key and value sizes, window and output gate inside the attention kernels
  * recurrences: `ops.linear_attn.DecayedState` over per-request fp32 states (`common/recurrent_state.py`)
  * the previous token of a sequence is found through the request table (`ops.BigramTable`)

Sizes that kernels cannot take are padded with zeros when the weights are loaded (width, attention head sizes and
feed-forward sizes to 64, recurrent head sizes to 16, everything narrow to 8).
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..common.infer_state import InferState
from ..common.recurrent_state import RecurrentStateMixin, RecurrentStates
from ..ops import moe as moe_ops
from ..ops import reference as ref
from ..ops.linear_attn import ChunkPlan, DecayedState
from .base import LayerWeights
from .registry import register_config, register_model
from .stream_lm import ACT_ALPHA, StreamLM
from .weights import get_shaped, kv_head_range, tp_range
from .weights import pad_zeros as _pad
from .weights import round_up as _up

RANDOM_DECAY_RANK = 16     # low-rank size of the decay projection for random weights (checkpoints bring their own)


@register_config("Libulorn")
def normalize_libulorn(cfg: dict) -> dict:
    """The keys the rest of the framework reads (HF spelling), next to the design's own."""
    layers = cfg["layers"]
    left = [l["mixer"]["left"] for l in layers if l["type"] == "parallel"]
    moe = [l["mlp"]["router"] for l in layers if l.get("mlp")]
    out = dict(cfg, model_type="libulorn", hidden_size=cfg["width"], vocab_size=cfg["vocab"],
               num_hidden_layers=len(layers),
               num_attention_heads=max([a["heads"] for a in left] or [1]),
               num_key_value_heads=max([a["kv_heads"] for a in left] or [1]),
               head_dim=max([a["dim"] for a in left] or [64]),
               kv_elems_per_token=sum(a["kv_heads"] * (_up(a["dim"], 64) + _up(a["vdim"], 64)) for a in left))
    if moe:
        out.update(num_experts=max(r["experts"] for r in moe), num_experts_per_tok=max(r["top"] for r in moe),
                   decoder_sparse_step=1, mlp_only_layers=[i for i, l in enumerate(layers) if not l.get("mlp")])
    return out


class AttentionSpec:
    def __init__(self, c: dict, tp):
        self.heads, self.kv_heads, self.dim, self.vdim = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
        self.scale = float(c["scale"])
        self.window = int((c.get("mask") or {}).get("size") or 0)
        self.rot = c.get("rot") or {"base": 10000.0, "dims": 0}
        self.dp, self.vp = _up(self.dim, 64), _up(self.vdim, 64)
        assert self.heads % tp.size == 0 and self.heads % self.kv_heads == 0, "attention heads must divide"
        self.kv_range = kv_head_range(self.kv_heads, tp.rank, tp.size)
        self.hq, self.hkv = self.heads // tp.size, self.kv_range[1] - self.kv_range[0]
        self.kv_row = self.hkv * (self.dp + self.vp)


class RecurrentSpec:
    def __init__(self, c: dict, kind: str, tp):
        self.kind = kind
        self.heads, self.dim, self.vdim = c["heads"], c["dim"], c["vdim"]
        self.tau, self.cap = float(c.get("tau") or 1.0), float(c.get("gate_cap") or 1.0)
        self.dp, self.vp = _up(self.dim, 16), _up(self.vdim, 16)
        assert self.heads % tp.size == 0, "recurrent heads must divide by tp"
        self.h = self.heads // tp.size
        self.state_elems = DecayedState.state_elems(kind, self.h, self.dp, self.vp)


class LayerSpec:
    """Sizes and constants of one layer."""

    def __init__(self, c: dict, tp):
        self.type = c["type"]
        m = c["mixer"]
        self.left = None
        if self.type == "parallel":
            self.left, self.rec = AttentionSpec(m["left"], tp), RecurrentSpec(m["right"], "gla", tp)
            self.left_scale, self.right_scale = float(m["left_scale"]), float(m["right_scale"])
        elif self.type == "mlstm":
            self.rec = RecurrentSpec(m, "mlstm", tp)
        else:
            raise ValueError(f"unknown mixer {self.type!r}")
        f = c.get("mlp")
        self.moe = f is not None
        if f is None:
            return
        if f["kind"] != "moe":
            raise ValueError(f"unknown feed-forward {f['kind']!r}")
        self.experts, self.top = f["router"]["experts"], f["router"]["top"]
        self.ff, self.clamp = f["expert"]["ff"], (ACT_ALPHA, float(f["expert"]["limit"]))
        s = f.get("shared")
        self.shared_ff = s["ff"] if s else 0
        self.shared_clamp = (ACT_ALPHA, float(s["limit"])) if s else None


@register_model("libulorn")
class LibulornLM(RecurrentStateMixin, StreamLM):
    model_type = "libulorn"
    native_units = ("attention", "attention_generic", "attention_tc", "gemm_f32", "gemm_tcgen05", "moe", "ops_basic",
                    "recurrent", "rms_stream", "sampling")

    # ------------------------------------------------------------------ config
    def _read_config(self, c: dict):
        self.hidden, self.vocab = c["width"], c["vocab"]
        self.hidden_p = _up(self.hidden, 64)
        self.specs = [LayerSpec(l, self.tp) for l in c["layers"]]
        self.num_layers = len(self.specs)
        self.eps = c["norm"]["eps"]
        self.bigram_cfg = (c.get("embedding") or {}).get("bigram")
        self.tie_embeddings = False
        # what the engine reads of any model
        left = [s.left for s in self.specs if s.left is not None]
        self.num_q_heads = max([a.heads for a in left] or [1])
        self.num_kv_heads = max([a.kv_heads for a in left] or [1])
        self.hq, self.hkv = max([a.hq for a in left] or [1]), max([a.hkv for a in left] or [1])
        self.head_dim = max([max(a.dp, a.vp) for a in left] or [64])
        self.rot_dim = 0
        self.inter = None
        self._check_options()

    # ------------------------------------------------------------------ weights
    def weight_shapes(self) -> Dict[str, tuple]:
        W = self.hidden
        s = {"embed": (self.vocab, W), "head": (self.vocab, W), "final.norm": (W,)}
        if self.bigram_cfg:
            s["bigram"] = (self.bigram_cfg["buckets"] + 1, W)

        def gated(p, ff):
            s.update({p + "gate": (ff, W), p + "up": (ff, W), p + "down": (W, ff)})

        def recurrent(p, r):
            k, v = r.heads * r.dim, r.heads * r.vdim
            s.update({p + "q": (k, W), p + "k": (k, W), p + "v": (v, W), p + "g": (v, W), p + "o": (W, v)})
            if r.kind == "gla":
                n = RANDOM_DECAY_RANK
                s.update({p + "norm": (r.vdim,), p + "a1": (n, W), p + "a2": (k, n), p + "a2.b": (k,)})
            else:
                s.update({p + "norm": (v,), p + "i": (r.heads, W), p + "i.b": (r.heads,), p + "f": (r.heads, W),
                          p + "f.b": (r.heads,)})

        for i, l in enumerate(self.specs):
            p, m = f"l{i}.", f"l{i}.mix."
            s[p + "norm1"] = (W,)
            if l.left is not None:
                a, q = l.left, m + "left."
                s.update({q + "q": (a.heads * a.dim, W), q + "k": (a.kv_heads * a.dim, W),
                          q + "v": (a.kv_heads * a.vdim, W), q + "q.norm": (a.dim,), q + "k.norm": (a.dim,),
                          q + "g": (a.heads, W), q + "o": (W, a.heads * a.vdim)})
                recurrent(m + "right.", l.rec)
            else:
                recurrent(m, l.rec)
            if l.moe:
                f = p + "mlp."
                s.update({p + "norm2": (W,), f + "router": (l.experts, W)})
                for e in range(l.experts):
                    gated(f"{f}e{e}.", l.ff)
                if l.shared_ff:
                    gated(f + "shared.", l.shared_ff)
        return s

    def weight_inits(self):
        """Random initialisation of what is not a matrix: unit norms, no biases."""
        def fill(value):
            return lambda shape, gen, device: torch.full(shape, value, dtype=self.dtype, device=device)

        return {n: fill(1.0 if "norm" in n else 0.0) for n, shape in self.weight_shapes().items() if len(shape) == 1}

    def _load_norm(self, src, name):
        return self._vec(get_shaped(src, name, self.hidden), self.hidden_p)

    def _load_weights(self, src):
        W, P = self.hidden, self.hidden_p
        self._load_embed_and_head(src)
        self.bigram = None
        if self.bigram_cfg:
            b = self.bigram_cfg
            n = b["buckets"] + 1
            self.bigram = ops.BigramTable(self._dev(_pad(get_shaped(src, "bigram", n, W), n, P)), b["buckets"],
                                          b["mul_prev"], b["mul_cur"])
        self.final_norm = self._load_norm(src, "final.norm")
        self.layers = []
        for i, l in enumerate(self.specs[: self.num_layers]):
            lw = LayerWeights()
            p, m = f"l{i}.", f"l{i}.mix."
            lw.spec = l
            lw.norm1 = self._load_norm(src, p + "norm1")
            rows, outs, cols = [], [], {}

            def add(name, w):
                at = sum(x.shape[0] for x in rows)
                rows.append(w)
                cols[name] = (at, w.shape[0])

            if l.left is not None:
                self._load_attention(lw, src, m + "left.", l.left, add, outs)
                self._load_recurrent(lw, src, m + "right.", l.rec, add, outs, l.right_scale)
            else:
                self._load_recurrent(lw, src, m, l.rec, add, outs, 1.0)
            lw.in_w, lw.cols = self._dev(torch.cat(rows)), cols
            lw.o_w = self._dev(torch.cat(outs, dim=1))
            if l.moe:
                lw.norm2 = self._load_norm(src, p + "norm2")
                self._load_moe(lw, src, p + "mlp.", l)
            self.layers.append(lw)

    def _load_attention(self, lw, src, p, a: AttentionSpec, add, outs):
        h0, h1 = tp_range(a.heads, self.tp.rank, self.tp.size)
        k0, k1 = a.kv_range
        add("qkv", torch.cat([self._heads(src, p + "q", a.heads, a.dim, a.dp, h0, h1),
                              self._heads(src, p + "k", a.kv_heads, a.dim, a.dp, k0, k1),
                              self._heads(src, p + "v", a.kv_heads, a.vdim, a.vp, k0, k1)]))
        add("gate", self._narrow(get_shaped(src, p + "g", a.heads, self.hidden)[h0:h1], h1 - h0))
        lw.q_norm = self._vec(get_shaped(src, p + "q.norm", a.dim), a.dp)
        lw.k_norm = self._vec(get_shaped(src, p + "k.norm", a.dim), a.dp)
        outs.append(self._out_heads(src, p + "o", a.heads, a.vdim, a.vp, h0, h1))

    def _load_recurrent(self, lw, src, p, s: RecurrentSpec, add, outs, out_scale):
        h0, h1 = tp_range(s.heads, self.tp.rank, self.tp.size)
        for n, size, padded in (("q", s.dim, s.dp), ("k", s.dim, s.dp), ("v", s.vdim, s.vp), ("g", s.vdim, s.vp)):
            add("r" + n, self._heads(src, p + n, s.heads, size, padded, h0, h1))
        kw = dict(eps=self.eps, out_scale=out_scale)
        if s.kind == "gla":
            rank = src.shape(p + "a1")[0]
            add("a1", self._narrow(get_shaped(src, p + "a1", rank, self.hidden), rank))
            a2 = get_shaped(src, p + "a2", s.heads * s.dim, rank).view(s.heads, s.dim, rank)[h0:h1]
            b = get_shaped(src, p + "a2.b", s.heads * s.dim).view(s.heads, s.dim)[h0:h1]
            rank8 = _up(rank, 8)
            kw.update(tau=s.tau, a2=self._dev(_pad(a2, s.h, s.dp, rank8).view(-1, rank8)),
                      a2_bias=self._vec(b, s.h, s.dp).view(-1),
                      weight=self._vec(get_shaped(src, p + "norm", s.vdim), s.vp))
        else:
            n8 = _up(2 * s.h, 8)
            gw = torch.cat([get_shaped(src, p + n, s.heads, self.hidden)[h0:h1] for n in "if"])
            gb = torch.cat([get_shaped(src, p + n + ".b", s.heads)[h0:h1] for n in "if"])
            lw.if_w, lw.if_b = self._dev(_pad(gw, n8, self.hidden_p)), self._dev(_pad(gb, n8))
            w = get_shaped(src, p + "norm", s.heads * s.vdim).view(s.heads, s.vdim)[h0:h1]
            kw.update(cap=s.cap, weight=self._vec(w, s.h, s.vp).view(-1))
        lw.rec = DecayedState(s.kind, s.h, s.dp, s.vp, s.dim, s.vdim, **kw)
        outs.append(self._out_heads(src, p + "o", s.heads, s.vdim, s.vp, h0, h1))

    def _load_moe(self, lw, src, p, l: LayerSpec):
        """Router, experts stacked as in `models/moe.py`, shared expert."""
        tp, r = self.tp.size, self.tp.rank
        lw.router_w = self._dev(self._narrow(get_shaped(src, p + "router", l.experts, self.hidden), l.experts))
        self._load_experts(lw, src, p, l.experts, l.ff)
        if l.shared_ff:
            a, b = self._load_gated(src, p + "shared.", l.shared_ff, *tp_range(l.shared_ff, r, tp))
            lw.shared_gate_up_w, lw.shared_down_w = self._dev(a), self._dev(b)

    def _init_rope(self):
        """Rotary tables of every attention layer (layers with the same rotation share them)."""
        self.cos = self.sin = None
        n, tables = max(self.max_seq_length + 8, 16), {}
        for lw in self.layers:
            a = lw.spec.left
            if a is None:
                continue
            s = a.rot.get("scaling")
            key = (a.rot["base"], a.rot["dims"], tuple(sorted(s.items())) if s else None)
            if key not in tables:
                scaling = s and dict(rope_type="llama3", factor=s["factor"], low_freq_factor=s["low"],
                                     high_freq_factor=s["high"], original_max_position_embeddings=s["original"])
                tables[key] = ref.build_rope_cache(n, a.rot["dims"], a.rot["base"], scaling, device=self.device)
            lw.cos, lw.sin = tables[key]

    # ------------------------------------------------------------------ memory
    def _kv_rows(self):
        return [s.left.kv_row for s in self.specs[: self.num_layers] if s.left is not None]

    def kv_bytes_per_token(self):
        return super().kv_bytes_per_token() + 4     # + its token id

    def _init_mem(self, max_total_token_num, mem_fraction):
        # the requests' recurrent states come out of the same budget: allocate them first
        self.states = RecurrentStates()
        kv = 0
        for i, lw in enumerate(self.layers):
            self.states.reserve(i, lw.spec.rec.state_elems)
            if lw.spec.left is not None:
                lw.kv_slot = kv
                kv += 1
        self.states.allocate(self.max_req_num + 1, self.device, int(self.extra.get("state_snapshot_slots") or 0))
        super()._init_mem(max_total_token_num, mem_fraction)
        if self.bigram is not None:
            self.bigram.slot_token = torch.zeros(self.mem_manager.size + 1, dtype=torch.int32, device=self.device)

    # ------------------------------------------------------------------ forward
    def _embed(self, ids, st):
        x, st.extra["stream_h"] = ops.embedding_pair(ids, self.embed_w, self.bigram, self.req_manager.req_to_token_indexs,
                                                     st.b_req_idx, st.seq_pos,
                                                     st.batch_of_token if st.is_prefill else None, st.mem_index)
        return x

    def _layers_forward(self, x, st: InferState):
        """x: the fp32 residual stream.  Returns the final norm's output."""
        h = st.extra.pop("stream_h")
        if st.is_prefill and self.device.type == "cuda" and self.dtype == torch.bfloat16:
            st.extra["chunk_plan"] = ChunkPlan(st.extra["q_len_cpu"], self.device)
        n = len(self.layers)
        for i, lw in enumerate(self.layers):
            after = self.final_norm if i + 1 == n else None
            y = self._reduced(self._mixer(i, lw, h, st), lw.o_w)
            h = ops.add_rms_(x, y, lw.norm1, self.hidden, self.eps, self.dtype, None if lw.spec.moe else after)
            if lw.spec.moe:
                h = self._moe(i, lw, h, x, after, st)
            if self.stream_tap is not None:
                self.stream_tap(i, x)
        st.extra["normed"] = True
        return h

    def _mixer(self, i, lw, h, st: InferState):
        """The mixer's heads, gated, side by side (input of the output projection)."""
        l, r = lw.spec, lw.rec
        proj = ops.gemm(h, lw.in_w)

        def part(name):
            at, n = lw.cols[name]
            return proj[:, at:at + n]

        rec = dict(q=part("rq"), k=part("rk"), v=part("rv"), g=part("rg"), state=self.states.view(i), st=st,
                   plan=st.extra.get("chunk_plan"))
        if l.left is None:
            z = ops.gemm(h, lw.if_w, epi="f32", bias=lw.if_b)
            return r(zi=z[:, : r.H], zf=z[:, r.H: 2 * r.H], **rec)
        a = l.left
        out = torch.empty((h.shape[0], lw.o_w.shape[1]), dtype=h.dtype, device=h.device)
        split = a.hq * a.vp
        qkv, kv_layer = part("qkv"), self._kv_layer(lw.kv_slot)
        ops.qk_norm_rope_scatter_(qkv, kv_layer, lw.cos, lw.sin, st.position_ids, st.mem_index, lw.q_norm, lw.k_norm,
                                  self.eps, a.hq, a.hkv, a.dp, a.dim, a.vp, a.rot["dims"])
        ops.window_attention(qkv[:, : a.hq * a.dp], kv_layer, self.req_manager.req_to_token_indexs, st, a.hq, a.hkv, a.dp,
                             a.vp, a.scale, a.window, part("gate")[:, : a.hq], l.left_scale, out[:, :split])
        r(a1=part("a1"), out=out[:, split:], **rec)
        return out

    def _moe(self, i, lw, h, x, after, st):
        l = lw.spec
        logits = ops.gemm(h, lw.router_w, epi="f32")[:, : l.experts]
        ids, weights = moe_ops.topk_softmax(logits, l.top, renorm=False)
        if self.route_capture is not None:
            self.route_capture.capture(i, ids, st.mem_index)
        shared = None
        if lw.shared_down_w is not None:
            shared = ops.gemm(ops.gemm(h, lw.shared_gate_up_w, epi="gated_clamp", clamp=l.shared_clamp), lw.shared_down_w)
        one = self.tp.size == 1
        out = moe_ops.routed_experts_rms_(h, ids, weights, lw.w13, lw.w2, l.clamp, shared, x if one else None,
                                          lw.norm2 if one else None, self.hidden, self.eps, after if one else None, lw.e0)
        if one:
            return out
        self.tp.all_reduce_(out)
        return ops.add_rms_(x, out, lw.norm2, self.hidden, self.eps, self.dtype, after)
