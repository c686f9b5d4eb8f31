"""Silupel: recurrent layers (minGRU), attention within chunks of positions and latent attention, each followed by a dense
feed-forward, around an fp32 residual stream; the mixers read a token-shifted layer norm, and a run of layers may be looped.

    stream = embed[token];  per layer: stream += mixer(shift(norm1(stream))), stream += ff(norm2(stream))   (a layer may have no ff)
    logits = head . final(stream)

Every layer has its own sizes and constants (`layers` in config.json); `loop` repeats layers start .. stop - 1 with the same
weights.  How it maps onto this package:

  * one pass adds a sublayer's output to the fp32 stream, normalises the sum and shifts it (`ops.norm_shift`); the norm of a
    sequence's last token is part of its recurrent state (`common/recurrent_state.py`), and so is minGRU's state
  * one GEMM gives every projection of a mixer.  minGRU: `ops.linear_attn.gated_scan`
  * chunked attention: paged keys and values; chunk, soft cap and elementwise gate inside the attention kernels
    (`ops.window_attention`).  A head's temperature is a factor on its queries, in the rotation pass (`ops.qk_norm_rope_scatter_`)
  * latents: `models/latent.py`; the pool row of a token is [latent | rotated key part]
  * a layer that runs several times has one set of weights, and pool rows and states for every run

Sizes that kernels cannot take are padded with zeros when the weights are loaded (width, head sizes, recurrent and feed-forward
sizes to 64, latents and the rotated part to 16, everything narrow to 8).
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import ops
from ..common.infer_state import InferState
from ..common.recurrent_state import RecurrentStateMixin, RecurrentStates
from ..ops import mla as mla_ops
from ..ops import reference as ref
from ..ops.linear_attn import gated_scan, scan_plan
from .base import LayerWeights
from .latent import LatentHeads
from .registry import register_config, register_model
from .stream_lm import StreamLM
from .weights import get_shaped, kv_head_range, tp_range
from .weights import pad_zeros as _pad
from .weights import round_up as _up

MINGRU, CHUNKED, LATENT = "mingru", "attention", "latent_attention"


def _kv_row(kind: str, m: dict, kv_heads: int) -> int:
    """Elements of a layer's pool row (0: it has none)."""
    if kind == LATENT:
        return _up(m["kv_rank"], 16) + _up(m["rot_dim"], 16)
    return kv_heads * (_up(m["dim"], 64) + _up(m["vdim"], 64)) if kind == CHUNKED else 0


def layer_order(n: int, loop) -> List[int]:
    """Layer numbers in the order in which they run, of a stack of n layers."""
    if not loop:
        return list(range(n))
    a, b, times = loop["start"], loop["stop"], loop["times"]
    if not (0 <= a <= b and times >= 0):
        raise ValueError("loop: start, stop and times name no run of layers")
    a, b = min(a, n), min(b, n)
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


@register_config("Silupel")
def normalize_silupel(cfg: dict) -> dict:
    """The keys the rest of the framework reads (HF spelling), next to the design's own."""
    layers = cfg["layers"]
    mix = [l["mixer"] for l in layers if l["type"] != MINGRU]
    order = layer_order(len(layers), cfg.get("loop"))
    return dict(cfg, model_type="silupel", hidden_size=cfg["width"], vocab_size=cfg["vocab"], num_hidden_layers=len(layers),
                num_attention_heads=max([m["heads"] for m in mix] or [1]),
                num_key_value_heads=max([m.get("kv_heads", 1) for m in mix] or [1]),
                head_dim=max([m["dim"] + m.get("rot_dim", 0) for m in mix] or [64]),
                kv_elems_per_token=sum(_kv_row(layers[i]["type"], layers[i]["mixer"], layers[i]["mixer"].get("kv_heads", 1))
                                       for i in order))


class LayerSpec:
    """Sizes and constants of one layer."""

    moe = False

    def __init__(self, c: dict, tp):
        self.type = c["type"]
        if self.type not in (MINGRU, CHUNKED, LATENT):
            raise ValueError(f"unknown mixer {self.type!r}")
        m = c["mixer"]
        f = c.get("mlp")
        if f is not None and f["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {f['kind']!r}")
        self.ff = f["ff"] if f is not None else 0
        self.heads = self.hq = self.kv_heads = self.kv_row = 0
        if self.type == MINGRU:
            self.size = m["width"]
            assert self.size % tp.size == 0, "the recurrent size must divide by tp"
            self.n = self.size // tp.size
            self.np = _up(self.n, 64)
            return
        self.heads, self.dim, self.vdim, self.scale = m["heads"], m["dim"], m["vdim"], float(m["scale"])
        assert self.heads % tp.size == 0, "attention heads must divide by tp"
        self.hq = self.heads // tp.size
        self.vp = _up(self.vdim, 64)
        self.rot = m.get("rot") or {"base": 10000.0, "dims": 0}
        if self.type == LATENT:
            self.rank, self.rot_dim, self.q_rank = m["kv_rank"], m["rot_dim"], m.get("q_rank")
            self.kv_heads = 1
            if self.rot["dims"] != self.rot_dim:
                raise ValueError("latent attention: rot.dims must be rot_dim")
            self.dp = _up(self.dim + self.rot_dim, 64)
        else:
            self.kv_heads = m["kv_heads"]
            assert self.heads % self.kv_heads == 0, "attention heads must divide by the key / value heads"
            self.kv_range = kv_head_range(self.kv_heads, tp.rank, tp.size)
            self.hkv = self.kv_range[1] - self.kv_range[0]
            self.dp = _up(self.dim, 64)
            self.chunk = int((m.get("mask") or {}).get("size") or 0)
            self.softcap = float(m.get("softcap") or 0.0)
        if self.rot["dims"] % 2 or self.rot["dims"] > max(self.dim, getattr(self, "rot_dim", 0)):
            raise ValueError("rot.dims must be even and fit the head")
        self.kv_row = _kv_row(self.type, m, 1 if self.type == LATENT else self.hkv)


class Run:
    """One run of a layer: its weights, its rows in the pool and its states."""

    def __init__(self, lw, index: int):
        self.lw, self.spec, self.index = lw, lw.spec, index
        self.kv_slot = None


@register_model("silupel")
class SilupelLM(RecurrentStateMixin, StreamLM):
    model_type = "silupel"
    native_units = ("attention", "attention_generic", "attention_tc", "gated_scan", "gemm_f32", "gemm_tcgen05", "latent_attn",
                    "norm_shift", "ops_basic", "sampling", "window_prefill_tc")

    # ------------------------------------------------------------------ config
    def _read_config(self, c: dict):
        self.hidden, self.vocab = c["width"], c["vocab"]
        self.hidden_p = _up(self.hidden, 64)
        self.specs = [LayerSpec(l, self.tp) for l in c["layers"]]
        self.num_layers = len(self.specs)
        self.loop = c.get("loop")
        self.eps = c["norm"]["eps"]
        self.tie_embeddings = False
        # what the engine reads of any model
        self.num_q_heads = max(max(s.heads for s in self.specs), 1)
        self.num_kv_heads = self.hkv = max(max(s.kv_heads for s in self.specs), 1)
        self.hq = max(max(s.hq for s in self.specs), 1)
        self.head_dim = max([max(s.dp, s.vp) for s in self.specs if s.heads] or [64])
        self.rot_dim = 0
        self.inter = None
        self._check_options()

    def _order(self) -> List[int]:
        return layer_order(self.num_layers, self.loop)

    # ------------------------------------------------------------------ weights
    def weight_shapes(self) -> Dict[str, tuple]:
        W = self.hidden
        s = {"embed": (self.vocab, W), "head": (self.vocab, W), "final.norm": (W,)}
        for i, l in enumerate(self.specs):
            p, m = f"l{i}.", f"l{i}.mix."
            s.update({p + "norm1": (W,), p + "shift": (W,)})
            if l.type == MINGRU:
                s.update({m + "z": (l.size, W), m + "z.b": (l.size,), m + "x": (l.size, W), m + "x.b": (l.size,),
                          m + "g": (l.size, W), m + "o": (W, l.size)})
            elif l.type == LATENT:
                qr = l.q_rank or l.rank
                s.update({m + "dq": (qr, W), m + "dq.norm": (qr,), m + "uq": (l.heads * (l.dim + l.rot_dim), qr),
                          m + "dkv": (l.rank + l.rot_dim, W), m + "dkv.norm": (l.rank,), m + "uk": (l.heads * l.dim, l.rank),
                          m + "uv": (l.heads * l.vdim, l.rank), m + "o": (W, l.heads * l.vdim)})
            else:
                for n, rows in (("q", l.heads * l.dim), ("k", l.kv_heads * l.dim), ("v", l.kv_heads * l.vdim)):
                    s.update({m + n: (rows, W), m + n + ".b": (rows,)})
                s.update({m + "temp": (l.heads,), m + "g": (l.heads * l.vdim, W), m + "o": (W, l.heads * l.vdim), m + "o.b": (W,)})
            if l.ff:
                f = p + "mlp."
                s.update({p + "norm2": (W,), f + "gate": (l.ff, W), f + "up": (l.ff, W), f + "down": (W, l.ff)})
        return s

    def weight_inits(self):
        """Random initialisation of what is not a matrix: unit norms and temperatures, half a shift, no biases."""
        def fill(value):
            return lambda shape, gen, device: torch.full(shape, value, dtype=self.dtype, device=device)

        def value(n):
            return 1.0 if "norm" in n or n.endswith("temp") else 0.5 if n.endswith("shift") else 0.0

        return {n: fill(value(n)) for n, shape in self.weight_shapes().items() if len(shape) == 1}

    def _load_norm(self, src, name):
        return self._vec(get_shaped(src, name, self.hidden), self.hidden_p)

    def _load_weights(self, src):
        self._load_embed_and_head(src)
        self.final_norm = self._load_norm(src, "final.norm")
        self.layers = []
        load = {MINGRU: self._load_mingru, CHUNKED: self._load_attention, LATENT: self._load_latent}
        for i, l in enumerate(self.specs[: self.num_layers]):
            lw = LayerWeights()
            p = f"l{i}."
            lw.spec = l
            lw.norm1, lw.shift = self._load_norm(src, p + "norm1"), self._load_norm(src, p + "shift")
            load[l.type](lw, src, p + "mix.", l)
            if l.ff:
                lw.norm2 = self._load_norm(src, p + "norm2")
                a, b = self._load_gated(src, p + "mlp.", l.ff, *tp_range(l.ff, self.tp.rank, self.tp.size))
                lw.gate_up_w, lw.down_w = self._dev(a), self._dev(b)
            self.layers.append(lw)
        self.runs = [Run(self.layers[i], r) for r, i in enumerate(self._order())]

    def _head_bias(self, src, name, heads, size, padded, h0, h1):
        return _pad(get_shaped(src, name, heads * size).view(heads, size)[h0:h1], h1 - h0, padded).reshape(-1)

    def _load_mingru(self, lw, src, m, l: LayerSpec):
        c0, c1 = tp_range(l.size, self.tp.rank, self.tp.size)
        mats = [_pad(get_shaped(src, m + n, l.size, self.hidden)[c0:c1], l.np, self.hidden_p) for n in "zxg"]
        bias = [_pad(get_shaped(src, m + n + ".b", l.size)[c0:c1], l.np) for n in "zx"]
        lw.in_w = self._dev(torch.cat(mats))
        lw.in_b = self._dev(torch.cat(bias + [torch.zeros_like(bias[0])]))
        lw.o_w = self._dev(_pad(get_shaped(src, m + "o", self.hidden, l.size)[:, c0:c1], self.hidden_p, l.np))

    def _load_attention(self, lw, src, m, l: LayerSpec):
        h0, h1 = tp_range(l.heads, self.tp.rank, self.tp.size)
        parts = [("q", l.heads, l.dim, l.dp, h0, h1), ("k", l.kv_heads, l.dim, l.dp, *l.kv_range),
                 ("v", l.kv_heads, l.vdim, l.vp, *l.kv_range)]
        gate = self._heads(src, m + "g", l.heads, l.vdim, l.vp, h0, h1)
        lw.in_w = self._dev(torch.cat([self._heads(src, m + n, *a) for n, *a in parts] + [gate]))
        bias = [self._head_bias(src, m + n + ".b", *a) for n, *a in parts]
        lw.in_b = self._dev(torch.cat(bias + [torch.zeros(gate.shape[0], dtype=bias[0].dtype, device=bias[0].device)]))
        lw.temp = self._vec(get_shaped(src, m + "temp", l.heads)[h0:h1], l.hq)
        lw.o_w = self._dev(self._out_heads(src, m + "o", l.heads, l.vdim, l.vp, h0, h1))
        if self.tp.rank == 0:       # a sum over the ranks follows
            lw.o_b = self._dev(_pad(get_shaped(src, m + "o.b", self.hidden), self.hidden_p))

    def _load_latent(self, lw, src, m, l: LayerSpec):
        h0, h1 = tp_range(l.heads, self.tp.rank, self.tp.size)
        W, per = self.hidden, l.dim + l.rot_dim
        qr = l.q_rank or src.shape(m + "dq")[0]
        q16 = _up(qr, 16)
        lat = lw.latent = LatentHeads(l.hq, l.dim, l.rot_dim, l.vdim, l.rank, l.scale, 0)
        dkv = get_shaped(src, m + "dkv", l.rank + l.rot_dim, W)
        lw.in_w = self._dev(torch.cat([self._narrow(get_shaped(src, m + "dq", qr, W), qr, 16),
                                       self._narrow(dkv[: l.rank], l.rank, 16), self._narrow(dkv[l.rank:], l.rot_dim, 16)]))
        lw.q_rank, lw.q_cols = qr, q16
        lw.q_norm = self._vec(get_shaped(src, m + "dq.norm", qr), q16)
        lw.kv_norm = self._vec(get_shaped(src, m + "dkv.norm", l.rank), lat.rp)
        uq = get_shaped(src, m + "uq", l.heads * per, qr).view(l.heads, per, qr)[h0:h1]
        lw.uq_w = self._dev(_pad(uq, l.hq, l.dp, q16).reshape(l.hq * l.dp, q16))
        uk = get_shaped(src, m + "uk", l.heads * l.dim, l.rank).view(l.heads, l.dim, l.rank)[h0:h1]
        uv = get_shaped(src, m + "uv", l.heads * l.vdim, l.rank).view(l.heads, l.vdim, l.rank)[h0:h1]
        lat.load(lw, self._dev, uk, uv)
        lw.o_w = self._dev(self._out_heads(src, m + "o", l.heads, l.vdim, l.vp, h0, h1))

    def _init_rope(self):
        """Rotary tables (layers with the same rotation share them)."""
        self.cos = self.sin = None
        n, tables = max(self.max_seq_length + 8, 16), {}
        for lw in self.layers:
            if lw.spec.type == MINGRU:
                continue
            rot = lw.spec.rot
            s = rot.get("scaling")
            key = (rot["base"], rot["dims"], tuple(sorted(s.items())) if s else None)
            if key not in tables:
                scaling = s and dict(rope_type="llama3", factor=s["factor"], low_freq_factor=s["low"],
                                     high_freq_factor=s["high"], original_max_position_embeddings=s["original"])
                tables[key] = ref.build_rope_cache(n, rot["dims"], rot["base"], scaling, device=self.device)
            lw.rope = mla_ops.LatentRope(*tables[key], rot["dims"], neighbours=False)

    # ------------------------------------------------------------------ memory
    def _kv_rows(self):
        return [r.spec.kv_row for r in self.runs if r.spec.kv_row]

    def _init_mem(self, max_total_token_num, mem_fraction):
        # the requests' recurrent states come out of the same budget: allocate them first
        self.states = RecurrentStates()
        kv = 0
        for r in self.runs:
            self.states.reserve(("shift", r.index), self.hidden_p)
            if r.spec.type == MINGRU:
                self.states.reserve(("scan", r.index), r.spec.np)
            else:
                r.kv_slot = kv
                kv += 1
        self.states.allocate(self.max_req_num + 1, self.device, int(self.extra.get("state_snapshot_slots") or 0))
        super()._init_mem(max_total_token_num, mem_fraction)

    # ------------------------------------------------------------------ forward
    def _norm(self, x, y, run, st: InferState, **kw):
        """(x + y, its norm ahead of the run's mixer; without a run: the final norm)."""
        if run is None:
            return ops.norm_shift(x, y, self.final_norm, self.hidden, self.eps, self.dtype, **kw)
        shift = ops.TokenShift(run.lw.shift, self.states.view(("shift", run.index)), st)
        return ops.norm_shift(x, y, run.lw.norm1, self.hidden, self.eps, self.dtype, shift, **kw)

    def _embed(self, ids, st):
        x, st.extra["first_normed"] = self._norm(None, self.embed_w, self.runs[0] if self.runs else None, st, ids=ids)
        return x

    def _layers_forward(self, x, st: InferState):
        """x: the fp32 residual stream.  Returns the final norm's output."""
        h = st.extra.pop("first_normed")
        mixers = {MINGRU: self._mingru_mixer, CHUNKED: self._attention_mixer, LATENT: self._latent_mixer}
        if st.is_prefill and any(r.spec.type == MINGRU for r in self.runs):
            st.extra["scan_plan"] = scan_plan(st.extra["q_len_cpu"], self.device)
        for i, run in enumerate(self.runs):
            lw = run.lw
            after = self.runs[i + 1] if i + 1 < len(self.runs) else None
            y = self._reduced(mixers[run.spec.type](run, h, st), lw.o_w, lw.o_b)
            if run.spec.ff:
                x, h = ops.norm_shift(x, y, lw.norm2, self.hidden, self.eps, self.dtype)
                y = self._reduced(ops.gemm(h, lw.gate_up_w, epi="gated_gelu"), lw.down_w)
            x, h = self._norm(x, y, after, st)
            if self.stream_tap is not None:
                self.stream_tap(i, x)
        st.extra["normed"] = True
        return h

    def _mingru_mixer(self, run, h, st: InferState):
        n = run.spec.np
        proj = ops.gemm(h, run.lw.in_w, bias=run.lw.in_b)        # [T, z | x | gate]
        return gated_scan(proj[:, :n], proj[:, n:2 * n], proj[:, 2 * n:], self.states.view(("scan", run.index)), st, self.dtype,
                          st.extra.get("scan_plan"))

    def _attention_mixer(self, run, h, st: InferState):
        l, lw = run.spec, run.lw
        proj = ops.gemm(h, lw.in_w, bias=lw.in_b)                # [T, q heads | k heads | v heads | gate]
        nq, at = l.hq * l.dp, l.hq * l.dp + l.hkv * (l.dp + l.vp)
        kv_layer = self._kv_layer(run.kv_slot)
        ops.qk_norm_rope_scatter_(proj[:, :at], kv_layer, lw.rope.cos, lw.rope.sin, st.position_ids, st.mem_index, None, None,
                                  self.eps, l.hq, l.hkv, l.dp, l.dim, l.vp, lw.rope.dims, norm=False, q_scale=lw.temp)
        return ops.window_attention(proj[:, :nq], kv_layer, self.req_manager.req_to_token_indexs, st, l.hq, l.hkv, l.dp, l.vp,
                                    l.scale, 0, gate=proj[:, at:], chunk=l.chunk, softcap=l.softcap)

    def _latent_mixer(self, run, h, st: InferState):
        l, lw, lat = run.spec, run.lw, run.lw.latent
        proj = ops.gemm(h, lw.in_w)                              # [T, query latent | latent | rotated part]
        kv_layer = self._kv_layer(run.kv_slot)
        cq = mla_ops.latent_prepare_(proj[:, lw.q_cols:], kv_layer, lw.kv_norm, st.mem_index, l.rank, lat.rp, self.eps, lw.rope,
                                     st.position_ids, proj[:, : lw.q_cols], lw.q_norm, lw.q_rank)
        q = ops.gemm(cq, lw.uq_w)
        ops.rope_heads_(q, lw.rope.cos, lw.rope.sin, st.position_ids, l.hq, l.dp, l.dim, lw.rope.dims, lw.rope.neighbours)
        return lat.attend(lw, q, kv_layer, self.req_manager.req_to_token_indexs, st)
