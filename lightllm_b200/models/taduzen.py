"""Taduzen: latent attention without positions through a sliding window, mixture-of-experts layers whose experts are
looked up by token id, and dynamic-tanh norms before and after every sublayer around an fp32 residual stream.

    stream = embedding row;  per layer: stream += post1(attention(pre1(stream))), stream += post2(ffn(pre2(stream)))
    (a layer may have no ffn);  logits = logit_scale * head . final(stream)

Every layer has its own sizes (`layers` in config.json).  How it maps onto this package:

  * residual stream and norms in fp32; a norm has no row statistics, so the output projection's GEMM epilogue applies
    the norm of its own result, adds it to the stream and applies the next sublayer's norm (`ops.gemm` epi "dyt");
    after an MoE layer the combine kernel does the same
  * one GEMM gives q and the new latents; the pool row of a token is the normalised latent (`MLAMemoryManager`)
  * attention: absorbed form in decode, expanded form (keys and values per head, tcgen05) in longer prompt passes
  * the experts of a token do not depend on activations: the expert-sorted layouts of all layers come from one launch at
    the start of the step (`ops.moe.TableRouting`)

Sizes that tensor-core kernels cannot take are padded with zeros when the weights are loaded (width, head sizes and
feed-forward sizes to 64, the latent to 16, the vocabulary to 8): zero rows and columns add nothing anywhere.
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..common.infer_state import InferState, ShardedLogits
from ..common.mem_manager import MLAMemoryManager
from ..ops import mla as mla_ops
from ..ops import moe as moe_ops
from ..ops import reference as ref
from .base import LayerWeights
from .latent import LatentHeads
from .registry import register_config, register_model
from .stream_lm import StreamLM
from .weights import get_shaped, tp_range
from .weights import pad_zeros as _pad
from .weights import round_up as _up


@register_config("Taduzen")
def normalize_taduzen(cfg: dict) -> dict:
    """The keys the rest of the framework reads (HF spelling), next to the design's own."""
    layers = cfg["layers"]
    moe = [l["mlp"]["router"] for l in layers if l.get("mlp") and l["mlp"]["kind"] == "moe"]
    out = dict(cfg, model_type="taduzen", hidden_size=cfg["width"], vocab_size=cfg["vocab"],
               num_hidden_layers=len(layers), num_attention_heads=max(l["mixer"]["heads"] for l in layers),
               kv_lora_rank=max(_up(l["mixer"]["kv_rank"], 16) for l in layers), qk_rope_head_dim=0)
    if moe:
        out.update(num_experts=max(r["experts"] for r in moe), num_experts_per_tok=max(r["top"] for r in moe),
                   decoder_sparse_step=1, mlp_only_layers=[i for i, l in enumerate(layers)
                                                           if not l.get("mlp") or l["mlp"]["kind"] != "moe"])
    return out


class LayerSpec:
    """Sizes and constants of one layer."""

    def __init__(self, c: dict):
        if c["type"] != "latent_attention":
            raise ValueError(f"unknown mixer {c['type']!r}")
        m = c["mixer"]
        self.heads, self.dim, self.vdim, self.rank = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        self.scale = float(m["scale"])
        self.window = int((m.get("mask") or {}).get("size") or 0)
        self.dp, self.vp, self.rp = _up(self.dim, 64), _up(self.vdim, 64), _up(self.rank, 16)
        f = c.get("mlp")
        self.kind = f["kind"] if f else None
        self.moe = self.kind == "moe"
        if self.kind not in (None, "dense", "moe"):
            raise ValueError(f"unknown feed-forward {self.kind!r}")
        if self.kind == "dense":
            self.ff = f["ff"]
        elif self.kind == "moe":
            self.experts, self.top = f["router"]["experts"], f["router"]["top"]
            self.ff = f["expert"]["ff"]
            self.shared_ff = (f.get("shared") or {}).get("ff") or 0


@register_model("taduzen")
class TaduzenLM(StreamLM):
    model_type = "taduzen"
    native_units = ("dyt", "gemm_f32", "gemm_tcgen05", "latent_attn", "moe", "ops_basic", "sampling",
                    "window_prefill_tc")

    # ------------------------------------------------------------------ config
    def _read_config(self, c: dict):
        self.hidden, self.vocab = c["width"], c["vocab"]
        self.hidden_p = _up(self.hidden, 64)
        self.specs = [LayerSpec(l) for l in c["layers"]]
        self.num_layers = len(self.specs)
        self.eps = c["norm"]["eps"]
        self.logit_scale = float(c.get("logit_scale", 1.0))
        self.tie_embeddings = False
        self.kv_row = max(s.rp for s in self.specs)
        tp = self.tp.size
        for s in self.specs:
            assert s.heads % tp == 0, "heads must divide by tp"
        # what the engine reads of any model
        self.num_q_heads = max(s.heads for s in self.specs)
        self.num_kv_heads = self.hkv = 1
        self.hq = self.num_q_heads // tp
        self.head_dim = self.kv_row
        self.rot_dim = 0
        self.inter = None
        self._check_options()

    # ------------------------------------------------------------------ weights
    def weight_shapes(self) -> Dict[str, tuple]:
        W = self.hidden
        s = {"embed": (self.vocab, W), "head": (self.vocab, W)}

        def norm(name):
            s.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})

        def gated(p, ff):
            s.update({p + "gate": (ff, W), p + "up": (ff, W), p + "down": (W, ff)})

        norm("final.norm")
        for i, l in enumerate(self.specs):
            p = f"l{i}."
            norm(p + "norm1")
            norm(p + "norm1b")
            m = p + "mix."
            s.update({m + "q": (l.heads * l.dim, W), m + "dkv": (l.rank, W), m + "dkv.norm": (l.rank,),
                      m + "uk": (l.heads * l.dim, l.rank), m + "uv": (l.heads * l.vdim, l.rank),
                      m + "o": (W, l.heads * l.vdim)})
            if l.kind is None:
                continue
            norm(p + "norm2")
            norm(p + "norm2b")
            f = p + "mlp."
            if l.kind == "dense":
                s.update({f + "up": (l.ff, W), f + "down": (W, l.ff)})
                continue
            s[f + "table"] = (self.vocab, l.top)
            for e in range(l.experts):
                gated(f"{f}e{e}.", l.ff)
            if l.shared_ff:
                gated(f + "shared.", l.shared_ff)
                s[f + "shared.sg"] = (1, W)
        return s

    def weight_inits(self):
        """Random initialisation of what is not a matrix: unit norms, and tables of distinct experts."""
        def ones(shape, gen, device):
            return torch.ones(shape, dtype=self.dtype, device=device)

        def zeros(shape, gen, device):
            return torch.zeros(shape, dtype=self.dtype, device=device)

        def table(experts):
            def make(shape, gen, device):
                r = torch.rand((shape[0], experts), generator=gen, device=device)
                return r.topk(shape[1], dim=-1)[1].to(torch.int32)
            return make

        out = {}
        for name, shape in self.weight_shapes().items():
            if name.endswith(".b"):
                out[name] = zeros
            elif ".norm" in name:
                out[name] = ones
            elif name.endswith(".table"):
                out[name] = table(self.specs[int(name[1:].split(".")[0])].experts)
        return out

    def _load_norm(self, src, name) -> ops.DytNorm:
        W, P = self.hidden, self.hidden_p
        return ops.DytNorm(_pad(get_shaped(src, name, W).float(), P).to(self.device),
                           _pad(get_shaped(src, name + ".b", W).float(), P).to(self.device),
                           float(get_shaped(src, name + ".alpha").float()))

    def _load_weights(self, src):
        tp, r = self.tp.size, self.tp.rank
        W, P = self.hidden, self.hidden_p
        self._load_embed_and_head(src)
        self.final_norm = self._load_norm(src, "final.norm")
        self.layers, tables = [], []
        for i, l in enumerate(self.specs[: self.num_layers]):
            lw = LayerWeights()
            p = f"l{i}."
            lw.spec = l
            lw.norm1, lw.norm1b = self._load_norm(src, p + "norm1"), self._load_norm(src, p + "norm1b")
            self._load_mixer(lw, src, p + "mix.", l)
            if l.kind is not None:
                lw.norm2, lw.norm2b = self._load_norm(src, p + "norm2"), self._load_norm(src, p + "norm2b")
            if l.kind == "dense":
                i0, i1 = tp_range(l.ff, r, tp)
                I = _up(i1 - i0, 64)
                lw.up_w = self._dev(_pad(get_shaped(src, p + "mlp.up", l.ff, W)[i0:i1], I, P))
                lw.down_w = self._dev(_pad(get_shaped(src, p + "mlp.down", W, l.ff)[:, i0:i1], P, I))
            elif l.kind == "moe":
                tables.append(self._load_moe(lw, src, p + "mlp.", l))
                lw.moe_index = len(tables) - 1
            self.layers.append(lw)
        self.routing = moe_ops.TableRouting(tables) if tables else None

    def _load_mixer(self, lw, src, m, l: LayerSpec):
        W, P = self.hidden, self.hidden_p
        h0, h1 = tp_range(l.heads, self.tp.rank, self.tp.size)
        lw.heads = h1 - h0
        q = self._heads(src, m + "q", l.heads, l.dim, l.dp, h0, h1)
        dkv = get_shaped(src, m + "dkv", l.rank, W)
        lw.qkv_w = self._dev(torch.cat([q, _pad(dkv, l.rp, P)]))
        lw.kv_norm = self._dev(get_shaped(src, m + "dkv.norm", l.rank), torch.float32)
        uk = get_shaped(src, m + "uk", l.heads * l.dim, l.rank).view(l.heads, l.dim, l.rank)[h0:h1]
        uv = get_shaped(src, m + "uv", l.heads * l.vdim, l.rank).view(l.heads, l.vdim, l.rank)[h0:h1]
        lw.latent = LatentHeads(h1 - h0, l.dim, 0, l.vdim, l.rank, l.scale, l.window)
        lw.latent.load(lw, self._dev, uk, uv)
        lw.o_w = self._dev(self._out_heads(src, m + "o", l.heads, l.vdim, l.vp, h0, h1))

    def _load_moe(self, lw, src, p, l: LayerSpec):
        """Experts stacked as in `models/moe.py`; returns the routing entry (table, first expert, experts) of this rank."""
        tp, r = self.tp.size, self.tp.rank
        e0, e1 = self._load_experts(lw, src, p, l.experts, l.ff)
        if l.shared_ff:
            s0, s1 = tp_range(l.shared_ff, r, tp)
            a, b = self._load_gated(src, p + "shared.", l.shared_ff, s0, s1)
            lw.shared_gate_up_w, lw.shared_down_w = self._dev(a), self._dev(b)
            sg = get_shaped(src, p + "shared.sg", 1, self.hidden).float().view(-1)
            lw.shared_gate_w = self._dev(_pad(sg, self.hidden_p), torch.float32)
        table = get_shaped(src, p + "table", self.vocab, l.top).to(torch.int32)
        if int(table.min()) < 0 or int(table.max()) >= l.experts:
            raise ValueError(f"{p}table names an expert outside 0 .. {l.experts - 1}")
        return table.to(self.device).contiguous(), e0, e1 - e0

    def _init_rope(self):
        self.cos = self.sin = None     # no positions

    # ------------------------------------------------------------------ memory
    def kv_bytes_per_token(self):
        return MLAMemoryManager.bytes_per_token(self.dtype, self.kv_row, 0, self.num_layers)

    def _make_mem_manager(self, size):
        if self.extra.get("kv_type") not in (None, "none", "None"):
            raise ValueError("--llm_kv_type: the latent cache has no quantised form here")
        return MLAMemoryManager(size, self.dtype, self.kv_row, 0, self.num_layers, self.device)

    # ------------------------------------------------------------------ forward
    def _embed(self, ids, st):
        x, st.extra["first_normed"] = ops.embedding_dyt(ids, self.embed_w, self.layers[0].norm1)
        if self.routing is not None:
            st.extra["layouts"] = self.routing.layouts(ids)
            st.extra["token_ids"] = ids
        return x

    def _layers_forward(self, x, st: InferState):
        """x: the fp32 residual stream.  Returns the final norm's output."""
        h = st.extra.pop("first_normed")
        tap = self.stream_tap
        n = len(self.layers)
        for i, lw in enumerate(self.layers):
            after = self.layers[i + 1].norm1 if i + 1 < n else self.final_norm
            kind = lw.spec.kind
            a = self._attention_block(i, lw, h, st)
            h = self._project_dyt(a, lw.o_w, x, lw.norm1b, lw.norm2 if kind else after)
            if kind == "dense":
                h = self._project_dyt(ops.gemm(h, lw.up_w, epi="relu2"), lw.down_w, x, lw.norm2b, after)
            elif kind == "moe":
                h = self._moe(i, lw, h, x, after, st)
            if tap is not None:
                tap(i, x)
        st.extra["normed"] = True
        return h

    def _project_dyt(self, a, w, x, post, nxt):
        """x += post(a . w^T, summed over the tensor-parallel ranks); returns nxt(x)."""
        if self.tp.size == 1:
            return ops.gemm(a, w, epi="dyt", x=x, dyt=(post, nxt))
        return self._reduce_dyt(ops.gemm(a, w, epi="f32"), x, post, nxt)

    def _reduce_dyt(self, y, x, post, nxt):
        self.tp.all_reduce_(y)
        return ops.add_dyt_(x, y, post, nxt, self.dtype)

    def _moe(self, i, lw, h, x, after, st):
        lay = st.extra["layouts"][lw.moe_index]
        rc = self.route_capture
        if rc is not None:
            rc.capture(i, self.routing.ids(lw.moe_index, st.extra["token_ids"]), st.mem_index)
        shared = None
        if lw.shared_down_w is not None:
            shared = ops.gemm(ops.gemm(h, lw.shared_gate_up_w, epi="gated_silu"), lw.shared_down_w)
        one = self.tp.size == 1
        out = moe_ops.uniform_experts_dyt_(h, lay, lw.w13, lw.w2, "silu", shared, lw.shared_gate_w, x if one else None,
                                           lw.norm2b if one else None, after if one else None, lw.e0)
        return out if one else self._reduce_dyt(out, x, lw.norm2b, after)

    def _attention_block(self, i, lw, h, st: InferState):
        l = lw.spec
        qc = ops.gemm(h, lw.qkv_w)                               # [T, heads * dim | latent]
        q = qc[:, : lw.heads * l.dp]
        kv_layer = self._kv_layer(i)
        mla_ops.latent_norm_scatter_(qc[:, lw.heads * l.dp:], kv_layer, lw.kv_norm, st.mem_index, l.rank, self.eps)
        return lw.latent.attend(lw, q, kv_layer, self.req_manager.req_to_token_indexs, st)

    def _lm_head(self, h, normed: bool = True):
        assert normed, "the layer stack returns normalised rows"
        v = self.vocab // self.tp.size
        logits = ops.gemm(h, self.lm_head_w, epi="f32", out_scale=self.logit_scale)[:, :v]
        if self.tp.size == 1:
            return logits
        return ShardedLogits(logits.contiguous(), self.tp, self.tp.rank * v, self.vocab)
