"""Plain, slow restatement of the Taduzen decoder, one function per mechanism, in the number format of its inputs.

It shares no code with the package: the tests compare the framework with it.  A model is a dict of tensors under the
checkpoint's names plus the config dict; a sequence is processed whole, with no cache.
"""
import torch


def dyt(x, w, b, alpha):
    """Dynamic tanh: elementwise, no statistics."""
    return torch.tanh(alpha * x) * w + b


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def visible(n_query, n_key, first_query, window):
    """[n_query, n_key] bool: a query sees its own position and the window - 1 before it; the first query stands at
    position first_query, the first key at 0."""
    i = torch.arange(first_query, first_query + n_query)[:, None]
    j = torch.arange(n_key)[None, :]
    d = i - j
    return (d >= 0) & (d < window)


def latent_of(h, w_dkv, w_norm, eps):
    return rms(h @ w_dkv.t(), w_norm, eps)


def latent_attention_core(q, c, w_uk, w_uv, heads, scale, mask):
    """q [n, heads * dim], c [m, rank] -> [n, heads * vdim]."""
    n, m = q.shape[0], c.shape[0]
    qh = q.view(n, heads, -1)
    k = (c @ w_uk.t()).view(m, heads, -1)
    v = (c @ w_uv.t()).view(m, heads, -1)
    s = torch.einsum("nhd,mhd->hnm", qh, k) * scale
    s = s.masked_fill(~mask[None], float("-inf"))
    p = torch.softmax(s, dim=-1)
    return torch.einsum("hnm,mhd->nhd", p, v).reshape(n, -1)


def latent_attention(t, p, h, cfg, eps):
    q = h @ t[p + "q"].t()
    c = latent_of(h, t[p + "dkv"], t[p + "dkv.norm"], eps)
    n = h.shape[0]
    size = (cfg.get("mask") or {}).get("size") or n
    o = latent_attention_core(q, c, t[p + "uk"], t[p + "uv"], cfg["heads"], cfg["scale"], visible(n, n, 0, size))
    return o @ t[p + "o"].t()


def relu_squared_mlp(h, up, down):
    a = torch.relu(h @ up.t())
    return (a * a) @ down.t()


def silu(z):
    return z / (1 + torch.exp(-z))


def gated_mlp(h, gate, up, down):
    return (silu(h @ gate.t()) * (h @ up.t())) @ down.t()


def table_experts(tokens, table):
    """Expert ids of every token: a row of the table per token id."""
    return table[tokens].long()


def moe(t, p, h, tokens, cfg):
    r = cfg["router"]
    ids = table_experts(tokens, t[p + "table"])
    out = torch.zeros_like(h)
    for n in range(h.shape[0]):
        for e in ids[n].tolist():
            q = f"{p}e{e}."
            out[n] += gated_mlp(h[n:n + 1], t[q + "gate"], t[q + "up"], t[q + "down"])[0] / r["top"]
    if cfg.get("shared"):
        q = p + "shared."
        g = torch.sigmoid(h @ t[q + "sg"].t())
        out = out + g * gated_mlp(h, t[q + "gate"], t[q + "up"], t[q + "down"])
    return out


def feed_forward(t, p, h, tokens, cfg):
    if cfg["kind"] == "dense":
        return relu_squared_mlp(h, t[p + "up"], t[p + "down"])
    return moe(t, p, h, tokens, cfg)


def norm(t, name, x):
    return dyt(x, t[name], t[name + ".b"], t[name + ".alpha"])


def forward(t, cfg, tokens, dtype=torch.float64, stream=None):
    """Logits [n, vocab] of one sequence; `stream` (a list) receives the residual stream after every layer."""
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in t.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = t["embed"][tokens]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = latent_attention(t, p + "mix.", norm(t, p + "norm1", x), layer["mixer"], cfg["norm"]["eps"])
        x = x + norm(t, p + "norm1b", m)
        if layer.get("mlp"):
            f = feed_forward(t, p + "mlp.", norm(t, p + "norm2", x), tokens, layer["mlp"])
            x = x + norm(t, p + "norm2b", f)
        if stream is not None:
            stream.append(x)
    return (norm(t, "final.norm", x) @ t["head"].t()) * cfg.get("logit_scale", 1.0)
