"""Plain, slow restatement of the Libulorn decoder: one function per mechanism, whole sequences, no cache, torch on the CPU.
Shares nothing with the package; the tests compare the package with it.

`w` maps checkpoint names to tensors; everything runs in the number format of `DT` (float64 by default)."""
import math

import torch

DT = torch.float64


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def linear(w, name, h):
    return h @ w[name].to(DT).t()


def bigram_rows(tokens, c):
    rows, prev = [], None
    for t in tokens:
        rows.append(c["buckets"] if prev is None else (prev * c["mul_prev"] + t * c["mul_cur"]) % c["buckets"])
        prev = t
    return rows


def embed(w, tokens, cfg):
    return w["embed"].to(DT)[list(tokens)] + w["bigram"].to(DT)[bigram_rows(tokens, cfg["embedding"]["bigram"])]


def frequencies(rot):
    n = rot["dims"] // 2
    out = []
    for i in range(n):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2 * math.pi / f
            if wave < s["original"] / s["high"]:
                pass
            elif wave > s["original"] / s["low"]:
                f = f / s["factor"]
            else:
                a = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - a) * f / s["factor"] + a * f
        out.append(f)
    return torch.tensor(out, dtype=DT)


def rotate(x, rot, pos0=0):
    """x [T, heads, dim]: the first rot.dims numbers of every head, as pairs (i, i + dims / 2)."""
    T, n = x.shape[0], rot["dims"] // 2
    ang = (torch.arange(pos0, pos0 + T, dtype=DT)[:, None] * frequencies(rot)).unsqueeze(1)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * ang.cos() - v * ang.sin(), v * ang.cos() + u * ang.sin(), x[..., 2 * n:]], -1)


def window_attention(q, k, v, scale, window):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]"""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=DT)
    for i in range(T):
        lo = max(0, i - window + 1)
        for h in range(H):
            s = (k[lo:i + 1, h // rep] @ q[i, h]) * scale
            out[i, h] = torch.softmax(s, 0) @ v[lo:i + 1, h // rep]
    return out


def window_attention_fast(q, k, v, scale, window):
    """The same with one mask (for long sequences)."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    hide = ~((j <= i) & (i - j < window))
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].t()) * scale
        out.append(torch.softmax(s.masked_fill(hide, float("-inf")), -1) @ v[:, h // rep])
    return torch.stack(out, 1)


def attention_mixer(w, p, h, c, eps):
    T = h.shape[0]
    q = linear(w, p + "q", h).view(T, c["heads"], c["dim"])
    k = linear(w, p + "k", h).view(T, c["kv_heads"], c["dim"])
    v = linear(w, p + "v", h).view(T, c["kv_heads"], c["vdim"])
    q = rotate(rms(q, eps) * w[p + "q.norm"].to(DT), c["rot"])
    k = rotate(rms(k, eps) * w[p + "k.norm"].to(DT), c["rot"])
    o = window_attention_fast(q, k, v, c["scale"], c["mask"]["size"])
    o = o * torch.sigmoid(linear(w, p + "g", h)).unsqueeze(-1)
    return linear(w, p + "o", o.reshape(T, -1))


def gated_linear_recurrence(q, k, v, decay, S=None):
    """q, k, decay [T, H, dim], v [T, H, vdim]; S [H, dim, vdim] -> (o [T, H, vdim], S)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=DT) if S is None else S.clone()
    out = []
    for t in range(T):
        S = decay[t].unsqueeze(-1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(1)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gated_linear_mixer(w, p, h, c, eps):
    T, H, D = h.shape[0], c["heads"], c["dim"]
    q = linear(w, p + "q", h).view(T, H, D) * D ** -0.5
    k = linear(w, p + "k", h).view(T, H, D)
    v = linear(w, p + "v", h).view(T, H, c["vdim"])
    z = linear(w, p + "a2", linear(w, p + "a1", h)) + w[p + "a2.b"].to(DT)
    decay = torch.sigmoid(z).pow(1.0 / c["tau"]).view(T, H, D)
    o, _ = gated_linear_recurrence(q, k, v, decay)
    o = (rms(o, eps) * w[p + "norm"].to(DT)).reshape(T, -1)
    g = linear(w, p + "g", h)
    return linear(w, p + "o", o * g * torch.sigmoid(g))


def parallel_mixer(w, p, h, c, eps):
    return c["left_scale"] * attention_mixer(w, p + "left.", h, c["left"], eps) + \
        c["right_scale"] * gated_linear_mixer(w, p + "right.", h, c["right"], eps)


def mlstm_recurrence(q, k, v, i, f, state=None):
    """q, k [T, H, dim], v [T, H, vdim], log gates i, f [T, H] -> (o, (S, n, m))."""
    T, H, D = q.shape
    if state is None:
        state = torch.zeros(H, D, v.shape[-1], dtype=DT), torch.zeros(H, D, dtype=DT), torch.zeros(H, dtype=DT)
    S, n, m = (s.clone() for s in state)
    out = []
    for t in range(T):
        m1 = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - m1)[:, None], torch.exp(i[t] - m1)[:, None]
        S = a.unsqueeze(-1) * S + (b * k[t]).unsqueeze(-1) * v[t].unsqueeze(1)
        n = a * n + b * k[t]
        m = m1
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None])
    return torch.stack(out), (S, n, m)


def mlstm_gates(zi, zf, cap):
    return cap * torch.tanh(zi / cap), torch.nn.functional.logsigmoid(cap * torch.tanh(zf / cap))


def mlstm_mixer(w, p, h, c, eps):
    T, H, D = h.shape[0], c["heads"], c["dim"]
    q = linear(w, p + "q", h).view(T, H, D) * D ** -0.5
    k = linear(w, p + "k", h).view(T, H, D)
    v = linear(w, p + "v", h).view(T, H, c["vdim"])
    i, f = mlstm_gates(linear(w, p + "i", h) + w[p + "i.b"].to(DT), linear(w, p + "f", h) + w[p + "f.b"].to(DT),
                       c["gate_cap"])
    o, _ = mlstm_recurrence(q, k, v, i, f)
    o = rms(o, eps).reshape(T, -1) * w[p + "norm"].to(DT)
    return linear(w, p + "o", o * torch.sigmoid(linear(w, p + "g", h)))


def expert(w, p, h, limit):
    g = linear(w, p + "gate", h).clamp(max=limit)
    u = linear(w, p + "up", h).clamp(-limit, limit)
    return linear(w, p + "down", g * torch.sigmoid(1.702 * g) * (u + 1))


def route(w, p, h, c):
    """(experts [T, top], their weights)"""
    s = torch.softmax(linear(w, p + "router", h), -1)
    val, ids = s.topk(c["top"], -1)
    return ids, val


def moe(w, p, h, c):
    ids, val = route(w, p, h, c["router"])
    y = torch.zeros_like(h)
    for e in range(c["router"]["experts"]):
        tok, slot = (ids == e).nonzero(as_tuple=True)
        if tok.numel():
            y.index_add_(0, tok, val[tok, slot, None] * expert(w, f"{p}e{e}.", h[tok], c["expert"]["limit"]))
    if c.get("shared"):
        y = y + expert(w, p + "shared.", h, c["shared"]["limit"])
    return y


MIXERS = {"parallel": parallel_mixer, "mlstm": mlstm_mixer}


def forward(w, cfg, tokens, streams=None):
    """Logits [T, vocab]; `streams` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = embed(w, tokens, cfg)
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + rms(MIXERS[l["type"]](w, p + "mix.", x, l["mixer"], eps), eps) * w[p + "norm1"].to(DT)
        if l.get("mlp"):
            x = x + rms(moe(w, p + "mlp.", x, l["mlp"]), eps) * w[p + "norm2"].to(DT)
        if streams is not None:
            streams.append(x)
    return linear(w, "head", rms(x, eps) * w["final.norm"].to(DT))
