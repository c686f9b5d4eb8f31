"""Plain, slow restatement of the Katarax decoder: one function per mechanism, whole sequences, no cache, torch on the CPU.
Shares nothing with the package; the tests compare the package with it.

`w` maps checkpoint names to tensors; everything runs in the number format of `DT` (float64 by default)."""
import math

import torch

DT = torch.float64


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(w, name, x, eps):
    """Norm whose stored weight is the distance from one."""
    return rms(x, eps) * (1 + w[name].to(DT))


def linear(w, name, h):
    return h @ w[name].to(DT).t()


def angles(rot, T, pos0=0):
    """[T, dims / 2]"""
    f = torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)], dtype=DT)
    return torch.arange(pos0, pos0 + T, dtype=DT)[:, None] * f


def turn(u, v, a):
    return u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()


def rotate_halves(x, rot, pos0=0):
    """x [T, heads, dim]: pairs (i, i + dims / 2) of the first rot.dims numbers of every head."""
    n = rot["dims"] // 2
    u, v = turn(x[..., :n], x[..., n:2 * n], angles(rot, x.shape[0], pos0)[:, None])
    return torch.cat([u, v, x[..., 2 * n:]], -1)


def rotate_neighbours(x, rot, pos0=0):
    """x [T, heads, dim]: pairs (2 i, 2 i + 1) of the first rot.dims numbers of every head."""
    n = rot["dims"]
    u, v = turn(x[..., 0:n:2], x[..., 1:n:2], angles(rot, x.shape[0], pos0)[:, None])
    return torch.cat([torch.stack([u, v], -1).flatten(-2), x[..., n:]], -1)


def visible(T, window=None, keep=0):
    """[T, T] mask: causal, through a window, the first `keep` positions always."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    m = j <= i
    return m if window is None else m & ((i - j < window) | (j < keep))


def bucket(n, rows, far):
    """Row of the distance table: one per distance up to half of the rows, the rest spaced by logarithm up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(table, T, far):
    """table [rows, H] -> [H, T, T] (entry [h, i, j] for key j at or before query i)."""
    rows = torch.tensor([bucket(n, table.shape[0], far) for n in range(T)])
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None]).clamp_min(0)
    return table.to(DT)[rows[dist]].permute(2, 0, 1)


def attend(q, k, v, scale, mask, bias=None):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim], mask [T, T], bias [H, T, T] or None -> [T, H, vdim]"""
    H, rep = q.shape[1], q.shape[1] // k.shape[1]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].t()) * scale
        if bias is not None:
            s = s + bias[h]
        out.append(torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ v[:, h // rep])
    return torch.stack(out, 1)


def mask_of(c, T):
    m = c.get("mask") or {}
    return visible(T, m.get("size"), m.get("keep_first", 0))


def keys_values(w, p, h, c, eps):
    T = h.shape[0]
    return (linear(w, p + "k", h).view(T, c["kv_heads"], c["dim"]), linear(w, p + "v", h).view(T, c["kv_heads"], c["vdim"]))


def biased_attention(w, p, h, c, eps, shared):
    T = h.shape[0]
    q = linear(w, p + "q", h).view(T, c["heads"], c["dim"])
    k, v = shared if shared is not None else keys_values(w, p, h, c, eps)
    o = attend(q, k, v, c["scale"], mask_of(c, T), distance_bias(w[p + "rel"], T, c["bias_max"]))
    return linear(w, p + "o", o.reshape(T, -1)), (k, v)


def rotated_attention(w, p, h, c, eps, shared):
    T = h.shape[0]

    def prepared(x):
        return rms(rotate_halves(x, c["rot"]), eps)

    q = prepared(linear(w, p + "q", h).view(T, c["heads"], c["dim"]))
    if shared is None:
        k, v = keys_values(w, p, h, c, eps)
        shared = prepared(k), v
    o = attend(q, *shared, c["scale"], mask_of(c, T))
    return linear(w, p + "o", o.reshape(T, -1)), shared


def latent_attention(w, p, h, c, eps, shared):
    T, H, D, R, rank = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    cq = rms(linear(w, p + "dq", h), eps) * w[p + "dq.norm"].to(DT)
    q = linear(w, p + "uq", cq).view(T, H, D + R)
    both = linear(w, p + "dkv", h)
    lat = rms(both[:, :rank], eps) * w[p + "dkv.norm"].to(DT)
    kr = rotate_neighbours(both[:, None, rank:], c["rot"])
    q = torch.cat([q[..., :D], rotate_neighbours(q[..., D:], c["rot"])], -1)
    k = torch.cat([linear(w, p + "uk", lat).view(T, H, D), kr.expand(T, H, R)], -1)
    v = linear(w, p + "uv", lat).view(T, H, c["vdim"])
    o = attend(q, k, v, c["scale"], mask_of(c, T)).reshape(T, -1)
    return linear(w, p + "o", o * torch.sigmoid(linear(w, p + "g", h))), None


def expert(w, p, h, limit):
    g = linear(w, p + "gate", h).clamp(max=limit)
    u = linear(w, p + "up", h).clamp(-limit, limit)
    return linear(w, p + "down", g * torch.sigmoid(1.702 * g) * (u + 1))


def route(w, p, h, c):
    """(experts [T, top], their weights)"""
    s = torch.sigmoid(linear(w, p + "router", h))
    choice = s + w[p + "correction"].to(DT)
    groups = choice.view(len(h), c["groups"]["count"], -1)
    best = groups.topk(2, -1)[0].sum(-1).topk(c["groups"]["keep"], -1)[1]
    closed = torch.ones(groups.shape[:2], dtype=torch.bool).scatter_(1, best, False)
    choice = groups.masked_fill(closed[..., None], float("-inf")).flatten(1)
    ids = choice.topk(c["top"], -1)[1]
    val = s.gather(1, ids)
    return ids, val / (val.sum(-1, keepdim=True) + 1e-20) * c["scale"]


def moe(w, p, h, c):
    ids, val = route(w, p, h, c["router"])
    y = torch.zeros_like(h)
    for e in range(c["router"]["experts"]):
        tok, slot = (ids == e).nonzero(as_tuple=True)
        if tok.numel():
            y.index_add_(0, tok, val[tok, slot, None] * expert(w, f"{p}e{e}.", h[tok], c["expert"]["limit"]))
    return y


MIXERS = {"attention": biased_attention, "attention_2": rotated_attention, "latent_attention": latent_attention}


def forward(w, cfg, tokens, streams=None):
    """Logits [T, vocab]; `streams` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"].to(DT)[list(tokens)]
    held = {}
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = centred_norm(w, p + "norm1", x, eps)
        y, held[i] = MIXERS[l["type"]](w, p + "mix.", h, l["mixer"], eps, held.get(l["mixer"].get("kv_from")))
        if l.get("mlp"):
            y = y + moe(w, p + "mlp.", h, l["mlp"])
        x = x + y
        if streams is not None:
            streams.append(x)
    z = linear(w, "head", centred_norm(w, "final.norm", x, eps))
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(z / cap)
