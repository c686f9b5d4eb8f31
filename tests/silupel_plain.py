"""Plain, slow restatement of the Silupel decoder: one function per mechanism, whole sequences, no cache, torch on the CPU.
Shares nothing with the package; the tests compare the package with it.

`w` maps checkpoint names to tensors; everything runs in the number format of `DT` (float64 by default)."""
import math

import torch

DT = torch.float64


def layer_norm(x, weight, eps):
    """Centred, divided by the root of the mean squared deviation, times a weight."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight.to(DT)


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight.to(DT)


def token_shift(h, mu):
    """Every element moves by its own share mu towards the row of the token before (zeros ahead of the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu.to(DT)


def linear(w, name, h):
    y = h @ w[name].to(DT).t()
    return y + w[name + ".b"].to(DT) if name + ".b" in w else y


def frequencies(rot):
    """[dims / 2] angles per position; long wavelengths are stretched when the rotation has a scaling."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            turns = s["original"] * f / (2 * math.pi)          # rotations within the original context
            if turns < s["low"]:
                f = f / s["factor"]
            elif turns <= s["high"]:
                t = (turns - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return torch.tensor(out, dtype=DT)


def rotate_halves(x, rot, pos0=0):
    """x [T, heads, dim]: pairs (i, i + dims / 2) of the first rot.dims numbers of every head."""
    n = rot["dims"] // 2
    a = (torch.arange(pos0, pos0 + x.shape[0], dtype=DT)[:, None] * frequencies(rot))[:, None]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), x[..., 2 * n:]], -1)


def visible(T, chunk=None):
    """[T, T] mask: causal, and inside the query's own chunk of positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    m = j <= i
    return m if chunk is None else m & (i // chunk == j // chunk)


def attend(q, k, v, scale, mask, cap=None):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim], scale: one number per head -> [T, H, vdim]"""
    H, rep = q.shape[1], q.shape[1] // k.shape[1]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].t()) * scale[h]
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        out.append(torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ v[:, h // rep])
    return torch.stack(out, 1)


def chunk_attention(w, p, h, c, eps):
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q = rotate_halves(linear(w, p + "q", h).view(T, H, c["dim"]), c["rot"])
    k = rotate_halves(linear(w, p + "k", h).view(T, G, c["dim"]), c["rot"])
    v = linear(w, p + "v", h).view(T, G, c["vdim"])
    o = attend(q, k, v, c["scale"] * w[p + "temp"].to(DT), visible(T, c["mask"]["size"]), c["softcap"])
    return linear(w, p + "o", o.reshape(T, -1) * torch.sigmoid(linear(w, p + "g", h)))


def latent_attention(w, p, h, c, eps):
    T, H, D, R, rank = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["kv_rank"]
    q = linear(w, p + "uq", rms_norm(linear(w, p + "dq", h), w[p + "dq.norm"], eps)).view(T, H, D + R)
    both = linear(w, p + "dkv", h)
    lat = rms_norm(both[:, :rank], w[p + "dkv.norm"], eps)
    shared = rotate_halves(both[:, None, rank:], c["rot"])
    q = torch.cat([q[..., :D], rotate_halves(q[..., D:], c["rot"])], -1)
    k = torch.cat([linear(w, p + "uk", lat).view(T, H, D), shared.expand(T, H, R)], -1)
    v = linear(w, p + "uv", lat).view(T, H, c["vdim"])
    return linear(w, p + "o", attend(q, k, v, [c["scale"]] * H, visible(T)).reshape(T, -1))


def mingru(w, p, h, c, eps):
    z = torch.sigmoid(linear(w, p + "z", h))
    u = linear(w, p + "x", h)
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    s, rows = torch.zeros_like(u[0]), []
    for t in range(h.shape[0]):
        s = (1 - z[t]) * s + z[t] * cand[t]
        rows.append(s)
    g = linear(w, p + "g", h)
    return linear(w, p + "o", torch.stack(rows) * g * torch.sigmoid(g))


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense(w, p, h):
    return linear(w, p + "down", gelu(linear(w, p + "gate", h)) * linear(w, p + "up", h))


def layer_order(cfg):
    """Layer indices in the order in which they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


MIXERS = {"mingru": mingru, "attention": chunk_attention, "latent_attention": latent_attention}


def forward(w, cfg, tokens, streams=None):
    """Logits [T, vocab]; `streams` (a list) receives the residual stream after every layer that runs."""
    eps = cfg["norm"]["eps"]
    x = w["embed"].to(DT)[list(tokens)]
    for i in layer_order(cfg):
        l, p = cfg["layers"][i], f"l{i}."
        h = token_shift(layer_norm(x, w[p + "norm1"], eps), w[p + "shift"])
        x = x + MIXERS[l["type"]](w, p + "mix.", h, l["mixer"], eps)
        if l.get("mlp"):
            x = x + dense(w, p + "mlp.", layer_norm(x, w[p + "norm2"], eps))
        if streams is not None:
            streams.append(x)
    return linear(w, "head", layer_norm(x, w["final.norm"], eps))
