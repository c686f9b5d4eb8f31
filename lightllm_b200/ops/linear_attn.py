"""Linear attention with matrix states.  First the Gated DeltaNet (Qwen3-Next / Qwen3.5 hybrid layers) on torch ops, with
its decode kernels; at the end of the file `DecayedState`: gated linear attention with a decay per key channel, and the
matrix memory of xLSTM (mLSTM), on the kernels of `csrc/recurrent.cu`.

Per head the layer keeps a matrix state S [dk, dv] and updates it token by token:

    S <- exp(g_t) * S                               (decay)
    d  = beta_t * (v_t - S^T k_t)                   (what the state does not predict yet)
    S <- S + k_t d^T ,   o_t = S^T q_t

with q, k l2-normalised and q scaled by dk^-1/2.  `gated_delta_step` is that recurrence for one token of every
request of a decode batch; `gated_delta_chunked` processes a whole prompt in chunks of 64 tokens with matrix
products: inside a chunk with start state S0 and cumulative log-decay G_i the corrections D solve the unit lower
triangular system (I + A) D = beta * (V - exp(G) * K S0), A_ij = beta_i exp(G_i - G_j) (k_i . k_j) for j < i; then
O = exp(G) * Q S0 + (M * Q K^T) D with M_ij = exp(G_i - G_j) for j <= i, and the chunk's end state is
exp(G_C) S0 + (exp(G_C - G) * K)^T D.  A depthwise causal convolution (kernel 4, SiLU) runs over q, k, v first; its
state is the last kernel-1 inputs.

Reference: lightllm/models/qwen3next/ (triton_kernel/fla/*, causal_conv1d) and the flash-linear-attention kernels
it wraps.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F


def l2norm(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    return x * torch.rsqrt((x * x).sum(-1, keepdim=True) + eps)


def causal_conv_prefill(x: torch.Tensor, state: torch.Tensor, w: torch.Tensor):
    """x [T, C] new inputs of one request, state [C, K-1] (previous inputs, zeros for a fresh request), w [C, K].
    Returns (silu(conv) [T, C], new state [C, K-1])."""
    K = w.shape[1]
    full = torch.cat([state.to(x.dtype), x.t()], dim=1)           # [C, K-1+T]
    y = F.conv1d(full.unsqueeze(0), w.to(x.dtype).unsqueeze(1), groups=w.shape[0])[0]   # [C, T]
    return F.silu(y).t(), full[:, -(K - 1):].contiguous()


def causal_conv_step(x: torch.Tensor, state: torch.Tensor, w: torch.Tensor):
    """One token per request: x [B, C], state [B, C, K-1] -> (silu(conv) [B, C], new state)."""
    full = torch.cat([state.to(x.dtype), x.unsqueeze(-1)], dim=-1)  # [B, C, K]
    y = (full * w.to(x.dtype).unsqueeze(0)).sum(-1)
    return F.silu(y), full[:, :, 1:].contiguous()


def gated_delta_naive(q, k, v, g, beta, S0=None):
    """Token-by-token recurrence (the definition): q, k [T, H, dk], v [T, H, dv], g, beta [T, H] -> (o [T, H, dv], S)."""
    T, H, dk = k.shape
    dv = v.shape[-1]
    q = l2norm(q.float()) * dk ** -0.5
    k = l2norm(k.float())
    v, g, beta = v.float(), g.float(), beta.float()
    S = torch.zeros(H, dk, dv, dtype=torch.float32, device=q.device) if S0 is None else S0.float().clone()
    o = torch.empty(T, H, dv, dtype=torch.float32, device=q.device)
    for t in range(T):
        S = S * g[t].exp().view(H, 1, 1)
        d = (v[t] - torch.einsum("hkv,hk->hv", S, k[t])) * beta[t].unsqueeze(-1)
        S = S + k[t].unsqueeze(-1) * d.unsqueeze(-2)
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o, S


def gated_delta_step(q, k, v, g, beta, S):
    """One token of each request: q, k [B, H, dk], v [B, H, dv], g, beta [B, H], S [B, H, dk, dv] fp32.
    Returns (o [B, H, dv] fp32, new S)."""
    dk = k.shape[-1]
    q = l2norm(q.float()) * dk ** -0.5
    k = l2norm(k.float())
    S = S * g.float().exp().unsqueeze(-1).unsqueeze(-1)
    d = (v.float() - torch.einsum("bhkv,bhk->bhv", S, k)) * beta.float().unsqueeze(-1)
    S = S + k.unsqueeze(-1) * d.unsqueeze(-2)
    return torch.einsum("bhkv,bhk->bhv", S, q), S


def gated_delta_chunked(q, k, v, g, beta, S0=None, chunk: int = 64):
    """A prompt (or a chunk of it) of one request: shapes as `gated_delta_naive`; S0 [H, dk, dv] fp32 or None."""
    T, H, dk = k.shape
    dv = v.shape[-1]
    dev = q.device
    q = (l2norm(q.float()) * dk ** -0.5).transpose(0, 1)   # [H, T, dk]
    k = l2norm(k.float()).transpose(0, 1)
    v = v.float().transpose(0, 1)
    g = g.float().t()                                       # [H, T]
    beta = beta.float().t()
    S = torch.zeros(H, dk, dv, dtype=torch.float32, device=dev) if S0 is None else S0.float().clone()
    out = torch.empty(H, T, dv, dtype=torch.float32, device=dev)
    for s in range(0, T, chunk):
        e = min(s + chunk, T)
        C = e - s
        qc, kc, vc, bc = q[:, s:e], k[:, s:e], v[:, s:e], beta[:, s:e]
        G = g[:, s:e].cumsum(-1)                                     # [H, C], <= 0 and decreasing
        ratio = (G.unsqueeze(-1) - G.unsqueeze(-2))                  # G_i - G_j
        lower = torch.tril(torch.ones(C, C, dtype=torch.bool, device=dev))
        M = torch.where(lower, ratio, torch.full_like(ratio, float("-inf"))).exp()   # exp(G_i - G_j), j <= i
        kk = kc @ kc.transpose(-1, -2)                               # k_i . k_j
        A = (bc.unsqueeze(-1) * M * kk).tril(-1)
        eG = G.exp().unsqueeze(-1)
        rhs = bc.unsqueeze(-1) * (vc - eG * (kc @ S))
        eye = torch.eye(C, dtype=torch.float32, device=dev).expand(H, C, C)
        D = torch.linalg.solve_triangular(eye + A, rhs, upper=False, unitriangular=True)
        out[:, s:e] = eG * (qc @ S) + (M * (qc @ kc.transpose(-1, -2))) @ D
        tail = (G[:, -1:] - G).exp().unsqueeze(-1)                   # exp(G_C - G_j)
        S = G[:, -1].exp().view(H, 1, 1) * S + (kc * tail).transpose(-1, -2) @ D
    return out.transpose(0, 1), S


def conv_and_delta_step(mixed, conv_state, conv_w_f32, ssm_state, req, g, beta, nk: int, nv: int, dk: int, dv: int):
    """The decode step of one Gated DeltaNet layer for a batch, two kernels (csrc/linear_attn.cu): convolution step
    over the q / k / v channels, then per (request, value head) the normalisation of q and k, the state update and the
    read-out, with the state row strips held in registers (one read and one write of the state).  Updates
    `conv_state [slots, C, K-1]` and `ssm_state [slots, nv, dk, dv]` (fp32 or bf16) in place at rows `req`.

    mixed [B, C] fp32, conv_w_f32 [C, K] fp32, req [B] int32, g / beta [B, nv] fp32 -> core [B, nv, dv] fp32."""
    import ctypes

    from . import _count
    from ._native import check, kernels, ptr, stream

    B, C = mixed.shape
    K = conv_w_f32.shape[1]
    assert mixed.dtype == torch.float32 and mixed.is_contiguous() and C == 2 * nk * dk + nv * dv
    assert conv_state.is_contiguous() and ssm_state.is_contiguous() and req.dtype == torch.int32
    assert conv_state.dtype in (torch.float32, torch.bfloat16) and ssm_state.dtype in (torch.float32, torch.bfloat16)
    g, beta = g.contiguous(), beta.contiguous()
    y = torch.empty_like(mixed)
    ci = ctypes.c_int
    check(kernels().llb_gdn_conv_step(ptr(mixed), ptr(conv_state), ci(int(conv_state.dtype == torch.bfloat16)),
                                      ptr(conv_w_f32), ptr(req), ptr(y), ci(B), ci(C), ci(K), stream()),
          "gdn_conv_step")
    core = torch.empty((B, nv, dv), dtype=torch.float32, device=mixed.device)
    check(kernels().llb_gdn_recurrent_step(ptr(y), ptr(g), ptr(beta), ptr(ssm_state),
                                           ci(int(ssm_state.dtype == torch.bfloat16)), ptr(req), ptr(core), ci(B),
                                           ci(nk), ci(nv), ci(dk), ci(dv), stream()), "gdn_recurrent_step")
    _count(2)
    return core


def step_kernel_supported(dk: int, dv: int, K: int) -> bool:
    """Shapes the decode-step kernels take: the value head fits a CTA in whole warps (dv a multiple of 32, at most
    256) and a thread's strip of a state column fits its registers (dk <= 64 x (256 // dv))."""
    return dv % 32 == 0 and 32 <= dv <= 256 and 1 <= K <= 16 and 1 <= dk <= 64 * (256 // dv)


def rmsnorm_gated(x: torch.Tensor, z: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """norm(x) * w * silu(z) over the last dimension (the norm sees x alone; z only gates)."""
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (w.float() * y * F.silu(z.float())).to(z.dtype)


# ---------------------------------------------------------------- states with decays (GLA, mLSTM)
CHUNK = 64


class ChunkPlan:
    """The chunks (64 tokens) of a prompt pass: first token row, length and request of every chunk, chunks of every request."""

    def __init__(self, q_len: torch.Tensor, device, size: int = CHUNK):
        q_len = q_len.to(torch.int64)
        n = (q_len + size - 1) // size
        zero = torch.zeros(1, dtype=torch.int64)
        cu_q, cu_c = torch.cat([zero, q_len.cumsum(0)]), torch.cat([zero, n.cumsum(0)])
        self.count = int(cu_c[-1])
        b = torch.repeat_interleave(torch.arange(len(q_len)), n)
        off = (torch.arange(self.count) - cu_c[b]) * size
        tok0, length = cu_q[b] + off, (q_len[b] - off).clamp_max(size)
        host = torch.cat([tok0, length, b, cu_c]).to(torch.int32)
        dev = host.to(device, non_blocking=True)
        self.tok0, self.len, self.req, self.cu_chunk = torch.split(dev, [self.count] * 3 + [len(q_len) + 1])


class DecayedState:
    """One layer's recurrence S_t = diag(a_t) S_(t-1) + b_t k_t v_t^T, o_t = dim^(-1/2) S_t^T q_t over per-request states,
    with its output step: RMS norm of every head over its values, times a weight, times silu(g) or sigmoid(g).

    kind "gla":    a = sigmoid(z)^(1 / tau) per key channel, z = a2 (a1 h) + bias; b = 1; silu(g).
    kind "mlstm":  log gates i = cap tanh(zi / cap), f = logsigmoid(cap tanh(zf / cap)) per head, a running maximum m (0 at
                   the start) that keeps the exponentials in range, a normaliser n; sigmoid(g).

    dk, dv: padded head sizes (multiples of 16), dim, vdim: the true ones.  weight: fp32 [dv] or [H * dv]."""

    def __init__(self, kind: str, H: int, dk: int, dv: int, dim: int, vdim: int, eps: float, weight: torch.Tensor,
                 tau: float = 1.0, a2=None, a2_bias=None, cap: float = 1.0, out_scale: float = 1.0):
        assert kind in ("gla", "mlstm") and dk % 16 == 0 and dv % 16 == 0
        self.kind, self.H, self.dk, self.dv, self.dim, self.vdim = kind, H, dk, dv, dim, vdim
        self.eps, self.tau, self.cap, self.out_scale = float(eps), float(tau), float(cap), float(out_scale)
        self.weight, self.a2, self.a2_bias = weight, a2, a2_bias
        assert weight.dtype == torch.float32 and weight.numel() in (dv, H * dv)
        self.w_stride = 0 if weight.numel() == dv else dv
        self.rank = 0 if a2 is None else a2.shape[1]

    @staticmethod
    def state_elems(kind: str, H: int, dk: int, dv: int) -> int:
        return H * dk * dv + (H * (dk + 1) if kind == "mlstm" else 0)

    @staticmethod
    def chunked_sizes(dk: int, dv: int, rank: int) -> bool:
        return dk <= 256 and dv <= 512 and rank <= 128 and rank % 8 == 0

    def __call__(self, q, k, v, g, state, st, a1=None, zi=None, zf=None, out=None, plan=None, token_by_token=False):
        """q, k [T, H * dk], v, g [T, H * dv] (columns of one matrix, or with its row pitch); a1 [T, rank] likewise; zi, zf
        fp32 [T, H] with one row pitch; state [slots, elems].  Prompt passes in bf16 run chunked (`plan`), everything else
        token by token."""
        T = q.shape[0]
        if out is None:
            out = torch.empty((T, self.H * self.dv), dtype=q.dtype, device=q.device)
        first = st.b_ready_cache_len if st.is_prefill else st.seq_pos
        if not q.is_cuda:
            return self._torch(q, k, v, g, state, st, a1, zi, zf, out)
        from . import DTYPE_CODES, _count
        from ._native import c_int, check, f32, i64, kernels, ptr, stream

        ld = q.stride(0)
        assert all(t.stride(0) == ld and t.stride(1) == 1 for t in (q, k, v, g)) and state.stride(1) == 1
        assert a1 is None or a1.stride(0) == ld
        ldz = 0 if zi is None else zi.stride(0)
        kind = 0 if self.kind == "gla" else 1
        common = (ptr(q), ptr(k), ptr(v), ptr(g), i64(ld), ptr(a1), ptr(self.a2), ptr(self.a2_bias), c_int(self.rank),
                  f32(1.0 / self.tau), ptr(zi), ptr(zf), i64(ldz), f32(self.cap), ptr(state), i64(state.stride(0)),
                  ptr(self.weight), c_int(self.w_stride), f32(self.eps), ptr(out), i64(out.stride(0)), f32(self.out_scale),
                  ptr(st.b_req_idx))
        sizes = (c_int(st.batch_size), c_int(self.H), c_int(self.dk), c_int(self.dv), c_int(self.dim), c_int(self.vdim),
                 stream())
        chunked = st.is_prefill and q.dtype == torch.bfloat16 and not token_by_token and \
            self.chunked_sizes(self.dk, self.dv, self.rank)
        if not chunked:
            check(kernels().llb_recurrent_scan(c_int(kind), c_int(DTYPE_CODES[q.dtype]), *common,
                                               ptr(st.cu_q if st.is_prefill else None), ptr(first), *sizes),
                  "recurrent_scan")
            _count()
            return out
        n, dev = plan.count, q.device
        decay = torch.empty(T * self.H * (self.dk if kind == 0 else 3), dtype=torch.float32, device=dev)
        total = torch.empty(n * self.H * (self.dk if kind == 0 else 1), dtype=torch.float32, device=dev)
        m_prev, norms = None, (None, None)
        if kind == 1:
            m_prev = torch.empty(n * self.H, dtype=torch.float32, device=dev)
            norms = torch.empty((2, n * self.H * self.dk), dtype=torch.float32, device=dev)
        local = torch.empty(n * self.H * self.dk * self.dv, dtype=torch.float32, device=dev)
        planes = torch.empty((2, n * self.H * self.dk * self.dv), dtype=torch.bfloat16, device=dev)
        check(kernels().llb_recurrent_chunks(c_int(kind), *common, ptr(first), ptr(plan.tok0), ptr(plan.len),
                                             ptr(plan.cu_chunk), ptr(decay), ptr(total), ptr(m_prev), ptr(norms[0]),
                                             ptr(norms[1]), ptr(local), ptr(planes[0]), ptr(planes[1]), c_int(T), c_int(n), *sizes),
              "recurrent_chunks")
        _count(4)
        return out

    def _torch(self, q, k, v, g, state, st, a1, zi, zf, out):
        """Token by token on torch ops (CPU tensors)."""
        H, dk, dv = self.H, self.dk, self.dv
        T = q.shape[0]
        qf, kf = q.float().view(T, H, dk) * self.dim ** -0.5, k.float().view(T, H, dk)
        vf, gf = v.float().view(T, H, dv), g.float().view(T, H, dv)
        if self.kind == "gla":
            z = a1.float() @ self.a2.float().t() + self.a2_bias
            decay = torch.exp(F.logsigmoid(z) / self.tau).view(T, H, dk)
        else:
            li = self.cap * torch.tanh(zi / self.cap)
            lf = F.logsigmoid(self.cap * torch.tanh(zf / self.cap))
        ends = st.cu_q.tolist() if st.is_prefill else list(range(T + 1))
        first = (st.b_ready_cache_len if st.is_prefill else st.seq_pos).tolist()
        weight = self.weight.view(-1, dv)
        o = torch.empty(T, H, dv)
        for b, r in enumerate(st.b_req_idx.tolist()):
            row = state[r]
            if first[b] == 0:
                row.zero_()
            S = row[: H * dk * dv].view(H, dk, dv)
            n, m = (row[H * dk * dv: H * dk * (dv + 1)].view(H, dk), row[H * dk * (dv + 1):]) \
                if self.kind == "mlstm" else (None, None)
            for t in range(ends[b], ends[b + 1]):
                if self.kind == "gla":
                    S.mul_(decay[t].unsqueeze(-1)).add_(kf[t].unsqueeze(-1) * vf[t].unsqueeze(1))
                    o[t] = torch.einsum("hdv,hd->hv", S, qf[t])
                    continue
                m1 = torch.maximum(lf[t] + m, li[t])
                a, kb = torch.exp(lf[t] + m - m1)[:, None], torch.exp(li[t] - m1)[:, None] * kf[t]
                S.mul_(a.unsqueeze(-1)).add_(kb.unsqueeze(-1) * vf[t].unsqueeze(1))
                n.mul_(a).add_(kb)
                m.copy_(m1)
                den = torch.maximum((n * qf[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
                o[t] = torch.einsum("hdv,hd->hv", S, qf[t]) / den[:, None]
        o = o * torch.rsqrt(o.square().sum(-1, keepdim=True) / self.vdim + self.eps) * weight * self.out_scale
        gate = torch.sigmoid(gf) * (gf if self.kind == "gla" else 1.0)
        out.copy_((o * gate).view(T, H * dv))
        return out


# ---------------------------------------------------------------- elementwise gated states (minGRU)
SHORT_SCAN = 16       # passes whose portions are at most this long run token by token
SCAN_CHUNKS = 128


def scan_plan(q_len: torch.Tensor, device):
    """Chunks of a prompt pass for `gated_scan`: at most SCAN_CHUNKS per request, so that composing the earlier ones stays cheap;
    None when all portions are short."""
    longest = int(q_len.max())
    return ChunkPlan(q_len, device, CHUNK * max(1, -(-longest // (SCAN_CHUNKS * CHUNK)))) if longest > SHORT_SCAN else None


def gated_scan(z, x, g, state, st, dtype, plan=None):
    """minGRU over per-request states: S = (1 - sigmoid(z)) S + sigmoid(z) c(x), c(x) = x + 1/2 where x >= 0, else sigmoid(x); returns
    S * silu(g) [T, n] in `dtype`.  z, x, g [T, n]: columns of one matrix; state fp32 [slots, n] (any row pitch); plan
    (`scan_plan`): the chunks of a prompt pass, None: token by token."""
    T, n = z.shape
    first = st.b_ready_cache_len if st.is_prefill else st.seq_pos
    if not z.is_cuda:
        zf, xf, gf = z.float(), x.float(), g.float()
        keep, add = torch.sigmoid(-zf), torch.sigmoid(zf) * torch.where(xf >= 0, xf + 0.5, torch.sigmoid(xf))
        ends = st.cu_q.tolist() if st.is_prefill else list(range(T + 1))
        s = torch.empty(T, n)
        for b, r in enumerate(st.b_req_idx.tolist()):
            row = state[r]
            if first[b] == 0:
                row.zero_()
            for t in range(ends[b], ends[b + 1]):
                row.mul_(keep[t]).add_(add[t])
                s[t] = row
        return (s * F.silu(gf)).to(dtype)
    from . import DTYPE_CODES, _count
    from ._native import c_int, check, i64, kernels, ptr, stream

    ld = z.stride(0)
    assert x.stride(0) == ld and g.stride(0) == ld and z.stride(1) == x.stride(1) == g.stride(1) == 1
    assert z.dtype == x.dtype == g.dtype and state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] == n
    out = torch.empty((T, n), dtype=dtype, device=z.device)
    common = (ptr(z), ptr(x), ptr(g), c_int(DTYPE_CODES[z.dtype]), i64(ld), ptr(out), c_int(DTYPE_CODES[dtype]), i64(n), ptr(state),
              i64(state.stride(0)), ptr(st.b_req_idx))
    if plan is None:
        check(kernels().llb_gated_scan(*common, ptr(st.cu_q if st.is_prefill else None), ptr(first), c_int(st.batch_size), c_int(n),
                                       stream()), "gated_scan")
        _count()
        return out
    steps = torch.empty((2 * plan.count + st.batch_size, n), dtype=torch.float32, device=z.device)
    check(kernels().llb_gated_chunks(*common, ptr(first), ptr(plan.tok0), ptr(plan.len), ptr(plan.cu_chunk), ptr(plan.req),
                                     ptr(steps), ptr(steps[plan.count:]), ptr(steps[2 * plan.count:]), c_int(plan.count), c_int(n),
                                     stream()), "gated_chunks")
    _count(2)
    return out
