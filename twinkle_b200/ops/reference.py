"""Plain-PyTorch fp32 restatement of every hand-written kernel.

These functions are (a) the oracle the CUDA kernels are tested against and
(b) the path taken on CPU tensors (gloo tests).  They favour clarity over
speed and never call a fused library kernel.
"""
from __future__ import annotations

import math
from typing import List, Optional, Tuple

import torch
import torch.nn.functional as F


# --------------------------------------------------------------------- norms
def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float = 1e-6, offset: float = 0.0) -> torch.Tensor:
    xf = x.float()
    inv = torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (xf * inv * (weight.float() + offset)).to(x.dtype)


def add_rmsnorm(x: torch.Tensor, residual: torch.Tensor, weight: torch.Tensor, eps: float = 1e-6,
                offset: float = 0.0) -> Tuple[torch.Tensor, torch.Tensor]:
    """``res' = x + residual`` (rounded to the storage dtype), ``y = rmsnorm(res')``."""
    new_res = (x.float() + residual.float()).to(x.dtype)
    return rmsnorm(new_res, weight, eps, offset), new_res


# ---------------------------------------------------------------------- rope
def rope_inv_freq(head_dim: int, theta: float, scaling: Optional[dict] = None, device=None,
                  seq_len: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, float]:
    """Inverse frequencies ``[head_dim/2]`` and the factor applied to cos/sin, for plain RoPE or a long-context variant
    given as a Hugging Face ``rope_scaling`` mapping (``rope_type`` / ``type``):

    * ``linear``: all frequencies ÷ ``factor``;
    * ``llama3``: wavelengths above ``original_max / low_freq_factor`` ÷ ``factor``, those below
      ``original_max / high_freq_factor`` unchanged, a linear blend between;
    * ``yarn``: per-dimension blend of interpolated (÷ ``factor``) and original frequencies along a ramp between the
      dimensions that complete ``beta_fast`` and ``beta_slow`` rotations over the original window; cos/sin scaled by
      ``attention_factor`` (default ``0.1·ln(factor) + 1``);
    * ``dynamic`` (NTK): the base grows with the sequence once it exceeds ``max_position_embeddings``:
      ``θ · (factor · L / max − (factor − 1)) ^ (d / (d − 2))``;
    * ``longrope`` (Phi-3 long-context): per-dimension divisors ``short_factor`` up to ``original_max_position_embeddings``
      tokens and ``long_factor`` beyond, cos/sin scaled by ``√(1 + ln(factor) / ln(original_max))``.

    The last two depend on the sequence length ``seq_len`` (a 0-dim tensor: largest position + 1, as Hugging Face takes
    it; chosen on the device, no host read); without it they give their short-sequence form.
    ``default`` / ``None`` give plain RoPE. Other types raise."""
    import math
    inv = 1.0 / (theta**(torch.arange(0, head_dim, 2, dtype=torch.float32, device=device) / head_dim))
    kind = (scaling or {}).get('rope_type', (scaling or {}).get('type', 'default'))
    if not scaling or kind in ('default', None):
        return inv, 1.0
    factor = float(scaling.get('factor', 1.0))
    if kind == 'linear':
        return inv / factor, 1.0
    if kind == 'llama3':
        lo, hi = float(scaling.get('low_freq_factor', 1.0)), float(scaling.get('high_freq_factor', 4.0))
        orig = float(scaling['original_max_position_embeddings'])
        wavelen = 2 * math.pi / inv
        smooth = ((orig / wavelen - lo) / (hi - lo)).clamp(0.0, 1.0)
        blended = (1 - smooth) * inv / factor + smooth * inv
        out = torch.where(wavelen > orig / lo, inv / factor, torch.where(wavelen < orig / hi, inv, blended))
        return out, 1.0
    if kind == 'yarn':
        orig = float(scaling.get('original_max_position_embeddings') or scaling.get('max_position_embeddings', 4096))
        fast, slow = float(scaling.get('beta_fast') or 32), float(scaling.get('beta_slow') or 1)
        att = scaling.get('attention_factor')
        if att is None:
            ms, ms_all = scaling.get('mscale'), scaling.get('mscale_all_dim')
            get = lambda sc, m=1.0: 1.0 if sc <= 1 else 0.1 * m * math.log(sc) + 1.0  # noqa: E731
            att = get(factor, ms) / get(factor, ms_all) if ms and ms_all else get(factor)

        def corr_dim(rot: float) -> float:
            return head_dim * math.log(orig / (rot * 2 * math.pi)) / (2 * math.log(theta))

        low, high = corr_dim(fast), corr_dim(slow)
        if scaling.get('truncate', True):
            low, high = math.floor(low), math.ceil(high)
        low, high = max(low, 0), min(high, head_dim - 1)
        if low == high:
            high += 0.001
        ramp = ((torch.arange(head_dim // 2, dtype=torch.float32, device=device) - low) / (high - low)).clamp(0, 1)
        keep = 1 - ramp                                  # 1 → original frequency, 0 → interpolated
        return inv / factor * (1 - keep) + inv * keep, float(att)
    if kind == 'dynamic':
        mx = float(scaling.get('max_position_embeddings', 0) or 0)
        if seq_len is None or mx <= 0 or head_dim <= 2:
            return inv, 1.0
        grow = (factor * seq_len.float().clamp_min(mx) / mx - (factor - 1.0))**(head_dim / (head_dim - 2))
        expo = torch.arange(0, head_dim, 2, dtype=torch.float32, device=device) / head_dim
        return 1.0 / ((theta * grow)**expo), 1.0
    if kind == 'longrope':
        orig = float(scaling.get('original_max_position_embeddings') or scaling.get('max_position_embeddings', 4096))
        short = torch.tensor(scaling['short_factor'], dtype=torch.float32, device=device)
        ext = short
        if seq_len is not None:
            ext = torch.where(seq_len > orig, torch.tensor(scaling['long_factor'], dtype=torch.float32, device=device), short)
        f = scaling.get('factor') or float(scaling.get('max_position_embeddings', orig)) / orig
        att = scaling.get('attention_factor')
        if att is None:
            att = 1.0 if f <= 1.0 else math.sqrt(1 + math.log(f) / math.log(orig))
        return inv / ext, float(att)
    raise NotImplementedError(f'rope scaling type {kind!r} is not supported (default, linear, llama3, yarn, dynamic, longrope are)')


def rope_tables(positions: torch.Tensor, head_dim: int, theta: float = 1e6, scaling: Optional[dict] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """cos/sin ``[T, head_dim/2]`` in fp32 for integer ``positions [T]`` (see :func:`rope_inv_freq` for ``scaling``)."""
    seq_len = None
    if scaling and scaling.get('rope_type', scaling.get('type')) in ('dynamic', 'longrope') and positions.numel():
        seq_len = positions.max() + 1
    inv_freq, att = rope_inv_freq(head_dim, theta, scaling, positions.device, seq_len)
    ang = positions.float()[:, None] * inv_freq[None, :]
    if att != 1.0:
        return ang.cos() * att, ang.sin() * att
    return ang.cos(), ang.sin()


def apply_rope(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """Rotate-half convention (HF Llama/Qwen): pairs are (i, i + R/2) inside the leading ``R = 2·cos.shape[-1]`` dims;
    dims past ``R`` pass through (partial rotary).  ``x [T, H, D]``."""
    rot = 2 * cos.shape[-1]
    xf = x.float()
    x1, x2 = xf[..., :rot // 2], xf[..., rot // 2:rot]
    c, s = cos[:, None, :], sin[:, None, :]
    parts = [x1 * c - x2 * s, x2 * c + x1 * s]
    if rot < x.shape[-1]:
        parts.append(xf[..., rot:])
    return torch.cat(parts, -1).to(x.dtype)


def qk_norm_rope(q: torch.Tensor, k: torch.Tensor, q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor],
                 cos: torch.Tensor, sin: torch.Tensor, eps: float = 1e-6, offset: float = 0.0) -> Tuple[torch.Tensor, torch.Tensor]:
    """Per-head RMSNorm on q and k (Qwen3; ``offset`` 1.0 for the "1 + w" form of Qwen3.5) followed by RoPE.
    ``q [T,Hq,D]``, ``k [T,Hkv,D]``."""
    if q_weight is not None:
        q = rmsnorm(q, q_weight, eps, offset)
        k = rmsnorm(k, k_weight, eps, offset)
    return apply_rope(q, cos, sin), apply_rope(k, cos, sin)


# ------------------------------------------- short convolution in front of attention
def short_conv(u: torch.Tensor, weight: Optional[torch.Tensor], positions: torch.Tensor, history: Optional[torch.Tensor] = None,
               slots: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal depth-wise convolution without bias, in fp32: row t is ``Σ_j w[:, taps−1−j] · u_{t−j}`` over the rows of its own
    sequence.  ``u [T, C]``, ``weight [C, taps]`` (None: ``u`` itself), ``positions [T]`` = place of every row in its sequence.
    Packed rows (``history`` None) find their predecessors in front of them and start at position 0; with ``history
    [slots, taps−1, C]`` every row stands alone and the row of position p lies in ``history[slots[t], p mod (taps−1)]``."""
    x = u.float()
    if weight is None:
        return x
    w = weight.float()
    taps = w.shape[1]
    y = x * w[:, taps - 1]
    for j in range(1, taps):
        if history is None:
            prev = F.pad(x, (0, 0, j, 0))[:x.shape[0]]
        else:
            prev = history[slots.long(), (positions - j) % (taps - 1)].float()
        y = y + torch.where((positions >= j)[:, None], prev * w[:, taps - 1 - j], torch.zeros((), device=x.device))
    return y


def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    """``1 + coef · ln(⌊(p + 1) / every⌋ + 1)`` in fp32."""
    return 1.0 + coef * torch.log(((positions + 1) // every + 1).float())


def conv_heads(proj: torch.Tensor, weight: Optional[torch.Tensor], positions: torch.Tensor, hq: int, hkv: int, d: int, e: int, eps: float,
               coef: float = 0.0, every: int = 0, v_first: Optional[torch.Tensor] = None, lam: Optional[torch.Tensor] = None,
               history: Optional[torch.Tensor] = None, slots: Optional[torch.Tensor] = None):
    """Leading ``[q | k | v]`` columns of a projection → ``(q [T,hq,d], k [T,hkv,d], v [T,hkv,e])``: short convolution, q and k
    over their root mean square per head, query temperature, values mixed as ``(1 − λ) v + λ v_first``.  fp32 inside; the
    results are rounded to the projection's dtype."""
    T = proj.shape[0]
    y = short_conv(proj[:, :hq * d + hkv * (d + e)], weight, positions, history, slots)
    q, k, v = y[:, :hq * d].reshape(T, hq, d), y[:, hq * d:(hq + hkv) * d].reshape(T, hkv, d), y[:, (hq + hkv) * d:].reshape(T, hkv, e)
    q = q * torch.rsqrt(q.pow(2).mean(-1, keepdim=True) + eps)
    k = k * torch.rsqrt(k.pow(2).mean(-1, keepdim=True) + eps)
    if every:
        q = q * query_temperature(positions, coef, every)[:, None, None]
    if v_first is not None:
        v = v + lam.float() * (v_first.reshape(v.shape).float() - v)
    return q.to(proj.dtype), k.to(proj.dtype), v.to(proj.dtype)


def stream_rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, out_dtype: torch.dtype, adds=(), mult: float = 1.0, offset: float = 0.0):
    """fp32 residual stream: ``x ← x + mult · Σ y_i ⊙ s_i`` over ``adds = [(y, s), …]``, then its RMS norm (weight ``offset + w``)
    in ``out_dtype``.  Returns ``(norm, x)``."""
    x = x.float()
    if adds:
        x = x + mult * sum(y.float() * sc.float() for y, sc in adds)
    return (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * (weight.float() + offset)).to(out_dtype), x


def stream_gated_rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, offset: float, result: torch.Tensor, gate: torch.Tensor, bias: torch.Tensor,
                         post: torch.Tensor, row_of: Optional[torch.Tensor] = None, share: Optional[torch.Tensor] = None):
    """fp32 residual stream: ``x ← x + norm(σ(gate + bias) ⊙ result; post)``, then the norm of the sum in ``weight``'s dtype; both
    norms have weights ``offset + w``.  ``result [T, W]``, or expert rows of which token t has ``Σ_j share[t, j] · result[row_of[t, j]]``."""
    y = result.float() if row_of is None else (result[row_of.long()].float() * share[..., None]).sum(1)
    y = torch.sigmoid(gate[:, :x.shape[1]].float() + bias.float()) * y
    x = x + y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + eps) * (post.float() + offset)
    return stream_rmsnorm(x, weight, eps, weight.dtype, offset=offset)


def stream_joined_rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, offset: float, result: torch.Tensor, row_of: Optional[torch.Tensor] = None,
                          share: Optional[torch.Tensor] = None, beside: Optional[torch.Tensor] = None, open: Optional[torch.Tensor] = None):
    """fp32 residual stream: ``x ← x + result + open · beside``, then the norm of the sum (weight ``offset + w``) in ``weight``'s dtype.  ``result
    [T, W]``, or expert rows of which token t has ``Σ_j share[t, j] · result[row_of[t, j]]``; ``open [T]``."""
    y = result.float() if row_of is None else (result[row_of.long()].float() * share[..., None]).sum(1)
    if beside is not None:
        y = y + open.float()[:, None] * beside.float()
    return stream_rmsnorm(x.float() + y, weight, eps, weight.dtype, offset=offset)


# ------------------------------------------- rotated heads
def rotary_table(positions: torch.Tensor, frequencies: torch.Tensor) -> torch.Tensor:
    """``(cos, sin)`` of position times frequency ``[n]`` (fp64) as fp32 ``[T, n, 2]``."""
    a = positions.double()[:, None] * frequencies
    return torch.stack([a.cos(), a.sin()], -1).float()


def rotate_pairs(x: torch.Tensor, table: torch.Tensor, interleaved: bool) -> torch.Tensor:
    """``x [T, H, D]`` fp32, ``table [T, n, 2]``: the leading ``2n`` dimensions turned pair by pair, pairs ``(2i, 2i + 1)`` or ``(i, i + n)``."""
    n = table.shape[1]
    c, s = table[:, None, :, 0], table[:, None, :, 1]
    a, b = (x[..., 0:2 * n:2], x[..., 1:2 * n:2]) if interleaved else (x[..., :n], x[..., n:2 * n])
    ra, rb = a * c - b * s, b * c + a * s
    return torch.cat([torch.stack([ra, rb], -1).flatten(-2) if interleaved else torch.cat([ra, rb], -1), x[..., 2 * n:]], -1)


def rotary_heads(proj: torch.Tensor, first: int, bias: Optional[torch.Tensor], q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor], table: torch.Tensor,
                 interleaved: bool, hq: int, hkv: int, d: int, e: int, eps: float):
    """Columns ``[q | k | v]`` from ``first`` on → ``(q [T,hq,d], k [T,hkv,d], v [T,hkv,e])`` (None without own keys): bias, RMS norm of q and k per
    head, rotation.  fp32 inside; the results are rounded to the projection's dtype."""
    T, n = proj.shape[0], hq * d + hkv * (d + e)
    y = proj[:, first:first + n].float()
    if bias is not None:
        y = y + bias.float()
    q, k, v = y[:, :hq * d].reshape(T, hq, d), y[:, hq * d:(hq + hkv) * d].reshape(T, hkv, d), y[:, (hq + hkv) * d:].reshape(T, hkv, e)
    if q_weight is not None:
        q = rmsnorm(q, q_weight, eps)
    q = rotate_pairs(q, table, interleaved).to(proj.dtype)
    if not hkv:
        return q, None, None
    if k_weight is not None:
        k = rmsnorm(k, k_weight, eps)
    return q, rotate_pairs(k, table, interleaved).to(proj.dtype), v.to(proj.dtype)


def latent_rotary(proj: torch.Tensor, q0: int, heads: int, d: int, r: int, c0: int, nc: int, wc: Optional[torch.Tensor], eps: float, table: Optional[torch.Tensor],
                  interleaved: bool):
    """Queries ``[d | r]`` per head from column ``q0`` and ``[latent | key part]`` from column ``c0`` (``nc`` 0: none) → ``(q [T, heads, d + r], kept
    [T, nc + r] | None)``: the ``r`` dimensions rotated, the latent RMS-normed."""
    T = proj.shape[0]
    q = proj[:, q0:q0 + heads * (d + r)].reshape(T, heads, d + r)
    kept = rmsnorm(proj[:, c0:c0 + nc], wc, eps) if nc else None
    if r:
        q = torch.cat([q[..., :d], rotate_pairs(q[..., d:].float(), table, interleaved).to(proj.dtype)], -1)
        if nc:
            kept = torch.cat([kept, rotate_pairs(proj[:, None, c0 + nc:c0 + nc + r].float(), table, interleaved)[:, 0].to(proj.dtype)], -1)
    return q, kept


# ------------------------------------------- layers with norms on their results
def position_waves(positions: torch.Tensor, frequencies: torch.Tensor, width: int) -> torch.Tensor:
    """``[T, width]`` fp32: sine and cosine of position times frequency side by side (angles in fp64)."""
    a = positions.double()[:, None] * frequencies
    return torch.stack([a.sin(), a.cos()], -1).flatten(1)[:, :width].float()


def stream_normed(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float, out_dtype: torch.dtype, y: torch.Tensor, bias: Optional[torch.Tensor], post: torch.Tensor,
                  inner: Optional[torch.Tensor] = None, beside: Optional[torch.Tensor] = None, beside_inner: Optional[torch.Tensor] = None):
    unit = lambda t: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps)  # noqa: E731
    z = y.float() if bias is None else y.float() + bias.float()
    if beside is not None:
        z = 0.5 * (unit(z) * inner.float() + unit(beside.float()) * beside_inner.float())
    x = x + unit(z) * post.float()
    return (x if weight is None else unit(x) * weight.float()).to(out_dtype), x


def plain_heads(proj: torch.Tensor, first: int, bias: Optional[torch.Tensor], q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor], value_norm: bool,
                values_are_keys: bool, hq: int, hkv: int, d: int, e: int, eps: float):
    T, sizes = proj.shape[0], (hq * d, hkv * d, 0 if values_are_keys else hkv * e)
    y = proj[:, first:first + sum(sizes)].float()
    q, k, v = (y if bias is None else y + bias.float()).split(sizes, -1)
    v = (k if values_are_keys else v).reshape(T, hkv, e)

    def normed(t, w, h):
        whole = w is not None and w.numel() == h * d and h > 1         # one head: the same thing
        t = t if whole else t.reshape(T, h, d)
        if w is not None:
            t = t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w.float()
        return t.reshape(T, h, d)
    if value_norm:
        v = v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)
    return tuple(t.to(proj.dtype) for t in (normed(q, q_weight, hq), normed(k, k_weight, hkv), v))


# ------------------------------------------- selective scan, matrix memory
def conv_silu(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, positions: torch.Tensor, history: Optional[torch.Tensor] = None, slots: Optional[torch.Tensor] = None):
    return F.silu(short_conv(x, weight, positions, history, slots) + bias.float()).to(x.dtype)


def selective_scan(u: torch.Tensor, dt: torch.Tensor, dt_bias: torch.Tensor, A_log: torch.Tensor, B: torch.Tensor, C: torch.Tensor, D: torch.Tensor, z: torch.Tensor,
                   bounds, states=None):
    """Sequences ``bounds`` of rows, from ``states`` (None: empty ones) → ``(y [T, inner], last states)``; token by token."""
    dtype, (u, B, C) = u.dtype, (t.float() for t in (u, B, C))
    step = F.softplus(dt.float() + dt_bias.float())
    A, du = -torch.exp(A_log.float()), step * u
    rows, last = [], []
    for n, (a, b) in enumerate(zip(bounds[:-1], bounds[1:])):
        S = A.new_zeros(A.shape) if states is None else states[n]
        for t in range(a, b):
            S = torch.exp(step[t][:, None] * A) * S + du[t][:, None] * B[t]
            rows.append(S @ C[t])
        last.append(S)
    y = torch.stack(rows) if rows else torch.zeros_like(u)
    return ((y + D.float() * u) * F.silu(z.float())).to(dtype), last


def matrix_memory_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor, state, chunk: int = 32):
    """One sequence ``q, k [T, H, d]``, ``v [T, H, e]``, log gates ``[T, H]``, from ``(S, n, m)`` → ``(o [T, H, e], last (S, n, m))``, in chunks: a token's
    weight on an earlier one is the exponential of summed log gates, taken relative to the running maximum."""
    S, n, m = state
    out = []
    for a in range(0, q.shape[0], chunk):
        qc, kc, vc, ic, fc = (t[a:a + chunk].transpose(0, 1) for t in (q, k, v, i, f))         # [H, L, ·], [H, L]
        F_ = fc.cumsum(-1)
        g = ic - F_                                                                              # what a token is worth at the chunk's start
        top = torch.maximum(m[:, None], g.cummax(-1).values) + F_                               # running maximum
        start = torch.exp(F_ + m[:, None] - top)                                                # weight of the state at the chunk's start
        w = torch.exp((F_ - top)[:, :, None] + g[:, None, :]).tril()                            # [H, L, L]
        A = (qc @ kc.transpose(1, 2)) * w
        num = A @ vc + start[..., None] * (qc @ S)
        den = A.sum(-1) + start * (qc @ n[..., None])[..., 0]
        out.append((num / (torch.maximum(den.abs(), torch.exp(-top)) + 1e-6)[..., None]).transpose(0, 1))
        end = w[:, -1, :, None] * kc
        S = start[:, -1, None, None] * S + end.transpose(1, 2) @ vc
        n = start[:, -1, None] * n + end.sum(1)
        m = top[:, -1]
    return (torch.cat(out) if out else torch.zeros_like(v)), (S, n, m)


def matrix_memory(proj: torch.Tensor, first: int, heads: int, dim: int, vdim: int, i_bias: torch.Tensor, f_bias: torch.Tensor, cap: float, weight: torch.Tensor, eps: float,
                  bounds, states=None):
    """Columns ``[q | k | v | gate | i | f]`` from ``first`` on → ``(o [T, heads · vdim], last states)``; a state is ``(S, n, m)``."""
    T, nd, ne = proj.shape[0], heads * dim, heads * vdim
    q, k, v, g, i, f = proj[:, first:first + 2 * nd + 2 * ne + 2 * heads].float().split([nd, nd, ne, ne, heads, heads], -1)
    q, k, v = q.reshape(T, heads, dim) * dim**-0.5, k.reshape(T, heads, dim), v.reshape(T, heads, vdim)
    i, f = cap * torch.tanh((i + i_bias.float()) / cap), F.logsigmoid(cap * torch.tanh((f + f_bias.float()) / cap))
    out, last = [], []
    for n, (a, b) in enumerate(zip(bounds[:-1], bounds[1:])):
        s = (q.new_zeros(heads, dim, vdim), q.new_zeros(heads, dim), q.new_zeros(heads)) if states is None else states[n]
        o, s = matrix_memory_scan(q[a:b], k[a:b], v[a:b], i[a:b], f[a:b], s)
        out.append(o)
        last.append(s)
    o = torch.cat(out)
    o = (o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, ne) * weight.float() * torch.sigmoid(g)
    return o.to(proj.dtype), last


# ------------------------------------------- latent attention, HGRN2
def latent_norms(proj: torch.Tensor, q0: int, nq: int, wq: torch.Tensor, c0: int, nc: int, wc: Optional[torch.Tensor], eps: float):
    """RMS norms of the query-bottleneck and latent column ranges of a projection (``nc`` 0: no latent)."""
    return rmsnorm(proj[:, q0:q0 + nq], wq, eps), rmsnorm(proj[:, c0:c0 + nc], wc, eps) if nc else None


def latent_decode(q: torch.Tensor, pool: torch.Tensor, table: torch.Tensor, lens: torch.Tensor, scale: float, sinks: Optional[torch.Tensor] = None,
                  gate: Optional[torch.Tensor] = None, rank: int = 0, window: int = 0):
    """``q [B, H, K]`` against the cached rows of every sequence, keys of all heads whose first ``rank`` columns (0: all) are the values →
    ``[B, H, rank]``."""
    o = paged_attention_decode(q, pool[..., :q.shape[-1]], pool[..., :rank or q.shape[-1]], table, lens, scale, window or None, sinks=sinks)
    return o if gate is None else (o.float() * torch.sigmoid(gate.float())[..., None]).to(o.dtype)


def hgrn2_gates(f: torch.Tensor, bias: torch.Tensor, lower: torch.Tensor) -> torch.Tensor:
    """What a channel lets in, ``1 − forget gate = (1 − lower) · σ(−(f + bias))``, in fp32 (small values keep their digits)."""
    return (1 - lower.float()) * torch.sigmoid(-(f.float() + bias.float()))


def hgrn2_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, state: torch.Tensor, chunk: int = 16):
    """``S ← (1 − k_t) ⊙ S + k_t v_tᵀ``, ``o_t = Sᵀ q_t`` over one sequence, fp32: ``q, k [T, H, d]``, ``v [T, H, e]``, ``state [H, d, e]`` →
    ``(o [T, H, e], state)``.  Inside a chunk by the decay between every two tokens, one step per chunk."""
    out = []
    for a in range(0, q.shape[0], chunk):
        qc, kc, vc = (t[a:a + chunk].transpose(0, 1) for t in (q, k, v))
        G = torch.log1p(-kc).clamp_min(-60.0).cumsum(1)                                   # log decay since the chunk's start
        n = G.shape[1]
        past = torch.ones(n, n, dtype=torch.bool, device=q.device).tril()
        D = (G[:, :, None] - G[:, None]).masked_fill(~past[None, :, :, None], float('-inf')).exp()       # [H, to, from, d]
        A = torch.einsum('hid,hijd,hjd->hij', qc, D, kc)
        out.append((A @ vc + (qc * G.exp()) @ state).transpose(0, 1))
        state = state * G[:, -1].exp()[..., None] + (kc * D[:, -1]).transpose(1, 2) @ vc
    return torch.cat(out), state


def hgrn2(proj: torch.Tensor, q0: int, f0: int, v0: int, heads: int, dim: int, vdim: int, bias: torch.Tensor, lower: torch.Tensor, weight: torch.Tensor,
          eps: float, bounds: List[int], states: Optional[List[torch.Tensor]] = None):
    """The mixer between its projections, for packed rows of sequences at ``bounds``: ``(norm(o) [T, heads·vdim], last states)``."""
    T, n, e = proj.shape[0], heads * dim, heads * vdim
    q = F.silu(proj[:, q0:q0 + n].float()).view(T, heads, dim)
    k = hgrn2_gates(proj[:, f0:f0 + n], bias, lower).view(T, heads, dim)
    v = proj[:, v0:v0 + e].float().view(T, heads, vdim)
    out, last = [], []
    for i, (a, b) in enumerate(zip(bounds[:-1], bounds[1:])):
        o, S = hgrn2_scan(q[a:b], k[a:b], v[a:b], states[i] if states is not None else q.new_zeros(heads, dim, vdim))
        out.append(o)
        last.append(S)
    return rmsnorm(torch.cat(out), weight, eps).reshape(T, e).to(proj.dtype), last


# -------------------------------------------------------------------- swiglu
def swiglu(gate_up: torch.Tensor) -> torch.Tensor:
    """``[T, 2I]`` laid out as ``[gate | up]`` → ``silu(gate) * up`` ``[T, I]``."""
    g, u = gate_up.float().chunk(2, dim=-1)
    return (F.silu(g) * u).to(gate_up.dtype)


def geglu(gate_up: torch.Tensor) -> torch.Tensor:
    g, u = gate_up.float().chunk(2, dim=-1)
    return (F.gelu(g, approximate='tanh') * u).to(gate_up.dtype)


def clamped_glu(gate_up: torch.Tensor, limit: float = 7.0, alpha: float = 1.702) -> torch.Tensor:
    """GPT-OSS expert activation on ``[gate | up]``: ``(up + 1) · gate · σ(α · gate)`` with ``gate ≤ limit`` and
    ``|up| ≤ limit``."""
    g, u = gate_up.float().chunk(2, dim=-1)
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return ((u + 1.0) * g * torch.sigmoid(alpha * g)).to(gate_up.dtype)


def relu2(x: torch.Tensor) -> torch.Tensor:
    return F.relu(x.float()).square().to(x.dtype)


# ----------------------------------------------------------------- attention
def attention_varlen(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_seqlens: torch.Tensor, causal: bool = True,
                     scale: Optional[float] = None, return_lse: bool = False, cu_seqlens_k: Optional[torch.Tensor] = None,
                     window: Optional[int] = None, softcap: Optional[float] = None, sinks: Optional[torch.Tensor] = None, chunk: int = 0, terms=None):
    """Packed attention.  ``q [T,Hq,D]``, ``k,v [Tk,Hkv,D]``, ``cu_seqlens`` int
    ``[n+1]``; tokens of different segments never attend to each other; GQA by
    repeating each kv head ``Hq/Hkv`` times.  With ``cu_seqlens_k`` the keys of a segment may be longer than its
    queries; the causal diagonal is then aligned bottom-right (query row r sees keys 0 … r + Lk − Lq).
    ``window``: a query sees only the last ``window`` keys up to and including its own position (sliding-window
    checkpoints); ``softcap``: scores pass through ``cap · tanh(s / cap)`` before the softmax (Gemma-2); ``sinks [Hq]``: a
    learned logit per head that takes part in the softmax and carries no value (GPT-OSS), i.e. it only enlarges the
    denominator; ``chunk``: a query sees only the keys of its own block of that many positions, counted from the sequence's start; ``terms``
    (an ``ops.ScoreTerms``): what else happens to a score."""
    T, Hq, D = q.shape
    Hkv = k.shape[1]
    rep = Hq // Hkv
    scale = 1.0 / math.sqrt(D) if scale is None else scale
    out = q.new_empty(T, Hq, v.shape[-1])          # values may be narrower than the score width (latent attention)
    lse = torch.empty(Hq, T, dtype=torch.float32, device=q.device)
    bounds = cu_seqlens.tolist()
    kb = bounds if cu_seqlens_k is None else cu_seqlens_k.tolist()
    for a, b, ka, kbnd in zip(bounds[:-1], bounds[1:], kb[:-1], kb[1:]):
        if b <= a:
            continue
        qs = q[a:b].float().transpose(0, 1)  # [Hq, L, D]
        ks = k[ka:kbnd].float().transpose(0, 1).repeat_interleave(rep, 0)
        vs = v[ka:kbnd].float().transpose(0, 1).repeat_interleave(rep, 0)
        s = qs @ ks.transpose(1, 2) * scale
        if softcap:
            s = torch.tanh(s / softcap) * softcap
        if terms is not None:
            s = terms.apply(s, torch.arange(b - a, device=q.device)[:, None] + (kbnd - ka - b + a) - torch.arange(kbnd - ka, device=q.device))
        if causal:
            L, Lk = b - a, kbnd - ka
            s = s.masked_fill(torch.ones(L, Lk, dtype=torch.bool, device=q.device).triu(1 + Lk - L), float('-inf'))
            if window and Lk > window:
                s = s.masked_fill(torch.ones(L, Lk, dtype=torch.bool, device=q.device).tril(Lk - L - window), float('-inf'))
            if chunk and Lk > chunk:
                block = torch.arange(Lk, device=q.device) // chunk
                s = s.masked_fill(block[Lk - L:, None] != block, float('-inf'))
        l = torch.logsumexp(s, -1)
        if sinks is not None:
            l = torch.logaddexp(l, sinks.float()[:, None])
        p = torch.exp(s - l[..., None])
        out[a:b] = (p @ vs).transpose(0, 1).to(q.dtype)
        lse[:, a:b] = l
    return (out, lse) if return_lse else out


def paged_attention_decode(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_tables: torch.Tensor,
                           seq_lens: torch.Tensor, scale: Optional[float] = None, window: Optional[int] = None,
                           softcap: Optional[float] = None, sinks: Optional[torch.Tensor] = None, chunk: int = 0, terms=None) -> torch.Tensor:
    """One query token per sequence against a paged KV cache.
    ``q [B,Hq,D]``; caches ``[num_blocks, block_size, Hkv, D]`` (values may have a width of their own); ``block_tables
    [B, max_blocks]`` int; ``seq_lens [B]`` (including the current token)."""
    B, Hq, D = q.shape
    bs, Hkv = k_cache.shape[1], k_cache.shape[2]
    rep = Hq // Hkv
    scale = 1.0 / math.sqrt(D) if scale is None else scale
    E = v_cache.shape[-1]
    out = q.new_zeros(B, Hq, E)
    for b in range(B):
        n = int(seq_lens[b])
        if n == 0:
            continue
        nb = (n + bs - 1) // bs
        blocks = block_tables[b, :nb].long()
        kk = k_cache[blocks].reshape(-1, Hkv, D)[:n].float().repeat_interleave(rep, 1)
        vv = v_cache[blocks].reshape(-1, Hkv, E)[:n].float().repeat_interleave(rep, 1)
        s = torch.einsum('hd,nhd->hn', q[b].float(), kk) * scale
        if softcap:
            s = torch.tanh(s / softcap) * softcap
        if terms is not None:
            s = terms.apply(s[:, None], n - 1 - torch.arange(n, device=q.device)[None])[:, 0]
        if window and n > window:
            s[:, :n - window] = float('-inf')
        if chunk:
            s[:, :(n - 1) // chunk * chunk] = float('-inf')
        if sinks is not None:
            l = torch.logaddexp(torch.logsumexp(s, -1), sinks.float())
            out[b] = torch.einsum('hn,nhd->hd', torch.exp(s - l[:, None]), vv).to(q.dtype)
            continue
        out[b] = torch.einsum('hn,nhd->hd', torch.softmax(s, -1), vv).to(q.dtype)
    return out


# ------------------------------------------------------------ logprob / loss
def logprob_from_logits(logits: torch.Tensor, labels: torch.Tensor, temperature: float = 1.0,
                        with_entropy: bool = False) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    x = logits.float() / temperature
    lse = torch.logsumexp(x, -1)
    lp = x.gather(-1, labels.long().unsqueeze(-1)).squeeze(-1) - lse
    ent = None
    if with_entropy:
        ent = lse - (torch.softmax(x, -1) * x).sum(-1)
    return lp, ent


def fused_linear_logprob(hidden: torch.Tensor, weight: torch.Tensor, labels: torch.Tensor, temperature: float = 1.0,
                         with_entropy: bool = False, chunk: int = 2048) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``log softmax(hidden @ weightᵀ / temperature)[labels]`` without keeping
    the ``[T, V]`` matrix (chunks over T).  Differentiable via autograd."""
    lps, ents = [], []
    for s in range(0, hidden.shape[0], chunk):
        logits = hidden[s:s + chunk].float() @ weight.float().t()
        lp, ent = logprob_from_logits(logits, labels[s:s + chunk], temperature, with_entropy)
        lps.append(lp)
        if with_entropy:
            ents.append(ent)
    return torch.cat(lps), (torch.cat(ents) if with_entropy else None)


# -------------------------------------------------------------------- adamw
def adamw_step(master: torch.Tensor, exp_avg: torch.Tensor, exp_avg_sq: torch.Tensor, grad: torch.Tensor,
               param_out: Optional[torch.Tensor], lr: float, beta1: float, beta2: float, eps: float, weight_decay: float,
               step: int, grad_scale: float = 1.0) -> None:
    """Decoupled weight decay Adam on fp32 master weights; ``grad_scale``
    multiplies the gradient first (1/num_tokens × clip coefficient);
    ``param_out`` (bf16 working copy) receives the rounded result."""
    g = grad.float() * grad_scale
    master.mul_(1.0 - lr * weight_decay)
    exp_avg.mul_(beta1).add_(g, alpha=1.0 - beta1)
    exp_avg_sq.mul_(beta2).addcmul_(g, g, value=1.0 - beta2)
    bc1 = 1.0 - beta1**step
    bc2 = 1.0 - beta2**step
    denom = (exp_avg_sq / bc2).sqrt_().add_(eps)
    master.addcdiv_(exp_avg / bc1, denom, value=-lr)
    if param_out is not None:
        param_out.copy_(master)


# --------------------------------------------------------------------- lora
def sgmv(x: torch.Tensor, lora_a: torch.Tensor, lora_b: torch.Tensor, seg_starts: torch.Tensor, seg_slots: torch.Tensor,
         seg_ranks: torch.Tensor, seg_scales: torch.Tensor) -> torch.Tensor:
    """Segmented multi-LoRA: rows ``seg_starts[i]:seg_starts[i+1]`` of ``x [T,K]``
    use slot ``seg_slots[i]`` (−1 = no adapter) with rank ``seg_ranks[i]`` and
    scale ``seg_scales[i]``.  ``lora_a [S, R, K]``, ``lora_b [S, N, R]``.
    Returns the delta ``[T, N]`` in x's dtype."""
    T = x.shape[0]
    out = torch.zeros(T, lora_b.shape[1], dtype=x.dtype, device=x.device)
    starts = seg_starts.tolist()
    for i in range(len(starts) - 1):
        slot, r = int(seg_slots[i]), int(seg_ranks[i])
        if slot < 0 or r == 0 or starts[i + 1] <= starts[i]:
            continue
        a = lora_a[slot, :r].float()
        b = lora_b[slot, :, :r].float()
        xs = x[starts[i]:starts[i + 1]].float()
        out[starts[i]:starts[i + 1]] = ((xs @ a.t()) @ b.t() * float(seg_scales[i])).to(x.dtype)
    return out


# ---------------------------------------------------------------------- moe
def moe_router(logits: torch.Tensor, top_k: int, renormalize: bool = True) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """fp32 softmax → top-k → optional renormalisation.  Returns (weights [T,k]
    fp32, indices [T,k] int64, full probabilities [T,E] fp32)."""
    probs = torch.softmax(logits.float(), -1)
    w, idx = probs.topk(top_k, -1)
    if renormalize:
        w = w / w.sum(-1, keepdim=True)
    return w, idx, probs


def moe_choice(z: torch.Tensor, k: int, forced: Optional[torch.Tensor] = None, groups: int = 0, keep: int = 0, factor: float = 1.0):
    """Weights ``[T, k]`` and experts ``[T, k]`` for router logits ``z [T, E]``.  ``groups`` 0: the k largest, a softmax over just those; otherwise a
    softmax over all, choice among the ``keep`` groups with the best experts, weights times ``factor``.  ``forced``: see ``ops.moe_topk``."""
    s = torch.softmax(z, -1)
    c = z
    if groups > 1:
        best = z.view(z.shape[0], groups, -1).amax(-1).topk(keep, -1)[1]
        allowed = torch.zeros(z.shape[0], groups, dtype=torch.bool, device=z.device).scatter_(1, best, True)
        c = z.masked_fill(~allowed.repeat_interleave(z.shape[1] // groups, 1), float('-inf'))
    idx = c.topk(k, -1)[1]
    if forced is not None:
        idx = torch.where(forced[:, :1] < 0, idx, forced.long())
    return (s.gather(1, idx) * factor if groups else torch.softmax(z.gather(1, idx), -1)), idx


def moe_aux_loss(probs: torch.Tensor, indices: torch.Tensor, num_experts: int) -> torch.Tensor:
    """Switch-style load-balance loss: ``E · Σ_e f_e · P_e`` with ``f_e`` the
    fraction of routed slots and ``P_e`` the mean router probability."""
    T, k = indices.shape
    f = torch.zeros(num_experts, dtype=torch.float32, device=probs.device)
    f.scatter_add_(0, indices.reshape(-1), torch.ones(T * k, device=probs.device))
    f = f / (T * k)
    return num_experts * (f * probs.mean(0)).sum()


def grouped_gemm(x: torch.Tensor, weight: torch.Tensor, offsets: torch.Tensor) -> torch.Tensor:
    """Rows ``offsets[e]:offsets[e+1]`` of ``x [R, K]`` times ``weight[e]ᵀ`` with
    ``weight [E, N, K]`` → ``[R, N]``."""
    out = torch.zeros(x.shape[0], weight.shape[1], dtype=x.dtype, device=x.device)
    off = offsets.tolist()
    for e in range(weight.shape[0]):
        a, b = off[e], off[e + 1]
        if b > a:
            out[a:b] = (x[a:b].float() @ weight[e].float().t()).to(x.dtype)
    return out


def moe_experts(x: torch.Tensor, weights: torch.Tensor, indices: torch.Tensor, w_gate_up: torch.Tensor,
                w_down: torch.Tensor) -> torch.Tensor:
    """Dense-math MoE FFN: ``Σ_k weights[t,k] · down_e(swiglu(gate_up_e(x_t)))``."""
    T, k = indices.shape
    out = torch.zeros(T, x.shape[1], dtype=torch.float32, device=x.device)
    for e in range(w_gate_up.shape[0]):
        tok, slot = (indices == e).nonzero(as_tuple=True)
        if tok.numel() == 0:
            continue
        h = swiglu((x[tok].float() @ w_gate_up[e].float().t()).to(x.dtype))
        y = h.float() @ w_down[e].float().t()
        out.index_add_(0, tok, y * weights[tok, slot, None].float())
    return out.to(x.dtype)


# ----------------------------------------------------------------- sampling
def sample_tokens(logits: torch.Tensor, temperature: float = 1.0, top_k: int = -1, top_p: float = 1.0,
                  generator: Optional[torch.Generator] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """Returns (token ids [B], logprob of the chosen token under the *processed*
    distribution [B])."""
    x = logits.float()
    if temperature <= 0:
        tok = x.argmax(-1)
        return tok, torch.zeros(x.shape[0], device=x.device)
    x = x / temperature
    if top_k and top_k > 0:
        kth = x.topk(min(top_k, x.shape[-1]), -1).values[..., -1:]
        x = x.masked_fill(x < kth, float('-inf'))
    if top_p < 1.0:
        sorted_x, order = x.sort(-1, descending=True)
        cum = torch.softmax(sorted_x, -1).cumsum(-1)
        drop = cum - torch.softmax(sorted_x, -1) >= top_p
        sorted_x = sorted_x.masked_fill(drop, float('-inf'))
        x = torch.full_like(x, float('-inf')).scatter(-1, order, sorted_x)
    logp = torch.log_softmax(x, -1)
    tok = torch.multinomial(logp.exp(), 1, generator=generator).squeeze(-1)
    return tok, logp.gather(-1, tok[:, None]).squeeze(-1)
