"""Operator layer: autograd-aware entry points for every hot op.

On CUDA tensors each op launches a hand-written sm_100a kernel from the
in-tree extension ``twinkle_b200/ops/_C*.so`` (sources in ``ops/csrc``); if the
extension cannot be loaded on a machine that has a GPU the import fails loudly
instead of falling back.  On CPU tensors the fp32 formulas of
``ops.reference`` run (used by gloo tests and as oracles).

Kernel ↔ reference-site map (what each op replaces in the reference project):
``linear`` → ``F.linear`` everywhere; ``flash_attn_varlen`` → flash-attn varlen
(``model/transformers/strategy/sequence_parallel/__init__.py:230-337``);
``rmsnorm``/``swiglu``/``qk_norm_rope`` → Liger kernels (``kernel/liger.py``);
``fused_linear_logprob`` → ``utils/torch_utils.py:61-137`` +
``loss/liger_fused_linear_cross_entropy.py``; ``adamw_step`` → ``torch.optim.AdamW``;
``sgmv`` → ``model/multi_lora.py:320-326``; ``moe_*`` →
``model/transformers/moe/expert_parallel.py``.
"""
from __future__ import annotations

import math
import os
from typing import NamedTuple, Optional, Tuple

import torch

from . import reference as ref

_EXT = None


def ext():
    """The compiled extension; loaded on first use."""
    global _EXT
    if _EXT is None:
        from .build import load_extension
        _EXT = load_extension()
    return _EXT


def has_ext() -> bool:
    try:
        return ext() is not None
    except Exception:
        return False


def _cuda(t: torch.Tensor) -> bool:
    return t.is_cuda


# ------------------------------------------------------------------ linear
class _DeadValues:
    """While a layer is re-run only to rebuild its autograd graph (activation recompute in backward), the values of
    its last operations are never read: their backward needs the operands, not the result.  Inside this context
    the operations that opt in return uninitialised tensors of the right shape instead of computing."""
    on = False


class dead_values:

    def __enter__(self):
        self.prev, _DeadValues.on = _DeadValues.on, True

    def __exit__(self, *exc):
        _DeadValues.on = self.prev
        return False


def dead_values_enabled() -> bool:
    return _DeadValues.on


class _AddDead(torch.autograd.Function):
    """``a + b`` whose value nobody reads: returns an uninitialised tensor, passes the gradient to both."""

    @staticmethod
    def forward(ctx, a, b):
        return torch.empty_like(a)

    @staticmethod
    def backward(ctx, g):
        return g, g


def add(a: torch.Tensor, b: torch.Tensor, value_unused: bool = False) -> torch.Tensor:
    if value_unused and _DeadValues.on and a.is_cuda:
        return _AddDead.apply(a, b)
    return a + b


class _Linear(torch.autograd.Function):
    """y = x @ Wᵀ with three tcgen05 GEMM layouts: NT forward, NN for dX, TN for dW."""

    @staticmethod
    def forward(ctx, x, weight, bias, wgrad_out, dead=False):
        ctx.save_for_backward(x, weight)
        ctx.has_bias = bias is not None
        ctx.wgrad_out = wgrad_out
        if dead:  # graph only: dX needs W and dW needs x, nobody needs x·Wᵀ
            return torch.empty(*x.shape[:-1], weight.shape[0], dtype=x.dtype, device=x.device)
        x2 = x.reshape(-1, x.shape[-1])
        # the result is allocated in its final shape (not returned as a view of a 2-D product): a later op may then
        # accumulate into it in place, which autograd refuses for views created inside a custom Function
        y = torch.empty(*x.shape[:-1], weight.shape[0], dtype=x.dtype, device=x.device)
        gemm(x2, weight, 'nt', out=y.view(-1, weight.shape[0]))
        if bias is not None:
            y += bias
        return y

    @staticmethod
    def backward(ctx, gy):
        x, weight = ctx.saved_tensors
        g2 = gy.reshape(-1, gy.shape[-1])
        if not g2.is_contiguous():
            g2 = g2.contiguous()
        x2 = x.reshape(-1, x.shape[-1])
        gx = gw = gb = None
        if ctx.needs_input_grad[0]:
            gx = gemm(g2, weight, 'nn').view(x.shape)
        if ctx.needs_input_grad[1]:
            if ctx.wgrad_out is not None:
                # accumulate straight into the flat gradient bucket (fp32 or bf16)
                gemm(g2, x2, 'tn', out=ctx.wgrad_out, accumulate=True)
                gw = None
            else:
                gw = gemm(g2, x2, 'tn')
        if ctx.has_bias and ctx.needs_input_grad[2]:
            gb = g2.float().sum(0).to(gy.dtype)
        return gx, gw, gb, None, None


def gemm(a: torch.Tensor, b: torch.Tensor, layout: str = 'nt', out: Optional[torch.Tensor] = None,
         accumulate: bool = False, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``nt``: a[M,K]·b[N,K]ᵀ; ``nn``: a[M,K]·b[K,N]; ``tn``: a[K,M]ᵀ·b[K,N].  bf16
    operands, fp32 accumulation in tensor memory, bf16 or fp32 output."""
    if _cuda(a) and a.dtype == torch.bfloat16:
        return ext().gemm(a, b, layout, out, accumulate, out_dtype)
    af, bf = a.float(), b.float()
    r = af @ bf.t() if layout == 'nt' else (af @ bf if layout == 'nn' else af.t() @ bf)
    if out is not None:
        if accumulate:
            out.add_(r.to(out.dtype))
        else:
            out.copy_(r)
        return out
    return r.to(out_dtype or a.dtype)


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None, wgrad_out: Optional[torch.Tensor] = None,
           value_unused: bool = False):
    """``value_unused``: the caller never reads the result when the graph is being rebuilt (see ``dead_values``)."""
    if _cuda(x) and x.dtype == torch.bfloat16:
        n, k = weight.shape
        if n % 8 or k % 8:      # TMA rows are whole 16-byte vectors: odd sizes are filled up with zero rows / columns
            y = _Linear.apply(torch.nn.functional.pad(x, (0, -k % 8)), torch.nn.functional.pad(weight, (0, -k % 8, 0, -n % 8)), None, None, False)[..., :n]
            return y if bias is None else y + bias
        return _Linear.apply(x, weight, bias, wgrad_out, value_unused and _DeadValues.on)
    return torch.nn.functional.linear(x, weight, bias)


def linear_f32(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``x Wᵀ`` of 16-bit operands with the fp32 sums kept (no gradient): an output head whose logits are not rounded."""
    if not (_cuda(x) and x.dtype == torch.bfloat16):
        return torch.nn.functional.linear(x, weight).float()
    n, k = weight.shape
    if k % 8:
        x, weight = torch.nn.functional.pad(x, (0, -k % 8)), torch.nn.functional.pad(weight, (0, -k % 8))
    out = torch.empty(x.shape[0], -(-n // 4) * 4, dtype=torch.float32, device=x.device)[:, :n]
    return gemm(x.contiguous(), weight, 'nt', out=out)


# ------------------------------------------------------------------- norms
class _RMSNorm(torch.autograd.Function):

    @staticmethod
    def forward(ctx, x, weight, eps, offset):
        x2 = x.reshape(-1, x.shape[-1]).contiguous()       # a column slice of a wider tensor arrives strided
        y, rstd = ext().rmsnorm_fwd(x2, weight, eps, offset)
        ctx.save_for_backward(x2, weight, rstd)
        ctx.offset = offset
        ctx.shape = x.shape
        return y.view(x.shape)

    @staticmethod
    def backward(ctx, gy):
        x2, weight, rstd = ctx.saved_tensors
        gx, gw = ext().rmsnorm_bwd(gy.reshape(x2.shape).contiguous(), x2, weight, rstd, ctx.offset)
        return gx.view(ctx.shape), gw.to(weight.dtype), None, None


def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float = 1e-6, offset: float = 0.0) -> torch.Tensor:
    if _cuda(x) and x.dtype == torch.bfloat16:
        return _RMSNorm.apply(x, weight, eps, offset)
    return ref.rmsnorm(x, weight, eps, offset)


class _AddRMSNorm(torch.autograd.Function):
    """``h = x + residual``; ``y = rmsnorm(h)`` in one kernel.  Backward: the gradient that reaches ``h`` directly (the
    residual stream) is added inside the RMSNorm backward kernel, and the sum is the gradient of both inputs."""

    @staticmethod
    def forward(ctx, x, residual, weight, eps, offset):
        x2 = x.reshape(-1, x.shape[-1])
        r2 = residual.reshape(-1, x.shape[-1])
        y, rstd, h = ext().rmsnorm_fwd(x2.contiguous(), weight, eps, offset, r2.contiguous())
        ctx.save_for_backward(h, weight, rstd)
        ctx.offset = offset
        ctx.shape = x.shape
        return y.view(x.shape), h.view(x.shape)

    @staticmethod
    def backward(ctx, gy, gh):
        h, weight, rstd = ctx.saved_tensors
        if gy is None:
            return gh, gh, None, None, None
        gadd = gh.reshape(h.shape).contiguous() if gh is not None else None
        gx, gw = ext().rmsnorm_bwd(gy.reshape(h.shape).contiguous(), h, weight, rstd, ctx.offset, gadd)
        gx = gx.view(ctx.shape)
        return gx, gx, gw.to(weight.dtype), None, None


def add_rmsnorm(x, residual, weight, eps: float = 1e-6, offset: float = 0.0):
    """Returns ``(rmsnorm(x + residual), x + residual)``; one kernel on CUDA (the add costs no pass of its own, forward
    or backward)."""
    if _cuda(x) and x.dtype == torch.bfloat16 and residual.dtype == torch.bfloat16:
        return _AddRMSNorm.apply(x, residual, weight, eps, offset)
    return ref.add_rmsnorm(x, residual, weight, eps, offset)


# -------------------------------------------------------------------- rope
class _QKNormRope(torch.autograd.Function):
    """In: fused qkv ``[T, (Hq+2Hkv)·D]``; out: q ``[T,Hq,D]``, k ``[T,Hkv,D]``,
    v ``[T,Hkv,D]`` — per-head RMSNorm on q,k then rotate-half RoPE, one pass."""

    @staticmethod
    def forward(ctx, qkv, q_weight, k_weight, cos, sin, hq, hkv, d, eps):
        q, k, v, rstd = ext().qk_norm_rope_fwd(qkv, q_weight, k_weight, cos, sin, hq, hkv, d, eps)
        ctx.save_for_backward(qkv, q_weight, k_weight, cos, sin, rstd)
        ctx.dims = (hq, hkv, d, eps)
        return q, k, v

    @staticmethod
    def backward(ctx, gq, gk, gv):
        qkv, qw, kw, cos, sin, rstd = ctx.saved_tensors
        hq, hkv, d, eps = ctx.dims
        gqkv, gqw, gkw = ext().qk_norm_rope_bwd(gq.contiguous(), gk.contiguous(), gv.contiguous(), qkv, qw, kw, cos, sin,
                                                rstd, hq, hkv, d)
        return gqkv, gqw.to(qw.dtype), gkw.to(kw.dtype), None, None, None, None, None, None


_WARNED_HEAD_DIM = set()


def _head_dim_ok(d: int) -> bool:
    """The training attention and q/k-norm + RoPE kernels are written for 128-wide heads (every Qwen3 / Llama-3 size). Other
    widths — the tiny presets used in tests, vision towers — run on the PyTorch restatement; said once per width."""
    if d == 128:
        return True
    if d not in _WARNED_HEAD_DIM:
        _WARNED_HEAD_DIM.add(d)
        import logging
        logging.getLogger('twinkle_b200').warning(f'head_dim {d}: training attention and q/k-norm + RoPE run on PyTorch ops (those sm_100a kernels are for head_dim 128)')
    return False


def qkv_norm_rope(qkv: torch.Tensor, q_weight, k_weight, cos, sin, hq: int, hkv: int, d: int, eps: float = 1e-6, offset: float = 0.0):
    """Split fused qkv, apply q/k RMSNorm (if weights given; ``offset`` 1.0 = "1 + w") and RoPE on the leading
    ``2·cos.shape[-1]`` dims of every head.  The fused kernel serves full rotary with plain norm weights."""
    if (_cuda(qkv) and qkv.dtype == torch.bfloat16 and q_weight is not None and _head_dim_ok(d) and offset == 0.0
            and 2 * cos.shape[-1] == d):
        return _QKNormRope.apply(qkv.contiguous(), q_weight, k_weight, cos, sin, hq, hkv, d, eps)
    T = qkv.shape[0]
    q, k, v = qkv.split([hq * d, hkv * d, hkv * d], dim=-1)
    q, k, v = q.reshape(T, hq, d), k.reshape(T, hkv, d), v.reshape(T, hkv, d)
    q, k = ref.qk_norm_rope(q, k, q_weight, k_weight, cos, sin, eps, offset)
    return q, k, v


def rope_tables(positions: torch.Tensor, head_dim: int, theta: float = 1e6, scaling: Optional[dict] = None):
    return ref.rope_tables(positions, head_dim, theta, scaling)


# ------------------------------------------- layers with a 32-bit residual stream
def _needs_grad(*ts) -> bool:
    return torch.is_grad_enabled() and any(t is not None and t.requires_grad for t in ts)


def stream_rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, adds=(), mult: float = 1.0, offset: float = 0.0):
    """fp32 residual stream ``x [T, W]``: ``x ← x + mult · Σ y_i ⊙ s_i`` for ``adds = [(y, s), …]`` (at most two) and its RMS
    norm (weight ``offset + w``) in ``weight``'s dtype, one kernel on CUDA.  Returns ``(norm, x)``; without gradients ``x`` is
    updated in place."""
    if not _cuda(x) or _needs_grad(x, weight, *[t for a in adds for t in a]):
        return ref.stream_rmsnorm(x, weight, eps, weight.dtype, adds, mult, offset)
    (y1, s1), (y2, s2) = (list(adds) + [(None, None)] * 2)[:2]
    return ext().stream_rmsnorm(x, weight, eps, None if y1 is None else y1.contiguous(), s1, None if y2 is None else y2.contiguous(), s2, mult, offset), x


def stream_gated_rmsnorm(x, weight, eps: float, offset: float, result, gate, bias, post, row_of=None, share=None):
    """fp32 residual stream ``x [T, W]``: ``x ← x + norm(σ(gate + bias) ⊙ result; post)`` and the norm of the sum in ``weight``'s
    dtype (both norms with weights ``offset + w``), one kernel on CUDA.  ``gate``: leading ``W`` columns of a projection.
    ``result``: ``[T, W]``, or expert rows combined on the way (``row_of [T, k]``, ``share [T, k]``).  Returns ``(norm, x)``; without
    gradients ``x`` is updated in place."""
    if not _cuda(x) or _needs_grad(x, weight, result, gate, bias, post, share):
        return ref.stream_gated_rmsnorm(x, weight, eps, offset, result, gate, bias, post, row_of, share)
    return ext().stream_gated_rmsnorm(x, weight, eps, offset, result.contiguous(), gate, bias, post, row_of, share), x


def stream_joined_rmsnorm(x, weight, eps: float, offset: float, result, row_of=None, share=None, beside=None, open=None):
    """fp32 residual stream ``x [T, W]``: ``x ← x + result + open · beside`` and the norm of the sum (weight ``offset + w``) in ``weight``'s dtype,
    one kernel on CUDA.  ``result``: ``[T, W]``, or expert rows combined on the way (``row_of [T, k]``, ``share [T, k]``); ``beside [T, W]`` with a
    weight ``open [T]`` per token, or None.  Returns ``(norm, x)``; without gradients ``x`` is updated in place."""
    if not _cuda(x) or _needs_grad(x, weight, result, share, beside, open):
        return ref.stream_joined_rmsnorm(x, weight, eps, offset, result, row_of, share, beside, open)
    return ext().stream_joined_rmsnorm(x, weight, eps, offset, result.contiguous(), row_of, share, None if beside is None else beside.contiguous(), open), x


def stream_normed(x, weight, eps: float, y, bias, post, inner=None, beside=None, beside_inner=None):
    """fp32 residual stream ``x [T, W]``: ``x ← x + norm(y + bias; post)``, or with a second result ``x ← x + norm(½ (norm(y + bias; inner) +
    norm(beside; beside_inner)); post)``, and the norm of the sum (``weight`` None: the sum itself) in ``y``'s dtype, one kernel on CUDA.  Returns
    ``(norm, x)``; without gradients ``x`` is updated in place."""
    if not _cuda(x) or _needs_grad(x, weight, y, bias, post, inner, beside, beside_inner):
        return ref.stream_normed(x, weight, eps, y.dtype, y, bias, post, inner, beside, beside_inner)
    return ext().stream_normed(x, weight, eps, y.contiguous(), bias, post, inner, None if beside is None else beside.contiguous(), beside_inner), x


def position_waves(positions, frequencies, width: int):
    """``[T, width]`` fp32: sine and cosine of position times frequency (fp64) side by side."""
    return ref.position_waves(positions, frequencies, width)


def embed_positions(ids, weight, positions, frequencies):
    """Rows of an embedding plus :func:`position_waves`, fp32; one kernel on CUDA (no gradient)."""
    if _cuda(weight):
        return ext().embed_positions(ids.contiguous(), weight, positions.contiguous(), frequencies)
    return torch.nn.functional.embedding(ids, weight).float() + ref.position_waves(positions, frequencies, weight.shape[1])


# ------------------------------------------- heads without a rotation
def plain_heads(proj, first: int, bias, q_weight, k_weight, value_norm: bool, values_are_keys: bool, hq: int, hkv: int, d: int, e: int, eps: float, view=None, layer: int = -1):
    """Columns ``[q | k | v]`` (``[q | k]`` when the values are the projected keys) of a fused projection from ``first`` on → ``(q [T,hq,d'], k
    [T,hkv,d'] | None, v [T,hkv,e'] | None)``: bias, RMS norm of q and k per head (weights ``[d]``) or over all heads together (``[hq · d]``, ``[hkv ·
    d]``), values over their root mean square per head (``value_norm``).  ``view`` and the widths ``d'``, ``e'``: see :func:`rotary_heads`."""
    step = view is not None and view.stepping
    pools = (view.cache.k[layer], view.cache.v[layer], view.rows) if view is not None else (None, None, None)
    if _cuda(proj) and not _needs_grad(proj, bias, q_weight, k_weight):
        out = ext().plain_heads(proj, first, bias, q_weight, k_weight, value_norm, values_are_keys, hq, hkv, d, e, eps, *pools, not step)
        return tuple(out) if len(out) == 3 else (out[0], None, None)
    q, k, v = ref.plain_heads(proj, first, bias, q_weight, k_weight, value_norm, values_are_keys, hq, hkv, d, e, eps)
    if _needs_grad(proj, bias, q_weight, k_weight):
        return q, k, v
    q, k, v = (torch.nn.functional.pad(t, (0, -t.shape[-1] % 8)) for t in (q, k, v))
    if pools[0] is not None:
        pools[0].view(-1, *k.shape[1:])[view.rows] = k
        pools[1].view(-1, *v.shape[1:])[view.rows] = v
    return (q, None, None) if step else (q, k, v)


class ScoreTerms(NamedTuple):
    """What happens to an attention score beyond its scale, in this order: times a number per head (``temp [H]``), ``softcap · tanh(s / softcap)``, and a number
    for the distance ``n`` between query and key: ``−slope[h] ln(1 + rate[h] n)``, or ``table[bucket[min(n, last)], h]``."""
    softcap: float = 0.0
    temp: Optional[torch.Tensor] = None
    slope: Optional[torch.Tensor] = None
    rate: Optional[torch.Tensor] = None
    table: Optional[torch.Tensor] = None        # [rows, H]
    bucket: Optional[torch.Tensor] = None       # [distances] int32

    def apply(self, s, distance):
        """Scores ``[H, Lq, Lk]`` (scaled) at distances ``[Lq, Lk]``."""
        n = distance.clamp(min=0)
        if self.temp is not None:
            s = s * self.temp.float()[:, None, None]
        if self.softcap:
            s = self.softcap * torch.tanh(s / self.softcap)
        if self.slope is not None:
            s = s - self.slope.float()[:, None, None] * torch.log1p(self.rate.float()[:, None, None] * n)
        if self.table is not None:
            s = s + self.table.float()[self.bucket[n.clamp(max=self.bucket.numel() - 1)].long()].permute(2, 0, 1)
        return s

    @property
    def tensors(self):
        return self.temp, self.slope, self.rate, self.table, self.bucket


def _score_args(terms: Optional[ScoreTerms], softcap: float = 0.0):
    """A kernel's arguments for ``terms`` (or just a cap)."""
    if terms is None:
        return float(softcap or 0.0), None, None, None, None, None
    return (float(terms.softcap), *terms.tensors)


def _open_gate(o, gate):
    """The output of heads ``[T, H, e]`` times the sigmoid of a gate per head ``[T, H]`` or per element ``[T, H · e]``."""
    if gate is None:
        return o
    g = torch.sigmoid(gate.float())
    if g.shape[1] == o.shape[1]:
        return (o.float() * g[..., None]).to(o.dtype)
    g = g.view(*o.shape[:2], -1)
    return (o.float() * torch.nn.functional.pad(g, (0, o.shape[-1] - g.shape[-1]))).to(o.dtype)      # rows may be filled up with zeros


# ------------------------------------------- selective scan, matrix memory
def conv_silu(proj, first: int, channels: int, weight, bias, positions, view=None, layer: int = -1):
    """Causal depth-wise convolution (``weight [channels, taps]``, ``bias``) and silu on columns of a projection → ``[T, channels]``.  ``view`` (a
    ``CacheView``): the last inputs are kept in the history pool, a ring over positions, and single steps take their past from it."""
    step = view is not None and view.stepping
    hist = view.cache.conv[layer] if view is not None else None
    if _cuda(proj) and not _needs_grad(proj, weight, bias):
        return ext().conv_silu(proj, first, weight, bias, positions, step, hist, *((view.slots, view.left) if view is not None else (None, None)))
    x = proj[:, first:first + channels]
    y = ref.conv_silu(x, weight, bias, positions, hist if step else None, view.slots if step else None)
    if hist is not None:
        n = hist.shape[1]
        keep = (view.left < n).nonzero(as_tuple=True)[0]
        hist[view.slots[keep].long(), positions[keep] % n] = x[keep]
    return y


def selective_scan(u, dt, dt_bias, A_log, proj, b0: int, c0: int, D, gate, z0: int, cu_seqlens=None, max_seqlen: int = 0, view=None, layer: int = -1):
    """The selective scan behind its projections: inputs ``u [T, inner]``, step sizes ``softplus(dt + dt_bias)``, ``B`` and ``C`` in columns ``b0``, ``c0`` of
    ``proj``, ``A = −e^A_log``, skip ``D``, output gate ``silu`` of columns ``z0 …`` of ``gate`` → ``[T, inner]``.  Prompts start from an empty
    state; ``view`` (a ``CacheView``) says where the last states go, and single steps continue from there."""
    inner, n = A_log.shape
    step = view is not None and view.stepping
    states = view.cache.state[layer] if view is not None else None
    if _cuda(u) and not _needs_grad(u, dt, dt_bias, A_log, proj, D, gate):
        args = (u, dt, dt_bias, A_log, proj, b0, c0, D, gate, z0)
        if step:
            return ext().selective_step(*args, states, view.slots)
        return ext().selective_prefill(*args, cu_seqlens.to(torch.int32), int(max_seqlen), states, None if view is None else view.slots)
    args = (u, dt, dt_bias, A_log, proj[:, b0:b0 + n], proj[:, c0:c0 + n], D, gate[:, z0:z0 + inner])
    if step:
        slots = view.slots.long()
        y, last = ref.selective_scan(*args, list(range(u.shape[0] + 1)), list(states[slots]))
        states[slots] = torch.stack(last)
        return y
    y, last = ref.selective_scan(*args, cu_seqlens.tolist())
    if states is not None:
        states[view.slots[cu_seqlens[:-1].long()].long()] = torch.stack(last)
    return y


def matrix_memory(proj, first: int, heads: int, dim: int, vdim: int, i_bias, f_bias, cap: float, weight, eps: float, cu_seqlens=None, max_seqlen: int = 0, view=None,
                  layer: int = -1):
    """The matrix memory between its projections: columns ``[q | k | v | gate | i | f]`` of ``proj`` from ``first`` on → the normed and gated output ``[T, heads · vdim]``.
    Prompts start from an empty state; ``view`` (a ``CacheView``) says where the last states go, and single steps continue from there.  A
    state is a row of ``[heads, ·]``: the matrix by rows, the normaliser, the running maximum, each from a 16-byte boundary on."""
    step = view is not None and view.stepping
    states = view.cache.state[layer] if view is not None else None
    args = (proj, first, heads, dim, vdim, i_bias, f_bias, cap, weight, eps)
    if _cuda(proj) and not _needs_grad(proj, i_bias, f_bias, weight):
        if step:
            return ext().mlstm_step(*args, states, view.slots)
        return ext().mlstm_prefill(*args, cu_seqlens.to(torch.int32), int(max_seqlen), states, None if view is None else view.slots)
    n0 = -(-dim * vdim // 4) * 4
    m0 = n0 + -(-dim // 4) * 4

    def keep(slots, last):
        for s, (S, n, m) in zip(slots.tolist(), last):
            states[s, :, :dim * vdim], states[s, :, n0:n0 + dim], states[s, :, m0] = S.flatten(1), n, m
    if step:
        old = [(s[:, :dim * vdim].view(heads, dim, vdim), s[:, n0:n0 + dim], s[:, m0]) for s in states[view.slots.long()]]
        o, last = ref.matrix_memory(*args, list(range(proj.shape[0] + 1)), old)
        keep(view.slots, last)
        return o
    o, last = ref.matrix_memory(*args, cu_seqlens.tolist())
    if states is not None:
        keep(view.slots[cu_seqlens[:-1].long()], last)
    return o


# ------------------------------------------- rotated heads
def rotary_table(positions, frequencies):
    """``(cos, sin)`` of position times frequency (fp64 ``[n]``) as one fp32 tensor ``[T, n, 2]``."""
    if _cuda(positions):
        return ext().rotary_table(positions.contiguous(), frequencies)
    return ref.rotary_table(positions, frequencies)


def rotary_heads(proj, first: int, bias, q_weight, k_weight, table, at: int, pairs: int, interleaved: bool, hq: int, hkv: int, d: int, e: int, eps: float,
                 view=None, layer: int = -1):
    """Columns ``[q | k | v]`` of a fused projection from ``first`` on → ``(q [T,hq,d'], k [T,hkv,d'] | None, v [T,hkv,e'] | None)``: bias, RMS norm
    of q and k per head (weights ``[d]``, None: none), rotation of the leading ``2 · pairs`` dimensions by columns ``at …`` of ``table``
    (``rotary_table``).  ``hkv`` 0: queries only.  ``view`` (a ``CacheView``): keys and values are written to the cache; single steps return
    queries only.  Widths ``d'``, ``e'`` are ``d``, ``e`` rounded up to multiples of 8, the rest zero; with gradients they are ``d`` and ``e``."""
    step = view is not None and view.stepping
    pools = (view.cache.k[layer], view.cache.v[layer], view.rows) if view is not None and hkv else (None, None, None)
    if _cuda(proj) and not _needs_grad(proj, bias, q_weight, k_weight):
        out = ext().rotary_heads(proj, first, bias, q_weight, k_weight, table, at, pairs, interleaved, hq, hkv, d, e, eps, *pools, not step)
        return tuple(out) if len(out) == 3 else (out[0], None, None)
    q, k, v = ref.rotary_heads(proj, first, bias, q_weight, k_weight, table[:, at:at + pairs], interleaved, hq, hkv, d, e, eps)
    if _needs_grad(proj, bias, q_weight, k_weight):
        return q, k, v
    q, k, v = (None if t is None else torch.nn.functional.pad(t, (0, -t.shape[-1] % 8)) for t in (q, k, v))
    if pools[0] is not None:
        pools[0].view(-1, *k.shape[1:])[view.rows] = k
        pools[1].view(-1, *v.shape[1:])[view.rows] = v
    return (q, None, None) if step else (q, k, v)


def latent_rotary(proj, q0: int, heads: int, d: int, r: int, c0: int, nc: int, wc, eps: float, table, at: int, pairs: int, interleaved: bool, rank: int, view=None,
                  layer: int = -1):
    """Queries ``[d | r]`` per head in columns ``q0 …`` and a latent with its key part ``[nc | r]`` in columns ``c0 …`` of a projection (``nc`` 0: the
    layer borrows) → ``(q [T, heads, d + r], kept, ql)``.  The rotated dimensions ``r`` are turned by columns ``at …`` of ``table``, the latent is
    RMS-normed; ``kept [T, n']`` is ``[latent | key part]`` (``n'``: rounded up to a multiple of 8, the rest zero), also written to the cache that
    ``view`` names.  Prompts get the rotated query (without gradients ``proj`` is changed in place); single steps get ``ql [T, heads, rank + r]``
    with the rotated part in its last ``r`` columns, ready for the rest of the query in latent space."""
    T, step = proj.shape[0], view is not None and view.stepping
    pool = view.cache.k[layer] if view is not None and nc else None
    if _cuda(proj) and not _needs_grad(proj, wc):
        ql = torch.empty(T, heads, rank + r, dtype=proj.dtype, device=proj.device) if step else None
        kept = ext().latent_rotary(proj, q0, heads, d, r, c0, nc, wc, eps, table, at, pairs, interleaved, ql, pool, None if pool is None else view.rows, not step)
        return proj[:, q0:q0 + heads * (d + r)].view(T, heads, d + r), (kept if nc and not step else None), ql
    q, kept = ref.latent_rotary(proj, q0, heads, d, r, c0, nc, wc, eps, None if table is None else table[:, at:at + pairs], interleaved)
    if _needs_grad(proj, wc):
        return q, kept, None
    if kept is not None:
        kept = torch.nn.functional.pad(kept, (0, -kept.shape[-1] % 8))
        if pool is not None:
            pool.view(-1, pool.shape[-1])[view.rows] = kept
    return q, kept, (torch.nn.functional.pad(q[..., d:], (rank, 0)) if step else None)


# ------------------------------------------- latent attention, HGRN2
def latent_norms(proj, q0: int, nq: int, wq, c0: int, nc: int, wc, eps: float, view=None, layer: int = -1):
    """Column ranges of a projection → the normed query bottleneck ``[T, nq]`` and the normed latent ``[T, nc']`` (``nc'``: ``nc`` rounded
    up to a multiple of 8, the rest zero; None for ``nc`` 0), which is also written to the cache that ``view`` names."""
    pool = view.cache.k[layer] if view is not None and nc else None
    if _cuda(proj) and not _needs_grad(proj, wq, wc):
        q, c = ext().latent_norms(proj, q0, nq, wq, c0, nc, wc, eps, None if pool is None else pool, None if pool is None else view.rows)
        return q, (c if nc else None)
    q, c = ref.latent_norms(proj, q0, nq, wq, c0, nc, wc, eps)
    if c is not None and not _needs_grad(proj, wq, wc):
        c = torch.nn.functional.pad(c, (0, -nc % 8))
        if pool is not None:
            pool.view(-1, pool.shape[-1])[view.rows] = c
    return q, c


def head_linear(x, weight, transposed: bool = False, out=None):
    """One small matrix per head: ``x [B, H, K]`` times ``weight[h]ᵀ`` for ``weight [H, N, K]``, or times ``weight[h]`` for ``[H, K, N]``
    (``transposed``) → ``[B, H, N]``.  ``out [B, H, ≥ N]``: the result goes into its leading columns, and it is returned."""
    n, k = (weight.shape[2], weight.shape[1]) if transposed else weight.shape[1:]
    if _cuda(x) and x.dtype == torch.bfloat16 and n % 8 == 0 and k % 8 == 0 and not _needs_grad(x, weight) and (out is None or out.shape[2] % 8 == 0):
        y = ext().head_gemm(x if _tma_rows(x) else x.contiguous(), weight, transposed, None if out is None else out[..., :n])
        return y if out is None else out
    w = weight if transposed else weight.transpose(1, 2)
    y = torch.bmm(x.transpose(0, 1), w).transpose(0, 1)
    if out is None:
        return y.contiguous()
    out[..., :n] = y
    return out


def latent_decode(q, pool, table, lens, scale: float, sinks=None, gate=None, rank: int = 0, window: int = 0):
    """One token per sequence, ``q [B, H, K]`` in latent space, against the cached rows ``pool [blocks, bs, 1, K']``, keys of every head whose
    first ``rank`` columns (0: all ``K``) are the values → ``[B, H, rank]``.  ``window``: only the last positions (0: all); sink logits
    ``[H]`` in the denominator, result times ``σ(gate [B, H])``."""
    rank = rank or q.shape[-1]
    if _cuda(q):
        return ext().latent_decode(q.contiguous(), pool, table.to(torch.int32), lens.to(torch.int32), scale, sinks, gate, rank, window)
    return ref.latent_decode(q, pool, table, lens, scale, sinks, gate, rank, window)


def hgrn2(proj, q0: int, f0: int, v0: int, heads: int, dim: int, vdim: int, bias, lower, weight, eps: float, cu_seqlens=None, max_seqlen: int = 0,
          view=None, layer: int = -1):
    """The HGRN2 mixer between its projections: column ranges ``q``, ``f``, ``v`` of ``proj`` → the normed output ``[T, heads · vdim]``.  Prompts
    start from an empty state; ``view`` (a ``CacheView``) says where the last states go, and single steps continue from there."""
    step = view is not None and view.stepping
    states = view.cache.state[layer] if view is not None else None
    if _cuda(proj) and not _needs_grad(proj, bias, lower, weight):
        args = (proj, q0, f0, v0, heads, dim, vdim, bias, lower, weight, eps)
        if step:
            return ext().hgrn2_step(*args, states, view.slots)
        return ext().hgrn2_prefill(*args, cu_seqlens.to(torch.int32), int(max_seqlen), states, None if view is None else view.slots)
    if step:
        slots = view.slots.long()
        o, last = ref.hgrn2(proj, q0, f0, v0, heads, dim, vdim, bias, lower, weight, eps, list(range(proj.shape[0] + 1)), list(states[slots]))
        states[slots] = torch.stack(last)
        return o
    bounds = cu_seqlens.tolist()
    o, last = ref.hgrn2(proj, q0, f0, v0, heads, dim, vdim, bias, lower, weight, eps, bounds)
    if states is not None:
        states[view.slots[cu_seqlens[:-1].long()].long()] = torch.stack(last)
    return o


def conv_heads(proj, weight, positions, hq: int, hkv: int, d: int, e: int, eps: float, coef: float = 0.0, every: int = 0, v_first=None, lam=None,
               view=None, layer: int = -1):
    """Leading ``[q | k | v]`` columns of a fused projection → ``(q [T,hq,d'], k [T,hkv,d'] | None, v [T,hkv,e'])``: causal depth-wise
    convolution (``weight [C, taps]`` or None), q and k over their root mean square per head, query temperature, value mixing.
    ``view`` (a ``CacheView``) says where the tokens live in the sampler's cache: keys, values and the convolution history are
    written there, and single steps take their history from it (then k is None).  Widths ``d'``, ``e'`` are ``d``, ``e`` rounded
    up to multiples of 8, the rest zero; with gradients (no ``view``) they are ``d`` and ``e``."""
    step = view is not None and view.stepping
    cache = view.cache if view is not None else None
    hist = cache.conv[layer] if cache is not None else None
    if _cuda(proj) and not _needs_grad(proj, weight, v_first, lam):
        if v_first is not None:
            v_first = torch.nn.functional.pad(v_first, (0, -(-e // 8) * 8 - v_first.shape[-1])).contiguous()
        out = ext().conv_heads(proj, weight, positions, hq, hkv, d, e, eps, coef, every, v_first, lam, step, hist,
                               *((view.slots, view.left, view.rows, cache.k[layer], cache.v[layer]) if view is not None else (None, ) * 5), not step)
        return (out[0], None, out[1]) if step else tuple(out)
    if v_first is not None:
        v_first = v_first[..., :e]
    q, k, v = ref.conv_heads(proj, weight, positions, hq, hkv, d, e, eps, coef, every, v_first, lam, hist if step else None, view.slots if step else None)
    if _needs_grad(proj, weight, v_first, lam):
        return q, k, v
    q, k, v = (torch.nn.functional.pad(t, (0, -t.shape[-1] % 8)) for t in (q, k, v))
    if view is not None:
        cache.k[layer].view(-1, *k.shape[1:])[view.rows] = k
        cache.v[layer].view(-1, *v.shape[1:])[view.rows] = v
        if hist is not None:
            n, C = hist.shape[1:]
            keep = (view.left < n).nonzero(as_tuple=True)[0]
            hist[view.slots[keep].long(), positions[keep] % n] = proj[keep, :C]
    return q, (None if step else k), v


def glu_columns(proj: torch.Tensor, gate: int, up: int, width: int, limit: float = 0.0, act: str = 'silu') -> torch.Tensor:
    """``act(proj[:, gate : gate+width], proj[:, up : up+width])`` without copying the column ranges: ``silu(g) · u``, ``gelu_tanh(g) · u``, or with a
    ``limit`` ``g σ(1.702 g) (u + 1)`` on ``g ≤ limit`` and ``|u| ≤ limit``."""
    if _cuda(proj) and not _needs_grad(proj):
        return ext().glu_columns(proj, gate, up, width, limit, act == 'gelu_tanh')
    gu = torch.cat([proj[:, gate:gate + width], proj[:, up:up + width]], -1)
    return ref.geglu(gu) if act == 'gelu_tanh' else ref.clamped_glu(gu, limit) if limit else ref.swiglu(gu)


def _tma_rows(t) -> bool:
    """Whether rows and heads of ``[T, H, D]`` start on 16-byte boundaries with unit stride inside a head (16-bit elements)."""
    return t.stride(2) == 1 and t.stride(1) % 8 == 0 and t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0


def attention_packed(q, k, v, cu_seqlens, max_seqlen: int, scale: float, sinks=None, gate=None, window: int = 0, chunk: int = 0, key_tail=None,
                     terms: Optional[ScoreTerms] = None):
    """Causal packed attention for any key / value widths up to 256: tensor-core kernel for bf16 heads (keys up to 192, values up to
    128 wide), an fp32-arithmetic kernel for wider heads and for 32-bit models.  ``sinks [Hq]``: a logit per head in the denominator;
    ``gate``: the output is multiplied by its sigmoid, per head ``[T, Hq]`` or per element ``[T, Hq · e]``.  A position sees its last ``window`` keys,
    or its own block of ``chunk`` positions (0: no bound).  ``k`` and ``v`` may be column ranges of one tensor; ``key_tail [T, r]``: further key
    dimensions that all heads share (queries are ``[… | r]`` wide).  ``terms``: what else happens to scores."""
    extra = terms.tensors if terms is not None else ()
    if not _cuda(q) or _needs_grad(q, k, v, sinks, gate, key_tail, *extra):
        if key_tail is not None:
            k = torch.cat([k, key_tail[:, None].expand(-1, k.shape[1], -1)], -1)
        if window or chunk or terms is not None:
            o = ref.attention_varlen(q, k, v, cu_seqlens, True, scale, window=window or None, sinks=sinks, chunk=chunk, terms=terms)
        else:
            o = flash_attn_varlen(q, k, v, cu_seqlens, max_seqlen, True, scale, sinks=sinks)
        return _open_gate(o, gate)
    cu = cu_seqlens.to(torch.int32)
    if key_tail is not None:
        d, r = k.shape[2], key_tail.shape[1]
        if not (_flash_widths(q, k, v, 192) and d % 8 == 0 and r % 8 == 0 and d <= 128 and r <= 64 and key_tail.stride(0) % 8 == 0 and key_tail.data_ptr() % 16 == 0):
            k, key_tail = torch.cat([k, key_tail[:, None].expand(-1, k.shape[1], -1)], -1), None
    if _flash_widths(q, k, v, 192):
        q, k, v = (t if _tma_rows(t) else t.contiguous() for t in (q, k, v))
        return ext().flash_attn_fwd(q, k, v, cu, int(max_seqlen), True, scale, None, sinks, gate, window, chunk, key_tail, *_score_args(terms))[0]
    return ext().attention_packed(q.contiguous(), k.contiguous(), v.contiguous(), cu, int(max_seqlen), scale, sinks, gate, window, chunk, *_score_args(terms))


# ------------------------------------------------------------------ swiglu
class _SwiGLU(torch.autograd.Function):

    @staticmethod
    def forward(ctx, gate_up):
        ctx.save_for_backward(gate_up)
        return ext().swiglu_fwd(gate_up)

    @staticmethod
    def backward(ctx, gy):
        (gate_up, ) = ctx.saved_tensors
        return ext().swiglu_bwd(gy.contiguous(), gate_up)


def swiglu(gate_up: torch.Tensor) -> torch.Tensor:
    if _cuda(gate_up) and gate_up.dtype == torch.bfloat16:
        return _SwiGLU.apply(gate_up)
    return ref.swiglu(gate_up)


class _GeGLU(torch.autograd.Function):

    @staticmethod
    def forward(ctx, gate_up):
        ctx.save_for_backward(gate_up)
        return ext().geglu_fwd(gate_up)

    @staticmethod
    def backward(ctx, gy):
        (gate_up, ) = ctx.saved_tensors
        return ext().geglu_bwd(gy.contiguous(), gate_up)


def geglu(gate_up: torch.Tensor) -> torch.Tensor:
    """``[T, 2I]`` laid out as ``[gate | up]`` → ``gelu_tanh(gate) * up`` (Gemma-family MLPs); same kernel family as
    :func:`swiglu` (reference ``kernel/liger_impls/swiglu.py:26-32``)."""
    if _cuda(gate_up) and gate_up.dtype == torch.bfloat16:
        lead = gate_up.shape[:-1]
        return _GeGLU.apply(gate_up.reshape(-1, gate_up.shape[-1])).reshape(*lead, -1)
    return ref.geglu(gate_up)


# --------------------------------------------------------------- attention
class _FlashAttnVarlen(torch.autograd.Function):

    @staticmethod
    def forward(ctx, q, k, v, cu_seqlens, max_seqlen, causal, scale, cu_k=None, max_seqlen_k=0):
        out, lse = ext().flash_attn_fwd(q, k, v, cu_seqlens, max_seqlen, causal, scale, cu_k)
        ctx.save_for_backward(q, k, v, out, lse, cu_seqlens, cu_k if cu_k is not None else cu_seqlens)
        ctx.args = (max_seqlen, causal, scale, cu_k is not None, max_seqlen_k)
        ctx.mark_non_differentiable(lse)
        return out, lse

    @staticmethod
    def backward(ctx, gout, _glse):
        q, k, v, out, lse, cu, cu_k = ctx.saved_tensors
        max_seqlen, causal, scale, has_k, max_k = ctx.args
        dq, dk, dv = ext().flash_attn_bwd(gout.contiguous(), q, k, v, out, lse, cu, max_seqlen, causal, scale, cu_k if has_k else None, max_k)
        return dq, dk, dv, None, None, None, None, None, None


class _FlashAttnReuse(torch.autograd.Function):
    """Forward returns an attention output computed earlier (with its log-sum-exp); backward is the normal
    flash backward.  Lets an activation-recompute pass skip the attention forward."""

    @staticmethod
    def forward(ctx, q, k, v, out, lse, cu_seqlens, max_seqlen, causal, scale):
        ctx.save_for_backward(q, k, v, out, lse, cu_seqlens)
        ctx.args = (max_seqlen, causal, scale)
        return out.view_as(out)

    @staticmethod
    def backward(ctx, gout):
        q, k, v, out, lse, cu = ctx.saved_tensors
        max_seqlen, causal, scale = ctx.args
        dq, dk, dv = ext().flash_attn_bwd(gout.contiguous(), q, k, v, out, lse, cu, max_seqlen, causal, scale)
        return dq, dk, dv, None, None, None, None, None, None


class AttentionStash:
    """``mode='save'``: every attention call in scope appends its (out, lse); ``mode='reuse'``: calls consume
    them in the same order instead of recomputing."""
    current = None

    def __init__(self, mode: str, items=None, exchanges=None):
        """``items``: attention outputs; ``exchanges``: tensors received by sequence-parallel exchanges of the same
        layer (``None`` = do not keep them: the recompute pass exchanges again)."""
        self.mode, self.items, self._i = mode, ([] if items is None else items), 0
        self.exchanges, self._j = exchanges, 0

    def __enter__(self):
        self._prev = AttentionStash.current
        AttentionStash.current = self
        return self

    def __exit__(self, *exc):
        AttentionStash.current = self._prev


def _flash_widths(q, k, v, widest: int = 128) -> bool:
    """Whether the forward kernel takes these heads (training also needs the backward kernel, which is for 128-wide heads)."""
    d, e = q.shape[-1], v.shape[-1]
    return q.dtype == torch.bfloat16 and v.dtype == torch.bfloat16 and d <= widest and e <= 128 and d % 8 == 0 and e % 8 == 0


def flash_attn_varlen(q, k, v, cu_seqlens, max_seqlen: int, causal: bool = True, scale: Optional[float] = None,
                      cu_seqlens_k=None, max_seqlen_k: int = 0, return_lse: bool = False, window: Optional[int] = None,
                      softcap: Optional[float] = None, sinks: Optional[torch.Tensor] = None):
    """Packed causal attention with GQA.  ``q [T,Hq,D]``, ``k,v [Tk,Hkv,D]``.  ``cu_seqlens_k``: the keys of every
    sequence are a (longer) range of their own; the causal diagonal is aligned bottom-right.  A sliding ``window`` shorter
    than the longest row, a score ``softcap`` or per-head ``sinks`` select the PyTorch form (the kernels compute plain causal attention)."""
    scale = 1.0 / math.sqrt(q.shape[-1]) if scale is None else scale
    if window is not None and window >= max(int(max_seqlen), int(max_seqlen_k)):
        window = None           # no row reaches past the window: plain causal attention
    if window is not None or softcap or sinks is not None:
        return ref.attention_varlen(q, k, v, cu_seqlens, causal, scale, return_lse, cu_seqlens_k, window, softcap, sinks)
    if cu_seqlens_k is not None or return_lse:
        if _cuda(q) and q.dtype == torch.bfloat16 and _head_dim_ok(q.shape[-1]):
            out, lse = _FlashAttnVarlen.apply(q.contiguous(), k.contiguous(), v.contiguous(), cu_seqlens.to(torch.int32), int(max_seqlen), causal,
                                              scale, None if cu_seqlens_k is None else cu_seqlens_k.to(torch.int32), int(max_seqlen_k))
        else:
            out, lse = ref.attention_varlen(q, k, v, cu_seqlens, causal, scale, True, cu_seqlens_k)
        return (out, lse) if return_lse else out
    if _cuda(q) and q.shape[-1] != 128 and _flash_widths(q, k, v) and not _needs_grad(q, k, v) and AttentionStash.current is None:
        return ext().flash_attn_fwd(q.contiguous(), k.contiguous(), v.contiguous(), cu_seqlens.to(torch.int32), int(max_seqlen), causal, scale)[0]
    if _cuda(q) and q.dtype == torch.bfloat16 and _head_dim_ok(q.shape[-1]):
        q, k, v = q.contiguous(), k.contiguous(), v.contiguous()
        cu = cu_seqlens.to(torch.int32)
        st = AttentionStash.current
        if st is not None and st.mode == 'save' and not torch.is_grad_enabled():
            out, lse = ext().flash_attn_fwd(q, k, v, cu, int(max_seqlen), causal, scale)
            st.items.append((out, lse))
            return out
        if st is not None and st.mode == 'reuse' and st._i < len(st.items):
            out, lse = st.items[st._i]
            st._i += 1
            return _FlashAttnReuse.apply(q, k, v, out, lse, cu, int(max_seqlen), causal, scale)
        return _FlashAttnVarlen.apply(q, k, v, cu, int(max_seqlen), causal, scale)[0]
    return ref.attention_varlen(q, k, v, cu_seqlens, causal, scale)


def paged_attention_decode(q, k_cache, v_cache, block_tables, seq_lens, scale: Optional[float] = None, window: Optional[int] = None,
                           softcap: Optional[float] = None, sinks: Optional[torch.Tensor] = None, chunk: int = 0, gate: Optional[torch.Tensor] = None,
                           terms: Optional[ScoreTerms] = None):
    """One query token per sequence against the paged cache.  It sees its last ``window`` keys, or its own block of ``chunk`` positions;
    ``sinks [Hq]``: a logit per head in the denominator; ``gate``: the output is multiplied by its sigmoid, per head ``[B, Hq]`` or per element ``[B,
    Hq · e]``; ``softcap`` alone or all of ``terms``: what else happens to scores."""
    scale = 1.0 / math.sqrt(q.shape[-1]) if scale is None else scale
    vec = 16 // q.element_size()
    if (_cuda(q) and q.dtype in (torch.bfloat16, torch.float32) and all(t.shape[-1] % vec == 0 and t.shape[-1] <= 256 for t in (q, v_cache))
            and (sinks is None or sinks.dtype == q.dtype)):
        return ext().paged_attn_decode(q.contiguous(), k_cache, v_cache, block_tables.to(torch.int32), seq_lens.to(torch.int32), scale, window or 0, chunk, sinks, gate,
                                       *_score_args(terms, softcap))
    return _open_gate(ref.paged_attention_decode(q, k_cache, v_cache, block_tables, seq_lens, scale, window, softcap, sinks, chunk, terms), gate)


# ------------------------------------------------------ gated delta net (linear attention)
def _segment_starts(cu_seqlens: torch.Tensor, total: int) -> torch.Tensor:
    """``[T]`` int32: for every packed token the index of the first token of its sequence."""
    cu = cu_seqlens.to(torch.int64)
    lens = cu[1:] - cu[:-1]
    return torch.repeat_interleave(cu[:-1], lens, output_size=total).to(torch.int32)


class _CausalConv1d(torch.autograd.Function):
    """Forward: one kernel (depth-wise taps + SiLU, no leakage across packed sequences).  Backward: the gradient of the
    same op formed by autograd on the PyTorch expression (the convolution is a small share of a layer's backward)."""

    @staticmethod
    def forward(ctx, x, weight, cu_seqlens, activation):
        ctx.save_for_backward(x, weight, cu_seqlens)
        ctx.activation = activation
        return ext().causal_conv1d_fwd(x, weight.to(x.dtype).contiguous(), _segment_starts(cu_seqlens, x.shape[0]), activation)

    @staticmethod
    def backward(ctx, gy):
        from ..models.linear_attention import causal_conv1d_varlen_torch
        x, weight, cu = ctx.saved_tensors
        with torch.enable_grad():
            xd, wd = x.detach().requires_grad_(True), weight.detach().requires_grad_(True)
            y = causal_conv1d_varlen_torch(xd, wd, cu, ctx.activation)
            gx, gw = torch.autograd.grad(y, (xd, wd), gy)
        return gx, gw, None, None


def causal_conv1d_varlen(x: torch.Tensor, weight: torch.Tensor, cu_seqlens: torch.Tensor, activation: bool = True) -> torch.Tensor:
    """Depth-wise causal convolution (+ SiLU) over packed tokens: ``x [T, C]``, ``weight [C, W]``."""
    from ..models.linear_attention import causal_conv1d_varlen_torch
    if (_cuda(x) and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0 and 2 <= weight.shape[1] <= 4 and x.stride(1) == 1
            and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0):
        return _CausalConv1d.apply(x, weight, cu_seqlens, activation)
    return causal_conv1d_varlen_torch(x, weight, cu_seqlens, activation)


def gdn_kernel_supported(q: torch.Tensor, v: torch.Tensor) -> bool:
    return (_cuda(q) and q.dtype == torch.bfloat16 and v.dtype == torch.bfloat16 and q.shape[-1] in (64, 128)
            and q.stride(2) == 1 and q.stride(1) == q.shape[2] and v.stride(2) == 1 and v.stride(1) == v.shape[2])


class _GatedDeltaRule(torch.autograd.Function):
    """Forward: the recurrent kernel (q / k L2 normalisation and the grouped-head repeat inside).  Backward: autograd
    through the chunk-parallel PyTorch evaluator of the same function, re-run from the saved inputs."""

    @staticmethod
    def forward(ctx, q, k, v, g, beta, cu_seqlens, scale, chunk):
        o, _ = ext().gdn_recurrent_fwd(q, k, v, g.float().contiguous(), beta.float().contiguous(), cu_seqlens.to(torch.int32).contiguous(),
                                       None, scale, False)
        ctx.save_for_backward(q, k, v, g, beta, cu_seqlens)
        ctx.scale, ctx.chunk = scale, chunk
        return o

    @staticmethod
    def backward(ctx, go):
        from ..models.linear_attention import gated_delta_rule_varlen_torch
        q, k, v, g, beta, cu = ctx.saved_tensors
        with torch.enable_grad():
            ins = [t.detach().requires_grad_(True) for t in (q, k, v, g, beta)]
            o = gated_delta_rule_varlen_torch(*ins, cu, ctx.scale, chunk=ctx.chunk, normalize=True)
            grads = torch.autograd.grad(o, ins, go)
        return (*grads, None, None, None)


def gated_delta_rule_varlen(q, k, v, g, beta, cu_seqlens, scale: Optional[float] = None, chunk: int = 64, init_state=None,
                            return_states: bool = False):
    """Gated delta rule over packed sequences with **unnormalised** ``q, k [T, Hk, dk]`` (they are L2-normalised per head
    inside), ``v [T, Hv, dv]`` (``Hv`` a multiple of ``Hk``), ``g`` (log decay) and ``beta [T, Hv]``.  Returns
    ``o [T, Hv, dv]`` and, with ``return_states``, the final state per sequence ``[n, Hv, dk, dv]`` (fp32).
    ``init_state`` continues from earlier tokens (decoding); it and ``return_states`` are inference-only."""
    from ..models.linear_attention import gated_delta_rule_varlen_torch
    scale = q.shape[-1] ** -0.5 if scale is None else scale
    if gdn_kernel_supported(q, v) and gdn_kernel_supported(k, v):
        if init_state is None and not return_states:
            return _GatedDeltaRule.apply(q, k, v, g, beta, cu_seqlens, scale, chunk)
        if not torch.is_grad_enabled() or not any(t.requires_grad for t in (q, k, v, g, beta)):
            o, fin = ext().gdn_recurrent_fwd(q, k, v, g.float().contiguous(), beta.float().contiguous(),
                                             cu_seqlens.to(torch.int32).contiguous(),
                                             init_state.float().contiguous() if init_state is not None else None, scale, return_states)
            return (o, fin) if return_states else o
    return gated_delta_rule_varlen_torch(q, k, v, g, beta, cu_seqlens, scale, chunk=chunk, normalize=True, init_state=init_state,
                                         return_states=return_states)


# ------------------------------------------------------------- logprob / CE
class _LogprobFromLogits(torch.autograd.Function):

    @staticmethod
    def forward(ctx, logits, labels, temperature, with_entropy):
        x = logits.reshape(-1, logits.shape[-1])
        lp, lse, ent = ext().logprob_fwd(x, labels.reshape(-1).to(torch.int64), temperature, with_entropy)
        ctx.save_for_backward(x, labels.reshape(-1).to(torch.int64), lse, ent if with_entropy else lse)
        ctx.temperature, ctx.with_entropy, ctx.shape = temperature, with_entropy, logits.shape
        out_shape = labels.shape
        return lp.view(out_shape), (ent.view(out_shape) if with_entropy else lp.new_zeros(()))

    @staticmethod
    def backward(ctx, glp, gent):
        x, labels, lse, ent = ctx.saved_tensors
        gent_flat = gent.reshape(-1).contiguous().float() if ctx.with_entropy else None
        gx = ext().logprob_bwd(x.clone(), labels, lse, ent if ctx.with_entropy else None, glp.reshape(-1).contiguous().float(), gent_flat,
                               ctx.temperature)
        return gx.view(ctx.shape), None, None, None


def logprob_from_logits(logits, labels, temperature: float = 1.0, with_entropy: bool = False):
    """(logps, entropy|None); differentiable w.r.t. logits."""
    if _cuda(logits) and logits.dtype in (torch.bfloat16, torch.float32):
        lp, ent = _LogprobFromLogits.apply(logits.contiguous(), labels, temperature, with_entropy)
        return lp, (ent if with_entropy else None)
    return ref.logprob_from_logits(logits, labels, temperature, with_entropy)


class _FusedLinearLogprob(torch.autograd.Function):
    """lm_head GEMM + online-softmax statistics, chunked over tokens so the
    ``[T, V]`` logits never exist; backward re-forms each chunk's logits,
    converts them in place to dlogits and feeds the two gradient GEMMs."""

    @staticmethod
    def forward(ctx, hidden, weight, labels, temperature, with_entropy, chunk, wgrad_out):
        T = hidden.shape[0]
        lp = torch.empty(T, dtype=torch.float32, device=hidden.device)
        lse = torch.empty_like(lp)
        ent = torch.empty_like(lp) if with_entropy else None
        labels = labels.to(torch.int64)
        for s in range(0, T, chunk):
            e = min(s + chunk, T)
            logits = gemm(hidden[s:e], weight, 'nt')
            a, b, c = ext().logprob_fwd(logits, labels[s:e], temperature, with_entropy)
            lp[s:e], lse[s:e] = a, b
            if with_entropy:
                ent[s:e] = c
        ctx.save_for_backward(hidden, weight, labels, lse, ent if with_entropy else lse)
        ctx.cfg = (temperature, with_entropy, chunk)
        ctx.wgrad_out = wgrad_out
        return lp, (ent if with_entropy else lp.new_zeros(()))

    @staticmethod
    def backward(ctx, glp, gent):
        hidden, weight, labels, lse, ent = ctx.saved_tensors
        temperature, with_entropy, chunk = ctx.cfg
        T = hidden.shape[0]
        glp = glp.contiguous().float()
        gent = gent.contiguous().float() if with_entropy else None
        gh = torch.empty_like(hidden) if ctx.needs_input_grad[0] else None
        need_w = ctx.needs_input_grad[1]
        gw = ctx.wgrad_out
        if need_w and gw is None:
            gw = torch.zeros(weight.shape, dtype=torch.float32, device=weight.device)
        for s in range(0, T, chunk):
            e = min(s + chunk, T)
            logits = gemm(hidden[s:e], weight, 'nt')
            dlogits = ext().logprob_bwd(logits, labels[s:e], lse[s:e], ent[s:e] if with_entropy else None, glp[s:e],
                                        gent[s:e] if with_entropy else None, temperature)
            if gh is not None:
                gemm(dlogits, weight, 'nn', out=gh[s:e])
            if need_w:
                gemm(dlogits, hidden[s:e], 'tn', out=gw, accumulate=True)
        gw_ret = None
        if need_w and ctx.wgrad_out is None:
            gw_ret = gw.to(weight.dtype)
        return gh, gw_ret, None, None, None, None, None


def fused_linear_logprob(hidden, weight, labels, temperature: float = 1.0, with_entropy: bool = False, chunk: int = 4096,
                         wgrad_out: Optional[torch.Tensor] = None):
    """(logps [T] fp32, entropy|None) of ``labels`` under ``softmax(hidden·Wᵀ/T)``."""
    if _cuda(hidden) and hidden.dtype == torch.bfloat16:
        lp, ent = _FusedLinearLogprob.apply(hidden, weight, labels, temperature, with_entropy, chunk, wgrad_out)
        return lp, (ent if with_entropy else None)
    return ref.fused_linear_logprob(hidden, weight, labels, temperature, with_entropy)


# ------------------------------------------------------------------- adamw
def adamw_step(master, exp_avg, exp_avg_sq, grad, param_out, lr, beta1, beta2, eps, weight_decay, step, grad_scale=1.0):
    if _cuda(master):
        ext().adamw_step(master, exp_avg, exp_avg_sq, grad, param_out, float(lr), float(beta1), float(beta2), float(eps),
                         float(weight_decay), int(step), float(grad_scale))
    else:
        ref.adamw_step(master, exp_avg, exp_avg_sq, grad, param_out, lr, beta1, beta2, eps, weight_decay, step, grad_scale)


def sumsq(t: torch.Tensor) -> torch.Tensor:
    """Σ t² in fp32 as a 0-d tensor (partial of an L2 grad norm)."""
    if _cuda(t) and t.dtype in (torch.bfloat16, torch.float32) and t.is_contiguous():
        return ext().sumsq(t)
    return t.float().pow(2).sum()


# -------------------------------------------------------------------- lora
class _SGMV(torch.autograd.Function):
    """Segmented multi-LoRA on the tensor cores: shrink and expand are two expert-grouped tcgen05 GEMMs in
    which a *segment of tokens* plays the role of an expert and ``seg_slots`` maps it to its adapter block
    (−1 = no adapter → rows stay zero).  The rank mask (``r`` ≤ pool rank) and the ``alpha/r`` scale are one
    small element-wise pass over the ``[T, R]`` intermediate.  Weight gradients are per-segment ``tn`` GEMMs
    over 64-row-aligned token windows whose rows outside the segment are zeroed."""

    @staticmethod
    def forward(ctx, x, lora_a, lora_b, seg_starts, seg_slots, seg_ranks, seg_scales, host_segments, y_in=None, repeat=1):
        """``y_in`` (optional): the base projection's output; the delta is accumulated into it by the expand GEMM's
        epilogue instead of being produced as a tensor of its own and added.  ``repeat``: the pools of ``repeat``
        fused projections stacked along the rank axis (``A [S, repeat·R, K]``, ``B`` block-diagonal) — the rank mask
        then repeats per block."""
        E = ext()
        R = lora_a.shape[1]
        rowmask = _sgmv_rowmask(host_segments, R // repeat, x.device, x.dtype, repeat)   # [T, R] = scale where col < rank else 0
        h = E.grouped_gemm(x, lora_a, seg_starts, 'nt', seg_slots)             # [T, R]
        hm = h * rowmask
        if y_in is not None:
            E.grouped_gemm(hm, lora_b, seg_starts, 'nt', seg_slots, y_in, True)
            ctx.mark_dirty(y_in)
            y = y_in
        else:
            y = E.grouped_gemm(hm, lora_b, seg_starts, 'nt', seg_slots)        # [T, N]
        ctx.save_for_backward(x, lora_a, lora_b, hm, rowmask, seg_starts, seg_slots)
        ctx.host_segments = host_segments
        ctx.has_y = y_in is not None
        return y

    @staticmethod
    def backward(ctx, gy):
        E = ext()
        x, a, b, hm, rowmask, st, sl = ctx.saved_tensors
        gy = gy.contiguous()
        ghm = E.grouped_gemm(gy, b, st, 'nn', sl)                               # [T, R]   (b[s] is [N, R] = [K, N_out])
        gh = ghm * rowmask
        gx = E.grouped_gemm(gh, a, st, 'nn', sl) if ctx.needs_input_grad[0] else None
        ga = torch.zeros_like(a, dtype=torch.float32)
        gb = torch.zeros_like(b, dtype=torch.float32)
        T = x.shape[0]
        for (lo, hi, slot, rank, scale) in ctx.host_segments:
            if slot < 0 or rank == 0 or hi <= lo:
                continue
            a0, b0 = lo // 64 * 64, min((hi + 63) // 64 * 64, T)
            if a0 == lo and (b0 == hi or hi == T):       # the segment fills its 64-row windows: no rows to blank out
                ghs, hms = gh[a0:b0], hm[a0:b0]
            else:
                ghs, hms = gh[a0:b0].clone(), hm[a0:b0].clone()
                ghs[:lo - a0].zero_(), ghs[hi - a0:].zero_()
                hms[:lo - a0].zero_(), hms[hi - a0:].zero_()
            n = b0 - a0
            if n >= 8192:
                # split-K: the outputs are a handful of tiles ([R, K] and [N, R]) over a reduction of n rows — as one
                # GEMM that is a few CTAs walking the whole batch.  The K-grouped kernel gives every 1/32 of the rows
                # its own CTAs; the partial sums are added afterwards (32 small fp32 tensors)
                off = _split_k_offsets(n, x.device)
                ga[slot] += E.grouped_gemm_wgrad(ghs, x[a0:b0], off, off.numel() - 1).sum(0)
                gb[slot] += E.grouped_gemm_wgrad(gy[a0:b0], hms, off, off.numel() - 1).sum(0)
            else:
                E.gemm(ghs, x[a0:b0], 'tn', ga[slot], True, None)               # dA[slot] += ghᵀ x
                E.gemm(gy[a0:b0], hms, 'tn', gb[slot], True, None)              # dB[slot] += gyᵀ h
        return gx, ga.to(a.dtype), gb.to(b.dtype), None, None, None, None, None, (gy if ctx.has_y else None), None


_ROWMASKS: 'dict' = {}
_SPLITK: 'dict' = {}


def _split_k_offsets(n: int, device) -> torch.Tensor:
    """int32 boundaries that cut ``n`` reduction rows into at most 32 chunks whose sizes are multiples of 64."""
    key = (n, str(device))
    hit = _SPLITK.get(key)
    if hit is None:
        chunk = max(1024, ((n + 31) // 32 + 63) // 64 * 64)
        cuts = list(range(0, n, chunk)) + [n]
        hit = torch.tensor(cuts, dtype=torch.int32, device=device)
        if len(_SPLITK) >= 64:
            _SPLITK.pop(next(iter(_SPLITK)))
        _SPLITK[key] = hit
    return hit


def _sgmv_rowmask(host_segments, R: int, device, dtype, repeat: int = 1) -> torch.Tensor:
    """``[T, R]``: the segment's scale in the first ``rank`` columns of its rows, zero elsewhere.  Every LoRA linear of
    every layer asks for the same mask during one forward/backward (and its recompute), so the last few are kept: the
    mask is built on the host and copied once instead of by a dozen small kernels per call."""
    key = (tuple(host_segments), R, str(device), dtype, repeat)
    hit = _ROWMASKS.get(key)
    if hit is not None:
        return hit
    if repeat > 1:
        mask = _sgmv_rowmask(host_segments, R, device, dtype).repeat(1, repeat)
        if len(_ROWMASKS) >= 16:
            _ROWMASKS.pop(next(iter(_ROWMASKS)))
        _ROWMASKS[key] = mask
        return mask
    per_seg = torch.zeros(max(len(host_segments), 1), R, dtype=torch.float32)
    lens = []
    for i, (lo, hi, slot, rank, scale) in enumerate(host_segments):
        if slot >= 0:
            per_seg[i, :rank] = scale
        lens.append(hi - lo)
    if host_segments:
        rep = torch.tensor(lens, dtype=torch.int64, device=device)
        mask = per_seg[:len(host_segments)].to(device=device, dtype=dtype).repeat_interleave(rep, dim=0, output_size=sum(lens))
    else:
        mask = torch.zeros(0, R, device=device, dtype=dtype)
    if len(_ROWMASKS) >= 16:
        _ROWMASKS.pop(next(iter(_ROWMASKS)))
    _ROWMASKS[key] = mask
    return mask


def sgmv_fused_supported(x: torch.Tensor) -> bool:
    """Whether :func:`sgmv` can accumulate into the base output (``out=``) and take rank-stacked pools (``repeat=``)."""
    return _cuda(x) and x.dtype == torch.bfloat16


def sgmv(x, lora_a, lora_b, seg_starts, seg_slots, seg_ranks, seg_scales, host_segments=None, out=None, repeat: int = 1):
    """Multi-tenant LoRA delta for a token-segmented batch (see ``reference.sgmv``).  ``host_segments`` =
    ``[(lo, hi, slot, rank, scale)]`` mirrors the device tensors so the CUDA path needs no device read.  On a GPU
    ``out`` (the base projection's output ``[T, N]``) receives the delta in place and is returned; ``repeat`` says that
    ``lora_a`` / ``lora_b`` stack that many projections' pools along the rank axis."""
    if _cuda(x) and x.dtype == torch.bfloat16:
        if host_segments is None:
            starts = seg_starts.tolist()
            host_segments = [(starts[i], starts[i + 1], int(s), int(r), float(c)) for i, (s, r, c) in enumerate(
                zip(seg_slots.tolist(), seg_ranks.tolist(), seg_scales.tolist()))]
        T = x.shape[0]
        if any(hi > T for (_, hi, _, _, _) in host_segments):  # an open-ended segment ("all remaining tokens")
            host_segments = [(lo, min(hi, T), s, r, c) for (lo, hi, s, r, c) in host_segments if lo < T]
            seg_starts = torch.tensor([h[0] for h in host_segments] + [host_segments[-1][1]], dtype=torch.int32, device=x.device)
            seg_slots = torch.tensor([h[2] for h in host_segments], dtype=torch.int32, device=x.device)
        return _SGMV.apply(x.contiguous(), lora_a, lora_b, seg_starts, seg_slots, seg_ranks, seg_scales, host_segments, out, repeat)
    assert out is None and repeat == 1, 'in-place / stacked form is for the CUDA path'
    return _sgmv_autograd_cpu(x, lora_a, lora_b, seg_starts, seg_slots, seg_ranks, seg_scales)


def _sgmv_autograd_cpu(x, lora_a, lora_b, seg_starts, seg_slots, seg_ranks, seg_scales):
    outs = []
    starts = seg_starts.tolist()
    for i in range(len(starts) - 1):
        xs = x[starts[i]:starts[i + 1]]
        slot, r = int(seg_slots[i]), int(seg_ranks[i])
        if slot < 0 or r == 0:
            outs.append(xs.new_zeros(xs.shape[0], lora_b.shape[1]))
        else:
            outs.append((xs @ lora_a[slot, :r].t().to(xs.dtype)) @ lora_b[slot, :, :r].t().to(xs.dtype) * float(seg_scales[i]))
    return torch.cat(outs, 0) if outs else x.new_zeros(0, lora_b.shape[1])


# --------------------------------------------------------------------- moe
class _Router(torch.autograd.Function):
    """Fused fp32 softmax + top-k + renormalisation + expert histogram.  Backward is the closed form on the
    ``[T, E]`` probabilities (a few element-wise passes over a small tensor)."""

    @staticmethod
    def forward(ctx, logits, top_k, renorm, forced):
        w, idx, probs, hist = ext().moe_router(logits.contiguous(), top_k, renorm)
        if forced is not None:  # router replay: keep the probabilities, take the given experts (rows of -1: no replay)
            forced = forced.to(idx.device).long()
            idx = torch.where(forced[:, :1] < 0, idx, forced)
            w = probs.gather(-1, idx)
            if renorm:
                w = w / w.sum(-1, keepdim=True)
            hist = torch.zeros_like(hist).scatter_add_(0, idx.reshape(-1), torch.ones(idx.numel(), dtype=hist.dtype, device=hist.device))
        ctx.save_for_backward(probs, idx, w)
        ctx.renorm = renorm
        ctx.mark_non_differentiable(idx, hist)
        return w, idx, probs, hist

    @staticmethod
    def backward(ctx, gw, _gidx, gprobs, _ghist):
        probs, idx, w = ctx.saved_tensors
        dp = gprobs.clone() if gprobs is not None else torch.zeros_like(probs)
        if gw is not None:
            if ctx.renorm:
                S = probs.gather(-1, idx).sum(-1, keepdim=True)
                g_sel = (gw - (gw * w).sum(-1, keepdim=True)) / S
            else:
                g_sel = gw
            dp.scatter_add_(-1, idx, g_sel)
        dlogits = probs * (dp - (probs * dp).sum(-1, keepdim=True))
        return dlogits, None, None, None


def moe_router(logits, top_k: int, renormalize: bool = True, forced=None):
    """(weights [T,k] fp32, indices [T,k] int64, probs [T,E] fp32, histogram [E] | None)."""
    if _cuda(logits):
        return _Router.apply(logits, top_k, renormalize, forced)
    probs = torch.softmax(logits.float(), -1)
    w, idx = probs.topk(top_k, -1)
    if forced is not None:  # rows of -1 keep the router's own choice (tokens the sampler did not record)
        forced = forced.long()
        idx = torch.where(forced[:, :1] < 0, idx, forced)
        w = probs.gather(-1, idx)
    if renormalize:
        w = w / w.sum(-1, keepdim=True)
    return w, idx, probs, None


class _GroupedGemm(torch.autograd.Function):

    @staticmethod
    def forward(ctx, x, weight, offsets):
        ctx.save_for_backward(x, weight, offsets)
        return ext().grouped_gemm(x, weight, offsets, 'nt', None)

    @staticmethod
    def backward(ctx, gy):
        x, weight, offsets = ctx.saved_tensors
        gy = gy.contiguous()
        gx = ext().grouped_gemm(gy, weight, offsets, 'nn', None) if ctx.needs_input_grad[0] else None
        gw = ext().grouped_gemm_wgrad(gy, x, offsets, weight.shape[0]).to(weight.dtype) if ctx.needs_input_grad[1] else None
        return gx, gw, None


def grouped_gemm(x, weight, offsets, act: Optional[str] = None):
    """Per-expert GEMM over expert-sorted rows (``offsets [E+1]`` int32 on device).  ``act='relu2'``: the square of relu in the
    epilogue (no gradient)."""
    if _cuda(x) and x.dtype == torch.bfloat16:
        n, k = weight.shape[1:]
        if n % 8 or k % 8:      # TMA rows are whole 16-byte vectors: odd sizes are filled up with zero rows / columns
            pad = torch.nn.functional.pad
            return grouped_gemm(pad(x, (0, -k % 8)), pad(weight, (0, -k % 8, 0, -n % 8)), offsets, act)[:, :n]
        if act is not None:
            return ext().grouped_gemm(x, weight, offsets.to(torch.int32), 'nt', None, None, False, None, None, act)
        return _GroupedGemm.apply(x, weight, offsets.to(torch.int32))
    if _cuda(x) and x.dtype == torch.float32 and not _needs_grad(x, weight):
        return ext().grouped_gemm_f32(x.contiguous(), weight, offsets.to(torch.int32), act == 'relu2')
    if act is not None:
        return ref.relu2(grouped_gemm(x, weight, offsets))
    outs = []
    off = offsets.tolist()
    for e in range(weight.shape[0]):
        outs.append(x[off[e]:off[e + 1]] @ weight[e].t().to(x.dtype))
    if off[-1] < x.shape[0]:        # rows behind the last expert belong to nobody
        outs.append(x.new_zeros(x.shape[0] - off[-1], weight.shape[1]))
    return torch.cat(outs, 0)


def moe_topk(logits, bias, k: int, forced=None, groups: int = 0, keep: int = 0, factor: float = 1.0, x=None, shared=None):
    """fp32 ``logits [T, E]`` (+ ``bias``) → weights ``[T, k]`` fp32, their experts ``[T, k]`` int64, and tokens per expert ``[E]`` int32.
    ``groups`` 0: the k largest, weighed by a softmax over just those.  Otherwise a softmax over all experts, the k largest inside the
    ``keep`` best of ``groups`` groups of neighbours (a group is as good as its best expert), weighed by that softmax times ``factor``.
    ``forced``: experts to take instead (rows of −1: none).  With ``shared [1, H]`` a fourth result is ``σ(x · shared)`` ``[T]`` fp32."""
    if _cuda(logits) and logits.shape[1] <= 256 and k <= 32:
        return tuple(ext().moe_topk(logits, bias, k, None if forced is None else forced.to(logits.device).long().contiguous(), groups, keep, factor,
                                    None if shared is None else x, shared))
    z = logits.float() + (bias.float() if bias is not None else 0.0)
    w, idx = ref.moe_choice(z, k, forced, groups, keep, factor)
    hist = torch.zeros(z.shape[1], dtype=torch.int32, device=z.device).scatter_add_(0, idx.reshape(-1), torch.ones(idx.numel(), dtype=torch.int32, device=z.device))
    return (w, idx, hist) if shared is None else (w, idx, hist, torch.sigmoid(x.float() @ shared.float().t())[:, 0])


def moe_group_rows(x, idx, hist):
    """Rows of ``x [T, H]`` once per chosen expert, those of an expert together and nothing between them: ``(rows [T·k, H], row_of [T, k]
    int32, offsets [E+1] int32)``."""
    if _cuda(x) and hist.numel() <= 256:
        return tuple(ext().moe_group_rows(x.contiguous(), idx, hist))
    order = torch.argsort(idx.reshape(-1), stable=True)
    row_of = torch.empty(idx.numel(), dtype=torch.int32, device=x.device)
    row_of[order] = torch.arange(idx.numel(), dtype=torch.int32, device=x.device)
    offsets = torch.nn.functional.pad(hist.cumsum(0), (1, 0)).to(torch.int32)
    return x[order // idx.shape[1]], row_of.view(idx.shape), offsets


# ------------------------------------------------------- moe token permutation
def moe_index_maps(order: torch.Tensor, rows: torch.Tensor, bound: int, k: int):
    """From the expert sort (``order[i]`` = flat (token, slot) index of the i-th sorted pair, ``rows[i]`` = its row in
    the expert-grouped layout) build the two gather maps: ``row_of [T, k]`` (row of every (token, slot)),
    ``src_tok [bound]`` (token feeding each row, −1 = padding) and ``slot_of_row [bound]`` (flat index, −1 = padding)."""
    n = order.numel()
    dev = order.device
    row_of = torch.empty(n, dtype=torch.int32, device=dev)
    row_of[order] = rows.to(torch.int32)
    slot_of_row = torch.full((bound, ), -1, dtype=torch.int32, device=dev)
    slot_of_row[rows] = order.to(torch.int32)
    src_tok = torch.where(slot_of_row >= 0, slot_of_row // k, slot_of_row)
    return row_of.view(-1, k), src_tok, slot_of_row


def _rows_gather(x, src, scale=None):
    if _cuda(x) and x.dtype == torch.bfloat16:
        return ext().moe_rows_gather(x.contiguous(), src, scale)
    out = x.index_select(0, src.clamp_min(0).long()) * (src >= 0).to(x.dtype).unsqueeze(-1)
    return out if scale is None else out * scale.to(x.dtype).unsqueeze(-1)


def _rows_combine(y, row_of, w=None):
    if _cuda(y) and y.dtype == torch.bfloat16:
        return ext().moe_rows_combine(y.contiguous(), row_of, None if w is None else w.float().contiguous())
    g = y.index_select(0, row_of.reshape(-1).clamp_min(0).long()).view(row_of.shape[0], row_of.shape[1], -1)
    m = (row_of >= 0).to(y.dtype)
    if w is not None:
        m = m * w.to(y.dtype)
    return (g * m.unsqueeze(-1)).sum(1)


class _MoEDispatch(torch.autograd.Function):

    @staticmethod
    def forward(ctx, x, src_tok, row_of):
        ctx.save_for_backward(row_of)
        return _rows_gather(x, src_tok)

    @staticmethod
    def backward(ctx, g):
        row_of, = ctx.saved_tensors
        return _rows_combine(g.contiguous(), row_of), None, None


class _MoECombine(torch.autograd.Function):

    @staticmethod
    def forward(ctx, y, w, row_of, src_tok, slot_of_row):
        ctx.save_for_backward(y, w, row_of, src_tok, slot_of_row)
        return _rows_combine(y, row_of, w)

    @staticmethod
    def backward(ctx, g):
        y, w, row_of, src_tok, slot_of_row = ctx.saved_tensors
        g = g.contiguous()
        w_row = w.reshape(-1).float().index_select(0, slot_of_row.clamp_min(0).long())
        gy = _rows_gather(g, src_tok, w_row)
        if _cuda(y) and y.dtype == torch.bfloat16:
            gw = ext().moe_combine_wgrad(g, y, row_of)
        else:
            yy = y.index_select(0, row_of.reshape(-1).clamp_min(0).long()).view(row_of.shape[0], row_of.shape[1], -1)
            gw = (yy.float() * g.float().unsqueeze(1)).sum(-1) * (row_of >= 0)
        return gy, gw.to(w.dtype), None, None, None


def moe_dispatch(x, src_tok, row_of):
    """Token rows → expert-grouped rows (zero padding rows); backward sums every token's k rows."""
    return _MoEDispatch.apply(x, src_tok, row_of)


def moe_combine(y, w, row_of, src_tok, slot_of_row):
    """``out[t] = Σ_j w[t, j] · y[row_of[t, j]]`` with gradients for ``y`` and the routing weights ``w``."""
    return _MoECombine.apply(y, w, row_of, src_tok, slot_of_row)


class _ExpertLinearLora(torch.autograd.Function):
    """``y = x Wᵀ + s · (x Aᵀ) Bᵀ`` per expert over expert-grouped rows.  The low-rank term rides in the base GEMM as a
    second operand pair (``[x | h] · [W | s·B]ᵀ`` summed in tensor memory), forward and input-gradient alike, so the
    ``[rows, out]`` / ``[rows, in]`` tensors are written once and never re-read by an accumulate pass.
    ``TWINKLE_EXPERT_LORA_SPLIT=1`` keeps the earlier form (a separate rank-r GEMM accumulating into the output)."""

    @staticmethod
    def forward(ctx, x, weight, a, b, offsets, scale):
        E = ext()
        h = E.grouped_gemm(x, a, offsets, 'nt', None)                     # [rows, r]
        bs = (b.float() * scale).to(b.dtype)                               # [E, out, r] — scale folded into the small operand
        if _EXPERT_LORA_SPLIT:
            y = E.grouped_gemm(x, weight, offsets, 'nt', None)
            E.grouped_gemm(h, bs, offsets, 'nt', None, y, True)
        else:
            y = E.grouped_gemm(x, weight, offsets, 'nt', None, None, False, h, bs)
        ctx.save_for_backward(x, weight, a, bs, h, offsets)
        ctx.scale = scale
        return y

    @staticmethod
    def backward(ctx, gy):
        E = ext()
        x, weight, a, bs, h, offsets = ctx.saved_tensors
        gy = gy.contiguous()
        n_e = weight.shape[0]
        gh = E.grouped_gemm(gy, bs, offsets, 'nn', None)                   # [rows, r] = gy · (s·B)
        gx = None
        if ctx.needs_input_grad[0]:
            if _EXPERT_LORA_SPLIT:
                gx = E.grouped_gemm(gy, weight, offsets, 'nn', None)
                E.grouped_gemm(gh, a, offsets, 'nn', None, gx, True)
            else:
                gx = E.grouped_gemm(gy, weight, offsets, 'nn', None, None, False, gh, a)
        gw = E.grouped_gemm_wgrad(gy, x, offsets, n_e).to(weight.dtype) if ctx.needs_input_grad[1] else None
        ga = E.grouped_gemm_wgrad(gh, x, offsets, n_e).to(a.dtype) if ctx.needs_input_grad[2] else None
        gb = (E.grouped_gemm_wgrad(gy, h, offsets, n_e) * ctx.scale).to(bs.dtype) if ctx.needs_input_grad[3] else None
        return gx, gw, ga, gb, None, None


_EXPERT_LORA_SPLIT = os.environ.get('TWINKLE_EXPERT_LORA_SPLIT', '0') == '1'


def expert_linear(x, weight, offsets, lora_a=None, lora_b=None, scale: float = 1.0):
    """Per-expert linear over expert-grouped rows with an optional per-expert LoRA pair (``lora_a [E, r, in]``,
    ``lora_b [E, out, r]``)."""
    if lora_a is None:
        return grouped_gemm(x, weight, offsets)
    if _cuda(x) and x.dtype == torch.bfloat16:
        r = lora_a.shape[1]
        if r % 8:  # TMA rows must be 16-byte multiples: pad the rank with zero rows / columns
            pad = 8 - r % 8
            lora_a = torch.nn.functional.pad(lora_a, (0, 0, 0, pad))
            lora_b = torch.nn.functional.pad(lora_b, (0, pad))
        return _ExpertLinearLora.apply(x, weight, lora_a.contiguous(), lora_b.contiguous(), offsets.to(torch.int32), float(scale))
    return grouped_gemm(x, weight, offsets) + grouped_gemm(grouped_gemm(x, lora_a, offsets), lora_b, offsets) * scale


def sample_tokens(logits, temperature=1.0, top_k=-1, top_p=1.0, generator=None, seeds=None):
    """(tokens [B], logprob of each under the processed distribution [B]).  On CUDA every row draws from its
    own counter-based stream keyed by ``seeds[row]`` (fresh seeds when none are given)."""
    if _cuda(logits):
        if seeds is None:
            seeds = torch.randint(0, 2**62, (logits.shape[0], ), device=logits.device, dtype=torch.int64, generator=generator)
        tok, lp = ext().sample_tokens(logits.float().contiguous(), float(temperature), int(top_k), float(top_p), seeds)
        return tok, lp
    return ref.sample_tokens(logits, temperature, top_k, top_p, generator)


__all__ = [n for n in dir() if not n.startswith('_')]
