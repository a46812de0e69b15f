"""Kernel micro-benchmarks: ``python -m twinkle_b200.ops.microbench --op gemm --m 8192 --n 4096 --k 4096``.

Each op is timed with CUDA events on the launching stream after warm-up, with a write over a buffer larger
than L2 between iterations, and reported as achieved TFLOP/s or GB/s next to the fraction of the measured
device peaks (``MEASURED_PEAKS.json`` at the repository root when present; the stated fallback otherwise).
``--iters 1 --warmup 0 --no-flush`` gives a minimal launch sequence suitable for a profiler capture of one kernel.
"""
from __future__ import annotations

import argparse
import json
import os
from typing import Callable, Dict, Tuple

import torch


def peaks() -> Dict[str, float]:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), 'MEASURED_PEAKS.json')
    if os.path.exists(path):
        with open(path) as f:
            d = json.load(f)
        return dict(hbm_gbs=float(d['hbm_gbs']), tflops=float(d['bf16_tflops']), source='measured')
    return dict(hbm_gbs=6650.0, tflops=1590.0, source='fallback')


def time_op(fn: Callable[[], None], iters: int, warmup: int, flush: bool) -> float:
    """Median milliseconds per call."""
    scratch = torch.empty(256 << 20, dtype=torch.uint8, device='cuda') if flush else None
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    times = []
    for _ in range(iters):
        if scratch is not None:
            scratch.fill_(1)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
    times.sort()
    return times[len(times) // 2]


def _score_terms(a, dt):
    """Score terms of the attention ops: ``--terms log`` (cap and logarithms) or ``table`` (cap, factor per head, a table of 32 rows up to 1024)."""
    from twinkle_b200 import ops
    if not a.terms:
        return None
    one = torch.ones(a.heads, device='cuda', dtype=dt)
    if a.terms == 'log':
        return ops.ScoreTerms(30.0, slope=one, rate=0.1 * one)
    return ops.ScoreTerms(50.0, temp=one, table=torch.randn(32, a.heads, device='cuda', dtype=dt), bucket=(torch.arange(1025, device='cuda') * 31 // 1024).int())


def make(op: str, a) -> Tuple[Callable[[], None], float, float]:
    """(callable, flops, algorithmic bytes)."""
    from twinkle_b200 import ops
    E = ops.ext()
    dev = 'cuda'
    bf = torch.bfloat16
    if op == 'gemm':
        M, N, K = a.m, a.n, a.k
        shapes = {'nt': ((M, K), (N, K)), 'nn': ((M, K), (K, N)), 'tn': ((K, M), (K, N))}[a.layout]
        x, w = (torch.randn(s, device=dev, dtype=bf) for s in shapes)
        return (lambda: E.gemm(x, w, a.layout)), 2.0 * M * N * K, 2.0 * (M * K + N * K + M * N)
    if op == 'torch_gemm':
        x, w = torch.randn(a.m, a.k, device=dev, dtype=bf), torch.randn(a.n, a.k, device=dev, dtype=bf)
        return (lambda: torch.nn.functional.linear(x, w)), 2.0 * a.m * a.n * a.k, 2.0 * (a.m * a.k + a.n * a.k + a.m * a.n)
    if op in ('attn_fwd', 'attn_bwd'):
        T, hq, hkv, d = a.tokens, a.heads, a.kv_heads, 128
        n_seq = max(T // a.seq, 1)
        cu = torch.arange(0, n_seq + 1, device=dev, dtype=torch.int32) * a.seq
        q = torch.randn(T, hq, d, device=dev, dtype=bf, requires_grad=True)
        k = torch.randn(T, hkv, d, device=dev, dtype=bf, requires_grad=True)
        v = torch.randn(T, hkv, d, device=dev, dtype=bf, requires_grad=True)
        flops_fwd = 4.0 * n_seq * a.seq * a.seq * hq * d / 2  # causal
        byts = 2.0 * (2 * T * hq * d + 2 * T * hkv * d)
        if op == 'attn_fwd':
            def f():
                with torch.no_grad():
                    ops.flash_attn_varlen(q, k, v, cu, a.seq, True)
            return f, flops_fwd, byts
        o = ops.flash_attn_varlen(q, k, v, cu, a.seq, True)
        g = torch.randn_like(o)
        return (lambda: torch.autograd.grad(o, (q, k, v), g, retain_graph=True)), 2.5 * flops_fwd, 2.5 * byts
    if op in ('rope', 'rope_bwd'):
        T, hq, hkv = a.tokens, a.heads, a.kv_heads
        qkv = torch.randn(T, (hq + 2 * hkv) * 128, device=dev, dtype=bf)
        qw, kw = torch.ones(128, device=dev, dtype=bf), torch.ones(128, device=dev, dtype=bf)
        pos = torch.arange(T, device=dev) % 8192
        cos, sin = ops.rope_tables(pos, 128, 1e6)
        byts = 2.0 * 2 * T * (hq + 2 * hkv) * 128
        if op == 'rope':
            return (lambda: E.qk_norm_rope_fwd(qkv, qw, kw, cos, sin, hq, hkv, 128, 1e-6)), 0.0, byts
        q, k, v, rstd = E.qk_norm_rope_fwd(qkv, qw, kw, cos, sin, hq, hkv, 128, 1e-6)
        gq, gk, gv = torch.randn_like(q), torch.randn_like(k), torch.randn_like(v)
        return (lambda: E.qk_norm_rope_bwd(gq, gk, gv, qkv, qw, kw, cos, sin, rstd, hq, hkv, 128)), 0.0, 1.5 * byts
    if op in ('conv_heads', 'conv_heads_step'):
        # the step between projection and attention of a listed-layer stack: [q | k | v] in front of [gate | up] columns; prompts of
        # --seq tokens written into a paged cache, or one token of --batch sequences
        hq, hkv, d, taps, bs = a.heads, a.kv_heads, a.width, 4, 16
        step = op.endswith('step')
        T = a.batch if step else a.tokens
        C = (hq + 2 * hkv) * d
        proj = torch.randn(T, C + 6 * a.hidden, device=dev, dtype=bf)
        w, lam, vf = torch.randn(C, taps, device=dev, dtype=bf), torch.rand(1, device=dev, dtype=bf), torch.randn(T, hkv, d, device=dev, dtype=bf)
        pos = torch.full((T, ), a.seq - 1, device=dev) if step else torch.arange(T, device=dev) % a.seq
        kp, vp = (torch.zeros(T * bs if step else T, hkv, d, device=dev, dtype=bf) for _ in range(2))
        rows = torch.arange(T, device=dev) * (bs if step else 1)
        hist = torch.zeros(T + 1, taps - 1, C, device=dev, dtype=bf)
        slot = (torch.arange(T, device=dev, dtype=torch.int32) if step else (torch.arange(T, device=dev) // a.seq).int()) + 1
        left = torch.zeros(T, device=dev, dtype=torch.int32) if step else (a.seq - 1 - pos).int()
        # projection in; q, values (and keys of prompts) out, both pools; mixed-in values; history (all of it read and one row
        # of it written by a step, negligible for prompts)
        byts = 2.0 * T * d * (hq + 2 * hkv + hq + hkv + (0 if step else hkv) + 2 * hkv + hkv) + (2.0 * T * C * taps if step else 0.0)
        return (lambda: E.conv_heads(proj, w, pos, hq, hkv, d, d, 1e-5, 0.1, 4096, vf, lam, step, hist, slot, left, rows, kp, vp, not step)), 0.0, byts
    if op in ('rotary_heads', 'rotary_heads_step'):
        # bias, per-head norm, rotation and cache writes between projection and attention (the like kernel: rope, which norms and rotates)
        hq, hkv, d, bs, step = a.heads, a.kv_heads, a.width, 16, op.endswith('step')
        T = a.batch if step else a.tokens
        C = (hq + 2 * hkv) * d
        proj, bias, w = torch.randn(T, C + hq, device=dev, dtype=bf), torch.zeros(C, device=dev, dtype=bf), torch.ones(d, device=dev, dtype=bf)
        pos = torch.full((T, ), a.seq - 1, device=dev) if step else torch.arange(T, device=dev) % a.seq
        table = E.rotary_table(pos, torch.rand(d // 2, device=dev, dtype=torch.float64))
        kp, vp = (torch.zeros(T * bs if step else T, hkv, d, device=dev, dtype=bf) for _ in range(2))
        rows = torch.arange(T, device=dev) * (bs if step else 1)
        byts = 2.0 * T * d * (2 * hq + 2 * hkv + (2 if step else 4) * hkv)      # in; q; both pools; keys and values of prompts
        return (lambda: E.rotary_heads(proj, 0, bias, w, w, table, 0, d // 2, False, hq, hkv, d, d, 1e-6, kp, vp, rows, not step)), 0.0, byts
    if op == 'rotary_table':
        pos, f = torch.arange(a.tokens, device=dev) % a.seq, torch.rand(160, device=dev, dtype=torch.float64)
        return (lambda: E.rotary_table(pos, f)), 0.0, 8.0 * a.tokens * 160
    if op in ('latent_rotary', 'latent_rotary_step'):
        # norm of the latents (--rank), rotated parts (--tail) of keys and queries, cache write (the like kernel: latent_norms)
        H, d, r, R, step = a.heads, a.width, a.tail or 64, a.rank, op.endswith('step')
        T = a.batch if step else a.tokens
        proj, w = torch.randn(T, H * (d + r) + R + r, device=dev, dtype=bf), torch.ones(R, device=dev, dtype=bf)
        table = E.rotary_table(torch.arange(T, device=dev), torch.rand(r // 2, device=dev, dtype=torch.float64))
        pool, rows = torch.zeros(T, 1, 1, R + r, device=dev, dtype=bf), torch.arange(T, device=dev)
        ql = torch.empty(T, H, R + r, device=dev, dtype=bf) if step else None
        return ((lambda: E.latent_rotary(proj, 0, H, d, r, H * (d + r), R, w, 1e-6, table, 0, r // 2, True, ql, pool, rows, not step)), 0.0,
                2.0 * T * (2 * H * r + (2 if step else 3) * (R + r)))
    if op in ('joined_norm', 'joined_norm_experts'):
        W, k = a.hidden, 8
        x, w, b = torch.zeros(a.tokens, W, device=dev), torch.ones(W, device=dev, dtype=bf), torch.randn(a.tokens, W, device=dev, dtype=bf)
        if op == 'joined_norm':
            return (lambda: E.stream_joined_rmsnorm(x, w, 1e-6, 0.0, b)), 0.0, 12.0 * a.tokens * W
        y, o = torch.randn(a.tokens * k, W, device=dev, dtype=bf), torch.rand(a.tokens, device=dev)
        row_of, share = torch.randperm(a.tokens * k, device=dev, dtype=torch.int32).view(-1, k), torch.full((a.tokens, k), 1 / k, device=dev)
        return (lambda: E.stream_joined_rmsnorm(x, w, 1e-6, 0.0, y, row_of, share, b, o)), 0.0, a.tokens * W * (12.0 + 2.0 * k)
    if op == 'moe_topk_grouped':
        T, k, Ex = a.tokens, 8, 128
        lg, x, w = torch.randn(T, Ex, device=dev), torch.randn(T, a.hidden, device=dev, dtype=bf), torch.randn(1, a.hidden, device=dev, dtype=bf)
        return (lambda: E.moe_topk(lg, None, k, None, 8, 4, 1.0, x, w)), 0.0, 4.0 * T * Ex + 12.0 * T * k + 2.0 * T * a.hidden
    if op in ('hgrn2', 'hgrn2_step', 'gdn_step'):
        # the recurrent mixer between its projections: --heads states of 128 x 128 (prompts of --seq tokens, or a token of --batch
        # sequences); gdn_step: the Gated DeltaNet recurrence on one token of every sequence
        H, d, step = a.heads, a.width, op != 'hgrn2'
        T = a.batch if step else a.tokens
        if op == 'gdn_step':
            q, k, v = (torch.randn(T, H, d, device=dev, dtype=bf) for _ in range(3))
            g, beta, S = -torch.rand(T, H, device=dev) * 0.1, torch.rand(T, H, device=dev), torch.zeros(T, H, d, d, device=dev)
            cu = torch.arange(T + 1, device=dev, dtype=torch.int32)
            return (lambda: ops.gated_delta_rule_varlen(q, k, v, g, beta, cu, init_state=S, return_states=True)), 0.0, 8.0 * T * H * d * d
        proj = torch.randn(T, a.hidden + 3 * H * d, device=dev, dtype=bf)
        bias, low, w = torch.zeros(H * d, device=dev, dtype=bf), torch.zeros(H * d, device=dev, dtype=bf), torch.ones(d, device=dev, dtype=bf)
        n_seq = T if step else max(T // a.seq, 1)
        pool = torch.zeros(n_seq + 1, H, d, d, device=dev)
        args = (proj, a.hidden, a.hidden + H * d, a.hidden + 2 * H * d, H, d, d, bias, low, w, 1e-6)
        if step:
            slot = torch.arange(T, device=dev, dtype=torch.int32) + 1
            return (lambda: E.hgrn2_step(*args, pool, slot)), 0.0, 8.0 * T * H * d * d + 8.0 * T * H * d
        cu = torch.arange(0, n_seq + 1, device=dev, dtype=torch.int32) * a.seq
        slot = (torch.arange(T, device=dev) // a.seq).int() + 1
        # flops as for 'gdn' per state element and token: a write (multiply, add) and a read (multiply, add)
        return (lambda: E.hgrn2_prefill(*args, cu, a.seq, pool, slot)), 2.0 * T * H * d * d * 2, 8.0 * T * H * d
    if op == 'latent_decode':
        # --heads heads against latents of --rank with --tail rotated key dimensions inside --window (the like kernel: paged_decode)
        B, bs, ctx, R = a.batch, 16, a.seq, a.rank
        K, seen = R + a.tail, min(ctx, a.window or ctx)
        nb = B * ((ctx + bs - 1) // bs) + 1
        pool = torch.randn(nb, bs, 1, K, device=dev, dtype=bf)
        tables = torch.arange(1, nb, device=dev, dtype=torch.int32).view(B, -1)
        lens = torch.full((B, ), ctx, device=dev, dtype=torch.int32)
        q, sinks, gate = torch.randn(B, a.heads, K, device=dev, dtype=bf), torch.zeros(a.heads, device=dev, dtype=bf), torch.zeros(B, a.heads, device=dev, dtype=bf)
        if a.tail:
            sinks = gate = None
        return ((lambda: E.latent_decode(q, pool, tables, lens, K**-0.5, sinks, gate, R, a.window)), 2.0 * B * seen * a.heads * (K + R),
                2.0 * B * seen * K + 2.0 * B * a.heads * (K + R))
    if op == 'latent_norms':
        p = torch.randn(a.tokens, a.hidden + 1536 + 32, device=dev, dtype=bf)
        wq, wc = torch.ones(1024, device=dev, dtype=bf), torch.ones(512, device=dev, dtype=bf)
        pool, rows = torch.zeros(a.tokens, 1, 1, 512, device=dev, dtype=bf), torch.arange(a.tokens, device=dev)
        return (lambda: E.latent_norms(p, a.hidden, 1024, wq, a.hidden + 1024, 512, wc, 1e-6, pool, rows)), 0.0, 2.0 * a.tokens * (2 * 1536 + 512)
    if op == 'head_gemm':
        # the query into latent space: --batch tokens, --heads products of --width x --rank
        x, w = torch.randn(a.batch, a.heads, a.width, device=dev, dtype=bf), torch.randn(a.heads, a.width, a.rank, device=dev, dtype=bf)
        return (lambda: E.head_gemm(x, w, True)), 2.0 * a.batch * a.heads * a.width * a.rank, 2.0 * (x.numel() + w.numel() + a.batch * a.heads * a.rank)
    if op in ('gated_norm', 'gated_norm_experts'):
        W, k = a.hidden, 8
        x, g, w = torch.zeros(a.tokens, W, device=dev), torch.randn(a.tokens, W + 4096, device=dev, dtype=bf), torch.zeros(W, device=dev, dtype=bf)
        y = torch.randn(a.tokens * (k if op.endswith('experts') else 1), W, device=dev, dtype=bf)
        row_of = torch.randperm(a.tokens * k, device=dev, dtype=torch.int32).view(-1, k) if op.endswith('experts') else None
        share = torch.full((a.tokens, k), 1 / k, device=dev) if op.endswith('experts') else None
        return (lambda: E.stream_gated_rmsnorm(x, w, 1e-6, 1.0, y, g, w, w, row_of, share)), 0.0, a.tokens * W * (12.0 + 2.0 * (k if op.endswith('experts') else 1))
    if op in ('moe_topk', 'moe_group', 'moe_layout', 'moe_combine'):
        # choice and grouping of --tokens rows of --hidden over 128 experts, top 8; moe_layout: sort, index maps and gather of the
        # training block, moe_combine: its weighted sum
        T, k, Ex = a.tokens, 8, 128
        lg, x = torch.randn(T, Ex, device=dev), torch.randn(T, a.hidden, device=dev, dtype=bf)
        if op == 'moe_topk':
            return (lambda: E.moe_topk(lg, None, k, None)), 0.0, 4.0 * T * Ex + 12.0 * T * k
        w, idx, hist = E.moe_topk(lg, None, k, None)
        byts = 2.0 * T * a.hidden * (1 + k)
        if op == 'moe_group':
            return (lambda: E.moe_group_rows(x, idx, hist)), 0.0, byts
        from twinkle_b200.parallel.expert import expert_layout

        def layout():
            order, rows, offsets, bound = expert_layout(idx.reshape(-1), Ex, 128, hist)
            maps = ops.moe_index_maps(order, rows, bound, k)
            return maps, ops.moe_dispatch(x, maps[1], maps[0])
        if op == 'moe_layout':
            return layout, 0.0, byts
        (row_of, src, slot_of), xs = layout()
        return (lambda: ops.moe_combine(xs, w, row_of, src, slot_of)), 0.0, byts
    if op in ('experts_relu2', 'experts_swiglu', 'experts_columns'):
        # both products of the experts of one layer: two matrices with the activation in the epilogue, or [gate | up] and down
        T, k, Ex, W = a.tokens, 8, 128, a.hidden
        ff = 1152 if op == 'experts_relu2' else 768
        up = torch.randn(Ex, ff if op == 'experts_relu2' else 2 * ff, W, device=dev, dtype=bf) * 0.02
        down = torch.randn(Ex, W, ff, device=dev, dtype=bf) * 0.02
        _, idx, hist = E.moe_topk(torch.randn(T, Ex, device=dev), None, k, None)
        xs, _, off = E.moe_group_rows(torch.randn(T, W, device=dev, dtype=bf), idx, hist)

        def f():
            with torch.no_grad():
                if op == 'experts_columns':          # the unit as generation runs it
                    h = ops.glu_columns(ops.grouped_gemm(xs, up, off), 0, ff, ff)
                else:
                    h = ops.grouped_gemm(xs, up, off, act='relu2') if op == 'experts_relu2' else ops.swiglu(ops.grouped_gemm(xs, up, off))
                ops.grouped_gemm(h, down, off)
        used = min(Ex, T * k)
        return f, 2.0 * T * k * (up.shape[1] * W + W * ff), 2.0 * used * (up.shape[1] * W + W * ff)
    if op in ('stream_norm', 'add_rmsnorm'):
        w, y = torch.ones(a.hidden, device=dev, dtype=bf), torch.randn(a.tokens, a.hidden, device=dev, dtype=bf)
        if op == 'add_rmsnorm':
            r = torch.randn_like(y)
            return (lambda: E.rmsnorm_fwd(y, w, 1e-6, 0.0, r)), 0.0, 8.0 * a.tokens * a.hidden
        x, y2 = torch.zeros(a.tokens, a.hidden, device=dev), torch.randn_like(y)
        return (lambda: E.stream_rmsnorm(x, w, 1e-6, y, w, y2, w, 0.5)), 0.0, 14.0 * a.tokens * a.hidden
    if op == 'glu_columns':
        p = torch.randn(a.tokens, 6144 + 2 * a.hidden, device=dev, dtype=bf)
        return (lambda: E.glu_columns(p, 6144, 6144 + a.hidden, a.hidden, a.limit, a.gelu)), 0.0, 6.0 * a.tokens * a.hidden
    if op in ('stream_normed', 'stream_normed_pair'):
        # a normed result (or half the sum of two) joins the fp32 stream; its 16-bit copy goes on
        w, y = torch.ones(a.hidden, device=dev, dtype=bf), torch.randn(a.tokens, a.hidden, device=dev, dtype=bf)
        x, y2 = torch.zeros(a.tokens, a.hidden, device=dev), torch.randn_like(y)
        more = (w, y2, w) if op == 'stream_normed_pair' else ()
        return (lambda: ops.stream_normed(x, None, 1e-6, y, w, w, *more)), 0.0, (14.0 if more else 12.0) * a.tokens * a.hidden
    if op == 'embed_positions':
        ids, pos = torch.randint(0, a.vocab, (a.tokens, ), device=dev), torch.arange(a.tokens, device=dev)
        emb = torch.randn(a.vocab, a.hidden, device=dev, dtype=bf)
        f = torch.tensor([10000.0**(-2 * i / a.hidden) for i in range(a.hidden // 2)], dtype=torch.float64, device=dev)
        return (lambda: ops.embed_positions(ids, emb, pos, f)), 0.0, 6.0 * a.tokens * a.hidden
    if op in ('plain_heads', 'shared_heads'):
        # bias, norms and cache rows of 128-wide heads: q, k and v normed head by head, or q and k over all heads with the keys as values
        T, hq, hkv, d, shared = a.tokens, a.heads, a.kv_heads, 128, op == 'shared_heads'
        C = (hq + hkv * (1 if shared else 2)) * d
        proj, bias = torch.randn(T, C + 4096, device=dev, dtype=bf), torch.randn(C, device=dev, dtype=bf)
        qw, kw = (torch.ones(n * d if shared else d, device=dev, dtype=bf) for n in (hq, hkv))
        pool, rows = torch.zeros(T // 16 + 1, 16, hkv, d, device=dev, dtype=bf), torch.arange(T, device=dev)
        vpool = torch.zeros_like(pool)
        step = T <= 1024          # a step needs no keys and values of its own
        return ((lambda: E.plain_heads(proj, 0, bias, qw, kw, not shared, shared, hq, hkv, d, d, 1e-6, pool, vpool, rows, not step)), 0.0,
                2.0 * T * (C + d * (hq + 2 * hkv * (1 if step else 2))))
    if op in ('conv_silu', 'conv_silu_step'):
        T, n = a.tokens, a.hidden
        x, w, b = torch.randn(T, 2 * n, device=dev, dtype=bf), torch.randn(n, 4, device=dev, dtype=bf), torch.randn(n, device=dev, dtype=bf)
        step = op == 'conv_silu_step'
        pos = torch.full((T, ), 99, device=dev) if step else torch.arange(T, device=dev) % a.seq
        hist, slot = torch.zeros(T + 1 if step else T // a.seq + 2, 3, n, device=dev, dtype=bf), torch.arange(T, device=dev, dtype=torch.int32) // (1 if step else a.seq) + 1
        left = torch.zeros(T, device=dev, dtype=torch.int32) if step else (a.seq - 1 - pos).int()
        return (lambda: E.conv_silu(x, 0, w, b, pos, step, hist, slot, left)), 0.0, (12.0 if step else 4.0) * T * n
    if op in ('selective', 'selective_step'):
        # selective scan of --hidden channels with --states each; one token of --tokens sequences, or prompts of --seq tokens
        T, n, N, step = a.tokens, a.hidden, a.states, op == 'selective_step'
        u, dt, z = (torch.randn(T, n, device=dev, dtype=bf) for _ in range(3))
        A, D, b = (torch.randn(n, N, device=dev) - 1).to(bf), torch.ones(n, device=dev, dtype=bf), (torch.randn(n, device=dev) - 3).to(bf)
        bc = torch.randn(T, 2 * N, device=dev, dtype=bf)
        n_seq = T if step else max(T // a.seq, 1)
        state, slot = torch.zeros(n_seq + 1, n, N, device=dev), torch.arange(T, device=dev, dtype=torch.int32) * n_seq // T + 1
        if step:
            return (lambda: E.selective_step(u, dt, b, A, bc, 0, N, D, z, 0, state, slot)), 0.0, T * n * (8.0 + 8.0 * N) + 2.0 * n * N
        cu = torch.arange(0, n_seq + 1, device=dev, dtype=torch.int32) * a.seq
        return (lambda: E.selective_prefill(u, dt, b, A, bc, 0, N, D, z, 0, cu, a.seq, state, slot)), 6.0 * T * n * N, 8.0 * T * n
    if op in ('mlstm', 'mlstm_step'):
        # matrix memory of --heads heads of 128 x --width; one token of --tokens sequences, or prompts of --seq tokens
        T, H, d, e, step = a.tokens, a.heads, 128, a.width, op == 'mlstm_step'
        C = 2 * H * (d + e + 1)
        p, w, b = torch.randn(T, C + -C % 8, device=dev, dtype=bf), torch.ones(H * e, device=dev, dtype=bf), torch.ones(H, device=dev, dtype=bf)
        n_seq = T if step else max(T // a.seq, 1)
        state, slot = torch.zeros(n_seq + 1, H, d * e + d + 4, device=dev), torch.arange(T, device=dev, dtype=torch.int32) * n_seq // T + 1
        if step:
            return (lambda: E.mlstm_step(p, 0, H, d, e, b, 4 * b, 15.0, w, 1e-6, state, slot)), 0.0, T * (8.0 * H * d * (e + 1) + 2.0 * (C + H * e))
        cu = torch.arange(0, n_seq + 1, device=dev, dtype=torch.int32) * a.seq
        return (lambda: E.mlstm_prefill(p, 0, H, d, e, b, 4 * b, 15.0, w, 1e-6, cu, a.seq, state, slot)), 4.0 * T * H * d * e, 2.0 * T * (C + H * e)
    if op in ('attn_packed', 'attn_packed32'):
        # prefill attention at any head width (--width): the tensor-core kernel up to 192 in bf16, fp32 arithmetic beyond / in 32-bit;
        # --window / --chunk bound what a position sees, --tail adds key dimensions that all heads share
        T, d, dt = a.tokens, a.width, bf if op == 'attn_packed' else torch.float32
        n_seq = max(T // a.seq, 1)
        cu = torch.arange(0, n_seq + 1, device=dev, dtype=torch.int32) * a.seq
        q, k, v = (torch.randn(T, h, w, device=dev, dtype=dt) for h, w in ((a.heads, d + a.tail), (a.kv_heads, d), (a.kv_heads, d)))
        tail = torch.randn(T, a.tail, device=dev, dtype=dt) if a.tail else None
        first = [max(0, i - a.window + 1) if a.window else (i // a.chunk * a.chunk if a.chunk else 0) for i in range(a.seq)]
        pairs = n_seq * sum(i + 1 - f for i, f in enumerate(first))
        sinks = torch.zeros(a.heads, device=dev, dtype=dt) if a.sinks else None
        gate = torch.zeros(T, a.heads * (d if a.terms == 'table' else 1), device=dev, dtype=dt) if a.sinks else None
        terms = _score_terms(a, dt)
        return ((lambda: ops.attention_packed(q, k, v, cu, a.seq, d**-0.5, sinks, gate, a.window, a.chunk, tail, terms)), 2.0 * pairs * a.heads * (2 * d + a.tail),
                float(q.element_size()) * T * (d * (2 * a.heads + 2 * a.kv_heads) + a.tail * (a.heads + 1)))
    if op == 'rmsnorm':
        x, w = torch.randn(a.tokens, a.hidden, device=dev, dtype=bf), torch.ones(a.hidden, device=dev, dtype=bf)

        def f():
            with torch.no_grad():
                ops.rmsnorm(x, w, 1e-6)
        return f, 0.0, 4.0 * a.tokens * a.hidden
    if op == 'rmsnorm_bwd':
        x, w = torch.randn(a.tokens, a.hidden, device=dev, dtype=bf), torch.ones(a.hidden, device=dev, dtype=bf)
        g = torch.randn_like(x)
        _, rstd = E.rmsnorm_fwd(x, w, 1e-6, 0.0)
        return (lambda: E.rmsnorm_bwd(g, x, w, rstd, 0.0)), 0.0, 6.0 * a.tokens * a.hidden
    if op == 'swiglu':
        gu = torch.randn(a.tokens, 2 * a.hidden, device=dev, dtype=bf)

        def f():
            with torch.no_grad():
                ops.swiglu(gu)
        return f, 0.0, 6.0 * a.tokens * a.hidden
    if op == 'logprob':
        x = torch.randn(a.tokens, a.vocab, device=dev, dtype=bf)
        y = torch.randint(0, a.vocab, (a.tokens, ), device=dev)

        def f():
            with torch.no_grad():
                ops.logprob_from_logits(x, y)
        return f, 0.0, 2.0 * a.tokens * a.vocab
    if op == 'adamw':
        n = a.numel
        p, g = torch.randn(n, device=dev), torch.randn(n, device=dev, dtype=bf)
        m, v, lo = torch.zeros(n, device=dev), torch.zeros(n, device=dev), torch.empty(n, device=dev, dtype=bf)
        return (lambda: ops.adamw_step(p, m, v, g, lo, 1e-4, 0.9, 0.95, 1e-8, 0.01, 1, 1.0)), 0.0, float(n) * (4 * 3 * 2 + 2 + 2)
    if op == 'sgmv':
        # four tenants share the batch: equal token segments, each on its own adapter slot (rank a.rank of a pool of 16)
        T, H, N, r = a.tokens, a.hidden, a.n, a.rank
        x = torch.randn(T, H, device=dev, dtype=bf)
        A = torch.randn(4, 16, H, device=dev, dtype=bf) * 0.02
        B = torch.randn(4, N, 16, device=dev, dtype=bf) * 0.02
        cuts = [T * i // 4 for i in range(5)]
        host = [(cuts[i], cuts[i + 1], i, r, 2.0) for i in range(4)]
        st = torch.tensor(cuts, dtype=torch.int32, device=dev)
        sl = torch.arange(4, dtype=torch.int32, device=dev)
        rk = torch.full((4, ), r, dtype=torch.int32, device=dev)
        sc = torch.full((4, ), 2.0, dtype=torch.float32, device=dev)

        def f():
            with torch.no_grad():
                ops.sgmv(x, A, B, st, sl, rk, sc, host)
        return f, 2.0 * T * r * (H + N), 2.0 * T * (H + N)
    if op == 'paged_decode':
        B, bs, ctx = a.batch, 16, a.seq
        nb = B * ((ctx + bs - 1) // bs)
        kc = torch.randn(nb, bs, a.kv_heads, a.width, device=dev, dtype=bf)
        vc = torch.randn_like(kc)
        tables = torch.arange(nb, device=dev, dtype=torch.int32).view(B, -1)
        lens = torch.full((B, ), ctx, device=dev, dtype=torch.int32)
        q = torch.randn(B, a.heads, a.width, device=dev, dtype=bf)
        sinks, gate = (torch.zeros(a.heads, device=dev, dtype=bf), torch.zeros(B, a.heads * (a.width if a.terms == 'table' else 1), device=dev, dtype=bf)) if a.sinks else (None, None)
        terms = _score_terms(a, bf)
        seen = min(ctx, a.window or ctx) if not a.chunk else (ctx - 1) % a.chunk + 1
        return ((lambda: ops.paged_attention_decode(q, kc, vc, tables, lens, window=a.window or None, chunk=a.chunk, sinks=sinks, gate=gate, terms=terms)), 0.0,
                2.0 * 2 * B * seen * a.kv_heads * a.width)
    if op == 'sample':
        lg = torch.randn(a.batch, a.vocab, device=dev)
        seeds = torch.arange(a.batch, device=dev, dtype=torch.int64)
        return (lambda: ops.sample_tokens(lg, 0.8, 50, 0.95, seeds=seeds)), 0.0, 4.0 * a.batch * a.vocab
    if op in ('expert_lora', 'expert_lora_split', 'expert_base'):
        # one expert projection of the Qwen3-30B-A3B block: rows = tokens x top-8 over 128 experts (128-row aligned
        # segments), 2048 -> 1536, rank-16 LoRA pair per expert.  expert_base: the grouped GEMM alone; expert_lora: the
        # low-rank term as a second operand pair of the same GEMM; expert_lora_split: shrink, base, then a separate
        # rank-16 GEMM accumulating into the output
        Eg, K, N, r = 128, 2048, 1536, 16
        per = (a.tokens * 8 // Eg + 127) // 128 * 128
        rows = per * Eg
        off = torch.arange(0, Eg + 1, device=dev, dtype=torch.int32) * per
        x = torch.randn(rows, K, device=dev, dtype=bf)
        w = torch.randn(Eg, N, K, device=dev, dtype=bf) * 0.02
        la = torch.randn(Eg, r, K, device=dev, dtype=bf) * 0.02
        lb = torch.randn(Eg, N, r, device=dev, dtype=bf) * 0.02
        flops = 2.0 * rows * K * N + (0.0 if op == 'expert_base' else 2.0 * rows * r * (K + N))
        byts = 2.0 * (rows * K + rows * N + Eg * N * K)
        if op == 'expert_base':
            return (lambda: E.grouped_gemm(x, w, off, 'nt', None)), flops, byts
        if op == 'expert_lora':
            def f():
                h = E.grouped_gemm(x, la, off, 'nt', None)
                E.grouped_gemm(x, w, off, 'nt', None, None, False, h, lb)
            return f, flops, byts

        def f2():
            y = E.grouped_gemm(x, w, off, 'nt', None)
            h = E.grouped_gemm(x, la, off, 'nt', None)
            E.grouped_gemm(h, lb, off, 'nt', None, y, True)
        return f2, flops, byts
    if op in ('gdn', 'gdn_torch'):
        # Gated DeltaNet forward: 16 key / 32 value heads of 128, packed documents of --seq tokens
        T, hk, hv, d = a.tokens, 16, 32, 128
        n_seq = max(T // a.seq, 1)
        cu = torch.arange(0, n_seq + 1, device=dev, dtype=torch.int32) * a.seq
        q, k = torch.randn(T, hk, d, device=dev, dtype=bf), torch.randn(T, hk, d, device=dev, dtype=bf)
        v = torch.randn(T, hv, d, device=dev, dtype=bf)
        g, beta = -torch.rand(T, hv, device=dev) * 0.1, torch.rand(T, hv, device=dev)
        byts = 2.0 * T * d * (2 * hk + 2 * hv) + 8.0 * T * hv
        flops = 2.0 * T * hv * d * d * 3            # S·k, S·q and the rank-1 update
        if op == 'gdn':
            def f():
                with torch.no_grad():
                    ops.gated_delta_rule_varlen(q, k, v, g, beta, cu)
        else:
            from twinkle_b200.models.linear_attention import gated_delta_rule_varlen_torch

            def f():
                with torch.no_grad():
                    gated_delta_rule_varlen_torch(q, k, v, g, beta, cu)
        return f, flops, byts
    if op == 'router':
        lg = torch.randn(a.tokens, 128, device=dev, dtype=bf)

        def f():
            with torch.no_grad():
                ops.moe_router(lg, 8, True)
        return f, 0.0, a.tokens * 128 * (2 + 4) + a.tokens * 8 * 12
    raise SystemExit(f'unknown op {op}')


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument('--op', required=True)
    ap.add_argument('--m', type=int, default=8192)
    ap.add_argument('--n', type=int, default=4096)
    ap.add_argument('--k', type=int, default=4096)
    ap.add_argument('--layout', default='nt')
    ap.add_argument('--tokens', type=int, default=32768)
    ap.add_argument('--seq', type=int, default=8192)
    ap.add_argument('--heads', type=int, default=32)
    ap.add_argument('--kv-heads', type=int, default=8)
    ap.add_argument('--width', type=int, default=128, help='head width')
    ap.add_argument('--sinks', action='store_true', help='attn_packed, paged_decode: with sink logits and output gates')
    ap.add_argument('--window', type=int, default=0, help='attention: the last positions that a position sees (0: all)')
    ap.add_argument('--chunk', type=int, default=0, help='attention: positions of a block that sees only itself (0: none)')
    ap.add_argument('--tail', type=int, default=0, help='attention: key dimensions that all heads share')
    ap.add_argument('--terms', default='', choices=['', 'log', 'table'], help='attention: score terms (see _score_terms); with --sinks, table has gates per element')
    ap.add_argument('--states', type=int, default=16, help='selective scan: states per channel')
    ap.add_argument('--gelu', action='store_true', help='glu_columns: gelu in its tanh form')
    ap.add_argument('--limit', type=float, default=0.0, help='glu_columns: bound of the clamped unit (0: silu)')
    ap.add_argument('--hidden', type=int, default=4096)
    ap.add_argument('--vocab', type=int, default=151936)
    ap.add_argument('--batch', type=int, default=256)
    ap.add_argument('--rank', type=int, default=16)
    ap.add_argument('--numel', type=int, default=1 << 28)
    ap.add_argument('--iters', type=int, default=10)
    ap.add_argument('--warmup', type=int, default=3)
    ap.add_argument('--no-flush', action='store_true')
    ap.add_argument('--staged', type=int, default=None, help='1: staged epilogue of the SM-pair GEMM (bf16 outputs)')
    ap.add_argument('--pair', type=int, default=None, help='1: SM-pair GEMM kernel, 0: single-CTA tiles (default: library setting)')
    a = ap.parse_args()
    torch.manual_seed(0)
    if a.staged is not None:
        from twinkle_b200 import ops as _ops2
        _ops2.ext().set_gemm_staged(a.staged)
    if a.pair is not None:
        from twinkle_b200 import ops as _ops
        _ops.ext().set_gemm_pair(a.pair)
    fn, flops, byts = make(a.op, a)
    ms = time_op(fn, a.iters, a.warmup, not a.no_flush)
    pk = peaks()
    from twinkle_b200 import ops
    err = ops.ext().read_and_clear_error()
    out = dict(op=a.op, ms=round(ms, 4), error_word=err, peaks=pk['source'])
    if flops:
        out['tflops'] = round(flops / ms / 1e9, 1)
        out['frac_of_gemm_peak'] = round(flops / ms / 1e9 / pk['tflops'], 3)
    out['gbs'] = round(byts / ms / 1e6, 1)
    out['frac_of_hbm_peak'] = round(byts / ms / 1e6 / pk['hbm_gbs'], 3)
    out['args'] = {k: v for k, v in vars(a).items() if k != 'op'}
    print(json.dumps(out))


if __name__ == '__main__':
    main()
