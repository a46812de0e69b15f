"""Serving throughput of the sampler's engine at the sizes of a real model (random weights, one GPU): prefill tokens/s and
decode tokens/s of a model preset, used by ``bench.py --config serve``.

Prefill: packed prompts through ``NativeEngine.prefill`` (host bookkeeping included).  Decode: ``NativeEngine.decode_step`` on
sequences whose context is already in the cache (captured steps).  Timed with CUDA events after warm-up; the weights read per
step exceed the L2 cache, so steps do not find them there.
"""
from __future__ import annotations

from typing import Any, Dict, List, Sequence, Tuple

import torch

from ..data_format import SamplingParams
from ..models.config import DecoderConfig
from ..models.decoder import build_model
from .engine import NativeEngine, _Seq


def _timed(fn, steps: int, warmup: int) -> float:
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


@torch.no_grad()
def measure(cfg: DecoderConfig, prompts: Sequence[Tuple[int, int]], batches: Sequence[Tuple[int, int]], steps: int = 8, warmup: int = 3) -> Dict[str, Any]:
    """``prompts``: (number, length) of packed prompts; ``batches``: (sequences, context) of decode steps."""
    model = build_model(cfg, device='cuda', dtype=torch.bfloat16)
    model.requires_grad_(False)
    tokens = max([n * ln for n, ln in prompts] + [b * (c + steps + warmup + 20) for b, c in batches])
    eng = NativeEngine(model, cfg, torch.device('cuda'), num_blocks=tokens // 16 + 1024, max_batch=max([n for n, _ in prompts] + [b for b, _ in batches]))
    g = torch.Generator().manual_seed(0)
    make = lambda n: _Seq(0, torch.randint(0, cfg.vocab_size, (n, ), generator=g).tolist(), SamplingParams(max_tokens=0))  # noqa: E731
    out: Dict[str, List[Dict[str, Any]]] = {'prefill': [], 'decode': []}
    for n, ln in prompts:
        seqs = [make(ln) for _ in range(n)]

        def once():
            eng.prefill(seqs)
            eng.release(seqs)
        ms = _timed(once, steps, warmup)
        out['prefill'].append({'prompts': n, 'tokens_each': ln, 'ms': round(ms, 3), 'tokens_per_s': round(n * ln / ms * 1e3)})
    for b, c in batches:
        seqs = [make(c) for _ in range(b)]
        for lo in range(0, b, 16):                  # prompts of a few sequences at a time: activations stay small
            eng.prefill(seqs[lo:lo + 16])
        last = torch.zeros(b, dtype=torch.long, device='cuda')

        def step():
            for s in seqs:
                s.tokens.append(0)
            eng.grow(seqs)
            eng.decode_step(seqs, last)
        ms = _timed(step, steps, warmup)
        replay = None
        if eng._graphs:                             # the captured step alone (device time without the host bookkeeping)
            replay = _timed(list(eng._graphs.values())[-1]['graph'].replay, steps, warmup)
        out['decode'].append({'sequences': b, 'context': c, 'ms': round(ms, 3), 'tokens_per_s': round(b / ms * 1e3),
                              'captured_ms': None if replay is None else round(replay, 3)})
        eng.release(seqs)
        eng._graphs.clear()
    del eng, model
    torch.cuda.empty_cache()
    return out
