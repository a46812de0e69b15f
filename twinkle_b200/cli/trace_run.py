"""``bin/trace_run`` / ``twinkle-trace``: feed given token ids through a model step by step and write logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is one step: ``{"step": n, "entries": [{"id", "tokens", "want"}, …], "end": [ids]}``.  The entries of a step
are one batch; they either all start (their tokens are the prompt) or all go on by one token.  ``want`` lists the places among
an entry's tokens whose logits are written to ``OUT/<step>.f32`` (32-bit floats, ``[wanted, vocab]``); requests named in ``end``
give their cache back afterwards.  After each step ``done <step>`` is printed.

The steps are the sampler engine's own (``sampler/engine.py``): prefill, captured decode, paged cache.  ``float32`` runs the
same kernels in 32-bit.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Any, Dict, List

MAX_LIVE = 1024     # sequences that may be live at a time


class TraceReplay:
    """The sampler's engine behind a step-by-step interface."""

    def __init__(self, model_dir: str, dtype: str = 'bfloat16', max_tokens: int = 0, device=None, block_size: int = 16):
        import torch
        from ..data_format import SamplingParams
        from ..sampler import TorchSampler
        from ..sampler.engine import _Seq
        live = max(1, min(max_tokens, MAX_LIVE)) if max_tokens else MAX_LIVE
        # every live sequence holds room for one token more than it has
        blocks = (max_tokens + live) // block_size + live + 2 if max_tokens else None
        self.sampler = TorchSampler(model_id=model_dir, device=device, enable_lora=False, dtype=dtype,
                                    engine_args={'num_blocks': blocks, 'block_size': block_size, 'max_batch': live})
        self.engine, self.model = self.sampler.engine, self.sampler.model
        self._new = lambda tokens: _Seq(0, tokens, SamplingParams(max_tokens=0))
        self._torch = torch
        self.live: Dict[str, Any] = {}

    def step(self, entries: List[Dict[str, Any]]):
        """Logits ``[wanted, vocab]`` (fp32, device) of one batch, or None when nothing is wanted."""
        torch = self._torch
        going = [e['id'] in self.live for e in entries]
        if not entries:
            return None
        if any(going) != all(going):
            raise ValueError('the requests of a step either all start or all go on')
        if not all(going):
            seqs = [self._new([int(t) for t in e['tokens']]) for e in entries]
            hidden = self.engine.prefill(seqs)
            self.live.update((e['id'], s) for e, s in zip(entries, seqs))
            rows, lo = [], 0
            for e in entries:
                rows += [lo + int(w) for w in e.get('want', [])]
                lo += len(e['tokens'])
            return self.model.logits(hidden[torch.tensor(rows, device=hidden.device)]).float() if rows else None
        seqs = [self.live[e['id']] for e in entries]
        for e, s in zip(entries, seqs):
            if len(e['tokens']) != 1:
                raise ValueError('requests that go on bring one token')
            s.tokens.append(int(e['tokens'][0]))
        self.engine.grow(seqs)
        logits = self.engine.decode_step(seqs, torch.tensor([s.tokens[-1] for s in seqs], device=self.engine.device))
        rows = [i for i, e in enumerate(entries) for _ in e.get('want', [])]
        return logits[torch.tensor(rows, device=logits.device)] if rows else None

    def end(self, ids: List[str]) -> None:
        self.engine.release([self.live.pop(i) for i in ids])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog='trace_run', description=__doc__.split('\n')[0])
    ap.add_argument('--model', required=True, help='folder with config.json and model.safetensors')
    ap.add_argument('--dtype', default='bfloat16', choices=['bfloat16', 'float32'])
    ap.add_argument('--out', required=True, help='folder for <step>.f32')
    ap.add_argument('--max-tokens', type=int, default=0, help='most tokens that live requests hold at any time (0: size the cache by free memory)')
    args = ap.parse_args(argv)
    import torch
    if not torch.cuda.is_available():
        print('trace_run: no CUDA device', file=sys.stderr)
        return 2
    torch.set_float32_matmul_precision('highest')
    torch.backends.cudnn.allow_tf32 = False
    from .. import ops
    from ..ops.build import prefer_serving
    from ..models.config import DecoderConfig
    cfg = DecoderConfig.from_pretrained(args.model)
    if cfg.layer_specs is not None:
        prefer_serving(cfg.kernel_parts())
    ops.ext()
    replay = TraceReplay(args.model, args.dtype, args.max_tokens)
    os.makedirs(args.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        logits = replay.step(msg.get('entries', []))
        if logits is not None:
            logits.cpu().numpy().astype('<f4').tofile(os.path.join(args.out, f"{msg['step']}.f32"))
        replay.end(msg.get('end', []))
        print(f"done {msg['step']}", flush=True)
    code = ops.ext().read_and_clear_error()
    if code:
        print(f'trace_run: a kernel gave up waiting (code {code})', file=sys.stderr)
        return 1
    return 0


if __name__ == '__main__':
    sys.exit(main())
