"""Puzonex stacks (layers listed one by one: norms on each sub-layer's result on a 32-bit stream, attention with capped scores and numbers for
distances, selective scans, attention beside a matrix memory) against ``tests/puzonex_oracle.py``.

Every case runs on the CPU in fp32 and, marked ``gpu``, on the kernels in fp32 and bf16."""
import json
import os

import pytest
import torch

from tests import puzonex_oracle as O
from tests.test_pomelix import BACKENDS, _packed, _t, go_on, ids, rel, replay, run_one, start, tol, worst_row

_MADE, _RUN = {}, {}


@pytest.fixture(scope='session')
def checkpoint(tmp_path_factory):
    """name → (directory, config, weights); made once per session."""
    def get(name, seed=0):
        if (name, seed) not in _MADE:
            cfg = O.CONFIGS[name]
            W = O.random_weights(cfg, seed)
            _MADE[name, seed] = (O.write_checkpoint(str(tmp_path_factory.mktemp(name)), cfg, W), cfg, W)
        return _MADE[name, seed]
    return get


def _rand(G, *shape):
    return torch.randn(*shape, generator=G).bfloat16().double()


def wanted(cfg, W, tokens, where):
    """The oracle's logits and residual streams, formed once per prompt, and how far operands that are off by a rounding to 16 bits move them, per
    position: some places of a random model (a query almost orthogonal to what a memory holds, a result almost zero in front of its
    norm) magnify any rounding."""
    key = id(W), tuple(tokens)
    if key not in _RUN:
        _RUN[key] = [W, O.forward(cfg, W, tokens), None]         # (W is kept so that its id stays its own)
    lg, trail = _RUN[key][1]
    if where[1] != 'bfloat16':
        return lg, trail, [torch.zeros(len(tokens))] * (1 + len(trail))
    if _RUN[key][2] is None:
        G = torch.Generator().manual_seed(1)
        worst = [torch.zeros(len(tokens))] * (1 + len(trail))
        for _ in range(3):
            V = {n: t.float() * (1 + torch.randn(t.shape, generator=G) / 512) if t.dim() > 1 else t for n, t in W.items()}
            l2, t2 = O.forward(cfg, V, tokens, torch.float32)
            worst = [torch.maximum(w, row_errors(a, b)) for w, a, b in zip(worst, [l2] + t2, [lg] + trail)]
        _RUN[key][2] = worst
    return lg, trail, _RUN[key][2]


def row_errors(got, want):
    return (got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1).mean()


def close(got, want, moved, where):
    """32-bit: every position; 16-bit: every position as far as rounding explains, and most of them well inside."""
    err = row_errors(got, want)
    if where[1] != 'bfloat16':
        assert float(err.max()) < 2 * tol(where), float(err.max())
        return
    assert bool((err < 2 * tol(where) + 6 * moved).all()), (float((err / (2 * tol(where) + 6 * moved)).max()), err.topk(min(3, len(err))))
    assert float(err.median()) < 0.01 + 2 * float(moved.median()), (float(err.median()), float(moved.median()))


def agrees(got, cfg, W, tokens, where):
    want, _, moved = wanted(cfg, W, tokens, where)
    assert got.shape == want.shape
    close(got, want, moved[0], where)


class _View:
    """The part of a cache view that the mechanisms look at."""

    def __init__(self, where, rows=None, slots=None, left=None, stepping=False, k=None, v=None, conv=None, state=None):
        dev = lambda t: None if t is None else torch.as_tensor(t).to(where[0])  # noqa: E731
        self.cache = type('C', (), {'k': [k], 'v': [v], 'conv': [conv], 'state': [state]})()
        self.rows, self.slots, self.left, self.stepping = dev(rows), dev(slots), dev(left), stepping


def _prompt_rows(lens, slots):
    """Slots and later tokens of every row of packed prompts."""
    return (torch.tensor([s for s, n in zip(slots, lens) for _ in range(n)], dtype=torch.int32),
            torch.tensor([i for n in lens for i in range(n - 1, -1, -1)], dtype=torch.int32))


# ------------------------------------------------------------------------------------------------ mechanisms
@BACKENDS
@pytest.mark.parametrize('width', [1, 7, 52, 328, 1024])
def test_embedding_with_waves_of_near_and_far_positions(where, width):
    from twinkle_b200 import ops
    pos = torch.tensor([0, 1, 2, 17, 1000, 65537, 3_000_001])
    tokens = torch.tensor([3, 0, 9, 9, 1, 5, 2])
    E = _rand(torch.Generator().manual_seed(width), 10, width)
    f = torch.tensor([10000.0 ** (-2 * i / width) for i in range((width + 1) // 2)], dtype=torch.float64)
    got = ops.embed_positions(tokens.to(where[0]), _t(where, E), pos.to(where[0]), f.to(where[0]))
    want = E[tokens] + O.waves(pos.tolist(), width)
    assert got.dtype == torch.float32 and float((got.double().cpu() - want).abs().max()) < 1e-6
    assert float((ops.position_waves(pos, f, width).double() - O.waves(pos.tolist(), width)).abs().max()) < 1e-6


HEADS = [(6, 2, 24, 40), (5, 1, 11, 9), (3, 3, 64, 64), (8, 2, 128, 72), (2, 1, 160, 136), (1, 1, 256, 256), (7, 7, 14, 5), (32, 4, 128, 128), (1, 1, 9, 9)]


@BACKENDS
@pytest.mark.parametrize('shared', [False, True])
@pytest.mark.parametrize('hq,hkv,d,e', HEADS)
def test_bias_norms_and_cache_rows(where, hq, hkv, d, e, shared):
    """The fused step between projection and attention: values of their own (normed or not) or the projected keys, norms per head, over all
    heads, or none; prompts and single steps."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d + e)
    e = d if shared else e
    dt, T, lead = getattr(torch, where[1]), 9, 8 if d % 8 == 0 else 3
    C = (hq + hkv) * d + (0 if shared else hkv * e)
    proj, bias = _rand(G, T, lead + C + 8), _rand(G, C)
    weights = {kind: [(1 + 0.3 * _rand(G, n)).bfloat16().double() for n in sizes] for kind, sizes in (('head', (d, d)), ('whole', (hq * d, hkv * d)))}
    up = lambda n: -(-n // 8) * 8  # noqa: E731

    def want(with_bias, kind, value_norm):
        y = proj[:, lead:lead + C] + (bias if with_bias else 0)
        q, k = y[:, :hq * d], y[:, hq * d:(hq + hkv) * d]
        v = k if shared else y[:, (hq + hkv) * d:]
        if kind == 'whole':
            q, k = (O.norm(t, w, 1e-3) for t, w in zip((q, k), weights[kind]))
        q, k, v = q.view(T, hq, d), k.reshape(T, hkv, d), v.reshape(T, hkv, e)
        if kind == 'head':
            q, k = (O.norm(t, w, 1e-3) for t, w in zip((q, k), weights[kind]))
        return q, k, O.over_rms(v, 1e-3) if value_norm else v

    def run(with_bias, kind, value_norm, view=None):
        qw, kw = (None, None) if kind is None else (_t(where, w) for w in weights[kind])
        with torch.no_grad():
            return ops.plain_heads(_t(where, proj), lead, _t(where, bias) if with_bias else None, qw, kw, value_norm, shared, hq, hkv, d, e, 1e-3, view, 0)

    lim = tol(where) / 4
    for how in ((False, None, False), (True, 'head', True), (True, 'whole', False), (False, 'whole', True), (True, None, True)):
        for got, ref, n in zip(run(*how), want(*how), (d, d, e)):
            assert got.shape[-1] == up(n) and not got[..., n:].any() and worst_row(got[..., :n].flatten(1), ref.flatten(1)) < lim
    how = (True, 'whole', False) if shared else (True, 'head', True)
    q, k, v = want(*how)
    rows = torch.tensor([9, 4, 20, 23, 5, 11, 7, 2, 30])
    for stepping in (False, True):
        pools = [torch.full((8, 4, hkv, up(n)), 5.0, device=where[0], dtype=dt) for n in (d, e)]
        got = run(*how, _View(where, rows, stepping=stepping, k=pools[0], v=pools[1]))
        assert (got[1] is None) == stepping and worst_row(got[0][..., :d].flatten(1), q.flatten(1)) < lim
        for pool, ref, n in zip(pools, (k, v), (d, e)):
            flat = pool.view(32, hkv, -1).cpu()
            left = torch.ones(32, dtype=torch.bool)
            left[rows] = False
            assert worst_row(flat[rows][..., :n].flatten(1), ref.flatten(1)) < lim and not flat[rows][..., n:].any() and bool((flat[left] == 5).all())


def test_buckets_of_distances():
    """Exact up to half the rows; distances on a boundary belong to the bucket that begins there; everything far shares the last."""
    from twinkle_b200.models.config import AttentionSpec
    from twinkle_b200.ops import ScoreTerms
    for rows, far in ((32, 128), (32, 256), (16, 512), (10, 37), (7, 20), (2, 4), (64, 333), (3, 2.5)):
        got = AttentionSpec(heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0, buckets=rows, bias_max=far).distance_buckets()
        assert got == [O.bucket(n, rows, far) for n in range(len(got))] and got[-1] == rows - 1 and len(got) - 1 >= far
        assert got[:rows // 2] == list(range(rows // 2)) and all(a <= b for a, b in zip(got, got[1:]))
    # half = 16, 256 / 16 = 16: the bucket changes at every 16 · 2^(k / 4); k = 4, 8, 12 are whole distances
    table = AttentionSpec(heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0, buckets=32, bias_max=256).distance_buckets()
    assert [table[n] for n in (15, 16, 31, 32, 63, 64, 127, 128, 255, 256)] == [15, 16, 19, 20, 23, 24, 27, 28, 31, 31]
    terms = ScoreTerms(table=torch.arange(32.0)[:, None], bucket=torch.tensor(table, dtype=torch.int32))
    assert terms.apply(torch.zeros(1, 1, 3), torch.tensor([[64, 300, 99999]])).flatten().tolist() == [24, 31, 31]
    for bad in (dict(buckets=1, bias_max=4), dict(buckets=8, bias_max=4), dict(buckets=8, bias_max=40, log_bias=True), dict(values_are_keys=True, vdim=7)):
        with pytest.raises(ValueError):
            AttentionSpec(**{**dict(heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0), **bad})


def _standing_out(q, k, window, lens):
    """Every third query looks for the first key it sees, every third for the one before that, the rest for whatever: a bound that is off by
    one shows."""
    at = 0
    for n in lens:
        for i in range(n):
            first = max(0, i - window + 1)
            j = (first, first - 1, None)[i % 3]
            if j is not None and j >= 0:
                for h in range(q.shape[1]):
                    q[at + i, h] = k[at + j, h // (q.shape[1] // k.shape[1])]
        at += n
    return q


def _numbers(G, hq, kind, rows=12, far=90):
    """(softcap, temp, slope, rate, table, bucket) of score terms and what they add to scores ``[H, T, T]``."""
    temp = (1 + 0.5 * _rand(G, hq).abs()).bfloat16().double()
    if kind == 'log':
        slope, rate = _rand(G, hq).abs(), (0.3 * _rand(G, hq).abs()).bfloat16().double()
        return (None, slope, rate, None, None), None, lambda T: O.log_bias(slope, rate, T)
    table = _rand(G, rows, hq)
    bucket = torch.tensor([O.bucket(n, rows, far) for n in range(far + 1)], dtype=torch.int32)
    return (temp, None, None, table, bucket), temp, lambda T: O.table_bias(table, far, T)


def _score_terms(where, cap, numbers):
    from twinkle_b200.ops import ScoreTerms
    move = lambda t: None if t is None else t.to(where[0]) if t.dtype == torch.int32 else _t(where, t)  # noqa: E731
    return ScoreTerms(cap, *(move(t) for t in numbers))


@BACKENDS
@pytest.mark.parametrize('kind', ['log', 'table'])
@pytest.mark.parametrize('window,cap', [(1, 3.0), (37, 1.0), (127, 50.0), (128, 6.0), (129, 20.0), (5000, 4.0), (64, 0.0)])
@pytest.mark.parametrize('hq,hkv,d,e', [(4, 2, 64, 40), (3, 1, 24, 24), (2, 2, 128, 128), (2, 1, 192, 72), (5, 5, 11, 7), (2, 1, 200, 200)])
def test_packed_attention_with_capped_scores_and_distances(where, kind, window, cap, hq, hkv, d, e):
    """Caps far above the scores and far below them, both kinds of distance numbers, sinks, gates per element."""
    from twinkle_b200 import ops
    if where[0] == 'cpu' and (d > 64 or window == 5000):
        pytest.skip('same formulas at every width')
    G = torch.Generator().manual_seed(d + window)
    lens = [1, 140, 33, 270]
    _, cu = _packed(lens)
    T = sum(lens)
    k, v, gate = _rand(G, T, hkv, d), _rand(G, T, hkv, e), _rand(G, T, 8 + hq * e + 3)
    q = _standing_out(_rand(G, T, hq, d), k, window, lens)
    sink, scale = (1 + _rand(G, hq)).bfloat16().double(), 6.0 / d
    numbers, temp, added = _numbers(G, hq, kind)
    terms = _score_terms(where, cap, numbers)
    with torch.no_grad():
        args = _t(where, q), _t(where, k), _t(where, v), cu.to(where[0]), max(lens), scale
        got = ops.attention_packed(*args, _t(where, sink), _t(where, gate)[:, 8:8 + hq * e], window=window, terms=terms)
        plain = ops.attention_packed(*args, window=window, terms=terms)
        headwise = ops.attention_packed(*args, None, _t(where, gate)[:, 1:1 + hq], window=window, terms=terms)
    for a, b in zip(cu[:-1], cu[1:]):
        n = int(b - a)
        run = lambda s: O.attend(q[a:b], k[a:b], v[a:b], scale, cap or 1e9, added(n), window, temp, s)  # noqa: E731
        want = run(sink) * O.sigmoid(gate[a:b, 8:8 + hq * e]).view(n, hq, e)
        assert worst_row(got[a:b].flatten(1), want.flatten(1)) < tol(where)
        assert worst_row(plain[a:b].flatten(1), run(None).flatten(1)) < tol(where)
        assert worst_row(headwise[a:b].flatten(1), (run(None) * O.sigmoid(gate[a:b, 1:1 + hq])[..., None]).flatten(1)) < tol(where)


@BACKENDS
@pytest.mark.parametrize('kind', ['log', 'table'])
@pytest.mark.parametrize('window,cap', [(1, 3.0), (16, 1.0), (33, 50.0), (9999, 5.0), (50, 0.0)])
@pytest.mark.parametrize('hq,hkv,d,e,bs', [(6, 2, 24, 40, 16), (4, 4, 128, 72, 16), (10, 1, 64, 64, 8), (2, 1, 160, 136, 4), (3, 1, 256, 8, 16), (8, 2, 128, 128, 16)])
def test_decode_attention_with_capped_scores_and_distances(where, kind, window, cap, hq, hkv, d, e, bs):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d + window)
    lens = [1, 16, 33, 0, 130, 201]
    nb = max(lens) // bs + 1
    blocks = torch.randperm(nb * len(lens), generator=G).view(len(lens), nb).to(torch.int32)
    kc, vc = _rand(G, nb * len(lens), bs, hkv, d), _rand(G, nb * len(lens), bs, hkv, e)
    q, gate, sink = _rand(G, len(lens), hq, d), _rand(G, len(lens), hq * e + 5), (1 + _rand(G, hq)).bfloat16().double()
    scale = 6.0 / d
    seq = lambda c, b, n: c[blocks[b].long()].flatten(0, 1)[:n]  # noqa: E731
    for b, n in enumerate(lens):
        j = max(0, n - window) - (b % 2)
        if n and j >= 0:                                     # looks for the first key it sees, or the one before
            q[b] = seq(kc, b, n)[j].repeat_interleave(hq // hkv, 0)
    numbers, temp, added = _numbers(G, hq, kind)
    terms = _score_terms(where, cap, numbers)
    with torch.no_grad():
        got = ops.paged_attention_decode(_t(where, q), _t(where, kc), _t(where, vc), blocks.to(where[0]), torch.tensor(lens, device=where[0]), scale, window=window,
                                         sinks=_t(where, sink), gate=_t(where, gate)[:, 3:3 + hq * e], terms=terms)
    for b, n in enumerate(lens):
        if not n:
            continue
        # the oracle runs the whole sequence; all queries but the last are of no interest
        full = torch.cat([torch.zeros(n - 1, hq, d, dtype=torch.float64), q[b:b + 1]])
        want = O.attend(full, seq(kc, b, n), seq(vc, b, n), scale, cap or 1e9, added(n), window, temp, sink)[-1] * O.sigmoid(gate[b, 3:3 + hq * e]).view(hq, e)
        assert worst_row(got[b].flatten()[None], want.flatten()[None]) < tol(where)


@BACKENDS
@pytest.mark.parametrize('cap', [0.5, 30.0])
def test_caps_are_exact_at_every_size_of_score(where, cap):
    """A query of one dimension against keys of sizes from tiny to far beyond the cap: differences of scores show in the weights."""
    from twinkle_b200 import ops
    if where[1] == 'bfloat16':
        pytest.skip('scores of one exact product: the 32-bit kernels, whose arithmetic the 16-bit ones share')
    n, d = 40, 8
    k = torch.zeros(n, 1, d, dtype=torch.float64)
    k[:, 0, 0] = torch.logspace(-4, 2, n, dtype=torch.float64).float().double() * (1 - 2 * (torch.arange(n) % 2))
    q, v = torch.zeros(n, 1, d, dtype=torch.float64), torch.eye(n, dtype=torch.float64).view(n, 1, n)
    q[:, 0, 0] = 1
    with torch.no_grad():
        got = ops.attention_packed(_t(where, q), _t(where, k), _t(where, v), torch.tensor([0, n], dtype=torch.int32, device=where[0]), n, 1.0, terms=ops.ScoreTerms(cap))
    want = O.attend(q, k, v, 1.0, cap, torch.zeros(1, n, n), n)
    assert float((got.double().cpu() / want - 1)[want > 1e-30].abs().max()) < 2e-5


@BACKENDS
@pytest.mark.parametrize('channels,taps', [(24, 1), (40, 2), (8, 3), (64, 4), (136, 5), (30, 4), (24, 6), (1032, 4)])
def test_convolution_in_prompts_and_steps(where, channels, taps):
    """Packed prompts shorter and longer than the filter, then single steps from the kept inputs, on slots used before."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(channels + taps)
    lens, more, slots, lead = [1, 9, 2, 33], 7, [3, 1, 4, 2], 8 if channels % 8 == 0 else 3
    xs = [_rand(G, n + more, channels) for n in lens]
    w, bias = _rand(G, channels, taps), _rand(G, channels)
    want = [O.silu(O.short_convolution(x, w, bias)) for x in xs]
    hist = torch.full((6, taps - 1, channels), 7.0, device=where[0], dtype=getattr(torch, where[1])) if taps > 1 else None
    slot, left = _prompt_rows(lens, slots)
    pos, _ = _packed(lens)
    wide = lambda x: torch.cat([torch.ones(x.shape[0], lead, dtype=x.dtype), x, torch.ones(x.shape[0], 5 if lead == 3 else 8, dtype=x.dtype)], 1)  # noqa: E731
    with torch.no_grad():
        run = lambda x, p, view: ops.conv_silu(_t(where, wide(x)), lead, channels, _t(where, w), _t(where, bias), p.to(where[0]), view, 0)  # noqa: E731
        got = run(torch.cat([x[:n] for x, n in zip(xs, lens)]), pos, _View(where, slots=slot, left=left, conv=hist))
        assert worst_row(got, torch.cat([y[:n] for y, n in zip(want, lens)])) < tol(where) / 2
        assert hist is None or bool((hist[[0, 5]] == 7).all())
        plain = run(torch.cat([x[:n] for x, n in zip(xs, lens)]), pos, None)
        assert torch.equal(plain, got)
        for j in range(more):
            view = _View(where, slots=torch.tensor(slots, dtype=torch.int32), left=torch.zeros(4, dtype=torch.int32), stepping=True, conv=hist)
            got = run(torch.stack([x[n + j] for x, n in zip(xs, lens)]), torch.tensor([n + j for n in lens]), view)
            assert worst_row(got, torch.stack([y[n + j] for y, n in zip(want, lens)])) < tol(where) / 2


SCANS = [(40, 4), (33, 5), (64, 16), (96, 12), (130, 32), (24, 64), (16, 130), (8, 1), (20, 256)]


def _scan_inputs(G, T, inner, N):
    u, dt, B, C, z = _rand(G, T, inner), _rand(G, T, inner), _rand(G, T, N), _rand(G, T, N), _rand(G, T, inner)
    return u, dt, B, C, z


@BACKENDS
@pytest.mark.parametrize('inner,N', SCANS)
def test_selective_scan_in_prompts_and_steps(where, inner, N):
    """Packed prompts, then single steps from the kept states, on slots used before; steps from near zero to several, decays from slow to
    immediate."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(inner + N)
    lens, more, slots = [1, 40, 2, 75], 5, [3, 1, 4, 2]
    A_log, D, dtb = (1.2 * _rand(G, inner, N) - 1).bfloat16().double(), _rand(G, inner), (2 * _rand(G, inner) - 2).bfloat16().double()
    seqs = [_scan_inputs(G, n + more, inner, N) for n in lens]
    want = []
    for u, dt, B, C, z in seqs:
        y, S = O.selective_scan(u, O.softplus(dt + dtb), -torch.exp(A_log), B, C, D)
        want.append((y * O.silu(z), S))
    state = torch.full((6, inner, N), 3.0, device=where[0])

    def run(parts, view, cu=None, longest=0):
        u, dt, B, C, z = (torch.cat(x) for x in zip(*parts))
        T = u.shape[0]
        proj, gate = torch.cat([torch.ones(T, 3, dtype=torch.float64), B, C], 1), torch.cat([torch.ones(T, 8, dtype=torch.float64), z], 1)
        with torch.no_grad():
            return ops.selective_scan(_t(where, u), _t(where, dt), _t(where, dtb), _t(where, A_log), _t(where, proj), 3, 3 + N, _t(where, D), _t(where, gate), 8, cu, longest, view, 0)

    slot, left = _prompt_rows(lens, slots)
    _, cu = _packed(lens)
    got = run([[t[:n] for t in s] for s, n in zip(seqs, lens)], _View(where, slots=slot, left=left, state=state), cu.to(where[0]), max(lens))
    assert worst_row(got, torch.cat([y[:n] for (y, _), n in zip(want, lens)])) < tol(where)
    assert bool((state[[0, 5]] == 3).all())
    for j in range(more):
        view = _View(where, slots=torch.tensor(slots, dtype=torch.int32), stepping=True, state=state)
        got = run([[t[n + j:n + j + 1] for t in s] for s, n in zip(seqs, lens)], view)
        assert worst_row(got, torch.stack([y[n + j] for (y, _), n in zip(want, lens)])) < tol(where)
    for s, (_, S) in zip(slots, want):
        assert rel(state[s], S) < 3e-5              # inputs are exact, the state is 32-bit whatever the model computes in
    assert bool((state[[0, 5]] == 3).all())


@BACKENDS
@pytest.mark.parametrize('inner,N,lens', [(40, 16, [700]), (72, 5, [300, 1, 1100, 64])])
def test_selective_scan_of_long_prompts(where, inner, N, lens):
    """Long sequences are cut into time segments on a GPU: slow decays carry over all of them."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(N)
    A_log, D, dtb = (0.5 * _rand(G, inner, N) - 5).bfloat16().double(), _rand(G, inner), (_rand(G, inner) - 2).bfloat16().double()
    seqs = [_scan_inputs(G, n, inner, N) for n in lens]
    state, (slot, _), (_, cu) = torch.zeros(6, inner, N, device=where[0]), _prompt_rows(lens, [4, 2, 1, 3]), _packed(lens)
    u, dt, B, C, z = (torch.cat(x) for x in zip(*seqs))
    with torch.no_grad():
        got = ops.selective_scan(_t(where, u), _t(where, dt), _t(where, dtb), _t(where, A_log), _t(where, torch.cat([B, C], 1)), 0, N, _t(where, D), _t(where, z), 0, cu.to(where[0]),
                                 max(lens), _View(where, slots=slot, state=state), 0)
    for (a, b), s, n in zip(zip(cu[:-1], cu[1:]), seqs, range(4)):
        y, S = O.selective_scan(s[0], O.softplus(s[1] + dtb), -torch.exp(A_log), s[2], s[3], D)
        assert worst_row(got[a:b], y * O.silu(s[4])) < tol(where) and rel(state[[4, 2, 1, 3][n]], S) < 3e-5


MEMORIES = [(1, 8, 8), (3, 16, 40), (2, 24, 136), (4, 64, 64), (2, 128, 128), (1, 128, 300), (1, 256, 72), (2, 7, 9), (5, 10, 3), (1, 1, 1), (2, 33, 20), (3, 40, 16), (1, 96, 24)]


def _memory_inputs(G, T, H, d, e, spread):
    """Columns [q | k | v | gate | i | f]."""
    return torch.cat([_rand(G, T, 2 * H * d + 2 * H * e), (spread * _rand(G, T, 2 * H)).bfloat16().double()], 1)


def _memory(x, H, d, e, ib, fb, cap, w, eps):
    T = x.shape[0]
    q, k, v, g, i, f = x.split([H * d, H * d, H * e, H * e, H, H], 1)
    o, (S, n, m) = O.matrix_memory(q.reshape(T, H, d) * d**-0.5, k.reshape(T, H, d), v.reshape(T, H, e), O.capped(i + ib, cap), O.log_sigmoid(O.capped(f + fb, cap)))
    return O.over_rms(o, eps).reshape(T, H * e) * w * O.sigmoid(g), S, n, m


def _memory_state(row, d, e):
    """A pool row ``[H, ·]`` → (S, n, m)."""
    n0 = -(-d * e // 4) * 4
    m0 = n0 + -(-d // 4) * 4
    return row[:, :d * e].view(-1, d, e), row[:, n0:n0 + d], row[:, m0]


def _same_state(row, d, e, S, n, m, lim):
    """States agree up to the choice of the maximum they are kept relative to, and in that."""
    a, b, c = (t.double().cpu() for t in _memory_state(row, d, e))
    assert rel(a, S) < lim and rel(b, n) < lim and float((c - m).abs().max()) < 1e-3


@BACKENDS
@pytest.mark.parametrize('spread', [1.0, 8.0])
@pytest.mark.parametrize('H,d,e', MEMORIES)
def test_matrix_memory_in_prompts_and_steps(where, H, d, e, spread):
    """Packed prompts around the kernel's steps of 64 tokens, then single steps from the kept states, on slots used before; gates that all but
    close and inputs that outweigh everything before them (``spread``)."""
    from twinkle_b200 import ops
    if spread > 1 and d > 128:
        pytest.skip('one size more is enough')
    G = torch.Generator().manual_seed(d + e)
    lens, more, slots, cap, eps, lead = [1, 64, 2, 150], 4, [3, 1, 4, 2], 6.0, 1e-4, 8 if d % 8 == 0 else 3
    ib, fb, w = _rand(G, H), (2 + _rand(G, H)).bfloat16().double(), _rand(G, H * e)
    seqs = [_memory_inputs(G, n + more, H, d, e, spread) for n in lens]
    want = [_memory(x, H, d, e, ib, fb, cap, w, eps) for x in seqs]
    first = [_memory(x[:n], H, d, e, ib, fb, cap, w, eps)[1:] for x, n in zip(seqs, lens)]
    N = -(-d * e // 4) * 4 + -(-d // 4) * 4 + 4
    state = torch.full((6, H, N), 3.0, device=where[0])

    def run(parts, view, cu=None, longest=0):
        x = torch.cat(parts)
        fill = -(lead + x.shape[1]) % 8
        x = torch.cat([torch.ones(x.shape[0], lead, dtype=x.dtype), x, torch.ones(x.shape[0], fill, dtype=x.dtype)], 1)
        with torch.no_grad():
            return ops.matrix_memory(_t(where, x), lead, H, d, e, _t(where, ib), _t(where, fb), cap, _t(where, w), eps, cu, longest, view, 0)

    slot, _ = _prompt_rows(lens, slots)
    _, cu = _packed(lens)
    lim = tol(where) / 2 if where[1] == 'bfloat16' else 1e-4
    got = run([x[:n] for x, n in zip(seqs, lens)], _View(where, slots=slot, state=state), cu.to(where[0]), max(lens))
    assert worst_row(got, torch.cat([y[:n] for (y, *_), n in zip(want, lens)])) < lim
    for s, kept in zip(slots, first):
        _same_state(state[s], d, e, *kept, 2e-4)
    for j in range(more):
        view = _View(where, slots=torch.tensor(slots, dtype=torch.int32), stepping=True, state=state)
        got = run([x[n + j:n + j + 1] for x, n in zip(seqs, lens)], view)
        assert worst_row(got, torch.stack([y[n + j] for (y, *_), n in zip(want, lens)])) < lim
    for s, (_, S, n, m) in zip(slots, want):
        _same_state(state[s], d, e, S, n, m, 2e-4)
    assert bool((state[[0, 5]] == 3).all())


@BACKENDS
@pytest.mark.parametrize('H,d,e,lens', [(2, 24, 40, [1300]), (1, 128, 136, [700, 1, 1027]), (3, 16, 8, [300, 65, 640, 512])])
def test_matrix_memory_of_long_prompts(where, H, d, e, lens):
    """Long sequences are cut into time segments on a GPU: open forget gates carry over all of them."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d)
    ib, fb, w = _rand(G, H), torch.full((H, ), 7.0, dtype=torch.float64), _rand(G, H * e)
    seqs = [_memory_inputs(G, n, H, d, e, 1.0) for n in lens]
    N, slots = -(-d * e // 4) * 4 + -(-d // 4) * 4 + 4, [4, 2, 1, 3]
    state, (slot, _), (_, cu) = torch.zeros(6, H, N, device=where[0]), _prompt_rows(lens, slots), _packed(lens)
    x = torch.cat(seqs)
    x = torch.cat([x, torch.ones(x.shape[0], -x.shape[1] % 8, dtype=x.dtype)], 1)
    with torch.no_grad():
        got = ops.matrix_memory(_t(where, x), 0, H, d, e, _t(where, ib), _t(where, fb), 15.0, _t(where, w), 1e-5, cu.to(where[0]), max(lens), _View(where, slots=slot, state=state), 0)
    for (a, b), s, sl in zip(zip(cu[:-1], cu[1:]), seqs, slots):
        y, S, n, m = _memory(s, H, d, e, ib, fb, 15.0, w, 1e-5)
        assert worst_row(got[a:b], y) < (tol(where) / 2 if where[1] == 'bfloat16' else 2e-4)
        _same_state(state[sl], d, e, S, n, m, 2e-4)


@BACKENDS
@pytest.mark.parametrize('width', [52, 64, 70, 2304, 4608, 8200])
@pytest.mark.parametrize('pair', [False, True])
def test_normed_results_join_the_stream(where, width, pair):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(width)
    T, eps = 5, 1e-3
    x, y, b, post, nxt, inner, beside, beside_inner = (_rand(G, *s) for s in ((T, width), (T, width), (width, ), (width, ), (width, ), (width, ), (T, width), (width, )))
    z = 0.5 * (O.norm(y + b, inner, eps) + O.norm(beside, beside_inner, eps)) if pair else O.norm(y + b, post, eps)
    want = x + (O.norm(z, post, eps) if pair else z)
    t = lambda v: _t(where, v)  # noqa: E731
    for weight in (None, nxt):
        with torch.no_grad():
            h, s = ops.stream_normed(x.float().to(where[0]), None if weight is None else t(weight), eps, t(y), t(b), t(post), *((t(inner), t(beside), t(beside_inner)) if pair else ()))
        assert s.dtype == torch.float32 and h.dtype == getattr(torch, where[1]) and rel(s, want) < 1e-6
        assert rel(h, want if weight is None else O.norm(want, nxt, eps)) < tol(where) / 4
    with torch.no_grad():
        _, s = ops.stream_normed(x.float().to(where[0]), None, eps, t(y), None, t(post))
    assert rel(s, x + O.norm(y, post, eps)) < 1e-6


@BACKENDS
@pytest.mark.parametrize('ff,lead', [(64, 0), (18, 5), (40, 8), (7, 0)])
def test_gelu_gated_unit(where, ff, lead):
    from twinkle_b200 import ops
    p = 2 * _rand(torch.Generator().manual_seed(ff), 33, lead + 2 * ff)
    p[0, lead:lead + ff], p[1, lead:lead + ff] = 30.0, -30.0
    with torch.no_grad():
        got = ops.glu_columns(_t(where, p), lead, lead + ff, ff, 0.0, 'gelu_tanh')
    assert rel(got, O.gelu_tanh(p[:, lead:lead + ff]) * p[:, lead + ff:]) < tol(where) / 4


# ------------------------------------------------------------------------------------------------ whole models
@BACKENDS
@pytest.mark.parametrize('name', list(O.CONFIGS))
def test_prompt_and_token_by_token(checkpoint, where, name):
    """A prompt at once, a prompt cut after 1 / 2 / 40 tokens and continued by single steps: all as the oracle has it."""
    path, cfg, W = checkpoint(name)
    tokens = ids(70, cfg['vocab'], 1)
    rp = replay(path, where)
    for n_prompt in (70, 1, 2, 40):
        agrees(run_one(rp, 'r', tokens, n_prompt), cfg, W, tokens, where)


@BACKENDS
@pytest.mark.parametrize('name', ['mixed', 'wide'])
def test_long_prompt(checkpoint, where, name):
    """Over several tiles, pages, windows and steps of the recurrences; the last tokens one by one."""
    path, cfg, W = checkpoint(name)
    tokens = ids(420, cfg['vocab'], 3)
    agrees(run_one(replay(path, where), 'r', tokens, 410), cfg, W, tokens, where)


@BACKENDS
def test_residual_stream_after_every_layer(checkpoint, where):
    from twinkle_b200.models.decoder import PackedBatch, Stream
    path, cfg, W = checkpoint('mixed')
    tokens = ids(29, cfg['vocab'], 2)
    _, trail, moved = wanted(cfg, W, tokens, where)
    rp = replay(path, where)
    T = len(tokens)
    batch = PackedBatch(torch.tensor(tokens, device=where[0]), torch.arange(T, device=where[0]), torch.tensor([0, T], dtype=torch.int32, device=where[0]), T)
    with torch.no_grad():
        st = Stream(rp.model.embed_positions(batch))
        assert rel(st.x, W['embed'].double()[tokens] + O.waves(range(T), cfg['width'])) < 1e-6
        for layer, want, spread in zip(rp.model.layers, trail, moved[1:]):
            st = layer.advance(st, batch)
            seen = Stream(st.x.clone(), normed=st.normed)
            seen.enter(rp.model.norm)
            assert seen.x.dtype == torch.float32
            close(seen.x, want, spread, where)


@BACKENDS
@pytest.mark.parametrize('name', ['mixed', 'odd'])
def test_batches_of_unequal_requests(checkpoint, where, name):
    """Requests of 1 to 66 tokens in one batch, decoded together, shorter ones ending earlier: each as it is alone."""
    path, cfg, W = checkpoint(name)
    lens = {'a': (66, 9), 'b': (1, 25), 'c': (16, 3), 'd': (3, 12), 'e': (41, 25)}
    toks = {n: ids(a + b, cfg['vocab'], 10 + i) for i, (n, (a, b)) in enumerate(lens.items())}
    rp = replay(path, where)
    rows = {n: [t] for n, t in start(rp, {n: toks[n][:a] for n, (a, _) in lens.items()}).items()}
    for step in range(25):
        now = {n: toks[n][a + step] for n, (a, b) in lens.items() if step < b}
        for n, r in go_on(rp, now).items():
            rows[n].append(r[None].clone())
        rp.end([n for n, (_, b) in lens.items() if step == b - 1])
    assert not rp.live
    for n in lens:
        agrees(torch.cat(rows[n]), cfg, W, toks[n], where)
        alone = run_one(rp, n, toks[n], lens[n][0])
        assert rel(torch.cat(rows[n]), alone) < (5e-2 if where[1] == 'bfloat16' else 2e-5)


@BACKENDS
def test_freed_pages_and_slots_are_used_again(checkpoint, where):
    """A cache of few blocks serves one request after another; what an ended request left does not show."""
    path, cfg, W = checkpoint('mixed')
    rp = replay(path, where, max_tokens=64, block_size=4)
    cache = rp.engine.cache
    blocks, slots = len(cache.free), len(cache.free_slots)
    for t in [t for t in cache.state + cache.conv if t is not None]:
        t[1:] = 50.0                                     # whatever lies in a slot before its first use
    for i, (n, n_prompt) in enumerate([(60, 50), (9, 1), (40, 2), (5, 1), (64, 64)]):
        tokens = ids(n, cfg['vocab'], 40 + i)
        agrees(run_one(rp, f'r{i}', tokens, n_prompt), cfg, W, tokens, where)
        assert len(cache.free) == blocks and len(cache.free_slots) == slots
    with pytest.raises(RuntimeError, match='exhausted'):
        for i in range(blocks + 1):
            start(rp, {f'x{i}': [1]})


@BACKENDS
def test_cache_holds_what_a_layer_keeps(checkpoint, where):
    for name in O.CONFIGS:
        path, cfg, W = checkpoint(name)
        c = replay(path, where, max_tokens=64).engine.cache
        up = lambda n, k=8: -(-n // k) * k  # noqa: E731
        for layer, k, v, h, s in zip(cfg['layers'], c.k, c.v, c.conv, c.state):
            m = layer['mixer']
            if layer['type'] == 'mamba1':
                assert k is None and v is None and tuple(s.shape[1:]) == (m['inner'], m['state'])
                assert h is None if m['conv'] == 1 else tuple(h.shape[1:]) == (m['conv'] - 1, m['inner'])
                continue
            a = m if layer['type'] == 'attention' else m['left']
            assert h is None and tuple(k.shape[2:]) == (a['kv_heads'], up(a['dim'])) and tuple(v.shape[2:]) == (a['kv_heads'], up(a['vdim']))
            if layer['type'] == 'parallel':
                r = m['right']
                assert tuple(s.shape[1:]) == (r['heads'], up(r['dim'] * r['vdim'], 4) + up(r['dim'], 4) + 4)
            else:
                assert s is None
        assert all(s is None or s.dtype == torch.float32 for s in c.state)


@BACKENDS
def test_long_decoding_over_page_borders(checkpoint, where):
    path, cfg, W = checkpoint('mixed')
    tokens = ids(203, cfg['vocab'], 7)
    agrees(run_one(replay(path, where, block_size=8), 'r', tokens, 2), cfg, W, tokens, where)


@BACKENDS
def test_first_tokens(checkpoint, where):
    path, cfg, W = checkpoint('mixed')
    rp = replay(path, where)
    for n in (1, 2, 3, 4):
        tokens = ids(n, cfg['vocab'], 90 + n)
        agrees(run_one(rp, 'r', tokens, n), cfg, W, tokens, where)
        agrees(run_one(rp, 'r', tokens, 1), cfg, W, tokens, where)


def _asking_model(kind, size):
    """One layer in which token 299 looks for token 298 and for nothing else: channel 0 of the stream marks the one, channel 1 the other (the first
    wave is the fastest, so both stand well above it), and the last dimension of queries and keys carries the marks."""
    width, H, d = 80, 4, 24
    if kind == 'attention':
        layers, rows, p = [O.attention(H, 2, d, 40, 1.0, size, 30.0)], [0], 'l0.mix.'
    else:
        layers, p = [O.parallel((H, 2, d, 1.0, size, 30.0, 16, 90), (2, 16, 24, 5.0))], 'l0.mix.left.'
        rows = [layers[0].pop('rows')]
    cfg = dict(architecture='Puzonex', vocab=300, width=width, norm={'eps': 1e-5}, layers=layers)
    W = O.random_weights(cfg, 3, rows)
    W['embed'][:, :2] = 0
    W['embed'][298, 0], W['embed'][299, 1] = 24, 24
    W[p + 'q'], W[p + 'q.b'] = torch.zeros_like(W[p + 'q']), torch.zeros_like(W[p + 'q.b'])
    W[p + 'q'].view(H, d, width)[:, d - 1, 1] = 2
    k = W[p + 'k'].view(2, d, width)
    k[:, d - 1], k[:, :, 0] = 0, 0
    k[:, d - 1, 0] = 2
    W[p + 'k.b'] = torch.zeros_like(W[p + 'k.b'])
    for n in ('q.norm', 'k.norm'):
        W[p + n] = torch.ones_like(W[p + n])
    if kind == 'parallel':
        W[p + 'rel'] = W[p + 'rel'] / 4
        W['l0.mix.right.out'] = W['l0.mix.right.out'] / 8        # (the memory would remember the token in any case)
    return cfg, W


@BACKENDS
@pytest.mark.parametrize('kind,size', [('attention', 100), ('attention', 128), ('attention', 33), ('parallel', 100), ('parallel', 129)])
def test_keys_just_inside_and_just_outside(tmp_path, where, kind, size):
    """What the last token looks for stands at the first place it sees, the one before, around page borders, in the middle.  Asked for in the
    prompt and in decoding; another token there changes the logits (much) if and only if it is seen."""
    cfg, W = _asking_model(kind, size)
    path = O.write_checkpoint(tmp_path / 'm', cfg, W)
    rp = replay(path, where)
    for last in (size - 1, size, 230, 256):
        n, edge = last + 1, max(0, last - size + 1)
        for at in sorted({edge, edge - 1, edge + 1, edge - 2, (last // 16) * 16, (last // 16) * 16 - 1, (edge + last) // 2, 0}):
            if not 0 <= at < last:
                continue
            base = ids(n, 297, at)
            base[-1] = 299
            seen, unseen = list(base), list(base)
            seen[at], unseen[at] = 298, 297
            want, other = O.forward(cfg, W, seen)[0][-1], O.forward(cfg, W, unseen)[0][-1]
            if at >= edge:
                assert rel(other, want) > 0.1                      # a key that is seen matters …
            else:
                assert rel(other, want) < (1e-12 if kind == 'attention' else 0.05)     # … another does not (on the attention's side)
            for n_prompt in (n, n - 1, n - 3):
                assert n_prompt < 1 or rel(run_one(rp, 'r', seen, n_prompt)[-1], want) < 2 * tol(where), (last, at, n_prompt)     # … here as well


@BACKENDS
def test_greedy_generation_through_the_sampler(checkpoint, where):
    """``TorchSampler.sample`` (its scheduler, batching and cache) gives the oracle's greedy continuation."""
    from twinkle_b200.data_format import SamplingParams
    from twinkle_b200.sampler import TorchSampler
    path, cfg, W = checkpoint('mixed')
    s = TorchSampler(model_id=path, device=where[0], dtype=where[1], enable_lora=False, engine_args={'num_blocks': 256, 'max_batch': 2})
    prompts = [ids(n, cfg['vocab'], 70 + n) for n in (19, 1, 45)]             # three prompts, groups of two
    out = s.sample([{'input_ids': p} for p in prompts], SamplingParams(max_tokens=10, temperature=0.0))
    for p, r in zip(prompts, out):
        got = r.sequences[0].tokens
        assert len(got) == 10
        lg, _, moved = wanted(cfg, W, p + got, where)
        for i, t in enumerate(got):
            at = len(p) + i - 1
            slack = 0.1 + 12 * float(moved[0][at]) if where[1] == 'bfloat16' else 1e-4
            assert float(lg[at].max() - lg[at, t]) <= slack * float(lg[at].std())      # the best, up to a tie within rounding
    if where[0] == 'cuda':
        assert s.engine.use_cuda_graphs and s.engine._graphs                  # decoding was captured, not run eagerly
    s.sleep()
    s.wake_up()
    again = s.sample([{'input_ids': p} for p in prompts], SamplingParams(max_tokens=10, temperature=0.0))
    assert [r.sequences[0].tokens for r in again] == [r.sequences[0].tokens for r in out]


# ------------------------------------------------------------------------------------------------ registry, files, training
def test_config_and_weights_round_trip(checkpoint, tmp_path):
    from safetensors.torch import load_file
    from twinkle_b200.model import TransformersModel
    from twinkle_b200.models.config import DecoderConfig, preset
    for name in O.CONFIGS:
        path, cfg, W = checkpoint(name)
        c = DecoderConfig.from_pretrained(path)
        assert DecoderConfig.from_hf(c.to_hf()) == c and c.model_type == 'puzonex'
        m = TransformersModel(model_id=path, device='cpu')
        assert sum(p.numel() for p in m.model.parameters()) == c.num_params() == sum(t.numel() for t in W.values())
        out = m.save('ckpt', output_dir=str(tmp_path / name))
        back = load_file(os.path.join(out, 'model.safetensors'))
        assert set(back) == set(W) and all(torch.equal(back[n].float(), W[n].float()) and back[n].shape == W[n].shape for n in W)
        with open(os.path.join(out, 'config.json')) as f:
            assert DecoderConfig.from_hf(json.load(f)) == c
        assert DecoderConfig.from_pretrained(out) == c
    assert preset('tiny-puzonex', num_hidden_layers=3).num_hidden_layers == 3
    assert DecoderConfig.from_pretrained(checkpoint('mixed')[0]).kernel_parts() == ['heads', 'memory', 'selective']

    def changed(**what):
        bad = json.loads(json.dumps(O.CONFIGS['mixed']))
        for where, value in what.items():
            *keys, last = where.split('__')
            d = bad['layers']
            for k in keys:
                d = d[int(k[1:])] if k[:1] == 'l' and k[1:].isdigit() else d[k]
            d[last] = value
        for layer in bad['layers']:
            if layer['type'] == 'parallel':
                layer['mixer']['left'].setdefault('buckets', 10)
        return bad
    assert DecoderConfig.from_hf(changed()).layer_specs[0].mixer.left.buckets == 10
    for bad in (changed(l0__type='something'), changed(l0__mlp={'kind': 'something'})):
        with pytest.raises(NotImplementedError):
            DecoderConfig.from_hf(bad)
    for bad in (changed(l2__mixer__heads=5), changed(l0__mixer__left__vdim=32), changed(l0__mixer__left__bias_max=5), changed(l1__mixer__conv=0), O.CONFIGS['mixed']):
        with pytest.raises(ValueError):
            DecoderConfig.from_hf(bad)


def test_gradients_reach_every_weight(checkpoint):
    """Autograd through a stack of such layers against finite differences of the oracle's loss."""
    from twinkle_b200.models.bridge import hf_to_internal
    from twinkle_b200.models.config import DecoderConfig
    from twinkle_b200.models.decoder import PackedBatch, build_model
    path, cfg, W = checkpoint('mixed')
    c = DecoderConfig.from_pretrained(path)
    model = build_model(c, init=False)
    with torch.no_grad():
        for n, p in model.named_parameters():
            p.copy_(hf_to_internal(n, c, W.__getitem__).float())
    tokens = ids(26, cfg['vocab'], 5)
    T = len(tokens)
    hidden = model(PackedBatch(torch.tensor(tokens), torch.arange(T), torch.tensor([0, T], dtype=torch.int32), T))
    loss = torch.nn.functional.cross_entropy(model.logits(hidden)[:-1], torch.tensor(tokens[1:]))
    loss.backward()
    names = dict(model.named_parameters())

    def oracle_loss(name, delta):
        V = {n: t.double() for n, t in W.items()}
        V[name] = V[name] + delta
        return float(torch.nn.functional.cross_entropy(O.forward(cfg, V, tokens)[0][:-1], torch.tensor(tokens[1:])))

    G = torch.Generator().manual_seed(1)
    every = slice(None)
    for hf, internal, rows in (('l0.mix.left.k', 'layers.0.mixer.in_proj.weight', slice(144, 192)), ('l0.mix.left.g', 'layers.0.mixer.in_proj.weight', slice(192, 336)),
                               ('l0.mix.left.k.b', 'layers.0.mixer.left.qkv_bias', slice(144, 192)), ('l0.mix.left.k.norm', 'layers.0.mixer.left.head_k_norm.weight', every),
                               ('l0.mix.left.rel', 'layers.0.mixer.left.distance_table', every), ('l0.mix.left.temp', 'layers.0.mixer.left.temperature', every),
                               ('l0.mix.left.o.b', 'layers.0.mixer.left.o_bias', every), ('l0.mix.left.out', 'layers.0.mixer.left_norm.weight', every),
                               ('l0.mix.right.k', 'layers.0.mixer.in_proj.weight', slice(384, 432)), ('l0.mix.right.i', 'layers.0.mixer.in_proj.weight', slice(672, 675)),
                               ('l0.mix.right.f.b', 'layers.0.mixer.right.f_bias', every), ('l0.mix.right.norm', 'layers.0.mixer.right.out_norm.weight', every),
                               ('l1.mix.A_log', 'layers.1.mixer.A_log', every), ('l1.mix.conv', 'layers.1.mixer.conv_weight', every), ('l1.mix.dt.b', 'layers.1.mixer.dt_bias', every),
                               ('l1.mix.x', 'layers.1.mixer.x_proj.weight', every), ('l3.mix.D', 'layers.3.mixer.D', every), ('l3.mix.in', 'layers.3.mixer.in_proj.weight', every),
                               ('l2.mix.r1', 'layers.2.mixer.log_slope', every), ('l2.mix.r2', 'layers.2.mixer.log_rate', every), ('l2.mix.sink', 'layers.2.mixer.sinks', every),
                               ('l2.mix.v.b', 'layers.2.mixer.qkv_bias', slice(216, 336)), ('l5.mix.q.norm', 'layers.5.mixer.head_q_norm.weight', every),
                               ('l5.norm1', 'layers.5.post_mixer_layernorm.weight', every), ('l1.norm2', 'layers.1.post_mlp_layernorm.weight', every),
                               ('l0.mlp.up', 'layers.0.mlp.in_proj.weight', slice(128, 256)), ('embed', 'embed_tokens.weight', every), ('head', 'lm_head.weight', every)):
        direction = torch.randn(W[hf].shape, generator=G).double()
        fd = (oracle_loss(hf, 1e-6 * direction) - oracle_loss(hf, -1e-6 * direction)) / 2e-6
        ad = float((names[internal].grad[rows].double().reshape(-1) * direction.reshape(-1)).sum())
        assert abs(fd - ad) < 2e-3 * max(1.0, abs(fd)), (hf, fd, ad)
    assert all(p.grad is not None for p in names.values())


@BACKENDS
def test_training_follows_the_oracle(checkpoint, where):
    """Loss of the training engine (activation recompute per layer) = the oracle's, and it falls."""
    from twinkle_b200.model import TransformersModel
    path, cfg, W = checkpoint('mixed')
    m = TransformersModel(model_id=path, device=where[0], mixed_precision='bf16' if where[1] == 'bfloat16' else 'no')
    m.set_optimizer('AdamW', lr=2e-3, weight_decay=0.0)
    feats, want, count = [], 0.0, 0
    for i, n in enumerate((43, 20)):
        seq = ids(n + 1, cfg['vocab'], 60 + i)
        feats.append({'input_ids': seq[:-1], 'labels': seq[1:]})
        lp = torch.log_softmax(O.forward(cfg, W, seq[:-1])[0], -1)
        want, count = want - sum(float(lp[j, t]) for j, t in enumerate(seq[1:])), count + n
    losses = []
    for _ in range(4):
        losses.append(float(m.forward_backward(inputs=feats)['loss']))
        m.clip_grad_and_step(max_grad_norm=1.0)
    assert abs(losses[0] - want / count) < (5e-2 if where[1] == 'bfloat16' else 1e-4), (losses, want / count)
    assert losses[-1] < losses[0] - 0.1, losses


def test_adapters_apply_to_joined_projections():
    from twinkle_b200.model import LoraConfig, TransformersModel
    m = TransformersModel(model_id='tiny-puzonex', device='cpu', max_loras=1, max_r=4)
    m.add_adapter_to_model('a', LoraConfig(r=4, lora_alpha=8, target_modules=['left_q_proj', 'right_v_proj', 'v_proj', 'x_proj', 'dt_proj', 'up_proj', 'o_proj']))
    m.set_optimizer('AdamW', lr=1e-2, adapter_name='a')
    seq = ids(40, 1024, 3)
    losses = []
    for _ in range(4):
        losses.append(float(m.forward_backward(inputs=[{'input_ids': seq[:-1], 'labels': seq[1:]}], adapter_name='a')['loss']))
        m.clip_grad_and_step(max_grad_norm=1.0, adapter_name='a')
    assert losses[-1] < losses[0] - 1e-3, losses


@pytest.mark.gpu
@pytest.mark.parametrize('dtype', ['bfloat16', 'float32'])
def test_trace_command(checkpoint, tmp_path, dtype):
    """The command line end to end in a process of its own: batch, steps, a step without wishes, ends, files and answers."""
    import subprocess
    import sys

    import numpy as np
    path, cfg, W = checkpoint('odd')
    a, b = ids(21, cfg['vocab'], 1), ids(6, cfg['vocab'], 2)
    steps = [{'step': 0, 'entries': [{'id': 'a', 'tokens': a[:19], 'want': [0, 18]}, {'id': 'b', 'tokens': b[:5], 'want': [2]}], 'end': []},
             {'step': 1, 'entries': [{'id': 'a', 'tokens': a[19:20], 'want': []}, {'id': 'b', 'tokens': b[5:], 'want': []}], 'end': ['b']},
             {'step': 2, 'entries': [{'id': 'a', 'tokens': a[20:], 'want': [0]}], 'end': ['a']}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, 'bin', 'trace_run'), '--model', path, '--dtype', dtype, '--out', str(tmp_path / 'out'), '--max-tokens', '64'],
                       input='\n'.join(json.dumps(s) for s in steps) + '\n', capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith('done')] == ['done 0', 'done 1', 'done 2']
    assert sorted(os.listdir(tmp_path / 'out')) == ['0.f32', '2.f32']
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / 'out' / f'{n}.f32', dtype='<f4')).view(-1, cfg['vocab'])  # noqa: E731
    wa, wb = O.forward(cfg, W, a)[0], O.forward(cfg, W, b)[0]
    lim = 2 * tol((0, dtype)) if dtype == 'float32' else 0.5
    assert worst_row(read(0), torch.stack([wa[0], wa[18], wb[2]])) < lim and worst_row(read(2), wa[20:21]) < lim
