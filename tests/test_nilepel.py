"""Nilepel stacks (layers listed one by one: pre-norm sub-layers on a 32-bit stream, rotated grouped and latent attention inside windows
and chunks, borrowed keys and values, clamped feed-forward blocks, group-limited experts beside a shared one) against
``tests/nilepel_oracle.py``.

Every case runs on the CPU in fp32 and, marked ``gpu``, on the kernels in fp32 and bf16."""
import json
import os

import pytest
import torch

from tests import nilepel_oracle as O
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


# a router's choice may flip under bf16 rounding: positions where that can happen are compared loosely
def close_calls(cfg, W, tokens, margin):
    """Logits, and per position whether some router (there or at an earlier token) sees the last that it takes and the first that it
    leaves, among groups or among experts, closer than ``margin``."""
    key = id(W), tuple(tokens), margin
    if key in _RUN:
        return _RUN[key][1:]
    near = torch.zeros(len(tokens), dtype=torch.bool)
    real = O.route

    def spy(z, r):
        g = r.get('groups') or {'count': 1, 'keep': 1}
        best = z.view(z.shape[0], g['count'], -1).amax(-1).sort(-1, descending=True)
        if g['keep'] < g['count']:
            near.logical_or_(best.values[:, g['keep'] - 1] - best.values[:, g['keep']] < margin)
        allowed = torch.stack([torch.cat([row.view(g['count'], -1)[n] for n in b[:g['keep']]]) for row, b in zip(z, best.indices)]).sort(-1, descending=True).values
        if allowed.shape[1] > r['top']:
            near.logical_or_(allowed[:, r['top'] - 1] - allowed[:, r['top']] < margin)
        return real(z, r)
    O.route = spy
    try:
        out = O.forward(cfg, W, tokens)[0]
    finally:
        O.route = real
    _RUN[key] = W, out, near.int().cummax(0).values.bool()         # (W is kept so that its id stays its own)
    return _RUN[key][1:]


def agrees(got, cfg, W, tokens, where):
    """Logits of every position; in bf16 those before the first close call of a router, and most of all others."""
    want, near = close_calls(cfg, W, tokens, 0.08 if where[1] == 'bfloat16' else 1e-5)
    n = int((~near).sum())
    assert got.shape == want.shape
    if where[1] != 'bfloat16':
        assert n == len(tokens) and worst_row(got, want) < 2 * tol(where)
        return
    err = (got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1).mean()
    assert n == 0 or float(err[:n].max()) < 4 * tol(where)
    assert len(tokens) < 8 or float(err.median()) < tol(where) * 1.5


# ------------------------------------------------------------------------------------------------ mechanisms
ROTATIONS = [O.rot(2, 10.0), O.rot(6, 40.0), O.rot(16, 500.0, O._LONG), O.rot(64, 1e6), O.rot(32, 1e4, (2.0, 0.5, 8.0, 100)), O.rot(128, 5e5, (32.0, 1.0, 4.0, 8192))]


def test_frequencies_on_every_side_of_the_scaling():
    from twinkle_b200.models.config import RotarySpec
    for r in ROTATIONS:
        spec = RotarySpec(**r)
        f, plain = torch.tensor(spec.frequencies()), torch.tensor(RotarySpec(r['dims'], r['base']).frequencies())
        assert torch.allclose(f, torch.tensor(O.frequencies(r)), rtol=1e-9)
        if 'scaling' in r and r['dims'] > 16:
            slow = plain / f
            assert float(slow.min()) == 1.0 and float(slow.max()) == r['scaling']['factor'] and bool(((slow > 1.0001) & (slow < r['scaling']['factor'] - 1e-3)).any())


@BACKENDS
def test_angles_of_far_positions(where):
    """Cosines and sines keep their digits for positions in the millions."""
    from twinkle_b200 import ops
    pos = torch.tensor([0, 1, 2, 1000, 65537, 3_000_001])
    f = torch.tensor([v for r in ROTATIONS for v in O.frequencies(r)], dtype=torch.float64)
    got = ops.rotary_table(pos.to(where[0]), f.to(where[0]))
    a = pos.double()[:, None] * f
    assert got.dtype == torch.float32 and float((got.double().cpu() - torch.stack([a.cos(), a.sin()], -1)).abs().max()) < 1e-6


class _View:
    """The part of a cache view that the mechanisms look at."""

    def __init__(self, k, v, rows, stepping):
        self.cache, self.rows, self.stepping = type('C', (), {'k': [k], 'v': [v]})(), rows, stepping


HEADS = [(6, 2, 24, 40, 16), (5, 1, 11, 9, 6), (3, 3, 64, 64, 64), (8, 2, 128, 72, 32), (2, 1, 160, 136, 96), (1, 1, 256, 256, 256), (7, 7, 14, 5, 2), (32, 4, 128, 128, 128),
         (4, 2, 48, 16, 24)]


@BACKENDS
@pytest.mark.parametrize('neighbours', [True, False])
@pytest.mark.parametrize('hq,hkv,d,e,dims', HEADS)
def test_bias_norm_rotation_and_cache_rows(where, hq, hkv, d, e, dims, neighbours):
    """The fused step between projection and attention: prompts, single steps, layers without keys of their own, with and without bias and
    norm."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d + e)
    dt, T, lead = getattr(torch, where[1]), 9, 8 if d % 8 == 0 else 3
    pos = torch.tensor([0, 1, 2, 3, 17, 400, 401, 5000, 12])
    other, mine = O.rot(8, 77.0), O.rot(dims, 1234.0, O._LONG)
    f = torch.tensor(O.frequencies(other) + O.frequencies(mine), dtype=torch.float64)
    table = ops.rotary_table(pos.to(where[0]), f.to(where[0]))
    C = (hq + hkv) * d + hkv * e
    proj, bias, qw, kw = _rand(G, T, lead + C + 8), _rand(G, C), (1 + _rand(G, d)).bfloat16().double(), (1 + _rand(G, d)).bfloat16().double()
    up = lambda n: -(-n // 8) * 8  # noqa: E731

    def want(with_bias, with_norm):
        y = proj[:, lead:lead + C] + (bias if with_bias else 0)
        q, k, v = y[:, :hq * d].view(T, hq, d), y[:, hq * d:(hq + hkv) * d].view(T, hkv, d), y[:, (hq + hkv) * d:].view(T, hkv, e)
        if with_norm:
            q, k = O.norm(q, qw, 1e-3), O.norm(k, kw, 1e-3)
        return O.rotate(q, mine, neighbours, pos), O.rotate(k, mine, neighbours, pos), v

    def run(with_bias, with_norm, view=None, kv=hkv, p=proj, b=bias):
        with torch.no_grad():
            return ops.rotary_heads(_t(where, p), lead, _t(where, b) if with_bias else None, _t(where, qw) if with_norm else None, _t(where, kw) if with_norm and kv else None,
                                    table, 4, dims // 2, neighbours, hq, kv, d, e, 1e-3, view, 0)

    lim = tol(where) / 4
    for with_bias, with_norm in ((False, False), (True, True), (True, False), (False, True)):
        for got, ref, n in zip(run(with_bias, with_norm), want(with_bias, with_norm), (d, d, e)):
            assert got.shape[-1] == up(n) and not got[..., n:].any() and worst_row(got[..., :n].flatten(1), ref.flatten(1)) < lim
    q, k, v = want(True, True)
    rows = torch.tensor([9, 4, 20, 23, 5, 11, 7, 2, 30])
    for stepping in (False, True):
        pools = [torch.full((8, 4, hkv, up(n)), 5.0, device=where[0], dtype=dt) for n in (d, e)]
        got = run(True, True, _View(*pools, rows.to(where[0]), stepping))
        assert (got[1] is None) == stepping and worst_row(got[0][..., :d].flatten(1), q.flatten(1)) < lim
        for pool, ref, n in zip(pools, (k, v), (d, e)):
            flat = pool.view(32, hkv, -1).cpu()
            left = torch.ones(32, dtype=torch.bool)
            left[rows] = False
            assert worst_row(flat[rows][..., :n].flatten(1), ref.flatten(1)) < lim and not flat[rows][..., n:].any() and bool((flat[left] == 5).all())
    got = run(True, True, None, 0, proj[:, :lead + hq * d].contiguous(), bias[:hq * d].contiguous())
    assert got[1] is None and got[2] is None and worst_row(got[0][..., :d].flatten(1), q.flatten(1)) < lim


@BACKENDS
@pytest.mark.parametrize('H,d,r,R', [(5, 24, 16, 48), (3, 7, 6, 13), (4, 128, 64, 264), (20, 64, 32, 512), (1, 9, 4, 5), (2, 16, 2, 8), (3, 8, 12, 24)])
def test_latent_rows_and_rotated_queries(where, H, d, r, R):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(R + r)
    dt, T, q0 = getattr(torch, where[1]), 7, 8 if d % 8 == 0 and r % 8 == 0 else 5
    pos = torch.tensor([3, 0, 1, 70, 999, 4, 123456])
    turn, wide = O.rot(r, 300.0), -(-(R + r) // 8) * 8
    table = ops.rotary_table(pos.to(where[0]), torch.tensor(O.frequencies(O.rot(6, 5.0)) + O.frequencies(turn), dtype=torch.float64, device=where[0]))
    c0 = q0 + H * (d + r)
    proj, w = _rand(G, T, c0 + R + r + (-(c0 + R + r) % 8)), (1 + _rand(G, R)).bfloat16().double()
    q = proj[:, q0:c0].view(T, H, d + r)
    q = torch.cat([q[..., :d], O.rotate(q[..., d:], turn, True, pos)], -1)
    kept = torch.cat([O.norm(proj[:, c0:c0 + R], w, 1e-3), O.rotate(proj[:, None, c0 + R:c0 + R + r], turn, True, pos)[:, 0]], -1)
    lim, rows = tol(where) / 4, torch.tensor([9, 4, 20, 23, 5, 11, 7])
    for stepping in (False, True):
        for own in (True, False):
            pool = torch.full((6, 4, 1, wide), 5.0, device=where[0], dtype=dt)
            with torch.no_grad():
                p = _t(where, proj).clone()
                gq, gk, ql = ops.latent_rotary(p, q0, H, d, r, c0, R if own else 0, _t(where, w) if own else None, 1e-3, table, 3, r // 2, True, R,
                                               _View(pool, None, rows.to(where[0]), stepping), 0)
            if stepping:
                assert ql.shape == (T, H, R + r) and worst_row(ql[..., R:].flatten(1), q[..., d:].flatten(1)) < lim and worst_row(gq[..., :d].flatten(1), q[..., :d].flatten(1)) < lim
            else:
                assert ql is None and worst_row(gq.flatten(1), q.flatten(1)) < lim
                assert (gk is None) == (not own)
            if own:
                flat = pool.view(24, -1).cpu()
                left = torch.ones(24, dtype=torch.bool)
                left[rows] = False
                assert worst_row(flat[rows][:, :R + r], kept) < lim and not flat[rows][:, R + r:].any() and bool((flat[left] == 5).all())
                if not stepping:
                    assert torch.equal(gk.cpu(), flat[rows])                     # the cache holds what prompts attend over
            else:
                assert bool((pool == 5).all())


def _standing_out(G, q, k, first, lens):
    """Every third query looks for the first key it sees, every third for the one before that, the rest for whatever: a bound that is off by
    one shows."""
    at = 0
    for n in lens:
        for i in range(n):
            a = first(i)
            j = (a, a - 1, None)[i % 3]
            if j is not None and j >= 0:
                for h in range(q.shape[1]):
                    q[at + i, h] = k[at + j, h // (q.shape[1] // k.shape[1])]
        at += n
    return q


BOUNDS = [('window', 1), ('window', 37), ('window', 127), ('window', 128), ('window', 129), ('chunk', 1), ('chunk', 30), ('chunk', 64), ('chunk', 128), ('chunk', 129), ('window', 5000),
          ('chunk', 5000)]


@BACKENDS
@pytest.mark.parametrize('kind,size', BOUNDS)
@pytest.mark.parametrize('hq,hkv,d,e', [(4, 2, 64, 40), (3, 1, 24, 24), (2, 2, 128, 128), (2, 1, 192, 72), (5, 5, 11, 7), (2, 1, 200, 200)])
def test_packed_attention_inside_bounds(where, kind, size, hq, hkv, d, e):
    from twinkle_b200 import ops
    if where[0] == 'cpu' and (d > 64 or size == 5000):
        pytest.skip('same formulas at every width')
    G = torch.Generator().manual_seed(d + size)
    lens = [1, 140, 33, 270]
    _, cu = _packed(lens)
    T = sum(lens)
    first = (lambda i: O.seen_in_window(i, size)) if kind == 'window' else (lambda i: O.seen_in_chunk(i, size))
    k, v, gate = _rand(G, T, hkv, d), _rand(G, T, hkv, e), _rand(G, T, hq + 3)
    q = _standing_out(G, _rand(G, T, hq, d), k, first, lens)
    sink, scale = (1 + _rand(G, hq)).bfloat16().double(), 6.0 / d
    with torch.no_grad():
        got = ops.attention_packed(_t(where, q), _t(where, k), _t(where, v), cu.to(where[0]), max(lens), scale, _t(where, sink), _t(where, gate)[:, 1:1 + hq],
                                   **{kind: size})
        plain = ops.attention_packed(_t(where, q), _t(where, k), _t(where, v), cu.to(where[0]), max(lens), scale, **{kind: size})
    for a, b in zip(cu[:-1], cu[1:]):
        want = O.attend(q[a:b], k[a:b], v[a:b], scale, first, sink) * O.sigmoid(gate[a:b, 1:1 + hq])[..., None]
        assert worst_row(got[a:b].flatten(0, 1), want.flatten(0, 1)) < 2 * tol(where)
        assert worst_row(plain[a:b].flatten(0, 1), O.attend(q[a:b], k[a:b], v[a:b], scale, first).flatten(0, 1)) < 2 * tol(where)


@BACKENDS
@pytest.mark.parametrize('H,d,r,e,window', [(4, 64, 32, 64, 37), (3, 128, 64, 128, 128), (5, 24, 16, 32, 129), (2, 40, 8, 24, 1), (3, 7, 6, 11, 30), (2, 128, 64, 72, 0), (1, 136, 64, 72, 50)])
def test_packed_attention_with_a_shared_key_part(where, H, d, r, e, window):
    """Keys and values as column ranges of one product, the rotated key part from a tensor of its own, queries as columns of a projection."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d + r)
    lens = [1, 140, 270]
    _, cu = _packed(lens)
    T = sum(lens)
    proj, kv, kept = _rand(G, T, 8 + H * (d + r) + 8), _rand(G, T, H * (d + e)), _rand(G, T, -(-(24 + r) // 8) * 8)
    q = proj[:, 8:8 + H * (d + r)].view(T, H, d + r)
    k, tail = kv[:, :H * d].view(T, H, d), kept[:, 24:24 + r]
    whole = torch.cat([k, tail[:, None].expand(T, H, r)], -1)
    first = (lambda i: O.seen_in_window(i, window)) if window else (lambda i: 0)
    _standing_out(G, q, whole, first, lens)                       # (writes into proj)
    scale = 5.0 / (d + r)
    pt, kvt, keptt = _t(where, proj), _t(where, kv), _t(where, kept)
    with torch.no_grad():
        got = ops.attention_packed(pt[:, 8:8 + H * (d + r)].view(T, H, d + r), kvt[:, :H * d].view(T, H, d), kvt[:, H * d:].view(T, H, e), cu.to(where[0]), max(lens), scale,
                                   window=window, key_tail=keptt[:, 24:24 + r])
    for a, b in zip(cu[:-1], cu[1:]):
        want = O.attend(q[a:b], whole[a:b], kv[a:b, H * d:].view(b - a, H, e), scale, first)
        assert worst_row(got[a:b].flatten(0, 1), want.flatten(0, 1)) < 2 * tol(where)


def _paged(G, lens, bs, *shapes):
    """Pools of random rows in shuffled pages, the table, and the rows of a sequence in order."""
    need = sum(-(-n // bs) for n in lens) + 1
    order = (torch.randperm(need, generator=G) + 1).tolist()
    pools = [_rand(G, need + 1, bs, *s) for s in shapes]
    table = torch.zeros(len(lens), -(-max(lens) // bs) + 1, dtype=torch.int32)
    for i, n in enumerate(lens):
        for j in range(-(-n // bs)):
            table[i, j] = order.pop()
    return pools, table, lambda pool, i: pool[table[i].long()].flatten(0, 1)[:lens[i]]


@BACKENDS
@pytest.mark.parametrize('kind,size', [('window', 1), ('window', 16), ('window', 33), ('chunk', 1), ('chunk', 16), ('chunk', 50), ('window', 9999)])
@pytest.mark.parametrize('hq,hkv,d,e,bs', [(6, 2, 24, 40, 16), (4, 4, 128, 72, 16), (10, 1, 64, 64, 8), (2, 1, 160, 136, 4), (3, 1, 256, 8, 16)])
def test_decode_attention_inside_bounds(where, kind, size, hq, hkv, d, e, bs):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d + size)
    lens = [1, bs - 1, bs, bs + 1, 0, size, size + 1, 200, 49, 51] if size < 1000 else [1, 0, 77]
    (kp, vp), table, rows = _paged(G, lens, bs, (hkv, d), (hkv, e))
    q, sink, gate = _rand(G, len(lens), hq, d), (1 + _rand(G, hq)).bfloat16().double(), _rand(G, len(lens), hq + 3)
    scale = 6.0 / d
    first = (lambda i: O.seen_in_window(i, size)) if kind == 'window' else (lambda i: O.seen_in_chunk(i, size))
    for i, n in enumerate(lens):
        if n:
            k = rows(kp, i)
            for h in range(hq):                      # looks for the first key it sees, or for the one before
                j = first(n - 1) - h % 2
                q[i, h] = k[max(j, 0), h // (hq // hkv)]
    dev = lambda x: _t(where, x)  # noqa: E731
    args = (dev(q), dev(kp), dev(vp), table.to(where[0]), torch.tensor(lens, dtype=torch.int32, device=where[0]), scale)
    with torch.no_grad():
        got = ops.paged_attention_decode(*args, sinks=dev(sink), gate=dev(gate)[:, 2:2 + hq], **{kind: size})
        plain = ops.paged_attention_decode(*args, **{kind: size})
    for i, n in enumerate(lens):
        if n == 0:
            assert not got[i].any() and not plain[i].any()
            continue
        k, v = rows(kp, i), rows(vp, i)
        at = first(n - 1)
        assert worst_row(got[i], _one(q[i], k[at:], v[at:], scale, sink) * O.sigmoid(gate[i, 2:2 + hq])[:, None]) < 2 * tol(where), n
        assert worst_row(plain[i], _one(q[i], k[at:], v[at:], scale, None)) < 2 * tol(where), n


def _one(q, k, v, scale, sink):
    """One query ``[H, d]`` over all of ``k [n, G, d]``."""
    share = q.shape[0] // k.shape[1]
    s = torch.einsum('hd,nhd->hn', q, k.repeat_interleave(share, 1) if k.shape[1] > 1 else k.expand(-1, share, -1)) * scale
    top = s.amax(-1) if sink is None else torch.maximum(s.amax(-1), sink)
    p = torch.exp(s - top[:, None])
    o = torch.einsum('hn,nhe->he', p, v.repeat_interleave(share, 1) if v.shape[1] > 1 else v.expand(-1, share, -1))
    return o / (p.sum(-1) + (0 if sink is None else torch.exp(sink - top)))[:, None]


@BACKENDS
@pytest.mark.parametrize('window', [0, 1, 100, 128, 129, 5000])
@pytest.mark.parametrize('H,R,r,bs', [(5, 48, 16, 16), (3, 13, 6, 4), (20, 264, 32, 16), (40, 512, 64, 16), (8, 256, 32, 64), (16, 64, 8, 8)])
def test_latent_decode_with_key_parts_inside_a_window(where, H, R, r, bs, window):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(R + H + window)
    lens = [1, bs, bs + 1, 0, 127, 128, 129, 257, 700]
    K = R + r
    (pool, ), table, rows = _paged(G, lens, bs, (1, -(-K // 8) * 8))
    pool[..., K:] = 0
    q, sink, gate, scale = _rand(G, len(lens), H, K), (1 + _rand(G, H)).bfloat16().double(), _rand(G, len(lens), H + 3), 4.0 / K
    for i, n in enumerate(lens):
        if n:
            a = max(0, n - window) if window else 0
            q[i, 0], q[i, 1 % H] = rows(pool, i)[a, 0, :K], rows(pool, i)[max(a - 1, 0), 0, :K]
    dev = lambda x: _t(where, x)  # noqa: E731
    args = (dev(q), dev(pool), table.to(where[0]), torch.tensor(lens, dtype=torch.int32, device=where[0]), scale)
    with torch.no_grad():
        got = ops.latent_decode(*args, rank=R, window=window)
        more = ops.latent_decode(*args, dev(sink), dev(gate)[:, 1:1 + H], rank=R, window=window)
    assert got.shape == (len(lens), H, R) and torch.isfinite(got).all() and not got[lens.index(0)].any()
    for i, n in enumerate(lens):
        if n:
            c = rows(pool, i)[max(0, n - window) if window else 0:, :, :K]
            assert worst_row(got[i], _one(q[i], c, c[..., :R], scale, None)) < 2 * tol(where), n
            assert worst_row(more[i], _one(q[i], c, c[..., :R], scale, sink) * O.sigmoid(gate[i, 1:1 + H])[:, None]) < 2 * tol(where), n


@BACKENDS
@pytest.mark.parametrize('B,H,d,r,N', [(1, 3, 24, 16, 40), (5, 4, 64, 32, 512), (130, 2, 40, 8, 264), (3, 5, 7, 6, 11)])
def test_product_per_head_into_columns(where, B, H, d, r, N):
    """Queries as columns of a projection, the result in front of what is already there."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(B)
    p, w, tail = _rand(G, B, 8 + H * (d + r)), _rand(G, H, d, N), _rand(G, B, H, r)
    out = torch.cat([torch.zeros(B, H, N, dtype=torch.float64), tail], -1)
    with torch.no_grad():
        got = ops.head_linear(_t(where, p)[:, 8:].view(B, H, d + r)[..., :d], _t(where, w), transposed=True, out=_t(where, out))
    assert rel(got[..., :N], torch.einsum('bhk,hkn->bhn', p[:, 8:].view(B, H, d + r)[..., :d], w)) < tol(where) / 2
    assert torch.equal(got[..., N:], _t(where, tail))


@BACKENDS
@pytest.mark.parametrize('width', [52, 64, 70, 2304, 4608, 8200])
@pytest.mark.parametrize('k,beside', [(0, False), (1, True), (3, False), (9, True)])
def test_results_join_the_stream(where, width, k, beside):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(width + k)
    T, eps = 5, 1e-4
    x, y = torch.randn(T, width, generator=G), _rand(G, T * max(k, 1) + (3 if k else 0), width)
    w, b, opened = (1 + _rand(G, width)).bfloat16().double(), _rand(G, T, width), torch.rand(T, generator=G)
    row_of = share = None
    total = y
    if k:
        row_of, share = torch.randperm(y.shape[0], generator=G)[:T * k].view(T, k), torch.rand(T, k, generator=G)
        total = (y[row_of] * share[..., None].double()).sum(1)
        row_of, share = row_of.int().to(where[0]), share.to(where[0])
    want = x.double() + total + (opened.double()[:, None] * b if beside else 0)
    with torch.no_grad():
        h, nx = ops.stream_joined_rmsnorm(x.to(where[0]).clone(), _t(where, w), eps, 0.0, _t(where, y), row_of, share, _t(where, b) if beside else None,
                                          opened.to(where[0]) if beside else None)
    assert nx.dtype == torch.float32 and rel(nx, want) < 1e-6          # the stream itself is never rounded
    assert rel(h, O.norm(want, w, eps)) < tol(where) / 4


@BACKENDS
@pytest.mark.parametrize('ff,lead', [(64, 0), (18, 5), (40, 8), (7, 0)])
@pytest.mark.parametrize('limit', [0.0, 0.3, 1.0, 7.0])
def test_clamped_gated_unit(where, ff, lead, limit):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(ff)
    p = 3 * _rand(G, 11, lead + 2 * ff + 8)
    p = p.bfloat16().double()
    g, u = p[:, lead:lead + ff], p[:, lead + ff:lead + 2 * ff]
    if limit:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
        want = g * O.sigmoid(1.702 * g) * (u + 1)
    else:
        want = O.silu(g) * u
    with torch.no_grad():
        got = ops.glu_columns(_t(where, p), lead, lead + ff, ff, limit)
    assert rel(got, want) < tol(where) / 4


@BACKENDS
@pytest.mark.parametrize('E,count,keep,k', [(1, 1, 1, 1), (6, 3, 2, 2), (8, 8, 3, 3), (12, 2, 1, 4), (64, 8, 3, 6), (96, 6, 6, 8), (160, 8, 3, 6), (256, 2, 1, 32), (256, 256, 5, 5)])
def test_choice_among_the_best_groups(where, E, count, keep, k):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(E + k)
    T, width = 70, 40 if k % 2 else 52
    logits, h, sg = torch.randn(T, E, generator=G) * 2, _rand(G, T, width), _rand(G, 1, width) / 4
    sg = sg.bfloat16().double()
    want_idx, want_w = O.route(logits.double(), {'experts': E, 'top': k, 'scale': 2.5, 'groups': {'count': count, 'keep': keep}})
    forced = torch.stack([torch.randperm(E, generator=G)[:k] for _ in range(T)])
    forced[0] = -1
    with torch.no_grad():
        w, idx, hist, opened = ops.moe_topk(logits.to(where[0]), None, k, groups=count, keep=keep, factor=2.5, x=_t(where, h), shared=_t(where, sg))
        wf, idf, _ = ops.moe_topk(logits.to(where[0]), None, k, forced.to(where[0]), count, keep, 2.5)
    assert torch.equal(idx.cpu(), want_idx) and rel(w, want_w) < 1e-5 and hist.tolist() == torch.bincount(want_idx.flatten(), minlength=E).tolist()
    assert rel(opened, O.sigmoid(h @ sg.t())[:, 0]) < 1e-5
    assert torch.equal(idf.cpu()[0], want_idx[0]) and torch.equal(idf.cpu()[1:], forced[1:])
    assert rel(wf[1:], 2.5 * torch.softmax(logits.double(), -1).gather(1, forced.clamp_min(0))[1:]) < 1e-5


@BACKENDS
@pytest.mark.parametrize('E,k,T,width,ff,shared', [(1, 1, 3, 24, 16, 0), (6, 2, 40, 96, 32, 40), (5, 3, 40, 52, 20, 12), (64, 6, 64, 128, 264, 64)])
def test_gated_experts_beside_a_shared_one(where, E, k, T, width, ff, shared):
    from twinkle_b200.models.config import DecoderConfig
    from twinkle_b200.models.decoder import MoEBlock
    G = torch.Generator().manual_seed(E)
    h = _rand(G, T, width)
    m = O.moe(E, k, ff, 1.5, None, shared or None)
    w = {n[len('l0.mlp.'):]: t.double() for n, t in O.random_weights(dict(vocab=2, width=width, layers=[O.chunked(1, 1, 8, 8, 1, 1, O.rot(2, 2.0), m)]), E).items() if n.startswith('l0.mlp.')}
    block = MoEBlock(DecoderConfig(hidden_size=width, num_experts=E, num_experts_per_tok=k, moe_intermediate_size=ff, router_scoring='softmax_grouped', norm_topk_prob=False,
                                   routed_scaling_factor=1.5, shared_expert_intermediate_size=shared), 0)
    with torch.no_grad():
        block.gate.weight.copy_(w['router'])
        for e in range(E):
            block.experts.gate_up_proj[e].copy_(torch.cat([w[f'e{e}.gate'], w[f'e{e}.up']]))
            block.experts.down_proj[e].copy_(w[f'e{e}.down'])
        if shared:
            block.shared_expert.gate_up_proj.weight.copy_(torch.cat([w['shared.gate'], w['shared.up']]))
            block.shared_expert.down_proj.weight.copy_(w['shared.down'])
            block.shared_expert_gate.weight.copy_(w['shared.sg'])
        block = block.to(where[0], getattr(torch, where[1]))
        assert block.rows_apply()
        y, row_of, share, opened = block.rows(_t(where, h))
        got = (y[row_of.long()].float() * share[..., None]).sum(1)
        if shared:
            got = got + opened[:, None] * block.shared_expert.serve(_t(where, h)).float()
    z = (h @ w['router'].t()).sort(-1, descending=True).values
    sure = z[:, k - 1] - z[:, k] > 0.05 if E > k else torch.ones(T, dtype=torch.bool)
    assert int(sure.sum()) > T // 2 and worst_row(got.cpu()[sure], O.mixture(h, m, w)[sure]) < 2 * tol(where)


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
    """Over several tiles, pages, windows and chunks; the last tokens by steps."""
    path, cfg, W = checkpoint(name)
    tokens = ids(420, cfg['vocab'], 3)
    agrees(run_one(replay(path, where), 'r', tokens, 410), cfg, W, tokens, where)


@BACKENDS
def test_residual_stream_after_every_layer(checkpoint, where):
    from twinkle_b200.models.decoder import PackedBatch, Stream
    path, cfg, W = checkpoint('mixed')
    tokens = ids(29, cfg['vocab'], 2)
    _, trail = O.forward(cfg, W, tokens)
    n = int((~close_calls(cfg, W, tokens, 0.08 if where[1] == 'bfloat16' else 1e-5)[1]).sum())
    rp = replay(path, where)
    T = len(tokens)
    batch = PackedBatch(torch.tensor(tokens, device=where[0]), torch.arange(T, device=where[0]), torch.tensor([0, T], dtype=torch.int32, device=where[0]), T)
    with torch.no_grad():
        batch.rotary = rp.model.rotary_table(batch.position_ids)
        st = Stream(rp.model.embed(batch).float())
        assert rel(st.x, W['embed'].double()[tokens] * cfg['embedding']['scale']) < 1e-6
        for layer, want in zip(rp.model.layers, trail):
            st = layer.advance(st, batch)
            seen = Stream(st.x.clone(), plain=st.plain)
            seen.enter(rp.model.norm)
            assert seen.x.dtype == torch.float32 and n > 2 and worst_row(seen.x[:n], want[:n]) < 2 * tol(where)


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
        assert rel(torch.cat(rows[n]), alone) < (0.1 if where[1] == 'bfloat16' else 2e-5)


@BACKENDS
def test_freed_pages_are_used_again(checkpoint, where):
    """A cache of few blocks serves one request after another; what an ended request left does not show."""
    path, cfg, W = checkpoint('mixed')
    rp = replay(path, where, max_tokens=64, block_size=4)
    cache = rp.engine.cache
    blocks = len(cache.free)
    for i, (n, n_prompt) in enumerate([(60, 50), (9, 1), (40, 2), (5, 1), (64, 64)]):
        tokens = ids(n, cfg['vocab'], 40 + i)
        agrees(run_one(rp, f'r{i}', tokens, n_prompt), cfg, W, tokens, where)
        assert len(cache.free) == blocks
    with pytest.raises(RuntimeError, match='exhausted'):
        for i in range(blocks + 1):
            start(rp, {f'x{i}': [1]})


@BACKENDS
def test_cache_holds_what_a_layer_has_of_its_own(checkpoint, where):
    for name in O.CONFIGS:
        path, cfg, W = checkpoint(name)
        c = replay(path, where, max_tokens=64).engine.cache
        up = lambda n: -(-n // 8) * 8  # noqa: E731
        for layer, k, v, s in zip(cfg['layers'], c.k, c.v, c.state):
            m = layer['mixer']
            assert s is None
            if 'kv_from' in m:
                assert k is None and v is None
            elif layer['type'] == 'latent_attention':
                assert v is None and tuple(k.shape[2:]) == (1, up(m['kv_rank'] + m['rot_dim']))
            else:
                assert tuple(k.shape[2:]) == (m['kv_heads'], up(m['dim'])) and tuple(v.shape[2:]) == (m['kv_heads'], up(m['vdim']))


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


def _asking_model(kind, size, borrow=False):
    """One layer (with ``borrow`` a second one on its keys, which does the asking) in which token 299 looks for token 298 and for nothing else:
    channel 0 of the stream marks the one, channel 1 the other, and the last unrotated dimension of queries and keys carries the marks."""
    width, H, d, e = 80, 4, 24, 40
    if kind == 'latent':
        layers = [O.latents(H, d, 8, e, 32, 0.6, size, 100.0)]
    elif kind == 'chunk':
        layers = [O.chunked(H, 2, d, e, 0.6, size, O.rot(8, 100.0))]
    else:
        layers = [O.windowed(H, 2, d, e, 0.6, size, O.rot(8, 100.0))] + ([O.windowed(H, 2, d, e, 0.6, size, O.rot(8, 100.0), kv_from=0)] if borrow else [])
    cfg = dict(architecture='Nilepel', vocab=300, width=width, norm={'eps': 1e-5}, embedding={'scale': 2.0}, layers=layers)
    W = O.random_weights(cfg, 3)
    W['embed'][:, :2] = 0
    W['embed'][298, 0], W['embed'][299, 1] = 6, 6
    last = f'l{len(layers) - 1}.'
    for n in [n for n in W if n.endswith(('norm1', 'q.norm', 'k.norm', 'dkv.norm'))]:
        W[n] = torch.ones_like(W[n])
    qk = d + 8 if kind == 'latent' else d
    W[last + 'mix.q'] = torch.zeros_like(W[last + 'mix.q'])
    W[last + 'mix.q'].view(H, qk, width)[:, d - 1, 1] = 4
    if kind == 'latent':
        W['l0.mix.dkv'][0], W['l0.mix.uk'] = 0, torch.zeros_like(W['l0.mix.uk'])
        W['l0.mix.dkv'][0, 0], W['l0.mix.dkv'][1:, 0] = 4, 0
        W['l0.mix.uk'].view(H, d, 32)[:, d - 1, 0] = 1
    else:
        W['l0.mix.k'].view(2, d, width)[:, d - 1] = 0
        W['l0.mix.k'].view(2, d, width)[:, :, 0] = 0
        W['l0.mix.k'].view(2, d, width)[:, d - 1, 0] = 4
        for n in [n for n in W if n.endswith(('q.b', 'k.b'))]:
            W[n] = torch.zeros_like(W[n])
    if borrow:                                          # the first layer adds little, so that the second still recognises the tokens
        W['l0.mix.o'] = W['l0.mix.o'] / 16
    return cfg, W


@BACKENDS
@pytest.mark.parametrize('kind,size,borrow', [('window', 100, False), ('window', 128, True), ('window', 33, True), ('latent', 100, False), ('latent', 129, False), ('chunk', 100, False),
                                              ('chunk', 64, False)])
def test_keys_just_inside_and_just_outside(tmp_path, where, kind, size, borrow):
    """What the last token looks for stands at the first place it sees, the one before, around page borders, in the middle.  Asked for in the
    prompt and in decoding; another token there changes the logits if and only if it is seen."""
    cfg, W = _asking_model(kind, size, borrow)
    path = O.write_checkpoint(tmp_path / 'm', cfg, W)
    rp = replay(path, where)
    lasts = (size, 2 * size - 1, 2 * size, 230) if kind == 'chunk' else (size - 1, size, 230, 256)
    for last in lasts:
        n, edge = last + 1, (last // size * size if kind == 'chunk' else max(0, last - size + 1))
        for at in sorted({edge, edge - 1, edge + 1, edge - 2, (last // 16) * 16, (last // 16) * 16 - 1, (edge + last) // 2, 0}):
            if not 0 <= at < last:
                continue
            base = ids(n, 297, at)
            base[-1] = 299
            seen, unseen = list(base), list(base)
            seen[at], unseen[at] = 298, 297
            want, other = O.forward(cfg, W, seen)[0][-1], O.forward(cfg, W, unseen)[0][-1]
            assert rel(other, want) > 0.1 if at >= edge else rel(other, want) < 1e-12          # a key that is seen matters, another does not …
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
        lg, near = close_calls(cfg, W, p + got, 0.08 if where[1] == 'bfloat16' else 1e-5)
        for i, t in enumerate(got):
            at = len(p) + i - 1
            slack = 0.05 if where[1] == 'bfloat16' and not near[at] else (0.6 if where[1] == 'bfloat16' else 1e-4)
            assert float(lg[at].max() - lg[at, t]) <= slack * float(lg[at].std())      # the best, up to a tie within rounding
    if where[0] == 'cuda':
        assert s.engine.use_cuda_graphs and s.engine._graphs                  # decoding was captured, not run eagerly
    s.sleep()
    s.wake_up()
    again = s.sample([{'input_ids': p} for p in prompts], SamplingParams(max_tokens=10, temperature=0.0))
    assert [r.sequences[0].tokens for r in again] == [r.sequences[0].tokens for r in out]


def test_routing_is_recorded_per_expert_layer(checkpoint):
    from twinkle_b200.data_format import SamplingParams
    from twinkle_b200.sampler import TorchSampler
    path, cfg, W = checkpoint('mixed')
    s = TorchSampler(model_id=path, device='cpu', enable_lora=False, engine_args={'num_blocks': 64, 'max_batch': 2})
    r = s.sample([{'input_ids': ids(6, cfg['vocab'], 1)}], SamplingParams(max_tokens=3, temperature=0.0), return_routed_experts=True)[0].sequences[0]
    tops = [layer['mlp']['router']['top'] for layer in cfg['layers'] if (layer['mlp'] or {}).get('kind') == 'moe']
    assert [tuple(t.shape) for t in r.routed_experts] == [(8, k) for k in tops]


# ------------------------------------------------------------------------------------------------ registry, files, training
def test_config_and_weights_round_trip(checkpoint, tmp_path):
    from safetensors.torch import load_file
    from twinkle_b200.model import TransformersModel
    from twinkle_b200.models.config import DecoderConfig, preset
    for name in O.CONFIGS:
        path, cfg, W = checkpoint(name)
        c = DecoderConfig.from_pretrained(path)
        assert DecoderConfig.from_hf(c.to_hf()) == c and c.model_type == 'nilepel'
        m = TransformersModel(model_id=path, device='cpu')
        assert sum(p.numel() for p in m.model.parameters()) == c.num_params() == sum(t.numel() for t in W.values())
        out = m.save('ckpt', output_dir=str(tmp_path / name))
        back = load_file(os.path.join(out, 'model.safetensors'))
        assert set(back) == set(W) and all(torch.equal(back[n].float(), W[n].float()) and back[n].shape == W[n].shape for n in W)
        with open(os.path.join(out, 'config.json')) as f:
            assert DecoderConfig.from_hf(json.load(f)) == c
    assert preset('tiny-nilepel', num_hidden_layers=3).num_hidden_layers == 3
    assert DecoderConfig.from_pretrained(checkpoint('mixed')[0]).kernel_parts() == ['experts', 'latent', 'rotary']

    def changed(**what):
        bad = json.loads(json.dumps(O.CONFIGS['mixed']))
        for where, value in what.items():
            *keys, last = where.split('__')
            d = bad['layers']
            for k in keys:
                d = d[int(k[1:])] if k[:1] == 'l' and k[1:].isdigit() else d[k]
            d[last] = value
        return bad
    for bad in (changed(l0__type='something'), changed(l0__mlp={'kind': 'something'})):
        with pytest.raises(NotImplementedError):
            DecoderConfig.from_hf(bad)
    for source in (1, 2, 3, 5, 4):          # latents, other sizes, borrowed ones, itself, not earlier
        with pytest.raises(ValueError, match='kv_from'):
            DecoderConfig.from_hf(changed(l3__mixer__kv_from=source))
    with pytest.raises(ValueError, match='kv_from'):                   # another rotation
        DecoderConfig.from_hf(changed(l3__mixer__rot=O.rot(16, 501.0, O._LONG)))
    for bad in (changed(l0__mlp__router__groups={'count': 4, 'keep': 2}), changed(l0__mlp__router__groups={'count': 3, 'keep': 4}), changed(l0__mlp__router__top=5),
                changed(l0__mixer__heads=5), changed(l0__mixer__rot=O.rot(26, 500.0)), changed(l1__mixer__rot_dim=8)):
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
    for hf, internal, rows in (('l0.mix.k', 'layers.0.mixer.in_proj.weight', slice(144, 192)), ('l0.mix.v.b', 'layers.0.mixer.qkv_bias', slice(192, 272)),
                               ('l0.mix.k.norm', 'layers.0.mixer.head_k_norm.weight', slice(None)), ('l3.mix.q', 'layers.3.mixer.in_proj.weight', slice(0, 96)),
                               ('l3.mix.q.norm', 'layers.3.mixer.head_q_norm.weight', slice(None)), ('l5.mix.g', 'layers.5.mixer.in_proj.weight', slice(48, 50)),
                               ('l2.mix.sink', 'layers.2.mixer.sinks', slice(None)), ('l1.mix.dkv', 'layers.1.mixer.in_proj.weight', slice(200, 264)),
                               ('l4.mix.uv', 'layers.4.mixer.kv_up', slice(120, None)), ('l4.mix.dkv.norm', 'layers.4.mixer.kv_norm.weight', slice(None)),
                               ('l0.mlp.shared.sg', 'layers.0.mlp.shared_expert_gate.weight', slice(None)), ('l0.mlp.shared.up', 'layers.0.mlp.shared_expert.gate_up_proj.weight', slice(40, 80)),
                               ('l2.mlp.router', 'layers.2.mlp.gate.weight', slice(None)), ('l1.mlp.up', 'layers.1.mlp.in_proj.weight', slice(64, 128)),
                               ('l1.norm2', 'layers.1.pre_mlp_layernorm.weight', slice(None)), ('embed', 'embed_tokens.weight', slice(None)), ('head', 'lm_head.weight', slice(None))):
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


def test_adapters_apply_to_fused_projections_and_experts():
    from twinkle_b200.model import LoraConfig, TransformersModel
    m = TransformersModel(model_id='tiny-nilepel', device='cpu', max_loras=1, max_r=4)
    m.add_adapter_to_model('a', LoraConfig(r=4, lora_alpha=8, target_modules=['q_proj', 'v_proj', 'dkv_proj', 'up_proj', 'o_proj', 'gate_up', 'down']))
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
    assert worst_row(read(0), torch.stack([wa[0], wa[18], wb[2]])) < lim and worst_row(read(2), wa[20:]) < lim
