"""Moronex stacks (layers listed one by one: norms around each sub-layer, gated results on a 32-bit stream, HGRN2 and latent
attention, dense and expert feed-forward blocks) against ``tests/moronex_oracle.py``.

Every case runs on the CPU in fp32 and, marked ``gpu``, on the kernels in fp32 and bf16."""
import json
import os

import pytest
import torch

from tests import moronex_oracle as O
from tests.test_pomelix import BACKENDS, _packed, _t, go_on, ids, rel, replay, run_one, start, tol, worst_row

_MADE = {}


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


# a router's choice between two experts may flip under bf16 rounding: positions where that can happen are compared loosely
def close_calls(cfg, W, tokens, margin):
    """Per position: whether some layer's router sees its last chosen and first left-out logit closer than ``margin``."""
    near = torch.zeros(len(tokens), dtype=torch.bool)
    real = O.route

    def spy(h, w, top):
        z = (h @ w['router'].t() + w['router.b']).sort(-1, descending=True).values
        if z.shape[1] > top:
            near.logical_or_(z[:, top - 1] - z[:, top] < margin)
        return real(h, w, top)
    O.route = spy
    try:
        out = O.forward(cfg, W, tokens)[0]
    finally:
        O.route = real
    return out, near.int().cummax(0).values.bool()         # what a token was given reaches every later one


def agrees(got, cfg, W, tokens, where):
    """Logits of every position; in bf16 those before the first close call of a router, and most of all others."""
    want, near = close_calls(cfg, W, tokens, 0.08 if where[1] == 'bfloat16' else 1e-4)
    n = int((~near).sum())
    assert got.shape == want.shape
    if where[1] != 'bfloat16':
        assert n == len(tokens) and worst_row(got, want) < 2 * tol(where)
        return
    # a head's norm divides by next to nothing where query and state nearly cancel: single rows may be far off without a fault
    err = (got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1).mean()
    assert n == 0 or float(err[:n].quantile(0.9)) < 4 * tol(where)
    assert len(tokens) < 8 or float(err.median()) < tol(where) * 1.5


# ------------------------------------------------------------------------------------------------ mechanisms
@BACKENDS
@pytest.mark.parametrize('width', [52, 64, 70, 2304, 4608, 8200])
@pytest.mark.parametrize('k', [0, 1, 3, 8])
def test_gated_norm_joins_the_stream(where, width, k):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(width + k)
    T, eps = 5, 1e-4
    x, gate = torch.randn(T, width, generator=G), _rand(G, T, width + 24)
    y = _rand(G, T * max(k, 1) + 3, width) if k else _rand(G, T, width)
    bias, post, nxt = _rand(G, width), 0.3 * _rand(G, width), 0.3 * _rand(G, width)
    post, nxt = post.bfloat16().double(), nxt.bfloat16().double()
    row_of = share = None
    result = y
    if k:
        row_of, share = torch.randperm(y.shape[0], generator=G)[:T * k].view(T, k), torch.rand(T, k, generator=G)
        result = (y[row_of] * share[..., None].double()).sum(1)
        row_of, share = row_of.int().to(where[0]), share.to(where[0])
    want = x.double() + O.norm_about_one(O.sigmoid(gate[:, :width] + bias) * result, post, eps)
    with torch.no_grad():
        h, nx = ops.stream_gated_rmsnorm(x.to(where[0]).clone(), _t(where, nxt), eps, 1.0, _t(where, y), _t(where, gate), _t(where, bias), _t(where, post), row_of, share)
    assert nx.dtype == torch.float32 and rel(nx, want) < 1e-6          # the stream itself is never rounded
    assert rel(h, O.norm_about_one(want, nxt, eps)) < tol(where) / 4


@BACKENDS
def test_norm_about_one_without_a_result(where):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(1)
    for width in (52, 64, 2304):
        x, w = torch.randn(3, width, generator=G), 0.3 * _rand(G, width)
        w = w.bfloat16().double()
        with torch.no_grad():
            h, nx = ops.stream_rmsnorm(x.to(where[0]).clone(), _t(where, w), 1e-3, offset=1.0)
        assert torch.equal(nx.cpu(), x) and rel(h, O.norm_about_one(x.double(), w, 1e-3)) < tol(where) / 4


HGRN2_SIZES = [(1, 1, 1), (3, 6, 9), (2, 24, 40), (5, 32, 56), (2, 33, 20), (2, 64, 128), (1, 72, 24), (2, 128, 128), (1, 128, 256), (2, 160, 136), (1, 256, 256)]


def _hgrn2_case(H, d, e, T, seed, shift=2.0):
    G = torch.Generator().manual_seed(seed)
    lead = 5 if d % 8 else 16                                       # columns in front that belong to others
    proj = _rand(G, T, lead + H * (2 * d + e) + 8)
    bias, lower = (shift + 3 * torch.randn(H * d, generator=G)).bfloat16().double(), (torch.rand(H * d, generator=G) * 0.9).bfloat16().double()
    weight = (1 + 0.2 * torch.randn(e, generator=G)).bfloat16().double()
    return proj, lead, bias, lower, weight


def _hgrn2_want(proj, lead, H, d, e, bias, lower):
    n = H * d
    q = O.silu(proj[:, lead:lead + n]).view(-1, H, d)
    f = (lower + (1 - lower) * O.sigmoid(proj[:, lead + n:lead + 2 * n] + bias)).view(-1, H, d)
    return q, f, proj[:, lead + 2 * n:lead + 2 * n + H * e].reshape(-1, H, e)


class _View:
    """The part of a cache view that the recurrent mixer looks at."""

    def __init__(self, states, slots, stepping):
        self.cache, self.slots, self.stepping = type('C', (), {'state': [states]})(), slots, stepping


@BACKENDS
@pytest.mark.parametrize('H,d,e', HGRN2_SIZES)
def test_hgrn2_prompts_states_and_steps(where, H, d, e):
    """Packed prompts (of one token, around a round of sixteen, long enough for time segments), their last states, and steps from there."""
    from twinkle_b200 import ops
    lens = [1, 15, 16, 17, 300, 2, 640]
    pos, cu = _packed(lens)
    proj, lead, bias, lower, weight = _hgrn2_case(H, d, e, sum(lens), d + e)
    n = H * d
    states = torch.full((len(lens) + 2, H, d, e), 7.0, device=where[0])           # what freed slots were left with
    slots = torch.tensor([len(lens) - i for i in range(len(lens))], dtype=torch.int32)
    per_token = torch.cat([s.expand(m) for s, m in zip(slots, lens)]).to(where[0])
    args = [_t(where, t) for t in (bias, lower, weight)]
    with torch.no_grad():
        got = ops.hgrn2(_t(where, proj), lead, lead + n, lead + 2 * n, H, d, e, *args, 1e-4, cu.to(where[0]), max(lens), _View(states, per_token, False), 0)
    finals = []
    for i, (a, b) in enumerate(zip(cu[:-1], cu[1:])):
        o, S = O.hgrn2_scan(*_hgrn2_want(proj[a:b], lead, H, d, e, bias, lower))
        finals.append(S)
        assert worst_row(got[a:b], O.norm(o, weight, 1e-4).flatten(1)) < tol(where), lens[i]
        assert rel(states[slots[i]], S) < 2e-5, lens[i]                            # the state is 32-bit whatever the inputs are
    more, _, _, _, _ = _hgrn2_case(H, d, e, 3 * len(lens), 99)
    for t in range(3):
        rows = more[t * len(lens):(t + 1) * len(lens)]
        with torch.no_grad():
            got = ops.hgrn2(_t(where, rows), lead, lead + n, lead + 2 * n, H, d, e, *args, 1e-4, view=_View(states, slots.to(where[0]), True), layer=0)
        q, f, v = _hgrn2_want(rows, lead, H, d, e, bias, lower)
        for i in range(len(lens)):
            finals[i] = f[i][:, :, None] * finals[i] + (1 - f[i])[:, :, None] * v[i][:, None]
            o = (q[i][:, :, None] * finals[i]).sum(1)
            assert rel(got[i], O.norm(o, weight, 1e-4).flatten()) < tol(where)
            assert rel(states[slots[i]], finals[i]) < 2e-5
    assert bool((states[[0, len(lens) + 1]] == 7.0).all())                         # nobody else's state is touched


@BACKENDS
@pytest.mark.parametrize('shift', [-20.0, 9.0, 30.0])
def test_hgrn2_gates_at_their_ends(where, shift):
    """Gates that forget everything, keep nearly everything for thousands of tokens, and keep it all."""
    from twinkle_b200 import ops
    H, d, e, T = 2, 16, 24, 3000
    proj, lead, bias, lower, weight = _hgrn2_case(H, d, e, T, 5, shift)
    lower[::2] = 0
    n = H * d
    states = torch.zeros(2, H, d, e, device=where[0])
    with torch.no_grad():
        got = ops.hgrn2(_t(where, proj), lead, lead + n, lead + 2 * n, H, d, e, *[_t(where, t) for t in (bias, lower, weight)], 1e-9,
                        torch.tensor([0, T], dtype=torch.int32, device=where[0]), T, _View(states, torch.ones(T, dtype=torch.int32, device=where[0]), False), 0)
    o, S = O.hgrn2_scan(*_hgrn2_want(proj, lead, H, d, e, bias, lower))
    assert rel(states[1], S) < 5e-5 and torch.isfinite(got).all()
    if shift < 30:
        assert worst_row(got, O.norm(o, weight, 1e-9).flatten(1)) < 3 * tol(where)


@pytest.mark.gpu
def test_rows_that_fill_up_a_batch_leave_states_alone():
    from twinkle_b200 import ops
    proj, lead, bias, lower, weight = _hgrn2_case(2, 16, 24, 3, 1)
    states = torch.ones(3, 2, 16, 24, device='cuda')
    slots = torch.tensor([0, 2, 0], dtype=torch.int32, device='cuda')
    o = ops.hgrn2(proj.float().cuda(), lead, lead + 32, lead + 64, 2, 16, 24, bias.float().cuda(), lower.float().cuda(), weight.float().cuda(), 1e-5,
                  view=_View(states, slots, True), layer=0)
    assert not o[[0, 2]].any() and o[1].any()
    assert bool((states[:2] == 1).all()) and not bool((states[2] == 1).all())


@BACKENDS
@pytest.mark.parametrize('nq,nc', [(9, 13), (56, 48), (40, 0), (1536, 512), (24, 7)])
def test_latent_norms_and_cache_rows(where, nq, nc):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(nq)
    T, q0 = 7, 3 if nq % 2 else 8
    proj, wq, wc = _rand(G, T, q0 + nq + nc + 4), _rand(G, nq), _rand(G, max(nc, 1))
    pool = torch.full((6, 4, 1, -(-nc // 8) * 8), 5.0, device=where[0], dtype=getattr(torch, where[1])) if nc else None
    rows = torch.tensor([9, 4, 20, 23, 5, 11, 7], device=where[0])
    view = type('V', (), {'cache': type('C', (), {'k': [pool]})(), 'rows': rows})()
    with torch.no_grad():
        q, c = ops.latent_norms(_t(where, proj), q0, nq, _t(where, wq), q0 + nq, nc, _t(where, wc) if nc else None, 1e-3, view, 0)
    assert rel(q, O.norm(proj[:, q0:q0 + nq], wq, 1e-3)) < tol(where) / 4
    if nc:
        want = O.norm(proj[:, q0 + nq:q0 + nq + nc], wc, 1e-3)
        assert rel(c[:, :nc], want) < tol(where) / 4 and not c[:, nc:].any()
        flat = pool.view(24, -1)
        assert torch.equal(flat[rows], c)                                         # the cache holds what prompts attend over
        left = torch.ones(24, dtype=torch.bool)
        left[rows.cpu()] = False
        assert bool((flat[left.to(where[0])] == 5).all())


def _sink_attention(q, k, v, scale, sink, gate):
    """One sequence, ``q [T, H, d]``, ``k [T, H, d]``, ``v [T, H, e]``."""
    out = torch.zeros(*q.shape[:2], v.shape[-1], dtype=torch.float64)
    for h in range(q.shape[1]):
        s = q[:, h] @ k[:, h].t() * scale
        for i in range(q.shape[0]):
            top = torch.maximum(s[i, :i + 1].max(), sink[h])
            p = torch.exp(s[i, :i + 1] - top)
            out[i, h] = p / (p.sum() + torch.exp(sink[h] - top)) @ v[:i + 1, h]
    return out * O.sigmoid(gate)[..., None]


@BACKENDS
@pytest.mark.parametrize('H,d,e', [(3, 24, 40), (4, 64, 64), (2, 72, 128), (2, 128, 56), (3, 7, 11), (1, 160, 256)])
def test_packed_attention_with_sinks_and_gates(where, H, d, e):
    """Keys and values as column ranges of one product; sinks that weigh nothing, something and nearly everything."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d + e)
    lens = [1, 31, 130, 64]
    _, cu = _packed(lens)
    T = sum(lens)
    q, kv, gate = _rand(G, T, H, d), _rand(G, T, H * (d + e)), _rand(G, T, H + 5)
    k, v = kv[:, :H * d].view(T, H, d), kv[:, H * d:].view(T, H, e)
    sink = torch.tensor([-30.0, 3.0, 9.0, 40.0][:H]).bfloat16().double()
    kvt = _t(where, kv)
    with torch.no_grad():
        got = ops.attention_packed(_t(where, q), kvt[:, :H * d].view(T, H, d), kvt[:, H * d:].view(T, H, e), cu.to(where[0]), max(lens), 0.21, _t(where, sink),
                                   _t(where, gate)[:, 2:2 + H])
    assert got.shape == (T, H, e)
    for a, b in zip(cu[:-1], cu[1:]):
        want = _sink_attention(q[a:b], k[a:b], v[a:b], 0.21, sink, gate[a:b, 2:2 + H])
        err = (got[a:b].double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)
        assert float(err.max()) < 2 * tol(where)


@BACKENDS
@pytest.mark.parametrize('H,R,bs', [(3, 13, 4), (5, 48, 16), (16, 64, 16), (4, 264, 16), (32, 512, 16), (20, 512, 32), (128, 128, 64), (8, 1000, 16), (7, 96, 128)])
def test_latent_decode(where, H, R, bs):
    """Contexts of one token, around a page's border, over several tiles; one score stands out at a page's edge."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(R + H)
    lens = [1, bs - 1, bs, bs + 1, 333, 0, 127, 128, 129, 1500]
    need = sum(-(-n // bs) for n in lens) + 1
    order = (torch.randperm(need, generator=G) + 1).tolist()
    pool = _rand(G, need + 1, bs, 1, -(-R // 8) * 8)
    pool[..., R:] = 0
    table = torch.zeros(len(lens), -(-max(lens) // bs) + 1, dtype=torch.int32)
    for i, n in enumerate(lens):
        for j in range(-(-n // bs)):
            table[i, j] = order.pop()
    q, sink, gate = _rand(G, len(lens), H, R), (2 + _rand(G, H)).bfloat16().double(), _rand(G, len(lens), H + 3)
    scale = 1.5 / R**0.5
    for i, n in enumerate(lens):                       # head 0 looks for the last key, head 1 for the one at a page's start
        if n:
            q[i, 0] = pool[table[i, (n - 1) // bs], (n - 1) % bs, 0, :R]
            q[i, 1 % H] = pool[table[i, (n - 1) // bs], 0, 0, :R]
    with torch.no_grad():
        got = ops.latent_decode(_t(where, q), _t(where, pool), table.to(where[0]), torch.tensor(lens, dtype=torch.int32, device=where[0]), scale, _t(where, sink),
                                _t(where, gate)[:, 1:1 + H])
    assert got.shape == (len(lens), H, R) and not got[lens.index(0)].any()
    for i, n in enumerate(lens):
        if n:
            c = torch.stack([pool[table[i, p // bs], p % bs, 0, :R] for p in range(n)])
            s = q[i] @ c.t() * scale
            top = torch.maximum(s.max(-1).values, sink)
            p = torch.exp(s - top[:, None])
            want = p @ c / (p.sum(-1) + torch.exp(sink - top))[:, None] * O.sigmoid(gate[i, 1:1 + H])[:, None]
            assert worst_row(got[i], want) < 2 * tol(where), n


@BACKENDS
@pytest.mark.parametrize('B,H,K,N', [(1, 3, 24, 40), (5, 4, 64, 512), (130, 2, 40, 264), (3, 5, 7, 11), (70, 8, 128, 128)])
def test_product_per_head(where, B, H, K, N):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(B)
    x, w = _rand(G, B, H, K), _rand(G, H, N, K)
    with torch.no_grad():
        got = ops.head_linear(_t(where, x), _t(where, w))
        got_t = ops.head_linear(_t(where, x), _t(where, w.transpose(1, 2).contiguous()), transposed=True)
    want = torch.einsum('bhk,hnk->bhn', x, w)
    assert rel(got, want) < tol(where) / 2 and rel(got_t, want) < tol(where) / 2


@BACKENDS
@pytest.mark.parametrize('E,k,T,width,ff', [(1, 1, 3, 24, 16), (6, 2, 1, 96, 32), (5, 5, 40, 52, 20), (12, 4, 300, 64, 48), (100, 8, 64, 128, 264), (256, 32, 70, 40, 8)])
def test_experts(where, E, k, T, width, ff):
    """Choice by logit plus bias, softmax over the chosen, rows grouped by expert, square of relu, weighted sum."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(E)
    h, bias = _rand(G, T, width), _rand(G, E)
    logits = torch.randn(T, E, generator=G) * 3
    up, down = (_rand(G, E, ff, width) / width**0.5).bfloat16().double(), (_rand(G, E, width, ff) / ff**0.5).bfloat16().double()
    want_idx, want_w = O.route(logits.double(), {'router': torch.eye(E, dtype=torch.float64), 'router.b': bias}, k)
    forced = torch.stack([torch.randperm(E, generator=G)[:k] for _ in range(T)])
    forced[0] = -1
    with torch.no_grad():
        w, idx, hist = ops.moe_topk(logits.to(where[0]), _t(where, bias), k)
        assert torch.equal(idx.cpu(), want_idx) and rel(w, want_w) < 1e-5 and hist.tolist() == torch.bincount(want_idx.flatten(), minlength=E).tolist()
        wf, idf, _ = ops.moe_topk(logits.to(where[0]), _t(where, bias), k, forced.to(where[0]))
        assert torch.equal(idf.cpu()[0], want_idx[0]) and torch.equal(idf.cpu()[1:], forced[1:])
        assert rel(wf[1:], torch.softmax((logits.double() + bias).gather(1, forced.clamp_min(0)), -1)[1:]) < 1e-5 if T > 1 else True
        xs, row_of, offsets = ops.moe_group_rows(_t(where, h), idx, hist)
        assert torch.equal(offsets.cpu().diff(), hist.cpu()) and sorted(row_of.flatten().tolist()) == list(range(T * k))
        assert torch.equal(xs[row_of.long()], _t(where, h)[:, None].expand(T, k, width))
        bounds = offsets.cpu()[idx.cpu()], offsets.cpu()[idx.cpu() + 1]
        assert bool(((row_of.cpu() >= bounds[0]) & (row_of.cpu() < bounds[1])).all())
        a = ops.grouped_gemm(xs, _t(where, up), offsets, act='relu2')
        y = ops.grouped_gemm(a, _t(where, down), offsets)
    got = (y[row_of.long()].double().cpu() * want_w[..., None]).sum(1)
    want = torch.stack([sum(p * O.expert(h[t], up[n], down[n]) for n, p in zip(want_idx[t].tolist(), want_w[t])) for t in range(T)])
    assert worst_row(got, want) < 2 * tol(where)


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
def test_long_prompt(checkpoint, where):
    """Over several time segments, tiles and pages."""
    path, cfg, W = checkpoint('mixed')
    tokens = ids(520, cfg['vocab'], 3)
    agrees(run_one(replay(path, where), 'r', tokens, 517), cfg, W, tokens, where)


@BACKENDS
def test_residual_stream_after_every_layer(checkpoint, where):
    from twinkle_b200.models.decoder import PackedBatch, Stream
    path, cfg, W = checkpoint('mixed')
    tokens = ids(9, cfg['vocab'], 2)
    _, trail = O.forward(cfg, W, tokens)
    n = int((~close_calls(cfg, W, tokens, 0.08 if where[1] == 'bfloat16' else 1e-4)[1]).sum())
    rp = replay(path, where)
    batch = PackedBatch(torch.tensor(tokens, device=where[0]), torch.arange(9, device=where[0]), torch.tensor([0, 9], dtype=torch.int32, device=where[0]), 9)
    with torch.no_grad():
        st = Stream(rp.model.embed(batch).float())
        for layer, want in zip(rp.model.layers, trail):
            st = layer.advance(st, batch)
            seen = Stream(st.x.clone(), gated=st.gated)
            seen.enter(rp.model.norm)
            assert seen.x.dtype == torch.float32 and n > 2 and worst_row(seen.x[:n], want[:n]) < 2 * tol(where)


@BACKENDS
@pytest.mark.parametrize('name', ['mixed', 'odd'])
def test_batches_of_unequal_requests(checkpoint, where, name):
    """Requests of 1 to 66 tokens in one batch, decoded together, shorter ones ending earlier: each as it is alone."""
    path, cfg, W = checkpoint(name)
    lens = {'a': (66, 9), 'b': (1, 20), 'c': (16, 3), 'd': (3, 12)}
    toks = {n: ids(a + b, cfg['vocab'], 10 + i) for i, (n, (a, b)) in enumerate(lens.items())}
    rp = replay(path, where)
    rows = {n: [t] for n, t in start(rp, {n: toks[n][:a] for n, (a, _) in lens.items()}).items()}
    for step in range(20):
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
def test_freed_pages_and_states_are_used_again(checkpoint, where):
    """A cache of few blocks and slots serves one request after another; what an ended request left does not show."""
    path, cfg, W = checkpoint('mixed')
    rp = replay(path, where, max_tokens=64, block_size=4)
    cache = rp.engine.cache
    blocks, slots = len(cache.free), len(cache.free_slots)
    for i, (n, n_prompt) in enumerate([(60, 50), (9, 1), (40, 2), (5, 1), (64, 64)]):
        tokens = ids(n, cfg['vocab'], 40 + i)
        agrees(run_one(rp, f'r{i}', tokens, n_prompt), cfg, W, tokens, where)
        assert (len(cache.free), len(cache.free_slots)) == (blocks, slots)
    with pytest.raises(RuntimeError, match='exhausted'):
        for i in range(slots + 1):
            start(rp, {f'x{i}': [1]})


@BACKENDS
def test_cache_holds_latents_and_states_only(checkpoint, where):
    path, cfg, W = checkpoint('mixed')
    c = replay(path, where).engine.cache
    for layer, k, v, s in zip(cfg['layers'], c.k, c.v, c.state):
        m = layer['mixer']
        own = layer['type'] == 'latent_attention' and 'kv_from' not in m
        assert v is None and (k is not None) == own and (s is not None) == (layer['type'] == 'hgrn2')
        assert k is None or tuple(k.shape[2:]) == (1, -(-m['kv_rank'] // 8) * 8)
        assert s is None or (s.dtype == torch.float32 and tuple(s.shape[1:]) == (m['heads'], m['dim'], m['vdim']))


@BACKENDS
def test_long_decoding_over_page_borders(checkpoint, where):
    path, cfg, W = checkpoint('mixed')
    tokens = ids(203, cfg['vocab'], 7)
    agrees(run_one(replay(path, where, block_size=8), 'r', tokens, 2), cfg, W, tokens, where)


def _asking_model(borrow):
    """Latent attention in which token 299 looks for token 298 and for little else: one far key's share shows.  With ``borrow`` the
    layer that looks is a second one, on the latents of the first."""
    layers = [O.latents(4, 40, 24, 48, 48, 0.5)] + ([O.latents(4, 40, 24, 48, 48, 0.5, kv_from=0)] if borrow else [])
    cfg = dict(architecture='Moronex', vocab=300, width=96, norm={'eps': 1e-5}, layers=layers)
    W = O.random_weights(cfg, 3)
    M = torch.randn(48, 48, generator=torch.Generator().manual_seed(1)).bfloat16() / 7
    last = f'l{len(layers) - 1}.'
    zero = torch.zeros(48, 48, dtype=torch.bfloat16)
    W['l0.mix.dkv'], W[last + 'mix.dq'] = torch.cat([zero, M], 1), torch.cat([M, zero], 1)       # keys from one half of the stream, queries from the other
    W[last + 'mix.dq.norm'] = W['l0.mix.dkv.norm'].clone()
    W[last + 'mix.uq'] = W[last + 'mix.uk'].clone()
    W['embed'][299, :48] = W['embed'][298, 48:]
    W['l0.norm1'], W[last + 'norm1'] = torch.zeros(96).bfloat16(), torch.zeros(96).bfloat16()
    if borrow:                                          # the first layer adds little, so that the second still recognises the tokens
        W['l0.norm1b'] = torch.full((96, ), -0.95).bfloat16()
    return cfg, W


@BACKENDS
@pytest.mark.parametrize('borrow', [False, True])
def test_far_keys_and_page_borders(tmp_path, where, borrow):
    """What the last token looks for stands at the first places, around page borders, in the middle.  Asked for in the prompt and
    in decoding; putting another token there changes the logits far beyond the tolerance."""
    cfg, W = _asking_model(borrow)
    path = O.write_checkpoint(tmp_path / 'm', cfg, W)
    rp = replay(path, where)
    n = 300
    for at in (0, 1, 15, 16, 17, 127, 128, 200):
        base = ids(n, 297, at)
        base[-1] = 299
        seen, unseen = list(base), list(base)
        seen[at], unseen[at] = 298, 297
        want, other = O.forward(cfg, W, seen)[0][-1], O.forward(cfg, W, unseen)[0][-1]
        assert rel(other, want) > 0.15                                        # the far key matters …
        for n_prompt in (n, n - 1, n - 3):
            assert rel(run_one(rp, 'r', seen, n_prompt)[-1], want) < 2 * tol(where), (at, n_prompt)     # … and is found


@BACKENDS
def test_far_writes_stay_in_the_state(tmp_path, where):
    """Tokens 298 and 299 open every gate and overwrite the state, all others leave it nearly alone: which of the two came last is seen
    hundreds of tokens later, over segments and steps."""
    cfg = dict(architecture='Moronex', vocab=300, width=80, norm={'eps': 1e-5}, layers=[O.recurrent(2, 24, 40)])
    W = O.random_weights(cfg, 4)
    W['embed'][:, 0] = 0
    W['embed'][298:, 0] = 8
    W['l0.norm1'][0] = 0
    W['l0.mix.f'] = torch.zeros_like(W['l0.mix.f'])
    W['l0.mix.f'][:, 0] = -6
    W['l0.mix.f.b'], W['l0.mix.lower'] = torch.full((48, ), 8.0).bfloat16(), torch.zeros(48).bfloat16()
    path = O.write_checkpoint(tmp_path / 'm', cfg, W)
    rp = replay(path, where)
    n = 300
    for at in (0, 1, 15, 16, 17, 127, 128, 143, 250):
        one, two = ids(n, 297, at), ids(n, 297, at)
        one[at], two[at] = 298, 299
        want, other = O.forward(cfg, W, one)[0][-1], O.forward(cfg, W, two)[0][-1]
        assert rel(other, want) > 0.15
        for n_prompt in (n, n - 1, max(at, 1), at + 1):
            assert rel(run_one(rp, 'r', one, n_prompt)[-1], want) < 2 * tol(where), (at, n_prompt)


@BACKENDS
def test_first_tokens(checkpoint, where):
    path, cfg, W = checkpoint('mixed')
    rp = replay(path, where)
    for n in (1, 2, 3, 4):
        tokens = ids(n, cfg['vocab'], 90 + n)
        agrees(run_one(rp, 'r', tokens, n), cfg, W, tokens, where)
        agrees(run_one(rp, 'r', tokens, 1), cfg, W, tokens, where)


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
        lg, near = close_calls(cfg, W, p + got, 0.08 if where[1] == 'bfloat16' else 1e-4)
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
        assert DecoderConfig.from_hf(c.to_hf()) == c and c.model_type == 'moronex'
        m = TransformersModel(model_id=path, device='cpu')
        assert sum(p.numel() for p in m.model.parameters()) == c.num_params() == sum(t.numel() for t in W.values())
        out = m.save('ckpt', output_dir=str(tmp_path / name))
        back = load_file(os.path.join(out, 'model.safetensors'))
        assert set(back) == set(W) and all(torch.equal(back[n].float(), W[n].float()) and back[n].shape == W[n].shape for n in W)
        with open(os.path.join(out, 'config.json')) as f:
            assert DecoderConfig.from_hf(json.load(f)) == c
    assert preset('tiny-moronex', num_hidden_layers=3).num_hidden_layers == 3
    for change in (('type', 'something'), ('mlp', {'kind': 'something'})):
        bad = json.loads(json.dumps(O.CONFIGS['mixed']))
        bad['layers'][0][change[0]] = change[1]
        with pytest.raises(NotImplementedError):
            DecoderConfig.from_hf(bad)
    for source, rank in ((4, 48), (0, 48), (3, 48), (1, 40), (6, 48)):      # another rank, no latents, borrowed ones, a wrong rank, not earlier
        bad = json.loads(json.dumps(O.CONFIGS['mixed']))
        bad['layers'][6]['mixer'].update(kv_from=source, kv_rank=rank)
        with pytest.raises(ValueError, match='kv_from'):
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
    tokens = ids(19, cfg['vocab'], 5)
    hidden = model(PackedBatch(torch.tensor(tokens), torch.arange(19), torch.tensor([0, 19], dtype=torch.int32), 19))
    loss = torch.nn.functional.cross_entropy(model.logits(hidden)[:-1], torch.tensor(tokens[1:]))
    loss.backward()
    names = dict(model.named_parameters())

    def oracle_loss(name, delta):
        V = {n: t.double() for n, t in W.items()}
        V[name] = V[name] + delta
        return float(torch.nn.functional.cross_entropy(O.forward(cfg, V, tokens)[0][:-1], torch.tensor(tokens[1:])))

    G = torch.Generator().manual_seed(1)
    w = cfg['width']
    for hf, internal, rows in (('l0.mix.f', 'layers.0.mixer.in_proj.weight', slice(w + 72, w + 144)), ('l0.mix.lower', 'layers.0.mixer.lower', slice(None)),
                               ('l2.mix.f.b', 'layers.2.mixer.f_bias', slice(None)), ('l1.mix.dkv', 'layers.1.mixer.in_proj.weight', slice(w + 56, w + 104)),
                               ('l1.mix.sink', 'layers.1.mixer.sinks', slice(None)), ('l3.mix.uk', 'layers.3.mixer.kv_up', slice(0, 80)),
                               ('l6.mix.g', 'layers.6.mixer.in_proj.weight', slice(w + 40, None)), ('l3.rg2', 'layers.3.mlp_gate.weight', slice(None)),
                               ('l1.norm1b', 'layers.1.post_mixer_layernorm.weight', slice(None)), ('l0.rg2.b', 'layers.0.mlp_gate_bias', slice(None)),
                               ('l5.mlp.router', 'layers.5.mlp.gate.weight', slice(None)), ('head', 'lm_head.weight', slice(None))):
        direction = torch.randn(W[hf].shape, generator=G).double()
        fd = (oracle_loss(hf, 1e-5 * direction) - oracle_loss(hf, -1e-5 * direction)) / 2e-5
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
    for i, n in enumerate((33, 20)):
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
    m = TransformersModel(model_id='tiny-moronex', device='cpu', max_loras=1, max_r=4)
    m.add_adapter_to_model('a', LoraConfig(r=4, lora_alpha=8, target_modules=['q_proj', 'dq_proj', 'up_proj', 'o_proj', 'up', 'down']))
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
