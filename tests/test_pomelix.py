"""Pomelix stacks (layers listed one by one: short convolution in front of attention, unit-rms q and k, query temperature,
value mixing, mixer and feed-forward side by side on a 32-bit stream) against ``tests/pomelix_oracle.py``.

Every case runs on the CPU in fp32 and, marked ``gpu``, on the kernels in fp32 and bf16."""
import json
import os

import pytest
import torch

from tests import pomelix_oracle as O

WHERE = [pytest.param(('cpu', 'float32'), id='cpu'), pytest.param(('cuda', 'float32'), id='cuda32', marks=pytest.mark.gpu),
         pytest.param(('cuda', 'bfloat16'), id='cuda16', marks=pytest.mark.gpu)]
BACKENDS = pytest.mark.parametrize('where', WHERE)


def tol(where):
    return 2e-2 if where[1] == 'bfloat16' else 3e-5


def rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-12))


def worst_row(a, b):
    """Largest error of a row relative to the typical size of a row."""
    a, b = a.double().cpu(), b.double().cpu()
    return float(((a - b).norm(dim=-1) / b.norm(dim=-1).mean()).max())


def ids(n, vocab, seed):
    return torch.randint(0, vocab, (n, ), generator=torch.Generator().manual_seed(seed)).tolist()


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


def replay(path, where, max_tokens=2048, block_size=16):
    from twinkle_b200.cli.trace_run import TraceReplay
    return TraceReplay(path, where[1], max_tokens, where[0], block_size)


def start(rp, reqs):
    """All logits of several prompts run as one batch, per request."""
    out = rp.step([{'id': n, 'tokens': t, 'want': list(range(len(t)))} for n, t in reqs.items()])
    return dict(zip(reqs, out.split([len(t) for t in reqs.values()])))


def go_on(rp, reqs):
    out = rp.step([{'id': n, 'tokens': [t], 'want': [0]} for n, t in reqs.items()])
    return dict(zip(reqs, out))


def run_one(rp, name, tokens, n_prompt):
    rows = [start(rp, {name: tokens[:n_prompt]})[name]] + [go_on(rp, {name: t})[name][None] for t in tokens[n_prompt:]]
    rp.end([name])
    return torch.cat(rows)


# ------------------------------------------------------------------------------------------------ mechanisms
def _t(where, x):
    return x.to(where[0], getattr(torch, where[1]))


def _packed(lens):
    return torch.cat([torch.arange(n) for n in lens]), torch.tensor([0] + lens).cumsum(0).to(torch.int32)


@BACKENDS
@pytest.mark.parametrize('taps,d,e', [(0, 16, 16), (1, 24, 8), (2, 16, 40), (3, 20, 12), (4, 128, 136), (5, 10, 7), (4, 256, 64)])
def test_convolution_norm_temperature_and_mixing(where, taps, d, e):
    """The fused step between projection and attention, on packed prompts (some shorter than the filter)."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(taps * 100 + d)
    hq, hkv, eps, coef, every, lens = 6, 2, 1e-3, 0.5, 4, [1, 9, 2, 33]
    pos, cu = _packed(lens)
    C, T = (hq + hkv) * d + hkv * e, sum(lens)
    proj = torch.randn(T, C + 24, generator=G).bfloat16().float()
    w = torch.randn(C, taps, generator=G).bfloat16().float() if taps else None
    vf, lam = torch.randn(T, hkv, e, generator=G).bfloat16().float(), torch.tensor([0.375])
    with torch.no_grad():
        q, k, v = ops.conv_heads(_t(where, proj), None if w is None else _t(where, w), pos.to(where[0]), hq, hkv, d, e, eps, coef, every,
                                 _t(where, vf), _t(where, lam))
    for got, n in ((q, d), (k, d), (v, e)):      # rows are filled up to whole vectors with zeros
        assert got.shape[-1] == -(-n // 8) * 8 and not got[..., n:].any()
    for a, b in zip(cu[:-1], cu[1:]):
        u = proj[a:b, :C].double()
        y = O.causal_conv(u, w.double()) if taps else u
        n = int(b - a)
        eq, ek, ev = y[:, :hq * d].view(n, hq, d), y[:, hq * d:(hq + hkv) * d].view(n, hkv, d), y[:, (hq + hkv) * d:].view(n, hkv, e)
        temp = torch.tensor([O.query_temperature(p, coef, every) for p in range(n)], dtype=torch.float64)
        assert rel(q[a:b, :, :d], O.rms(eq, eps) * temp[:, None, None]) < tol(where) / 4
        assert rel(k[a:b, :, :d], O.rms(ek, eps)) < tol(where) / 4
        assert rel(v[a:b, :, :e], O.mix_values(ev, vf[a:b].double(), 0.375)) < tol(where) / 4


@BACKENDS
def test_temperature_changes_exactly_at_its_steps(where):
    from twinkle_b200 import ops
    pos = torch.tensor([0, 1, 5, 6, 7, 13, 14, 6999999, 7000000 - 2, 7000000 - 1])
    for every in (1, 7):
        one = torch.ones(len(pos), 8 * 3)
        with torch.no_grad():
            q, _, _ = ops.conv_heads(_t(where, one), None, pos.to(where[0]), 1, 1, 8, 8, 1e-9, 0.5, every)
        want = torch.tensor([O.query_temperature(int(p), 0.5, every) for p in pos])
        assert torch.allclose(q[:, 0, 0].float().cpu(), want, rtol=4e-3 if where[1] == 'bfloat16' else 1e-6)


@BACKENDS
@pytest.mark.parametrize('hq,hkv,d,e', [(4, 1, 24, 40), (3, 3, 64, 64), (6, 2, 72, 128), (2, 1, 128, 56), (10, 2, 16, 8), (2, 1, 160, 256)])
def test_packed_attention(where, hq, hkv, d, e):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d + e)
    lens = [1, 31, 130, 64]
    _, cu = _packed(lens)
    q, k, v = (torch.randn(sum(lens), h, n, generator=G).bfloat16().double() for h, n in ((hq, d), (hkv, d), (hkv, e)))
    with torch.no_grad():
        got = ops.attention_packed(_t(where, q), _t(where, k), _t(where, v), cu.to(where[0]), max(lens), 0.21)
    assert got.shape == (sum(lens), hq, e)
    for a, b in zip(cu[:-1], cu[1:]):
        assert worst_row(got[a:b].flatten(1), O.attention(q[a:b], k[a:b], v[a:b], 0.21).flatten(1)) < tol(where)


@BACKENDS
@pytest.mark.parametrize('hq,hkv,d,e,bs', [(4, 1, 24, 40, 16), (3, 1, 64, 64, 4), (6, 2, 72, 128, 16), (5, 1, 128, 56, 8), (8, 8, 16, 8, 16), (8, 1, 160, 256, 16)])
def test_paged_decode_attention(where, hq, hkv, d, e, bs):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(d * e)
    lens = [1, bs - 1, bs, bs + 1, 77, 0]
    blocks = torch.randperm(64, generator=G)
    table, free = torch.zeros(len(lens), 32, dtype=torch.int32), iter(blocks.tolist())
    kc, vc = torch.randn(64, bs, hkv, d, generator=G).bfloat16().double(), torch.randn(64, bs, hkv, e, generator=G).bfloat16().double()
    for i, n in enumerate(lens):
        for j in range(-(-n // bs)):
            table[i, j] = next(free)
    q = torch.randn(len(lens), hq, d, generator=G).bfloat16().double()
    with torch.no_grad():
        got = ops.paged_attention_decode(_t(where, q), _t(where, kc), _t(where, vc), table.to(where[0]), torch.tensor(lens, dtype=torch.int32, device=where[0]), 0.3)
    assert got.shape == (len(lens), hq, e) and not got[-1].any()
    for i, n in enumerate(lens[:-1]):
        k = torch.stack([kc[table[i, p // bs], p % bs] for p in range(n)])
        v = torch.stack([vc[table[i, p // bs], p % bs] for p in range(n)])
        want = O.attention(q[i:i + 1].expand(n, -1, -1), k, v, 0.3)[-1]          # the last row sees every key
        assert rel(got[i], want) < tol(where)


@BACKENDS
@pytest.mark.parametrize('width', [52, 64, 70, 2304, 4608, 8200])
def test_stream_update_and_norm(where, width):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(width)
    x = torch.randn(5, width, generator=G)
    y1, y2 = (torch.randn(5, width, generator=G).bfloat16() for _ in range(2))
    s1, s2, w = (torch.randn(width, generator=G).bfloat16() for _ in range(3))
    for adds in ((), ((y1, s1), ), ((y1, s1), (y2, s2))):
        want = x.double() + 0.7 * sum(y.double() * s.double() for y, s in adds)
        with torch.no_grad():
            h, nx = ops.stream_rmsnorm(x.to(where[0]).clone(), _t(where, w), 1e-4, [(_t(where, y), _t(where, s)) for y, s in adds], 0.7)
        assert nx.dtype == torch.float32 and rel(nx, want) < 1e-6          # the stream itself is never rounded
        assert h.dtype == w.to(getattr(torch, where[1])).dtype and rel(h, O.rms_norm(want, w.double(), 1e-4)) < tol(where) / 4


@BACKENDS
def test_gated_columns(where):
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(5)
    for n, gate, up, I in ((100, 20, 60, 36), (256, 64, 160, 96)):
        p = torch.randn(7, n, generator=G).bfloat16().double() * 4
        z, u = p[:, gate:gate + I], p[:, up:up + I]
        with torch.no_grad():
            assert rel(ops.glu_columns(_t(where, p), gate, up, I), z * torch.sigmoid(z) * u) < tol(where) / 4


# ------------------------------------------------------------------------------------------------ whole models
@BACKENDS
@pytest.mark.parametrize('name', list(O.CONFIGS))
def test_prompt_and_token_by_token(checkpoint, where, name):
    """A prompt at once, a prompt cut after 1 / 2 / 40 tokens and continued by single steps: all as the oracle has it."""
    path, cfg, W = checkpoint(name)
    tokens = ids(70, cfg['vocab'], 1)
    want, _ = O.forward(cfg, W, tokens)
    rp = replay(path, where)
    for n_prompt in (70, 1, 2, 40):
        assert worst_row(run_one(rp, 'r', tokens, n_prompt), want) < 2 * tol(where), n_prompt


@BACKENDS
def test_residual_stream_after_every_layer(checkpoint, where):
    from twinkle_b200 import ops
    from twinkle_b200.models.decoder import PackedBatch, Stream
    path, cfg, W = checkpoint('mixed')
    tokens = ids(37, cfg['vocab'], 2)
    _, trail = O.forward(cfg, W, tokens)
    rp = replay(path, where)
    batch = PackedBatch(torch.tensor(tokens, device=where[0]), torch.arange(37, device=where[0]), torch.tensor([0, 37], dtype=torch.int32, device=where[0]), 37)
    with torch.no_grad():
        st = Stream(rp.model.embed(batch).float())
        for layer, want in zip(rp.model.layers, trail):
            st = layer.advance(st, batch)
            x = ops.stream_rmsnorm(st.x.clone(), rp.model.norm.weight, 1e-5, st.adds, cfg['residual_mult'])[1]
            assert worst_row(x, want) < tol(where)


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
            rows[n].append(r[None])
        rp.end([n for n, (_, b) in lens.items() if step == b - 1])
    assert not rp.live
    for n in lens:
        assert worst_row(torch.cat(rows[n]), O.forward(cfg, W, toks[n])[0]) < 2 * tol(where), n


@BACKENDS
def test_freed_pages_and_history_are_used_again(checkpoint, where):
    """A cache of few blocks and slots serves one request after another; what an ended request left does not show, also when
    the next one is shorter than the convolution."""
    path, cfg, W = checkpoint('mixed')
    rp = replay(path, where, max_tokens=64, block_size=4)
    cache = rp.engine.cache
    blocks, slots = len(cache.free), len(cache.free_slots)
    for i, (n, n_prompt) in enumerate([(60, 50), (9, 1), (40, 2), (5, 1), (64, 64)]):
        tokens = ids(n, cfg['vocab'], 40 + i)
        assert worst_row(run_one(rp, f'r{i}', tokens, n_prompt), O.forward(cfg, W, tokens)[0]) < 2 * tol(where), i
        assert (len(cache.free), len(cache.free_slots)) == (blocks, slots)
    with pytest.raises(RuntimeError, match='exhausted'):
        for i in range(slots + 1):
            start(rp, {f'x{i}': [1]})


@BACKENDS
def test_long_decoding_over_page_borders(checkpoint, where):
    path, cfg, W = checkpoint('mixed')
    tokens = ids(203, cfg['vocab'], 7)
    got = run_one(replay(path, where, block_size=8), 'r', tokens, 2)
    assert worst_row(got, O.forward(cfg, W, tokens)[0]) < 2 * tol(where)


def _match_model():
    """One layer in which a token's query fits the keys of its own token and little else: the share of one far key shows."""
    cfg = dict(architecture='Pomelix', vocab=300, width=80, norm={'eps': 1e-5}, residual_mult=1.0,
               layers=[O.spec(4, 2, 40, 24, 3, 0.5, False, (0.2, 50))])
    W = O.random_weights(cfg, 3)
    k = W['l0.mix.k'].view(2, 1, 40, 80)
    W['l0.mix.q'] = k.expand(2, 2, 40, 80).reshape(160, 80).contiguous()        # query heads of a group look for what its key head shows
    for n in ('q', 'k'):
        W[f'l0.mix.{n}.conv'] = torch.tensor([0.05, 0.1, 1.0]).expand(W[f'l0.mix.{n}.conv'].shape[0], 3).bfloat16()
    return cfg, W


@BACKENDS
def test_far_keys_and_page_borders(tmp_path, where):
    """The last token occurs once before: at the first places, around page borders, in the middle.  Asked for in the prompt
    and in decoding; moving the earlier occurrence to another token changes the logits far beyond the tolerance."""
    cfg, W = _match_model()
    path = O.write_checkpoint(tmp_path / 'm', cfg, W)
    rp = replay(path, where)
    n, special = 300, 299
    for at in (0, 1, 2, 15, 16, 17, 127, 128, 129, 200):
        base = ids(n, 298, at)
        base[-1] = special
        seen, unseen = list(base), list(base)
        seen[at], unseen[at] = special, 298
        want, other = O.forward(cfg, W, seen)[0][-1], O.forward(cfg, W, unseen)[0][-1]
        assert rel(other, want) > 0.15                                        # the far key matters …
        for n_prompt in (n, n - 1, n - 3):
            assert rel(run_one(rp, 'r', seen, n_prompt)[-1], want) < 2 * tol(where), (at, n_prompt)     # … and is found


@BACKENDS
def test_first_tokens_and_convolution_edges(checkpoint, where):
    """A token reaches the convolution of exactly the next ``taps − 1`` places; nothing precedes the first token."""
    from twinkle_b200 import ops
    G = torch.Generator().manual_seed(0)
    d = 8
    for taps in (2, 3, 4, 6):
        w = torch.rand(3 * d, taps, generator=G).bfloat16().float() + 1
        u = torch.randn(12, 3 * d, generator=G).bfloat16().float()
        u2 = u.clone()
        u2[5] += 3
        with torch.no_grad():
            run = lambda x: ops.conv_heads(_t(where, x), _t(where, w), torch.arange(12, device=where[0]), 1, 1, d, d, 1e-5)[2]  # noqa: E731
            changed = (run(u) != run(u2)).flatten(1).any(1).tolist()
        assert changed == [5 <= t < 5 + taps for t in range(12)]
    path, cfg, W = checkpoint('mixed')
    rp = replay(path, where)
    for n in (1, 2, 3, 4):
        tokens = ids(n, cfg['vocab'], 90 + n)
        assert worst_row(run_one(rp, 'r', tokens, n), O.forward(cfg, W, tokens)[0]) < 2 * tol(where)


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
        seq, got = list(p), r.sequences[0].tokens
        assert len(got) == 10
        for t in got:
            lg = O.forward(cfg, W, seq)[0][-1]
            assert float(lg.max() - lg[t]) <= (0.05 if where[1] == 'bfloat16' else 1e-4) * float(lg.std())    # the best, up to a tie within rounding
            seq.append(t)
    scored = s.sample([{'input_ids': prompts[2]}], SamplingParams(max_tokens=0, prompt_logprobs=0))[0].prompt_logprobs
    lp = torch.log_softmax(O.forward(cfg, W, prompts[2])[0], -1)
    want = torch.tensor([float(lp[i, t]) for i, t in enumerate(prompts[2][1:])])
    assert float((torch.tensor(scored[1:]) - want).abs().max()) < tol(where) * 2 * float(lp.std())
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
        assert DecoderConfig.from_hf(c.to_hf()) == c and c.model_type == 'pomelix'
        m = TransformersModel(model_id=path, device='cpu')
        assert sum(p.numel() for p in m.model.parameters()) == c.num_params() == sum(t.numel() for t in W.values())
        out = m.save('ckpt', output_dir=str(tmp_path / name))
        back = load_file(os.path.join(out, 'model.safetensors'))
        assert set(back) == set(W) and all(torch.equal(back[n].float(), W[n].float()) and back[n].shape == W[n].shape for n in W)
        with open(os.path.join(out, 'config.json')) as f:
            assert DecoderConfig.from_hf(json.load(f)) == c
    assert preset('tiny-pomelix', num_hidden_layers=5).num_hidden_layers == 5
    bad = json.loads(json.dumps(O.CONFIGS['mixed']))
    bad['layers'][0]['type'] = 'something'
    with pytest.raises(NotImplementedError):
        DecoderConfig.from_hf(bad)


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
    assert abs(losses[0] - want / count) < (3e-2 if where[1] == 'bfloat16' else 1e-4), (losses, want / count)
    assert losses[-1] < losses[0] - 0.1, losses


def test_gradients_reach_every_weight(checkpoint):
    """Autograd through a stack of such layers against finite differences of the oracle's loss."""
    from twinkle_b200.models.config import DecoderConfig
    from twinkle_b200.models.decoder import PackedBatch, build_model
    from twinkle_b200.models.bridge import hf_to_internal
    path, cfg, W = checkpoint('mixed')
    c = DecoderConfig.from_pretrained(path)
    model = build_model(c, init=False)
    with torch.no_grad():
        for n, p in model.named_parameters():
            p.copy_(hf_to_internal(n, c, W.__getitem__).float())
    tokens = ids(11, cfg['vocab'], 5)
    hidden = model(PackedBatch(torch.tensor(tokens), torch.arange(11), torch.tensor([0, 11], dtype=torch.int32), 11))
    z = model.logits(hidden)
    loss = torch.nn.functional.cross_entropy(z[:-1], torch.tensor(tokens[1:]))
    loss.backward()
    names = dict(model.named_parameters())

    def oracle_loss(name, delta):
        V = {n: t.double() for n, t in W.items()}
        V[name] = V[name] + delta
        return float(torch.nn.functional.cross_entropy(O.forward(cfg, V, tokens)[0][:-1], torch.tensor(tokens[1:])))

    G = torch.Generator().manual_seed(1)
    for hf, internal, rows in (('l1.mix.v', 'layers.1.in_proj.weight', slice(4 * 32 + 4 * 32, None)), ('l0.mix.q.conv', 'layers.0.conv_weight', slice(0, 144)),
                               ('l2.mix.vmix', 'layers.2.v_lambda', slice(None)), ('l2.ls1', 'layers.2.mixer_scale', slice(None)),
                               ('l0.mlp.down', 'layers.0.down_proj.weight', slice(None)), ('l0.norm1', 'layers.0.input_layernorm.weight', slice(None))):
        direction = torch.randn(W[hf].shape, generator=G).double()
        fd = (oracle_loss(hf, 1e-4 * direction) - oracle_loss(hf, -1e-4 * direction)) / 2e-4
        ad = float((names[internal].grad[rows].double().reshape(-1) * direction.reshape(-1)).sum())
        assert abs(fd - ad) < 1e-3 * max(1.0, abs(fd)), (hf, fd, ad)
    assert all(p.grad is not None for n, p in names.items() if n != 'layers.1.v_lambda')      # the giving layer's own λ is unused


def test_adapters_apply_to_the_fused_projection():
    from twinkle_b200.model import LoraConfig, TransformersModel
    m = TransformersModel(model_id='tiny-pomelix', device='cpu', max_loras=1, max_r=4)
    m.add_adapter_to_model('a', LoraConfig(r=4, lora_alpha=8, target_modules=['q_proj', 'up_proj', 'o_proj']))
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
    import numpy as np
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / 'out' / f'{n}.f32', dtype='<f4')).view(-1, cfg['vocab'])  # noqa: E731
    wa, wb = O.forward(cfg, W, a)[0], O.forward(cfg, W, b)[0]
    lim = 2 * tol((0, dtype))
    assert worst_row(read(0), torch.stack([wa[0], wa[18], wb[2]])) < lim and worst_row(read(2), wa[20:]) < lim
