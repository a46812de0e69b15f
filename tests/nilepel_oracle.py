"""A plain, slow evaluation of the Nilepel decoder: one function per mechanism, one sequence at a time, whole sequence from its first
token, loops over heads, experts and pairs of dimensions where that is the clearest statement.  It shares no code with the package.

Weights come as a mapping from checkpoint names to tensors; a configuration is the checkpoint's ``config.json`` mapping.
"""
import math

import torch


def norm(x, w, eps):
    """RMS norm with a plain weight over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ------------------------------------------------------------------------------------------------ positions
def frequencies(rot):
    """One angular frequency per rotated pair; long wavelengths slowed down where ``scaling`` asks for it."""
    out = []
    sc = rot.get('scaling')
    for i in range(rot['dims'] // 2):
        f = rot['base'] ** (-2 * i / rot['dims'])
        if sc:
            length = 2 * math.pi / f
            if length > sc['original'] / sc['low']:
                f = f / sc['factor']
            elif length >= sc['original'] / sc['high']:
                mix = (sc['original'] / length - sc['low']) / (sc['high'] - sc['low'])
                f = (1 - mix) * f / sc['factor'] + mix * f
        out.append(f)
    return out


def rotate(x, rot, neighbours, positions=None):
    """``x [T, heads, n]``: the leading ``rot.dims`` dimensions turned by position times frequency.  ``neighbours``: a pair is
    ``(2i, 2i + 1)``, otherwise ``(i, i + dims / 2)``."""
    y, half = x.clone(), rot['dims'] // 2
    p = torch.arange(x.shape[0], dtype=x.dtype) if positions is None else positions.to(x.dtype)
    for i, f in enumerate(frequencies(rot)):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + half)
        c, s = torch.cos(p * f)[:, None], torch.sin(p * f)[:, None]
        y[..., a] = x[..., a] * c - x[..., b] * s
        y[..., b] = x[..., b] * c + x[..., a] * s
    return y


# ------------------------------------------------------------------------------------------------ attention
def seen_in_window(i, size):
    return max(0, i - size + 1)


def seen_in_chunk(i, size):
    return i // size * size


def attend(q, k, v, scale, first, sink=None):
    """One sequence: ``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, e]``; position i sees ``first(i) … i``.  ``sink [H]``: a logit in the
    denominator that belongs to no key."""
    T, H = q.shape[:2]
    j = torch.arange(T)
    seen = (j[None] <= j[:, None]) & (j[None] >= torch.tensor([first(i) for i in range(T)])[:, None])
    out = q.new_zeros(T, H, v.shape[-1])
    for h in range(H):
        g = h // (H // k.shape[1])
        s = (q[:, h] @ k[:, g].t() * scale).masked_fill(~seen, -math.inf)
        top = s.amax(-1) if sink is None else torch.maximum(s.amax(-1), sink[h])
        p = torch.exp(s - top[:, None])
        total = p.sum(-1) if sink is None else p.sum(-1) + torch.exp(sink[h] - top)
        out[:, h] = p @ v[:, g] / total[:, None]
    return out


def heads_of(h, w, name, count, width):
    y = h @ w[name].t()
    if name + '.b' in w:
        y = y + w[name + '.b']
    return y.view(h.shape[0], count, width)


def chunked_keys(h, m, w, eps):
    """What an 'attention' layer keeps: rotated keys and values."""
    return (rotate(heads_of(h, w, 'k', m['kv_heads'], m['dim']), m['rot'], True), heads_of(h, w, 'v', m['kv_heads'], m['vdim']))


def chunked_attention(h, kv, m, w, eps):
    T = h.shape[0]
    q = rotate(heads_of(h, w, 'q', m['heads'], m['dim']), m['rot'], True)
    o = attend(q, *kv, m['scale'], lambda i: seen_in_chunk(i, m['mask']['size']), w['sink'])
    return o.reshape(T, -1) @ w['o'].t()


def windowed_keys(h, m, w, eps):
    """What an 'attention_2' layer keeps: normed and rotated keys, and values."""
    k = norm(heads_of(h, w, 'k', m['kv_heads'], m['dim']), w['k.norm'], eps)
    return rotate(k, m['rot'], False), heads_of(h, w, 'v', m['kv_heads'], m['vdim'])


def windowed_attention(h, kv, m, w, eps):
    T = h.shape[0]
    q = rotate(norm(heads_of(h, w, 'q', m['heads'], m['dim']), w['q.norm'], eps), m['rot'], False)
    o = attend(q, *kv, m['scale'], lambda i: seen_in_window(i, m['mask']['size']), w['sink'])
    return (o * sigmoid(h @ w['g'].t())[:, :, None]).reshape(T, -1) @ w['o'].t()


def latent_keys(h, m, w, eps):
    """What a 'latent_attention' layer keeps: the normed latent and the rotated key part all heads share."""
    c = h @ w['dkv'].t()
    return norm(c[:, :m['kv_rank']], w['dkv.norm'], eps), rotate(c[:, None, m['kv_rank']:], m['rot'], True)[:, 0]


def latent_attention(h, kept, m, w, eps):
    T, H, d, r = h.shape[0], m['heads'], m['dim'], m['rot_dim']
    c, kr = kept
    q = (h @ w['q'].t()).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], m['rot'], True)], -1)
    k = torch.cat([(c @ w['uk'].t()).view(T, H, d), kr[:, None].expand(T, H, r)], -1)
    o = attend(q, k, (c @ w['uv'].t()).view(T, H, m['vdim']), m['scale'], lambda i: seen_in_window(i, m['mask']['size']))
    return o.reshape(T, -1) @ w['o'].t()


MIXERS = {'attention': (chunked_keys, chunked_attention), 'attention_2': (windowed_keys, windowed_attention), 'latent_attention': (latent_keys, latent_attention)}


# ------------------------------------------------------------------------------------------------ feed-forward
def limited_feed_forward(h, w, limit):
    g = torch.clamp(h @ w['gate'].t(), max=limit)
    u = torch.clamp(h @ w['up'].t(), min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w['down'].t()


def expert(x, gate, up, down):
    return (silu(x @ gate.t()) * (x @ up.t())) @ down.t()


def route(z, r):
    """Logits ``[T, experts]`` → chosen experts of every token, best first, and their weights."""
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    idx, share = [], []
    groups = r.get('groups') or {'count': 1, 'keep': 1}
    size = r['experts'] // groups['count']
    for row in s:
        best = sorted(range(groups['count']), key=lambda n: -float(row[n * size:(n + 1) * size].max()))[:groups['keep']]
        allowed = [x for n in best for x in range(n * size, (n + 1) * size)]
        chosen = sorted(allowed, key=lambda x: -float(row[x]))[:r['top']]
        idx.append(chosen)
        share.append(row[chosen] * r.get('scale', 1.0))
    return torch.tensor(idx), torch.stack(share)


def mixture(h, m, w):
    idx, share = route(h @ w['router'].t(), m['router'])
    out = torch.zeros_like(h)
    for n in range(m['router']['experts']):
        p = (share * (idx == n)).sum(-1, keepdim=True)          # 0 for tokens that did not choose it
        out = out + p * expert(h, w[f'e{n}.gate'], w[f'e{n}.up'], w[f'e{n}.down'])
    if m.get('shared'):
        out = out + sigmoid(h @ w['shared.sg'].t()) * expert(h, w['shared.gate'], w['shared.up'], w['shared.down'])
    return out


# ------------------------------------------------------------------------------------------------ the stack
def part(W, prefix):
    return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits ``[T, vocab]`` and the residual stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg['norm']['eps']
    x = W['embed'][torch.as_tensor(tokens)] * cfg['embedding']['scale']
    kept, trail = {}, []
    for i, layer in enumerate(cfg['layers']):
        p, m = f'l{i}.', layer['mixer']
        keys, mixer = MIXERS[layer['type']]
        w = part(W, p + 'mix.')
        h = norm(x, W[p + 'norm1'], eps)
        source = m.get('kv_from')
        if source is None:
            kept[i] = keys(h, m, w, eps)
        x = x + mixer(h, kept[i if source is None else source], m, w, eps)
        f = layer.get('mlp')
        if f:
            h = norm(x, W[p + 'norm2'], eps)
            w = part(W, p + 'mlp.')
            x = x + (mixture(h, f, w) if f['kind'] == 'moe' else limited_feed_forward(h, w, f['limit']))
        trail.append(x)
    return norm(x, W['final.norm'], eps) @ W['head'].t(), trail


# ---------------------------------------------------------------- models for the tests
def rot(dims, base, scaling=None):
    r = {'dims': dims, 'base': base}
    if scaling:
        r['scaling'] = dict(zip(('factor', 'low', 'high', 'original'), scaling))
    return r


def chunked(heads, kv_heads, dim, vdim, scale, size, r, mlp=None):
    return {'type': 'attention', 'mixer': {'heads': heads, 'kv_heads': kv_heads, 'dim': dim, 'vdim': vdim, 'scale': scale, 'mask': {'size': size}, 'rot': r}, 'mlp': mlp}


def windowed(heads, kv_heads, dim, vdim, scale, size, r, mlp=None, kv_from=None):
    layer = dict(chunked(heads, kv_heads, dim, vdim, scale, size, r, mlp), type='attention_2')
    if kv_from is not None:
        layer['mixer']['kv_from'] = kv_from
    return layer


def latents(heads, dim, rot_dim, vdim, kv_rank, scale, size, base, mlp=None):
    return {'type': 'latent_attention', 'mixer': {'heads': heads, 'dim': dim, 'rot_dim': rot_dim, 'vdim': vdim, 'kv_rank': kv_rank, 'scale': scale, 'mask': {'size': size},
                                                  'rot': rot(rot_dim, base)}, 'mlp': mlp}


def dense(ff, limit):
    return {'kind': 'dense', 'ff': ff, 'limit': limit}


def moe(experts, top, ff, scale=1.0, groups=None, shared=None):
    r = {'experts': experts, 'top': top, 'scale': scale}
    if groups:
        r['groups'] = dict(zip(('count', 'keep'), groups))
    m = {'kind': 'moe', 'expert': {'ff': ff}, 'router': r}
    if shared:
        m['shared'] = {'ff': shared}
    return m


_LONG = (8.0, 1.0, 4.0, 64)        # wavelengths on both sides of 16 and 64 positions
CONFIGS = {
    # layers of unequal sizes, every kind of feed-forward, two layers that borrow (one over a distance)
    'mixed': dict(vocab=120, width=96, norm={'eps': 1e-4}, embedding={'scale': 3.0},
                  layers=[windowed(6, 2, 24, 40, 0.25, 19, rot(16, 500.0, _LONG), moe(6, 2, 32, 1.5, (3, 2), 40)), latents(5, 24, 16, 32, 48, 0.2, 23, 1000.0, dense(64, 1.5)),
                          chunked(6, 3, 32, 24, 0.2, 21, rot(24, 300.0), moe(8, 3, 24, 2.5, (4, 2))), windowed(4, 2, 24, 40, 0.3, 33, rot(16, 500.0, _LONG), kv_from=0),
                          latents(3, 40, 8, 24, 64, 0.15, 70, 200.0, moe(4, 4, 16, 0.5, (2, 2), 24)),
                          windowed(2, 2, 24, 40, 0.2, 7, rot(16, 500.0, _LONG), dense(40, 0.7), kv_from=0)]),
    # sizes that are no whole vectors, one head, one expert, groups of one, heads in fives, a window of one, a chunk of one
    'odd': dict(vocab=97, width=52, norm={'eps': 1e-3}, embedding={'scale': 0.75},
                layers=[latents(3, 7, 6, 11, 13, 0.4, 30, 50.0, moe(3, 1, 20, 1.0, (3, 1), 12)), chunked(5, 1, 11, 9, 0.3, 13, rot(6, 40.0), dense(18, 2.0)),
                        windowed(1, 1, 10, 7, 0.35, 17, rot(10, 30.0), moe(1, 1, 36)), windowed(3, 1, 10, 7, 0.35, 1, rot(10, 30.0), kv_from=2),
                        chunked(2, 2, 14, 5, 0.3, 1, rot(2, 10.0), moe(5, 2, 12, 3.0)), latents(1, 9, 4, 6, 5, 0.5, 8, 20.0)]),
    # head widths on both sides of 64, 128 and 192, ranks up to 512, bounds around a tile of 128
    'wide': dict(vocab=64, width=72, norm={'eps': 1e-6}, embedding={'scale': 2.0},
                 layers=[chunked(2, 1, 160, 136, 0.06, 129, rot(96, 1e4), dense(40, 1.0)), latents(4, 128, 64, 128, 264, 0.06, 128, 1e4, moe(8, 3, 24, 2.0, (2, 1), 16)),
                         windowed(4, 2, 128, 72, 0.08, 127, rot(128, 1e5, (4.0, 1.0, 4.0, 512)), moe(16, 5, 16, 1.0, (4, 3))), windowed(3, 3, 200, 64, 0.06, 130, rot(64, 1e3)),
                         latents(20, 64, 32, 64, 512, 0.08, 250, 1e4, dense(24, 3.0)), windowed(8, 2, 128, 72, 0.08, 300, rot(128, 1e5, (4.0, 1.0, 4.0, 512)), kv_from=2)]),
}
for _c in CONFIGS.values():
    _c['architecture'] = 'Nilepel'


def random_weights(cfg, seed=0):
    """Weights under their checkpoint names, every value representable in bfloat16.  Sinks weigh as much as a few keys."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    mat = lambda o, i: rnd(o, i) / i**0.5  # noqa: E731
    width = cfg['width']
    W = {'embed': rnd(cfg['vocab'], width), 'final.norm': 1 + 0.2 * rnd(width), 'head': mat(cfg['vocab'], width)}
    for i, layer in enumerate(cfg['layers']):
        p, m, f = f'l{i}.', layer['mixer'], layer['mlp']
        H, d, e = m['heads'], m['dim'], m['vdim']
        own = m.get('kv_from') is None
        for n in ('1', '2') if f else ('1', ):
            W[p + f'norm{n}'] = 1 + 0.2 * rnd(width)
        if layer['type'] == 'latent_attention':
            r = m['kv_rank']
            W[p + 'mix.q'], W[p + 'mix.dkv'], W[p + 'mix.dkv.norm'] = mat(H * (d + m['rot_dim']), width), mat(r + m['rot_dim'], width), 1 + 0.2 * rnd(r)
            W[p + 'mix.uk'], W[p + 'mix.uv'] = mat(H * d, r), mat(H * e, r)
        else:
            G = m['kv_heads']
            W[p + 'mix.q'], W[p + 'mix.sink'] = mat(H * d, width), 1 + rnd(H)
            if own:
                W[p + 'mix.k'], W[p + 'mix.v'] = mat(G * d, width), mat(G * e, width)
            if layer['type'] == 'attention_2':
                W[p + 'mix.q.b'], W[p + 'mix.q.norm'], W[p + 'mix.g'] = rnd(H * d), 1 + 0.2 * rnd(d), mat(H, width)
                if own:
                    W[p + 'mix.k.b'], W[p + 'mix.v.b'], W[p + 'mix.k.norm'] = rnd(G * d), rnd(G * e), 1 + 0.2 * rnd(d)
        W[p + 'mix.o'] = mat(width, H * e)
        if f and f['kind'] == 'dense':
            W[p + 'mlp.gate'], W[p + 'mlp.up'], W[p + 'mlp.down'] = mat(f['ff'], width), mat(f['ff'], width), mat(width, f['ff'])
        elif f:
            n, ff = f['router']['experts'], f['expert']['ff']
            W[p + 'mlp.router'] = 2 * mat(n, width)
            for x in range(n):
                W[p + f'mlp.e{x}.gate'], W[p + f'mlp.e{x}.up'], W[p + f'mlp.e{x}.down'] = mat(ff, width), mat(ff, width), mat(width, ff)
            if f.get('shared'):
                ff = f['shared']['ff']
                W[p + 'mlp.shared.gate'], W[p + 'mlp.shared.up'], W[p + 'mlp.shared.down'], W[p + 'mlp.shared.sg'] = mat(ff, width), mat(ff, width), mat(width, ff), mat(1, width)
    return {n: t.to(torch.bfloat16) for n, t in W.items()}


def write_checkpoint(path, cfg, weights):
    import json
    import os
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, 'config.json'), 'w') as f:
        json.dump(cfg, f)
    save_file({n: t.contiguous() for n, t in weights.items()}, os.path.join(path, 'model.safetensors'))
    return str(path)
