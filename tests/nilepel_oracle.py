"""A plain, slow evaluation of the Nilepel decoder: one function per mechanism, one sequence at a time, whole sequence from its first
token, loops over positions, heads and experts where that is the clearest statement.  It shares no code with the package.

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
    out = q.new_zeros(T, H, v.shape[-1])
    for h in range(H):
        g = h // (H // k.shape[1])
        for i in range(T):
            a = first(i)
            s = (k[a:i + 1, g] @ q[i, h]) * scale
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            p = torch.exp(s - top)
            total = p.sum() if sink is None else p.sum() + torch.exp(sink[h] - top)
            out[i, h] = p @ v[a:i + 1, g] / total
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
    for t in range(h.shape[0]):
        for n, p in zip(idx[t].tolist(), share[t]):
            out[t] += p * expert(h[t], w[f'e{n}.gate'], w[f'e{n}.up'], w[f'e{n}.down'])
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
