"""A plain, slow evaluation of the Puzonex decoder: one function per mechanism, one sequence at a time, whole sequence from its first
token, recurrences token by token.  It shares no code with the package.

Weights come as a mapping from checkpoint names to tensors; a configuration is the checkpoint's ``config.json`` mapping.
"""
import math

import torch


def over_rms(x, eps):
    """The last dimension divided by its root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return over_rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def log_sigmoid(z):
    return -softplus(-z)


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z**3)))


def project(h, w, name):
    """``W h``, plus a bias where there is one."""
    y = h @ w[name].t()
    return y + w[name + '.b'] if name + '.b' in w else y


# ------------------------------------------------------------------------------------------------ positions
def waves(positions, width, dtype=torch.float64):
    """Sine and cosine of a position, side by side, at geometrically falling frequencies."""
    out = torch.empty(len(positions), width, dtype=dtype)
    for c in range(width):
        a = torch.as_tensor(positions, dtype=torch.float64) * 10000.0 ** (-2 * (c // 2) / width)
        out[:, c] = (torch.cos(a) if c % 2 else torch.sin(a)).to(dtype)
    return out


def bucket(n, rows, far):
    """Bucket of a distance: exact up to half the rows, then wider and wider ones up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    # tolerance: distances that lie on a boundary belong to the bucket that begins there
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9))


def table_bias(rel, far, T):
    """``[H, T, T]``: the learned number of (head, bucket of i − j)."""
    per = torch.stack([rel[bucket(n, rel.shape[0], far)] for n in range(T)])             # [T, H]
    d = (torch.arange(T)[:, None] - torch.arange(T)[None]).clamp(min=0)
    return per[d].permute(2, 0, 1)


def log_bias(r1, r2, T):
    """``[H, T, T]``: minus a logarithm of the distance per head."""
    d = (torch.arange(T)[:, None] - torch.arange(T)[None]).clamp(min=0).to(r1.dtype)
    return -r1[:, None, None] * torch.log(1 + r2[:, None, None] * d)


# ------------------------------------------------------------------------------------------------ attention
def attend(q, k, v, scale, cap, bias, window, temp=None, sink=None):
    """One sequence: ``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, e]``; position i sees its last ``window`` positions.  ``temp [H]`` multiplies
    scores in front of the cap, ``bias [H, T, T]`` joins them behind it; ``sink [H]``: a logit in the denominator that belongs to no key."""
    T, H = q.shape[:2]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    seen = (j <= i) & (i - j < window)
    out = q.new_zeros(T, H, v.shape[-1])
    for h in range(H):
        g = h // (H // k.shape[1])
        s = q[:, h] @ k[:, g].t() * scale
        if temp is not None:
            s = s * temp[h]
        s = (capped(s, cap) + bias[h]).masked_fill(~seen, -math.inf)
        top = s.amax(-1) if sink is None else torch.maximum(s.amax(-1), sink[h])
        p = torch.exp(s - top[:, None])
        total = p.sum(-1) if sink is None else p.sum(-1) + torch.exp(sink[h] - top)
        out[:, h] = p @ v[:, g] / total[:, None]
    return out


def sink_heads(h, m, w, eps):
    """q, k and v of an 'attention' layer: q and k normed per head, v over its root mean square."""
    T, H, G = h.shape[0], m['heads'], m['kv_heads']
    q = norm(project(h, w, 'q').view(T, H, m['dim']), w['q.norm'], eps)
    k = norm(project(h, w, 'k').view(T, G, m['dim']), w['k.norm'], eps)
    return q, k, over_rms(project(h, w, 'v').view(T, G, m['vdim']), eps)


def sink_attention(h, m, w, eps):
    T = h.shape[0]
    q, k, v = sink_heads(h, m, w, eps)
    o = attend(q, k, v, m['scale'], m['softcap'], log_bias(w['r1'], w['r2'], T), m['mask']['size'], sink=w['sink'])
    return project(o.reshape(T, -1), w, 'o')


def shared_heads(h, m, w, eps):
    """q, k and v of the left side of a 'parallel' layer: values are the keys before their norm, which runs over all heads together."""
    T, H, G = h.shape[0], m['heads'], m['kv_heads']
    q, k = project(h, w, 'q'), project(h, w, 'k')
    v = k.view(T, G, m['vdim'])
    return norm(q, w['q.norm'], eps).view(T, H, m['dim']), norm(k, w['k.norm'], eps).view(T, G, m['dim']), v


def shared_attention(h, m, w, eps):
    T = h.shape[0]
    q, k, v = shared_heads(h, m, w, eps)
    o = attend(q, k, v, m['scale'], m['softcap'], table_bias(w['rel'], m['bias_max'], T), m['mask']['size'], temp=w['temp'])
    return project(o.reshape(T, -1) * sigmoid(h @ w['g'].t()), w, 'o')


# ------------------------------------------------------------------------------------------------ recurrences
def short_convolution(x, taps, bias):
    """Causal, per channel; the last tap is the current token's; nothing before the start."""
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        y[t] = bias
        for j in range(n):
            at = t - (n - 1 - j)
            if at >= 0:
                y[t] = y[t] + taps[:, j] * x[at]
    return y


def selective_scan(x, dt, A, B, C, D, S=None):
    """``x, dt [T, inner]``, ``A [inner, state]``, ``B, C [T, state]`` → outputs ``[T, inner]`` and the last state ``[inner, state]``."""
    S = torch.zeros_like(A) if S is None else S
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba(h, m, w, eps=None):
    n, r, s = m['inner'], m['dt_rank'], m['state']
    xz = h @ w['in'].t()
    x = silu(short_convolution(xz[:, :n], w['conv'], w['conv.b']))
    p = x @ w['x'].t()
    dt = softplus(p[:, :r] @ w['dt'].t() + w['dt.b'])
    y, _ = selective_scan(x, dt, -torch.exp(w['A_log']), p[:, r:r + s], p[:, r + s:], w['D'])
    return (y * silu(xz[:, n:])) @ w['o'].t()


def matrix_memory(q, k, v, i, f, state=None):
    """``q, k [T, H, d]``, ``v [T, H, e]``, log gates ``i, f [T, H]`` → outputs ``[T, H, e]`` and the last ``(S [H, d, e], n [H, d], m [H])``."""
    T, H, d = q.shape
    S, n, m = state if state is not None else (q.new_zeros(H, d, v.shape[-1]), q.new_zeros(H, d), q.new_zeros(H))
    out = torch.zeros_like(v)
    for t in range(T):
        top = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = top
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / den[:, None]
    return out, (S, n, m)


def memory_gates(h, w, cap):
    """Log input and log forget gate ``[T, H]``."""
    return capped(project(h, w, 'i'), cap), log_sigmoid(capped(project(h, w, 'f'), cap))


def memory_mixer(h, m, w, eps):
    T, H, d, e = h.shape[0], m['heads'], m['dim'], m['vdim']
    q, k, v = ((h @ w[n].t()).view(T, H, -1) for n in 'qkv')
    o, _ = matrix_memory(q * d**-0.5, k, v, *memory_gates(h, w, m['gate_cap']))
    return (over_rms(o, eps).reshape(T, H * e) * w['norm'] * sigmoid(h @ w['g'].t())) @ w['o'].t()


def side_by_side(h, m, w, eps):
    """Half the sum of the normed results of two mixers."""
    a = shared_attention(h, m['left'], part(w, 'left.'), eps)
    b = memory_mixer(h, m['right'], part(w, 'right.'), eps)
    return 0.5 * (norm(a, w['left.out'], eps) + norm(b, w['right.out'], eps))


MIXERS = {'attention': sink_attention, 'mamba1': mamba, 'parallel': side_by_side}


# ------------------------------------------------------------------------------------------------ the stack
def feed_forward(h, w):
    return (gelu_tanh(h @ w['gate'].t()) * (h @ w['up'].t())) @ w['down'].t()


def part(W, prefix):
    return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits ``[T, vocab]`` and the residual stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg['norm']['eps']
    x = W['embed'][torch.as_tensor(tokens)] + waves(range(len(tokens)), cfg['width'], dtype)
    trail = []
    for i, layer in enumerate(cfg['layers']):
        p = f'l{i}.'
        x = x + norm(MIXERS[layer['type']](x, layer['mixer'], part(W, p + 'mix.'), eps), W[p + 'norm1'], eps)
        if layer.get('mlp'):
            x = x + norm(feed_forward(x, part(W, p + 'mlp.')), W[p + 'norm2'], eps)
        trail.append(x)
    return norm(x, W['final.norm'], eps) @ W['head'].t(), trail


# ---------------------------------------------------------------- models for the tests
def attention(heads, kv_heads, dim, vdim, scale, size, cap, ff=None):
    return {'type': 'attention', 'mixer': {'heads': heads, 'kv_heads': kv_heads, 'dim': dim, 'vdim': vdim, 'scale': scale, 'softcap': cap, 'mask': {'size': size}}, 'mlp': dense(ff)}


def mamba1(inner, state, dt_rank, conv, ff=None):
    return {'type': 'mamba1', 'mixer': {'inner': inner, 'state': state, 'dt_rank': dt_rank, 'conv': conv}, 'mlp': dense(ff)}


def parallel(left, right, ff=None):
    """``left``: heads, kv_heads, dim, scale, window, softcap, rows of the distance table, its last distance; ``right``: heads, dim, vdim, gate cap."""
    heads, kv_heads, dim, scale, size, cap, rows, far = left
    h, d, e, gate_cap = right
    return {'type': 'parallel', 'mlp': dense(ff),
            'mixer': {'left': {'heads': heads, 'kv_heads': kv_heads, 'dim': dim, 'vdim': dim, 'scale': scale, 'softcap': cap, 'bias_max': far, 'mask': {'size': size}},
                      'right': {'heads': h, 'dim': d, 'vdim': e, 'gate_cap': gate_cap}}, 'rows': rows}


def dense(ff):
    return None if ff is None else {'kind': 'dense', 'ff': ff}


CONFIGS = {
    # every kind of layer twice, of unequal sizes, with and without a feed-forward block
    'mixed': dict(vocab=120, width=96, norm={'eps': 1e-4},
                  layers=[parallel((6, 2, 24, 0.25, 19, 6.0, 10, 37), (3, 16, 40, 4.0), 128), mamba1(80, 12, 8, 3, 72), attention(6, 3, 24, 40, 0.3, 23, 5.0),
                          mamba1(64, 16, 24, 4), parallel((4, 4, 40, 0.2, 70, 20.0, 32, 128), (2, 24, 32, 9.0)), attention(8, 2, 16, 16, 0.4, 33, 3.0, 96)]),
    # sizes that are no whole vectors, one head, windows of one, a table of two rows, filters of one and of six taps, odd numbers of states
    'odd': dict(vocab=97, width=52, norm={'eps': 1e-3},
                layers=[mamba1(30, 5, 3, 2, 18), parallel((3, 1, 11, 0.3, 13, 2.5, 7, 20), (1, 10, 7, 3.0), 20), attention(5, 1, 10, 7, 0.35, 1, 4.0, 9), mamba1(21, 1, 1, 1),
                        attention(1, 1, 14, 5, 0.3, 17, 8.0), mamba1(12, 9, 5, 6, 33), parallel((2, 2, 9, 0.3, 30, 30.0, 2, 4), (5, 3, 9, 1.5)), parallel((1, 1, 6, 0.4, 1, 1.0, 5, 3), (2, 5, 12, 6.0), 11)]),
    # head widths on both sides of 64 and 128, values in several blocks, many states, windows around a tile of 128
    'wide': dict(vocab=64, width=72, norm={'eps': 1e-6},
                 layers=[attention(8, 1, 128, 72, 0.06, 129, 30.0, 40), parallel((4, 2, 160, 0.05, 128, 15.0, 16, 100), (2, 128, 136, 15.0)), mamba1(136, 64, 8, 4),
                         parallel((4, 4, 128, 0.07, 250, 50.0, 64, 333), (1, 256, 64, 7.0), 48), attention(3, 3, 200, 136, 0.06, 127, 10.0), mamba1(64, 130, 16, 5, 24)]),
}
_ROWS = {}
for _n, _c in CONFIGS.items():
    _c['architecture'] = 'Puzonex'
    _ROWS[_n] = [layer.pop('rows', 0) for layer in _c['layers']]


def random_weights(cfg, seed=0, rows=None):
    """Weights under their checkpoint names, every value representable in bfloat16.  Sinks weigh as much as a few keys, distances shift scores by
    about one, forget gates are mostly open, and a scan's steps reach from a few tokens to hundreds."""
    rows = rows if rows is not None else next((_ROWS[n] for n, c in CONFIGS.items() if c is cfg), None)
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    mat = lambda o, i: rnd(o, i) / i**0.5  # noqa: E731
    ones = lambda n: 1 + 0.2 * rnd(n)  # noqa: E731
    width = cfg['width']
    W = {'embed': rnd(cfg['vocab'], width), 'final.norm': ones(width), 'head': mat(cfg['vocab'], width)}

    def heads(p, m, own_values, norms):
        H, G, d, e = m['heads'], m['kv_heads'], m['dim'], m['vdim']
        W[p + 'q'], W[p + 'q.b'], W[p + 'k'], W[p + 'k.b'] = mat(H * d, width), 0.5 * rnd(H * d), mat(G * d, width), 0.5 * rnd(G * d)
        if own_values:
            W[p + 'v'], W[p + 'v.b'] = mat(G * e, width), 0.5 * rnd(G * e)
        W[p + 'q.norm'], W[p + 'k.norm'], W[p + 'o'] = ones(norms * H if norms > 1 else d), ones(norms * G if norms > 1 else d), mat(width, H * e)
    for i, layer in enumerate(cfg['layers']):
        p, m, f = f'l{i}.', layer['mixer'], layer['mlp']
        W[p + 'norm1'] = ones(width)
        if f:
            W[p + 'norm2'] = ones(width)
            W[p + 'mlp.gate'], W[p + 'mlp.up'], W[p + 'mlp.down'] = mat(f['ff'], width), mat(f['ff'], width), mat(width, f['ff'])
        if layer['type'] == 'attention':
            heads(p + 'mix.', m, True, 1)
            H = m['heads']
            W[p + 'mix.sink'], W[p + 'mix.r1'], W[p + 'mix.r2'] = 1 + rnd(H), rnd(H).abs(), 0.5 * rnd(H).abs()
        elif layer['type'] == 'mamba1':
            n, s, r = m['inner'], m['state'], m['dt_rank']
            W[p + 'mix.in'], W[p + 'mix.o'], W[p + 'mix.x'], W[p + 'mix.dt'] = mat(2 * n, width), mat(width, n), mat(r + 2 * s, n), mat(n, r)
            W[p + 'mix.conv'], W[p + 'mix.conv.b'], W[p + 'mix.dt.b'] = mat(n, m['conv']), 0.3 * rnd(n), rnd(n) - 2
            W[p + 'mix.A_log'], W[p + 'mix.D'] = 1.2 * rnd(n, s) - 1.5, ones(n)
        else:
            left, right, q = m['left'], m['right'], p + 'mix.left.'
            heads(q, left, False, left['dim'])
            H = left['heads']
            W[q + 'o.b'], W[q + 'g'], W[q + 'temp'], W[q + 'rel'] = 0.5 * rnd(width), mat(H * left['vdim'], width), 1 + 0.3 * rnd(H).abs(), rnd(rows[i], H)
            if W[q + 'q.norm'].numel() != H * left['dim']:      # one head of one dimension
                raise AssertionError
            q, h, d, e = p + 'mix.right.', right['heads'], right['dim'], right['vdim']
            W[q + 'q'], W[q + 'k'], W[q + 'v'], W[q + 'g'], W[q + 'o'] = mat(h * d, width), mat(h * d, width), mat(h * e, width), mat(h * e, width), mat(width, h * e)
            W[q + 'norm'], W[q + 'i'], W[q + 'i.b'], W[q + 'f'], W[q + 'f.b'] = ones(h * e), 2 * mat(h, width), rnd(h), mat(h, width), 3 + rnd(h)
            W[p + 'mix.left.out'], W[p + 'mix.right.out'] = ones(width), ones(width)
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
