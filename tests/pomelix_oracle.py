"""A plain, slow evaluation of the Pomelix decoder: one function per mechanism, one sequence at a time, whole sequence from
its first token, loops over positions where that is the clearest statement.  It shares no code with the package.

Weights come as a mapping from checkpoint names to tensors; a configuration is the checkpoint's ``config.json`` mapping.
"""
import math

import torch


def rms(x, eps):
    """x / sqrt(mean of squares + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def causal_conv(u, w):
    """``u [T, C]``, ``w [C, taps]``: y_t is the weighted sum of the last ``taps`` rows, the newest under the last weight."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y[t] += w[:, j] * u[src]
    return y


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1)


def attention(q, k, v, scale):
    """``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, e]`` → ``[T, H, e]``: causal softmax, query head h reads group h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = q.new_zeros(T, H, v.shape[-1])
    for h in range(H):
        g = h // per
        s = (q[:, h] @ k[:, g].t()) * scale
        for i in range(T):
            out[i, h] = torch.softmax(s[i, :i + 1], 0) @ v[:i + 1, g]
    return out


def mix_values(v, v_first, lam):
    return (1 - lam) * v + lam * v_first


def gated_feed_forward(h, gate, up, down):
    z = h @ gate.t()
    return (z * torch.sigmoid(z) * (h @ up.t())) @ down.t()


def mixer(h, m, w, eps, v_first):
    """One attention sub-layer on ``h [T, width]``; returns its result and the (unmixed) values."""
    T, H, G, d, e = h.shape[0], m['heads'], m['kv_heads'], m['dim'], m['vdim']
    q, k, v = (causal_conv(h @ w[n].t(), w[n + '.conv']) for n in 'qkv')
    q, k, v = rms(q.view(T, H, d), eps), rms(k.view(T, G, d), eps), v.view(T, G, e)
    qt = m.get('q_temp')
    if qt:
        for p in range(T):
            q[p] = q[p] * query_temperature(p, qt['coef'], qt['every'])
    own = v
    if m.get('v_mix') and v_first is not None:
        v = mix_values(v, v_first, w['vmix'])
    o = attention(q, k, v, m['scale'])
    return o.reshape(T, H * e) @ w['o'].t(), own


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits ``[T, vocab]`` and the residual stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps, mult = cfg['norm']['eps'], cfg['residual_mult']
    x = W['embed'][torch.as_tensor(tokens)]
    v_first, trail = None, []
    for i, layer in enumerate(cfg['layers']):
        p = f'l{i}.'
        mine = {n[len(p) + 4:]: t for n, t in W.items() if n.startswith(p + 'mix.')}
        h = rms_norm(x, W[p + 'norm1'], eps)
        a, v = mixer(h, layer['mixer'], mine, eps, v_first)
        if layer['mixer'].get('v_mix') and v_first is None:
            v_first = v
        add = a * W[p + 'ls1']
        if layer.get('mlp'):
            add = add + gated_feed_forward(h, W[p + 'mlp.gate'], W[p + 'mlp.up'], W[p + 'mlp.down']) * W[p + 'ls2']
        x = x + mult * add
        trail.append(x)
    return rms_norm(x, W['final.norm'], eps) @ W['embed'].t(), trail


# ---------------------------------------------------------------- models for the tests
def spec(heads, kv_heads, dim, vdim, conv, scale, v_mix=False, temp=None, ff=0):
    m = {'heads': heads, 'kv_heads': kv_heads, 'dim': dim, 'vdim': vdim, 'conv': conv, 'scale': scale, 'v_mix': v_mix}
    if temp:
        m['q_temp'] = {'coef': temp[0], 'every': temp[1]}
    return {'type': 'attention', 'mixer': m, 'mlp': {'kind': 'dense', 'ff': ff} if ff else None}


CONFIGS = {
    # layers of unequal sizes; the first does not mix values, the second gives them and has no feed-forward block
    'mixed': dict(vocab=120, width=96, norm={'eps': 1e-5}, residual_mult=0.6,
                  layers=[spec(6, 2, 24, 40, 3, 0.31, False, (0.25, 7), 64), spec(4, 4, 32, 16, 4, 0.2, True, (0.4, 20)),
                          spec(8, 4, 16, 16, 2, 0.35, True, (0.1, 5), 88)]),
    # widths that are no whole vectors, more taps than the vector kernel takes, groups of three and five, no temperature
    'odd': dict(vocab=97, width=52, norm={'eps': 1e-3}, residual_mult=0.9,
                layers=[spec(3, 1, 20, 12, 5, 0.4, True, (0.3, 3), 36), spec(5, 1, 7, 12, 1, 0.5, True, None, 20), spec(10, 2, 9, 11, 3, 0.3, False, (0.2, 1))]),
    # heads on both sides of 64, 128 and at 256
    'wide': dict(vocab=64, width=72, norm={'eps': 1e-6}, residual_mult=1.0,
                 layers=[spec(2, 1, 160, 256, 4, 0.08, False, (0.2, 11), 40), spec(4, 2, 128, 128, 4, 0.09, True, (0.2, 11), 48),
                         spec(2, 2, 64, 128, 2, 0.12, True), spec(3, 1, 72, 64, 3, 0.12)]),
}
for _c in CONFIGS.values():
    _c['architecture'] = 'Pomelix'


def random_weights(cfg, seed=0):
    """Weights under their checkpoint names, every value representable in bfloat16."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    mat = lambda o, i: rnd(o, i) / i**0.5  # noqa: E731
    width = cfg['width']
    W = {'embed': rnd(cfg['vocab'], width), 'final.norm': 1 + 0.2 * rnd(width)}
    for i, layer in enumerate(cfg['layers']):
        p, m = f'l{i}.', layer['mixer']
        sizes = {'q': m['heads'] * m['dim'], 'k': m['kv_heads'] * m['dim'], 'v': m['kv_heads'] * m['vdim']}
        W[p + 'norm1'], W[p + 'ls1'] = 1 + 0.2 * rnd(width), 1 + 0.3 * rnd(width)
        for n, s in sizes.items():
            W[p + f'mix.{n}'], W[p + f'mix.{n}.conv'] = mat(s, width), 0.6 * rnd(s, m['conv'])
        W[p + 'mix.o'] = mat(width, m['heads'] * m['vdim'])
        if m['v_mix']:
            W[p + 'mix.vmix'] = torch.rand((), generator=g) * 0.6 + 0.2
        if layer['mlp']:
            ff = layer['mlp']['ff']
            W[p + 'mlp.gate'], W[p + 'mlp.up'], W[p + 'mlp.down'], W[p + 'ls2'] = mat(ff, width), mat(ff, width), mat(width, ff), 1 + 0.3 * rnd(width)
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
