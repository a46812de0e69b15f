"""A plain, slow evaluation of the Moronex decoder: one function per mechanism, one sequence at a time, whole sequence from its
first token, loops over positions, heads and experts where that is the clearest statement.  It shares no code with the package.

Weights come as a mapping from checkpoint names to tensors; a configuration is the checkpoint's ``config.json`` mapping.
"""
import torch


def unit(x, eps):
    """x / sqrt(mean of squares + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """RMS norm with a plain weight."""
    return unit(x, eps) * w


def norm_about_one(x, w, eps):
    """RMS norm whose stored weight is the difference from one."""
    return unit(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def latent(h, m, w, eps):
    """What a latent-attention layer stores per token: ``[T, kv_rank]``."""
    return norm(h @ w['dkv'].t(), w['dkv.norm'], eps)


def latent_attention(h, c, m, w, eps):
    """``h [T, width]``, ``c [T, kv_rank]`` (this layer's or the one it borrows from) → ``[T, width]``."""
    T, H, d, e = h.shape[0], m['heads'], m['dim'], m['vdim']
    q = (norm(h @ w['dq'].t(), w['dq.norm'], eps) @ w['uq'].t()).view(T, H, d)
    k, v = (c @ w['uk'].t()).view(T, H, d), (c @ w['uv'].t()).view(T, H, e)
    gate = sigmoid(h @ w['g'].t())
    out = h.new_zeros(T, H, e)
    for n in range(H):
        s = (q[:, n] @ k[:, n].t()) * m['scale']
        for i in range(T):
            row, sink = s[i, :i + 1], w['sink'][n]
            top = torch.maximum(row.max(), sink)
            p = torch.exp(row - top)
            out[i, n] = (p / (p.sum() + torch.exp(sink - top))) @ v[:i + 1, n]
    return (out * gate[:, :, None]).reshape(T, H * e) @ w['o'].t()


def hgrn2_gates(h, m, w):
    """Forget gates ``[T, heads, dim]``."""
    low = w['lower']
    return (low + (1 - low) * sigmoid(h @ w['f'].t() + w['f.b'])).view(h.shape[0], m['heads'], m['dim'])


def hgrn2_scan(q, f, v):
    """``q, f [T, H, d]``, ``v [T, H, e]`` → outputs ``[T, H, e]`` and the last state ``[H, d, e]``."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append((q[t][:, :, None] * S).sum(1))
    return torch.stack(out), S


def hgrn2(h, m, w, eps):
    T, H = h.shape[0], m['heads']
    q, v = silu(h @ w['q'].t()).view(T, H, m['dim']), (h @ w['v'].t()).view(T, H, m['vdim'])
    o, _ = hgrn2_scan(q, hgrn2_gates(h, m, w), v)
    return norm(o, w['norm'], eps).reshape(T, -1) @ w['o'].t()


def gated_feed_forward(h, w):
    return (silu(h @ w['gate'].t()) * (h @ w['up'].t())) @ w['down'].t()


def expert(x, up, down):
    return torch.clamp(x @ up.t(), min=0) ** 2 @ down.t()


def route(h, w, top):
    """Chosen experts of every token, best first, and their weights."""
    best, idx = (h @ w['router'].t() + w['router.b']).topk(top, -1)
    e = torch.exp(best - best[:, :1])
    return idx, e / e.sum(-1, keepdim=True)


def mixture(h, m, w):
    idx, share = route(h, w, m['router']['top'])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for n, p in zip(idx[t].tolist(), share[t]):
            out[t] += p * expert(h[t], w[f'e{n}.up'], w[f'e{n}.down'])
    return out


def join(x, result, h, gate, bias, w, eps):
    """The residual stream after a sub-layer: its result gated by what it read, normed, added."""
    return x + norm_about_one(sigmoid(h @ gate.t() + bias) * result, w, eps)


def part(W, prefix):
    return {n[len(prefix):]: t for n, t in W.items() if n.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64):
    """Logits ``[T, vocab]`` and the residual stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg['norm']['eps']
    x = W['embed'][torch.as_tensor(tokens)]
    held, trail = {}, []
    for i, layer in enumerate(cfg['layers']):
        p, m = f'l{i}.', layer['mixer']
        w = part(W, p + 'mix.')
        h = norm_about_one(x, W[p + 'norm1'], eps)
        if layer['type'] == 'hgrn2':
            y = hgrn2(h, m, w, eps)
        else:
            if m.get('kv_from') is None:
                held[i] = latent(h, m, w, eps)
            y = latent_attention(h, held[m['kv_from'] if m.get('kv_from') is not None else i], m, w, eps)
        x = join(x, y, h, W[p + 'rg1'], W[p + 'rg1.b'], W[p + 'norm1b'], eps)
        if layer.get('mlp'):
            h = norm_about_one(x, W[p + 'norm2'], eps)
            w = part(W, p + 'mlp.')
            y = mixture(h, layer['mlp'], w) if layer['mlp']['kind'] == 'moe' else gated_feed_forward(h, w)
            x = join(x, y, h, W[p + 'rg2'], W[p + 'rg2.b'], W[p + 'norm2b'], eps)
        trail.append(x)
    return norm_about_one(x, W['final.norm'], eps) @ W['head'].t(), trail


# ---------------------------------------------------------------- models for the tests
def recurrent(heads, dim, vdim, mlp=None):
    return {'type': 'hgrn2', 'mixer': {'heads': heads, 'dim': dim, 'vdim': vdim}, 'mlp': mlp}


def latents(heads, dim, vdim, q_rank, kv_rank, scale, mlp=None, kv_from=None):
    m = {'heads': heads, 'dim': dim, 'vdim': vdim, 'q_rank': q_rank, 'kv_rank': kv_rank, 'scale': scale}
    if kv_from is not None:
        m['kv_from'] = kv_from
    return {'type': 'latent_attention', 'mixer': m, 'mlp': mlp}


def dense(ff):
    return {'kind': 'dense', 'ff': ff}


def moe(experts, top, ff):
    return {'kind': 'moe', 'expert': {'ff': ff}, 'router': {'experts': experts, 'top': top}}


CONFIGS = {
    # layers of unequal sizes and every kind of feed-forward; two layers borrow latents, one of them over a distance
    'mixed': dict(vocab=120, width=96, norm={'eps': 1e-5},
                  layers=[recurrent(3, 24, 40, dense(64)), latents(5, 24, 40, 56, 48, 0.3, moe(6, 2, 32)), recurrent(4, 32, 16),
                          latents(2, 40, 24, 24, 48, 0.25, moe(5, 3, 40), kv_from=1), latents(4, 16, 32, 32, 64, 0.4), recurrent(2, 16, 64, moe(4, 4, 16)),
                          latents(3, 32, 16, 40, 48, 0.2, dense(56), kv_from=1)]),
    # sizes that are no whole vectors, attention first, one head, one expert, ranks below the head width
    'odd': dict(vocab=97, width=52, norm={'eps': 1e-3},
                layers=[latents(3, 7, 11, 9, 13, 0.5, moe(3, 1, 20)), recurrent(5, 6, 9, moe(1, 1, 36)), latents(1, 12, 5, 4, 13, 0.4, dense(18), kv_from=0),
                        recurrent(1, 4, 6), recurrent(2, 33, 20, dense(12))]),
    # head widths on both sides of 64, 128 and at 256, ranks up to 512
    'wide': dict(vocab=64, width=72, norm={'eps': 1e-6},
                 layers=[recurrent(1, 160, 256, dense(40)), latents(2, 160, 136, 40, 264, 0.08, moe(8, 3, 24)), recurrent(2, 128, 128), recurrent(2, 64, 136, dense(24)),
                         latents(20, 64, 128, 96, 512, 0.1), latents(3, 128, 72, 96, 512, 0.09, kv_from=4)]),
}
for _c in CONFIGS.values():
    _c['architecture'] = 'Moronex'


def random_weights(cfg, seed=0):
    """Weights under their checkpoint names, every value representable in bfloat16.  Forget gates reach from nearly open to nearly
    closed, sinks weigh as much as a few keys."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    mat = lambda o, i: rnd(o, i) / i**0.5  # noqa: E731
    width = cfg['width']
    W = {'embed': rnd(cfg['vocab'], width), 'final.norm': 0.2 * rnd(width), 'head': mat(cfg['vocab'], width)}
    for i, layer in enumerate(cfg['layers']):
        p, m, f = f'l{i}.', layer['mixer'], layer['mlp']
        H, d, e = m['heads'], m['dim'], m['vdim']
        for n in ('1', '2') if f else ('1', ):
            W[p + f'norm{n}'], W[p + f'norm{n}b'] = 0.2 * rnd(width), 0.2 * rnd(width)
            W[p + f'rg{n}'], W[p + f'rg{n}.b'] = mat(width, width), rnd(width)
        if layer['type'] == 'hgrn2':
            W[p + 'mix.q'], W[p + 'mix.f'], W[p + 'mix.v'] = mat(H * d, width), mat(H * d, width), mat(H * e, width)
            W[p + 'mix.f.b'], W[p + 'mix.lower'] = 2 + 3 * rnd(H * d), torch.rand(H * d, generator=g) * 0.9
            W[p + 'mix.norm'] = 1 + 0.2 * rnd(e)
        else:
            r = m['kv_rank']
            W[p + 'mix.dq'], W[p + 'mix.dq.norm'], W[p + 'mix.uq'] = mat(m['q_rank'], width), 1 + 0.2 * rnd(m['q_rank']), mat(H * d, m['q_rank'])
            if m.get('kv_from') is None:
                W[p + 'mix.dkv'], W[p + 'mix.dkv.norm'] = mat(r, width), 1 + 0.2 * rnd(r)
            W[p + 'mix.uk'], W[p + 'mix.uv'], W[p + 'mix.sink'], W[p + 'mix.g'] = mat(H * d, r), mat(H * e, r), 2 + rnd(H), mat(H, width)
        W[p + 'mix.o'] = mat(width, H * e)
        if f and f['kind'] == 'dense':
            W[p + 'mlp.gate'], W[p + 'mlp.up'], W[p + 'mlp.down'] = mat(f['ff'], width), mat(f['ff'], width), mat(width, f['ff'])
        elif f:
            n, ff = f['router']['experts'], f['expert']['ff']
            W[p + 'mlp.router'], W[p + 'mlp.router.b'] = 2 * mat(n, width), 0.5 * rnd(n)
            for x in range(n):
                W[p + f'mlp.e{x}.up'], W[p + f'mlp.e{x}.down'] = mat(ff, width), mat(width, ff)
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
