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
