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
