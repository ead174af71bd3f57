"""Plain, slow restatement of the Gugezen decoder (torch on the CPU, float32 or float64), one function per mechanism.

It shares no code with the CUDA path: the tests build small random checkpoints, run both and compare. A sequence is processed
whole, token loops where the design is recurrent, no cache and no state object.

Notation: X [S, T, W] = S residual streams, all c E[tok] at the start; N(v; g) = v / sqrt(mean(v^2) + eps) * g, model gains g = 1 + w.
A sublayer f with input weights a [S], transfer matrix M [from, to] and output weights b [S] acts on all streams at once:
    y = f(N(sum_s a_s X_s; 1 + w));    X_t <- sum_s M[s, t] X_s + b_t y
A layer is a mixer sublayer, then (where it has one) a feed-forward sublayer. A layer can borrow all tensors of another one. Mixers:
  'parallel'  r_l left(h) + r_r right(h). left: grouped-query attention with projection biases, neighbour pairs of numbers turned by
              wavelength-dependent frequencies, a learned per-head sink in the softmax denominator, an element-wise sigmoid gate. right:
              linear attention whose matrix state decays by one fixed factor per head, silu on q, k and v, one RMS norm over all heads
              together, an element-wise sigmoid gate;
  'mamba2'    state-space duality: a short convolution with bias and silu over x, B and C, a state [N, vdim] per head that decays by a
              token-dependent step, a skip term, the silu gate BEFORE a norm in equal parts.
Feed-forwards: W_down (gelu_tanh(W_gate h) * W_up h), or a mixture of W_down gelu(W_up h) units behind a softmax router plus a shared
unit. Output: logits = k E N(sum_s X_s; 1 + w). cfg is the parsed config.json (a dict), w the tensor dict of the checkpoint.
"""
import math

import torch


def rms_norm(v, g, eps):
    v = v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)
    return v if g is None else v * g


def silu(v):
    return v * torch.sigmoid(v)


def gelu_tanh(v):
    return 0.5 * v * (1 + torch.tanh(math.sqrt(2 / math.pi) * (v + 0.044715 * v ** 3)))


def gelu_erf(v):
    return 0.5 * v * (1 + torch.erf(v / math.sqrt(2)))


# ------------------------------------------------------------------------------------------------ residual streams
def read_streams(X, a):
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + a[s] * X[s]
    return u


def write_streams(X, M, b, y):
    out = []
    for t in range(X.shape[0]):
        v = b[t] * y
        for s in range(X.shape[0]):
            v = v + M[s, t] * X[s]
        out.append(v)
    return torch.stack(out)


# ------------------------------------------------------------------------------------------------ attention half
def stretched_frequencies(rot):
    """angle per position of every neighbour pair. Pairs whose wavelength is below original / high keep base^(-2i/dims), those above
    original / low are slowed by the factor, in between the two are mixed by where original / wavelength lies between low and high"""
    dims = int(rot['dims'])
    out = []
    for i in range(dims // 2):
        f = float(rot['base']) ** (-2 * i / dims)
        sc = rot.get('scaling')
        if sc:
            turns = float(sc['original']) * f / (2 * math.pi)                  # original / wavelength
            if turns < float(sc['low']):
                f = f / float(sc['factor'])
            elif turns <= float(sc['high']):
                s = (turns - float(sc['low'])) / (float(sc['high']) - float(sc['low']))
                f = (1 - s) * f / float(sc['factor']) + s * f
        out.append(f)
    return out


def rotate_neighbours(v, pos, rot):
    """v [T, heads, d]: numbers 2i and 2i + 1 turn together, the numbers from dims on stay as they are"""
    out = v.clone()
    for i, f in enumerate(stretched_frequencies(rot)):
        c, s = torch.cos(pos.to(v.dtype) * f)[:, None], torch.sin(pos.to(v.dtype) * f)[:, None]
        out[..., 2 * i] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = v[..., 2 * i + 1] * c + v[..., 2 * i] * s
    return out


def softmax_with_sink(s, vis, sink):
    """rows of s over the visible keys; exp(sink) joins the denominator only"""
    s = s.masked_fill(~vis, float('-inf'))
    sink = torch.as_tensor(sink, dtype=s.dtype)
    m = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def attention(h, w, p, mc):
    T = h.shape[0]
    H, G, d = int(mc['heads']), int(mc.get('kv_heads', mc['heads'])), int(mc['dim'])
    dv = int(mc.get('vdim', d))
    lin = lambda n: h @ w[p + n].T + w[p + n + '.b']
    pos = torch.arange(T)
    q, k, v = lin('q').view(T, H, d), lin('k').view(T, G, d), lin('v').view(T, G, dv)
    if mc.get('rot'):
        q, k = rotate_neighbours(q, pos, mc['rot']), rotate_neighbours(k, pos, mc['rot'])
    vis = pos[None, :] <= pos[:, None]
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        out[:, hh] = softmax_with_sink(q[:, hh] @ k[:, g].T * float(mc['scale']), vis, w[p + 'sink'][hh]) @ v[:, g]
    return (out.reshape(T, H * dv) * torch.sigmoid(h @ w[p + 'g'].T)) @ w[p + 'o'].T


# ------------------------------------------------------------------------------------------------ recurrent half
def decayed_memory(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv], decay [T, H] -> read-outs [T, H, dv]; the state S [d, dv] of a head starts at zero"""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[-1], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o


def lightning(h, w, p, mc, eps):
    T, H, d = h.shape[0], int(mc['heads']), int(mc['dim'])
    dv = int(mc.get('vdim', d))
    act = lambda n, size: silu(h @ w[p + n].T).view(T, H, size)
    decay = torch.tensor([float(x) for x in mc['decay']], dtype=torch.float64).to(h.dtype).expand(T, H)
    o = decayed_memory(act('q', d), act('k', d), act('v', dv), decay)
    o = rms_norm(o.reshape(T, H * dv), w[p + 'norm'], eps)
    return (o * torch.sigmoid(h @ w[p + 'g'].T)) @ w[p + 'o'].T


def parallel(h, w, p, mc, eps):
    return (float(mc.get('left_scale', 1.0)) * attention(h, w, p + 'left.', mc['left'])
            + float(mc.get('right_scale', 1.0)) * lightning(h, w, p + 'right.', mc['right'], eps))


# ------------------------------------------------------------------------------------------------ state-space mixer
def short_conv(z, cw, bias):
    """z [T, C], cw [C, taps]: each channel over time, the last column of cw meets the current token, zeros before the start"""
    T, taps = z.shape[0], cw.shape[1]
    out = torch.zeros_like(z) + bias
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                out[t] += cw[:, j] * z[s]
    return out


def parts_norm(v, parts, gain, eps):
    T, n = v.shape
    return rms_norm(v.view(T, parts, n // parts), None, eps).reshape(T, n) * gain


def mamba2(h, w, p, mc, eps):
    T, H, dv, N, G = h.shape[0], int(mc['heads']), int(mc['vdim']), int(mc['state']), int(mc['groups'])
    inner = H * dv
    z, xbc, dt = torch.split(h @ w[p + 'in'].T, [inner, inner + 2 * G * N, H], -1)
    xbc = silu(short_conv(xbc, w[p + 'conv'], w[p + 'conv.b']))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    of_head = [hh // (H // G) for hh in range(H)]
    x, B, C = x.reshape(T, H, dv), B.reshape(T, G, N)[:, of_head], C.reshape(T, G, N)[:, of_head]
    dt = torch.nn.functional.softplus(dt + w[p + 'dt_bias'], threshold=1e9)
    decay = torch.exp(-torch.exp(w[p + 'A_log']) * dt)
    y = decayed_memory(C, B, dt[..., None] * x, decay) + w[p + 'D'][:, None] * x
    y = parts_norm(y.reshape(T, inner) * silu(z), int(mc['norm_groups']), w[p + 'norm'], eps)
    return y @ w[p + 'o'].T


# ------------------------------------------------------------------------------------------------ feed-forwards
def dense_ff(h, w, p):
    return (gelu_tanh(h @ w[p + 'gate'].T) * (h @ w[p + 'up'].T)) @ w[p + 'down'].T


def unit(h, w, p):
    return gelu_erf(h @ w[p + 'up'].T) @ w[p + 'down'].T


def moe_ff(h, w, p, fc):
    top = int(fc['router']['top'])
    s = torch.softmax(h @ w[p + 'router'].T, -1)
    y = unit(h, w, p + 'shared.') if fc.get('shared') else torch.zeros_like(h)
    for t in range(h.shape[0]):
        best = torch.argsort(-s[t], stable=True)[:top]
        total = s[t, best].sum() + 1e-20
        for e in best.tolist():
            y[t] += s[t, e] / total * unit(h[t:t + 1], w, f'{p}e{e}.')[0]
    return y


# ------------------------------------------------------------------------------------------------ the stack
def forward(cfg, weights, tokens, dtype=torch.float32, trace=None):
    """token ids of ONE sequence -> logits [T, vocab]; `trace` (a list) receives the sum of the streams after every layer"""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = float(cfg['norm']['eps'])
    emb = w['embed'][torch.tensor([int(t) for t in tokens])] * float(cfg['embedding']['scale'])
    X = torch.stack([emb] * int(cfg['streams']))
    for i, lc in enumerate(cfg['layers']):
        own = i
        while cfg['layers'][own].get('weights_of') is not None:
            own = int(cfg['layers'][own]['weights_of'])
        p = f'l{own}.'

        def sublayer(X, q, f):
            u = read_streams(X, w[f'{p}hc{q}.in'])
            return write_streams(X, w[f'{p}hc{q}.mix'], w[f'{p}hc{q}.out'], f(rms_norm(u, 1 + w[f'{p}norm{q}'], eps)))

        mixer = {'parallel': parallel, 'mamba2': mamba2}[lc['type']]
        X = sublayer(X, 1, lambda h: mixer(h, w, p + 'mix.', lc['mixer'], eps))
        fc = lc.get('mlp')
        if fc is not None:
            X = sublayer(X, 2, lambda h: dense_ff(h, w, p + 'mlp.') if fc['kind'] == 'dense' else moe_ff(h, w, p + 'mlp.', fc))
        if trace is not None:
            trace.append(X.sum(0))
    return rms_norm(X.sum(0), 1 + w['final.norm'], eps) @ w['embed'].T * float(cfg.get('logit_scale', 1.0))
