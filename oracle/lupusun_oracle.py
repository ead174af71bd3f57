"""Plain, slow restatement of the Lupusun decoder (torch on the CPU, float32 or float64), one function per mechanism.

It shares no code with the CUDA path: the tests build small random checkpoints, run both and compare. A sequence is processed
whole, token loops where the design is recurrent, no cache and no state object.

Notation: x residual stream [T, W]; N(v; g) = v / sqrt(mean(v^2) + eps) * g; m the residual factor. The stream starts as
    x = e = N(E[tok]; g_e)
and a layer is
    x <- x + m mixer(N(x; g1));   x <- x + m ff(N(x; g2))         (the second line only where the layer has a feed-forward)
A block of layers can run several times in a row; e is added to x ahead of every pass of the block but the first. Mixers:
  'delta'      gated delta rule: a matrix state per head that decays, is corrected towards the current value at the current key and
               is then read by the query; short causal convolutions with silu in front, unit-length queries and keys shared by groups
               of heads, a head norm and a silu gate behind;
  'attention'  grouped-query attention with projection biases, a partial rotation with blended frequencies (numbers i and
               i + dims / 2 turn together), a per-head unit norm of queries and keys AFTER the rotation, keys limited to the
               query's own chunk of positions, a learned per-head sink in the softmax denominator.
Feed-forward: W_down (relu(W_gate h) * (W_up h)). cfg is the parsed config.json (a dict), w the tensor dict of the checkpoint.
"""
import math

import torch


def rms_norm(v, g, eps):
    v = v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)
    return v if g is None else v * g


def embed(tokens, w, eps, dtype):
    rows = w['embed'][torch.tensor([int(t) for t in tokens])].to(dtype)
    return rms_norm(rows, w['embed.norm'].to(dtype), eps)


# ------------------------------------------------------------------------------------------------ attention
def blended_frequencies(rot):
    """(angle per position of every turning pair, factor on cos and sin). Pair i of n = dims / 2 turns by base^(-i/n); pairs that turn
    slowly over the original context are divided by the factor, fast ones are not, a linear ramp in between"""
    n, base = int(rot['dims']) // 2, float(rot['base'])
    plain = [base ** (-i / n) for i in range(n)]
    sc = rot.get('scaling')
    if not sc:
        return plain, 1.0
    where = lambda turns: n * math.log(float(sc['original']) / (turns * 2 * math.pi)) / math.log(base)
    a, b = math.floor(where(float(sc['fast']))), math.ceil(where(float(sc['slow'])))
    a, b = (0 if a < 0 else a), (2 * n - 1 if b > 2 * n - 1 else b)
    width = b - a if b - a > 0.001 else 0.001
    out = []
    for i, f in enumerate(plain):
        slow = (i - a) / width
        slow = 0.0 if slow < 0 else 1.0 if slow > 1 else slow
        out.append((1 - slow) * f + slow * f / float(sc['factor']))
    return out, 1.0 + 0.1 * math.log(float(sc['factor']))


def rotate_halves(v, pos, rot):
    """v [T, heads, d]: numbers i and i + dims / 2 turn together, the numbers from dims on stay as they are"""
    freq, mag = blended_frequencies(rot)
    n = len(freq)
    ang = pos.to(v.dtype)[:, None] * torch.tensor(freq, dtype=torch.float64).to(v.dtype)[None, :]
    c, s = (torch.cos(ang) * mag)[:, None, :], (torch.sin(ang) * mag)[:, None, :]
    a, b = v[..., :n], v[..., n:2 * n]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., 2 * n:]], -1)


def same_chunk(T, size):
    """[T, T] bool: query i sees key j when j <= i and both lie in the same run of `size` positions (size 0: no runs)"""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    vis = j <= i
    return vis & (torch.div(i, size, rounding_mode='floor') == torch.div(j, size, rounding_mode='floor')) if size else vis


def softmax_with_sink(s, vis, sink):
    """rows of s over the visible keys; exp(sink) joins the denominator only"""
    s = s.masked_fill(~vis, float('-inf'))
    sink = torch.as_tensor(sink, dtype=s.dtype)
    m = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def chunked_attention(h, w, p, mc, eps):
    T = h.shape[0]
    H, G, d = int(mc['heads']), int(mc.get('kv_heads', mc['heads'])), int(mc['dim'])
    dv = int(mc.get('vdim', d))
    lin = lambda n: h @ w[p + n].to(h.dtype).T + w[p + n + '.b'].to(h.dtype)
    pos = torch.arange(T)
    q, k, v = lin('q').view(T, H, d), lin('k').view(T, G, d), lin('v').view(T, G, dv)
    if mc.get('rot'):
        q, k = rotate_halves(q, pos, mc['rot']), rotate_halves(k, pos, mc['rot'])
    q, k = rms_norm(q, None, eps), rms_norm(k, None, eps)
    vis = same_chunk(T, int((mc.get('mask') or {}).get('size') or 0))
    sink = w[p + 'sink'].to(h.dtype)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        out[:, hh] = softmax_with_sink(q[:, hh] @ k[:, g].T * float(mc['scale']), vis, sink[hh]) @ v[:, g]
    return out.reshape(T, H * dv) @ w[p + 'o'].to(h.dtype).T


# ------------------------------------------------------------------------------------------------ gated delta rule
def short_conv(z, cw):
    """z [T, C], cw [C, taps]: each channel over time, the last column of cw meets the current token, zeros before the start"""
    T, taps = z.shape[0], cw.shape[1]
    out = torch.zeros_like(z)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                out[t] += cw[:, j] * z[s]
    return out


def unit(v):
    return v / torch.sqrt((v * v).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, decay, beta):
    """q, k [T, H, d], v [T, H, dv], decay and beta [T, H] -> read-outs [T, H, dv]; the state S [d, dv] of a head starts at zero"""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = S * decay[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum('hdv,hd->hv', S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum('hdv,hd->hv', S, q[t])
    return o


def gated_delta(h, w, p, mc, eps):
    T = h.shape[0]
    H, G, d = int(mc['heads']), int(mc.get('kv_heads', mc['heads'])), int(mc['dim'])
    dv = int(mc.get('vdim', d))
    silu = torch.nn.functional.silu
    lin = lambda n: h @ w[p + n].to(h.dtype).T
    conv = lambda n: silu(short_conv(lin(n), w[p + n + '.conv'].to(h.dtype)))
    of_head = [hh // (H // G) for hh in range(H)]
    q = (unit(conv('q').view(T, G, d)) * d ** -0.5)[:, of_head]
    k = unit(conv('k').view(T, G, d))[:, of_head]
    v = conv('v').view(T, H, dv)
    beta = torch.sigmoid(lin('b'))
    rate = torch.nn.functional.softplus(lin('a') + w[p + 'dt_bias'].to(h.dtype), threshold=1e9)
    decay = torch.exp(-torch.exp(w[p + 'A_log'].to(h.dtype)) * rate)
    o = rms_norm(delta_rule(q, k, v, decay, beta), w[p + 'norm'].to(h.dtype), eps)
    return (o.reshape(T, H * dv) * silu(lin('g'))) @ w[p + 'o'].to(h.dtype).T


def dense_ff(h, w, p):
    return (torch.relu(h @ w[p + 'gate'].to(h.dtype).T) * (h @ w[p + 'up'].to(h.dtype).T)) @ w[p + 'down'].to(h.dtype).T


# ------------------------------------------------------------------------------------------------ the stack
def layer_runs(cfg):
    """[(layer index, add the embedding output first?), ...] in the order the layers run"""
    n, lp = len(cfg['layers']), cfg.get('loop')
    if not lp:
        return [(i, False) for i in range(n)]
    out = [(i, False) for i in range(int(lp['start']))]
    for t in range(int(lp['times'])):
        out += [(i, t > 0 and i == int(lp['start'])) for i in range(int(lp['start']), int(lp['stop']))]
    return out + [(i, False) for i in range(int(lp['stop']), n)]


def forward(cfg, weights, tokens, dtype=torch.float32, trace=None):
    """token ids of ONE sequence -> logits [T, vocab]; `trace` (a list) receives the residual stream after every layer run"""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps, m = float(cfg['norm']['eps']), float(cfg.get('residual_mult', 1.0))
    first = embed(tokens, w, eps, dtype)
    x = first
    for i, again in layer_runs(cfg):
        lc, p = cfg['layers'][i], f'l{i}.'
        if again:
            x = x + first
        mixer = {'delta': gated_delta, 'attention': chunked_attention}[lc['type']]
        x = x + m * mixer(rms_norm(x, w[p + 'norm1'], eps), w, p + 'mix.', lc['mixer'], eps)
        if lc.get('mlp') is not None:
            if lc['mlp']['kind'] != 'dense':
                raise NotImplementedError(lc['mlp']['kind'])
            x = x + m * dense_ff(rms_norm(x, w[p + 'norm2'], eps), w, p + 'mlp.')
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, w['final.norm'], eps) @ w['head'].T
