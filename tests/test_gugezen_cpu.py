"""Host-side parts of the Gugezen integration that need no GPU: config parsing, the registry, checkpoint shapes, what the page pool
allocates per layer, the wavelength-dependent frequencies, the oracle's own mechanisms on hand-made inputs, and the power of the test
weights to show a mistake (planted in the oracle)."""
import math

import pytest
import torch

import phi3_b200  # noqa: F401
from phi3_b200 import configs, registry, weights
from phi3_b200.paged import PagePool, PAGE
from oracle import gugezen_oracle as O

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    d = configs.tiny_gugezen()
    c = configs.GugezenConfig(d)
    assert (c.vocab_size, c.width, c.eps, c.embed_scale, c.streams, c.logit_scale, c.num_hidden_layers) == (300, 96, 1e-5, 0.7, 3, 1.5, 6)
    assert [l.mixer.kind for l in c.layers] == ['parallel', 'mamba2', 'parallel', 'mamba2', 'parallel', 'mamba2']
    assert c.sources == [0, 1, 0, 3, 4, 1]
    p, m = c.layers[0].mixer, c.layers[3].mixer
    assert (p.att.heads, p.att.kv_heads, p.att.dim, p.att.vdim, p.att.scale) == (6, 3, 24, 40, 2.0 * 24 ** -0.5)
    assert (p.mem.heads, p.mem.dim, p.mem.vdim, p.att_scale, p.mem_scale) == (3, 24, 40, 0.8, 1.1) and p.mem.decay == d['layers'][0]['mixer']['right']['decay']
    r = p.att.rot
    assert (r.base, r.dims, r.scaling.factor, r.scaling.low, r.scaling.high, r.scaling.original) == (10000.0, 16, 4.0, 1.0, 4.0, 64.0)
    assert c.layers[4].mixer.att.rot.scaling is None
    assert (m.heads, m.vdim, m.state, m.groups, m.taps, m.norm_groups, m.inner, m.channels) == (4, 40, 24, 4, 3, 2, 160, 160 + 2 * 4 * 24)
    f = c.layers[0].ff
    assert (f.kind, f.ff, f.experts, f.top, f.shared_ff) == ('moe', 40, 5, 2, 72) and c.layers[4].ff.shared_ff == 0
    assert c.layers[1].ff.kind == 'dense' and c.layers[1].ff.ff == 136 and c.layers[3].ff is None
    assert c.kv_layout() == [(3, 24, 40), (0, 0, 0), (3, 24, 40), (0, 0, 0), (1, 40, 24), (0, 0, 0)]
    bare = configs.tiny_gugezen(layers=[configs.tiny_gugezen()['layers'][i] for i in (0, 1)])
    for k in ('embedding', 'streams', 'logit_scale'):
        del bare[k]
    for k in ('kv_heads', 'vdim', 'rot'):
        del bare['layers'][0]['mixer']['left'][k]
    for k in ('left_scale', 'right_scale'):
        del bare['layers'][0]['mixer'][k]
    del bare['layers'][0]['mixer']['right']['vdim']
    for k in ('groups', 'norm_groups'):
        del bare['layers'][1]['mixer'][k]
    b = configs.GugezenConfig(bare)
    b0, b1 = (l.mixer for l in b.layers)
    assert (b.embed_scale, b.streams, b.logit_scale) == (1.0, 1, 1.0) and (b0.att.kv_heads, b0.att.vdim, b0.att.rot) == (6, 24, None)
    assert (b0.att_scale, b0.mem_scale, b0.mem.vdim, b1.groups, b1.norm_groups) == (1.0, 1.0, 24, 1, 1)


@pytest.mark.parametrize('key,val,err', [
    (('layers', 1, 'type'), 'recurrent', NotImplementedError), (('layers', 3, 'mlp'), {'kind': 'none'}, NotImplementedError),
    (('layers', 4, 'mixer', 'left', 'rot', 'dims'), 7, ValueError), (('layers', 4, 'mixer', 'left', 'rot', 'dims'), 42, ValueError),
    (('layers', 4, 'mixer', 'left', 'kv_heads'), 3, ValueError), (('layers', 4, 'mixer', 'left', 'vdim'), 5000, NotImplementedError),
    (('layers', 4, 'mixer', 'right', 'decay'), [0.5], ValueError), (('layers', 4, 'mixer', 'right', 'dim'), 600, NotImplementedError),
    (('layers', 3, 'mixer', 'groups'), 3, ValueError), (('layers', 3, 'mixer', 'norm_groups'), 3, ValueError),
    (('layers', 3, 'mixer', 'conv'), 0, ValueError), (('layers', 3, 'mixer', 'state'), 513, NotImplementedError),
    (('layers', 4, 'mlp', 'router', 'top'), 5, ValueError), (('layers', 4, 'mlp', 'router', 'experts'), 1025, NotImplementedError),
    (('layers', 2, 'weights_of'), 2, ValueError), (('layers', 2, 'weights_of'), 6, ValueError), (('layers', 2, 'weights_of'), 1, ValueError),
    (('streams',), -1, ValueError), (('streams',), 17, NotImplementedError)])
def test_config_refuses_what_it_cannot_mean(key, val, err):
    import copy
    bad = copy.deepcopy(configs.tiny_gugezen())               # layers that share tensors also share their sub-dicts
    node = bad
    for k in key[:-1]:
        node = node[k]
    node[key[-1]] = val
    with pytest.raises(err):
        configs.GugezenConfig(bad)


def test_registry_and_checkpoint_shapes():
    ent = registry.entry_for({'architecture': 'Gugezen'})
    assert ent.engine == 'paged' and isinstance(ent.config(configs.tiny_gugezen()), configs.GugezenConfig)
    d = configs.tiny_gugezen()
    shapes, w = weights.gugezen_tensor_shapes(d), weights.random_gugezen_weights(d, 0)
    assert set(shapes) == set(w) and all(tuple(w[k].shape) == tuple(v) for k, v in shapes.items())
    assert shapes['embed'] == (300, 96) and 'head' not in shapes and shapes['l0.mix.left.q'] == (144, 96) and shapes['l0.mix.left.v.b'] == (120,)
    assert shapes['l0.mix.left.g'] == (240, 96) and shapes['l0.mix.right.o'] == (96, 120) and shapes['l0.mix.right.norm'] == (120,)
    assert shapes['l1.mix.in'] == (2 * 144 + 2 * 2 * 40 + 6, 96) and shapes['l1.mix.conv'] == (304, 4) and shapes['l1.mix.D'] == (6,)
    assert shapes['l0.mlp.e4.up'] == (40, 96) and 'l0.mlp.e5.up' not in shapes and shapes['l0.mlp.shared.down'] == (96, 72)
    assert not any(k.startswith(('l2.', 'l5.')) for k in shapes) and 'l3.norm2' not in shapes and 'l3.hc2.in' not in shapes
    assert shapes['l3.hc1.mix'] == (3, 3) and shapes['l4.hc2.out'] == (3,) and 'l4.mlp.shared.up' not in shapes


def test_page_pool_holds_a_cache_and_a_state_per_layer():
    c = configs.GugezenConfig(configs.tiny_gugezen())
    pool = PagePool(c.kv_layout(), 2 * PAGE, 2, torch.float32, 'cpu', state_layout=[3 * 24 * 40, 6 * 24 * 40, 3 * 304])
    assert [t.numel() for t in pool.k] == [2 * 3 * 64 * 24, 0, 2 * 3 * 64 * 24, 0, 2 * 64 * 40, 0]
    assert pool.k[0].data_ptr() != pool.k[2].data_ptr()       # layers that share tensors keep caches of their own


@pytest.mark.parametrize('rot', [{'base': 10000.0, 'dims': 16, 'scaling': {'factor': 4.0, 'low': 1.0, 'high': 4.0, 'original': 64}},
                                 {'base': 500.0, 'dims': 2, 'scaling': {'factor': 32.0, 'low': 0.5, 'high': 3.0, 'original': 4096}},
                                 {'base': 1e6, 'dims': 48, 'scaling': {'factor': 1.0, 'low': 1.0, 'high': 2.0, 'original': 100}},
                                 {'base': 100.0, 'dims': 12, 'scaling': {'factor': 2.5, 'low': 2.0, 'high': 9.0, 'original': 20}},
                                 {'base': 100.0, 'dims': 12}])
def test_frequencies_of_the_product_and_the_oracle_agree(rot):
    from types import SimpleNamespace
    sc = rot.get('scaling')
    got = configs.wavelength_frequencies(SimpleNamespace(base=rot['base'], dims=rot['dims'], scaling=SimpleNamespace(**sc) if sc else None))
    want = O.stretched_frequencies(rot)
    assert len(got) == rot['dims'] // 2 and all(abs(a - b) <= 1e-12 * b for a, b in zip(got, want))


# ------------------------------------------------------------------------------------------------ the oracle's mechanisms
def test_oracle_frequencies_by_hand():
    # base 100, four pairs: 1, 0.316, 0.1, 0.0316; wavelengths 6.3, 19.9, 62.8, 198.7; original 60: borders 15 (high 4) and 60 (low 1)
    f = O.stretched_frequencies({'base': 100.0, 'dims': 8, 'scaling': {'factor': 5.0, 'low': 1.0, 'high': 4.0, 'original': 60}})
    assert f[0] == 1.0 and abs(f[2] - 0.1 / 5) < 1e-15 and abs(f[3] - 100 ** -0.75 / 5) < 1e-15
    f1 = 100 ** -0.25
    s = (60 / (2 * math.pi / f1) - 1) / 3
    assert 0 < s < 1 and abs(f[1] - ((1 - s) * f1 / 5 + s * f1)) < 1e-15
    assert O.stretched_frequencies({'base': 100.0, 'dims': 4}) == [1.0, 0.1]


def test_oracle_rotation_pairs_neighbours_and_is_partial():
    rot = {'base': 100.0, 'dims': 4}
    v = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0, 6.0]]], dtype=F64).repeat(2, 1, 1)
    out = O.rotate_neighbours(v, torch.tensor([0, 3]), rot)
    assert torch.equal(out[0, 0], v[0, 0])
    a, b = 3.0, 0.3                                           # numbers 0 and 1 turn by 1 per position, 2 and 3 by 0.1; 4 and 5 pass
    want = [math.cos(a) - 2 * math.sin(a), 2 * math.cos(a) + math.sin(a), 3 * math.cos(b) - 4 * math.sin(b), 4 * math.cos(b) + 3 * math.sin(b), 5.0, 6.0]
    assert torch.allclose(out[1, 0], torch.tensor(want, dtype=F64))


def test_oracle_sink_counts_once_and_has_no_value():
    p = O.softmax_with_sink(torch.tensor([[0.3, -1.0, 2.0]], dtype=F64), torch.tensor([[True, False, True]]), 0.7)
    den = math.exp(0.3) + math.exp(2.0) + math.exp(0.7)
    assert torch.allclose(p, torch.tensor([[math.exp(0.3) / den, 0.0, math.exp(2.0) / den]], dtype=F64))


def test_oracle_attention_against_a_token_loop():
    torch.manual_seed(1)
    T, W, H, G, d, dv = 9, 8, 4, 2, 6, 5
    mc = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=0.7, rot={'base': 50.0, 'dims': 4})
    w = {'p.' + n: torch.randn(s, dtype=F64) for n, s in
         {'q': (H * d, W), 'k': (G * d, W), 'v': (G * dv, W), 'g': (H * dv, W), 'o': (W, H * dv), 'q.b': (H * d,), 'k.b': (G * d,), 'v.b': (G * dv,),
          'sink': (H,)}.items()}
    h = torch.randn(T, W, dtype=F64)
    got = O.attention(h, w, 'p.', mc)
    q, k = (h @ w['p.q'].T + w['p.q.b']).view(T, H, d), (h @ w['p.k'].T + w['p.k.b']).view(T, G, d)
    v = (h @ w['p.v'].T + w['p.v.b']).view(T, G, dv)
    pos = torch.arange(T)
    q, k = O.rotate_neighbours(q, pos, mc['rot']), O.rotate_neighbours(k, pos, mc['rot'])
    heads = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        for t in range(T):
            e = torch.exp(torch.stack([q[t, hh] @ k[j, hh // 2] * 0.7 for j in range(t + 1)]))
            heads[t, hh] = (e[:, None] * v[:t + 1, hh // 2]).sum(0) / (e.sum() + torch.exp(w['p.sink'][hh]))
    want = (heads.reshape(T, -1) / (1 + torch.exp(-(h @ w['p.g'].T)))) @ w['p.o'].T
    assert torch.allclose(got, want)


def test_oracle_memory_is_a_decayed_sum():
    torch.manual_seed(2)
    T, H, d, dv = 7, 2, 3, 4
    q, k, v = torch.randn(T, H, d, dtype=F64), torch.randn(T, H, d, dtype=F64), torch.randn(T, H, dv, dtype=F64)
    decay = torch.rand(T, H, dtype=F64)
    got = O.decayed_memory(q, k, v, decay)
    for t in range(T):
        for h in range(H):
            want = sum(torch.prod(decay[j + 1:t + 1, h]) * (k[j, h] @ q[t, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(got[t, h], want)


def test_oracle_linear_half_norms_all_heads_together():
    torch.manual_seed(3)
    T, W, H, d, dv, eps = 6, 5, 3, 4, 2, 1e-2
    mc = dict(heads=H, dim=d, vdim=dv, decay=[0.5, 0.9, 1.0])
    w = {'p.' + n: torch.randn(s, dtype=F64) for n, s in {'q': (H * d, W), 'k': (H * d, W), 'v': (H * dv, W), 'g': (H * dv, W), 'o': (W, H * dv),
                                                           'norm': (H * dv,)}.items()}
    h = torch.randn(T, W, dtype=F64)
    act = lambda n, s: torch.nn.functional.silu(h @ w['p.' + n].T).view(T, H, s)
    o = O.decayed_memory(act('q', d), act('k', d), act('v', dv), torch.tensor(mc['decay'], dtype=F64).expand(T, H)).reshape(T, H * dv)
    n = torch.stack([r / torch.sqrt((r * r).mean() + eps) for r in o]) * w['p.norm']
    assert torch.allclose(O.lightning(h, w, 'p.', mc, eps), (n * torch.sigmoid(h @ w['p.g'].T)) @ w['p.o'].T)


def test_oracle_state_space_mixer_against_a_token_loop():
    torch.manual_seed(4)
    T, W, H, dv, N, G, taps, parts, eps = 8, 6, 4, 3, 5, 2, 3, 3, 1e-2
    inner, C = H * dv, H * dv + 2 * G * N
    mc = dict(heads=H, vdim=dv, state=N, groups=G, conv=taps, norm_groups=parts)
    w = {'p.' + n: torch.randn(s, dtype=F64) for n, s in {'in': (inner + C + H, W), 'conv': (C, taps), 'conv.b': (C,), 'dt_bias': (H,), 'A_log': (H,),
                                                           'D': (H,), 'norm': (inner,), 'o': (W, inner)}.items()}
    h = torch.randn(T, W, dtype=F64)
    p = h @ w['p.in'].T
    S = torch.zeros(H, N, dv, dtype=F64)
    rows = []
    for t in range(T):
        z, dt = p[t, :inner], p[t, inner + C:]
        c = w['p.conv.b'].clone()
        for j in range(taps):                                 # taps[:, -1] meets token t itself
            if t - j >= 0:
                c = c + w['p.conv'][:, taps - 1 - j] * p[t - j, inner:inner + C]
        c = c / (1 + torch.exp(-c))
        y = torch.zeros(inner, dtype=F64)
        for hh in range(H):
            g = hh // (H // G)
            x, B, Cc = c[hh * dv:(hh + 1) * dv], c[inner + g * N:inner + (g + 1) * N], c[inner + G * N + g * N:inner + G * N + (g + 1) * N]
            step = torch.log(1 + torch.exp(dt[hh] + w['p.dt_bias'][hh]))
            S[hh] = torch.exp(-torch.exp(w['p.A_log'][hh]) * step) * S[hh] + step * B[:, None] * x[None, :]
            y[hh * dv:(hh + 1) * dv] = Cc @ S[hh] + w['p.D'][hh] * x
        y = y * z / (1 + torch.exp(-z))                       # gated first, normed in parts after that
        n = inner // parts
        rows.append(torch.cat([y[i * n:(i + 1) * n] / torch.sqrt((y[i * n:(i + 1) * n] ** 2).mean() + eps) for i in range(parts)]) * w['p.norm'])
    assert torch.allclose(O.mamba2(h, w, 'p.', mc, eps), torch.stack(rows) @ w['p.o'].T)


def test_oracle_streams_all_move_from_the_old_ones():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=F64)               # two streams of one token
    M, b, y = torch.tensor([[0.5, 2.0], [3.0, 0.25]], dtype=F64), torch.tensor([1.0, -1.0], dtype=F64), torch.tensor([[100.0, 200.0]], dtype=F64)
    out = O.write_streams(X, M, b, y)
    assert out[0].tolist() == [[0.5 + 30 + 100, 1 + 60 + 200]] and out[1].tolist() == [[2 + 2.5 - 100, 4 + 5 - 200]]   # M[from, to]
    assert O.read_streams(X, torch.tensor([2.0, 0.5], dtype=F64)).tolist() == [[7.0, 14.0]]


def test_oracle_gelus_and_mixture():
    z = torch.tensor([-3.0, -0.5, 0.0, 1.0, 4.0], dtype=F64)
    assert torch.allclose(O.gelu_erf(z), torch.nn.functional.gelu(z)) and torch.allclose(O.gelu_tanh(z), torch.nn.functional.gelu(z, approximate='tanh'))
    torch.manual_seed(5)
    W, ff, E = 4, 3, 5
    w = {f'm.e{e}.{n}': torch.randn(s, dtype=F64) for e in range(E) for n, s in (('up', (ff, W)), ('down', (W, ff)))}
    w['m.router'] = torch.randn(E, W, dtype=F64)
    w['m.shared.up'], w['m.shared.down'] = torch.randn(2, W, dtype=F64), torch.randn(W, 2, dtype=F64)
    h = torch.randn(6, W, dtype=F64)
    got = O.moe_ff(h, w, 'm.', {'kind': 'moe', 'expert': {'ff': ff}, 'router': {'experts': E, 'top': 2}, 'shared': {'ff': 2}})
    for t in range(6):
        s = torch.softmax(w['m.router'] @ h[t], 0)
        a, b = s.topk(2).indices.tolist()
        u = lambda n: w[n + 'down'] @ torch.nn.functional.gelu(w[n + 'up'] @ h[t])
        want = (s[a] * u(f'm.e{a}.') + s[b] * u(f'm.e{b}.')) / (s[a] + s[b]) + u('m.shared.')
        assert torch.allclose(got[t], want)


# ------------------------------------------------------------------------------------------------ mistakes planted in the oracle
def _plain(cfg, w, toks):
    return O.forward(cfg, w, toks, F64)


def _patch(monkeypatch, name, fn):
    monkeypatch.setattr(O, name, fn)


MISTAKES = {
    'sink left out': lambda mp: _patch(mp, 'softmax_with_sink', lambda s, vis, sink: torch.softmax(s.masked_fill(~vis, float('-inf')), -1)),
    'half pairs': lambda mp: _patch(mp, 'rotate_neighbours', lambda v, pos, rot: torch.cat([
        v[..., :rot['dims'] // 2] * torch.cos(pos[:, None] * torch.tensor(O.stretched_frequencies(rot), dtype=v.dtype))[:, None]
        - v[..., rot['dims'] // 2:rot['dims']] * torch.sin(pos[:, None] * torch.tensor(O.stretched_frequencies(rot), dtype=v.dtype))[:, None],
        v[..., rot['dims'] // 2:rot['dims']] * torch.cos(pos[:, None] * torch.tensor(O.stretched_frequencies(rot), dtype=v.dtype))[:, None]
        + v[..., :rot['dims'] // 2] * torch.sin(pos[:, None] * torch.tensor(O.stretched_frequencies(rot), dtype=v.dtype))[:, None],
        v[..., rot['dims']:]], -1)),
    'frequencies not stretched': lambda mp: _patch(mp, 'stretched_frequencies', lambda rot: [rot['base'] ** (-2 * i / rot['dims']) for i in range(rot['dims'] // 2)]),
    'decay lost': lambda mp: _patch(mp, 'decayed_memory', lambda q, k, v, decay, f=O.decayed_memory: f(q, k, v, torch.ones_like(decay))),
    'taps reversed': lambda mp: _patch(mp, 'short_conv', lambda z, cw, b, f=O.short_conv: f(z, cw.flip(1), b)),
    'convolution bias lost': lambda mp: _patch(mp, 'short_conv', lambda z, cw, b, f=O.short_conv: f(z, cw, 0 * b)),
    'one norm over all parts': lambda mp: _patch(mp, 'parts_norm', lambda v, parts, g, eps: O.rms_norm(v, g, eps)),
    'streams mixed the other way': lambda mp: _patch(mp, 'write_streams', lambda X, M, b, y, f=O.write_streams: f(X, M.T, b, y)),
    'only the first stream read': lambda mp: _patch(mp, 'read_streams', lambda X, a: a[0] * X[0]),
    'relu in the experts': lambda mp: _patch(mp, 'gelu_erf', lambda v: torch.relu(v)),
}


@pytest.mark.parametrize('name', list(MISTAKES))
def test_a_mistake_shows_in_the_logits(monkeypatch, name):
    """the random test weights make every mechanism count: a planted mistake moves the logits by at least a hundred times the fp32
    tolerance of the GPU tests"""
    cfg = configs.tiny_gugezen()
    w = weights.random_gugezen_weights(cfg, 1)
    toks = torch.randint(0, cfg['vocab'], (40,), generator=torch.Generator().manual_seed(2)).tolist()
    ref = _plain(cfg, w, toks)
    MISTAKES[name](monkeypatch)
    d = _plain(cfg, w, toks) - ref
    d = d - d.mean(-1, keepdim=True)
    assert float(d.pow(2).mean(-1).sqrt().max() / ref.std()) > 100 * 2e-4
