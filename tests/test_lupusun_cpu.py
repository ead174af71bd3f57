"""Host-side parts of the Lupusun integration that need no GPU: config parsing, the registry, checkpoint shapes, what the page pool
allocates per layer run, the frequencies of the blended rotation, the oracle's own mechanisms on hand-made inputs, and the power of the
test weights to show a mistake (planted in the oracle)."""
import math

import pytest
import torch

import phi3_b200  # noqa: F401
from phi3_b200 import configs, registry, weights
from phi3_b200.paged import PagePool, PAGE
from oracle import lupusun_oracle as O

F64 = torch.float64


def test_config_reads_every_size_and_constant():
    d = configs.tiny_lupusun()
    c = configs.LupusunConfig(d)
    assert c.vocab_size == 300 and c.width == 96 and c.eps == 1e-5 and c.residual_mult == 0.8 and c.num_hidden_layers == 4
    assert [l.mixer.kind for l in c.layers] == ['delta', 'attention', 'delta', 'attention']
    d0, a1, d2, a3 = (l.mixer for l in c.layers)
    assert (d0.heads, d0.kv_heads, d0.dim, d0.vdim, d0.taps) == (4, 2, 24, 40, 4) and (d2.taps, d2.kv_heads) == (3, 3)
    assert (a1.heads, a1.kv_heads, a1.dim, a1.vdim, a1.chunk, a1.scale) == (6, 3, 40, 24, 50, 2.0 * 40 ** -0.5)
    assert (a1.rot.base, a1.rot.dims) == (10000.0, 16)
    assert (a1.rot.scaling.factor, a1.rot.scaling.original, a1.rot.scaling.fast, a1.rot.scaling.slow) == (4.0, 64.0, 16.0, 1.5)
    assert a3.chunk == 0 and a3.rot.scaling is None and c.layers[2].ff is None and c.layers[0].ff.ff == 136
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 2)
    assert c.runs == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    # every run has a cache of its own; a recurrent run caches nothing
    assert c.kv_layout() == [(0, 0, 0), (3, 40, 24), (0, 0, 0), (3, 40, 24), (0, 0, 0), (1, 24, 56)]
    plain = configs.LupusunConfig(configs.tiny_lupusun(loop=None))
    assert plain.loop is None and plain.runs == [(i, False) for i in range(4)]
    bare = configs.tiny_lupusun()
    for k in ('rot', 'mask', 'vdim', 'kv_heads'):
        bare['layers'][1]['mixer'].pop(k)
    del bare['residual_mult']
    cb = configs.LupusunConfig(bare)
    b1 = cb.layers[1].mixer
    assert (b1.rot, b1.chunk, b1.vdim, b1.kv_heads) == (None, 0, 40, 6) and cb.residual_mult == 1.0
    for key, val, err in ((('layers', 0, 'type'), 'recurrent', NotImplementedError), (('layers', 0, 'mlp', 'kind'), 'moe', NotImplementedError),
                          (('layers', 1, 'mixer', 'rot', 'dims'), 7, ValueError), (('layers', 1, 'mixer', 'rot', 'dims'), 42, ValueError),
                          (('layers', 1, 'mixer', 'kv_heads'), 4, ValueError), (('layers', 0, 'mixer', 'kv_heads'), 3, ValueError),
                          (('layers', 0, 'mixer', 'conv'), 0, ValueError), (('layers', 0, 'mixer', 'dim'), 600, NotImplementedError),
                          (('layers', 1, 'mixer', 'mask', 'size'), -1, ValueError), (('layers', 1, 'mixer', 'vdim'), 5000, NotImplementedError),
                          (('loop', 'stop'), 5, ValueError), (('loop', 'start'), 3, ValueError), (('loop', 'times'), 0, ValueError)):
        bad = configs.tiny_lupusun()
        node = bad
        for k in key[:-1]:
            node = node[k]
        node[key[-1]] = val
        with pytest.raises(err):
            configs.LupusunConfig(bad)


def test_registry_and_checkpoint_shapes():
    ent = registry.entry_for({'architecture': 'Lupusun'})
    assert ent.engine == 'paged' and isinstance(ent.config(configs.tiny_lupusun()), configs.LupusunConfig)
    d = configs.tiny_lupusun()
    shapes, w = weights.lupusun_tensor_shapes(d), weights.random_lupusun_weights(d, 0)
    assert set(shapes) == set(w) and all(tuple(w[k].shape) == tuple(v) for k, v in shapes.items())
    assert shapes['embed'] == (300, 96) and shapes['embed.norm'] == (96,) and shapes['head'] == (300, 96)
    assert shapes['l0.mix.q'] == (48, 96) and shapes['l0.mix.v'] == (160, 96) and shapes['l0.mix.k.conv'] == (48, 4)
    assert shapes['l0.mix.v.conv'] == (160, 4) and shapes['l0.mix.b'] == (4, 96) and shapes['l0.mix.A_log'] == (4,)
    assert shapes['l0.mix.norm'] == (40,) and shapes['l0.mix.g'] == (160, 96) and shapes['l0.mlp.gate'] == (136, 96)
    assert shapes['l1.mix.q.b'] == (240,) and shapes['l1.mix.v'] == (72, 96) and shapes['l1.mix.sink'] == (6,) and shapes['l1.mix.o'] == (96, 144)
    assert 'l2.norm2' not in shapes and 'l0.mix.q.b' not in shapes and shapes['l3.mlp.down'] == (96, 88)


def test_page_pool_holds_a_cache_or_a_state_per_layer_run():
    c = configs.LupusunConfig(configs.tiny_lupusun())
    hist = [(m.taps - 1) * (2 * m.kv_heads * m.dim + m.heads * m.vdim) for m in (c.layers[0].mixer, c.layers[2].mixer)]
    mats = [m.heads * m.dim * m.vdim for m in (c.layers[0].mixer, c.layers[2].mixer)]
    pool = PagePool(c.kv_layout(), 3 * PAGE, 2, torch.float32, 'cpu', state_layout=[mats[0], hist[0], mats[1], hist[1], mats[1], 0])
    assert [t.numel() for t in pool.k] == [0, 3 * 3 * 64 * 40, 0, 3 * 3 * 64 * 40, 0, 3 * 64 * 24]
    assert [tuple(s.shape) for s in pool.state] == [(2, 3840), (2, 768), (2, 1920), (2, 576), (2, 1920), (2, 0)]
    assert pool.k[1].data_ptr() != pool.k[3].data_ptr()


@pytest.mark.parametrize('rot', [{'base': 10000.0, 'dims': 16, 'scaling': {'factor': 4.0, 'original': 64, 'fast': 16.0, 'slow': 1.5}},
                                 {'base': 500.0, 'dims': 2, 'scaling': {'factor': 32.0, 'original': 4096, 'fast': 32.0, 'slow': 1.0}},
                                 {'base': 1e6, 'dims': 48, 'scaling': {'factor': 1.0, 'original': 100, 'fast': 3.0, 'slow': 3.0}},
                                 {'base': 100.0, 'dims': 12, 'scaling': {'factor': 2.5, 'original': 20, 'fast': 0.01, 'slow': 0.001}},
                                 {'base': 100.0, 'dims': 12}])
def test_blended_frequencies_of_the_product_and_the_oracle_agree(rot):
    from types import SimpleNamespace
    sc = rot.get('scaling')
    ns = SimpleNamespace(base=rot['base'], dims=rot['dims'], scaling=SimpleNamespace(**sc) if sc else None)
    got, mag = configs.yarn_frequencies(ns)
    want, wmag = O.blended_frequencies(rot)
    assert len(got) == rot['dims'] // 2 and all(abs(a - b) <= 1e-12 * b for a, b in zip(got, want)) and abs(mag - wmag) < 1e-15


# ------------------------------------------------------------------------------------------------ the oracle's mechanisms
def test_oracle_blended_frequencies_by_hand():
    rot = {'base': 10000.0, 'dims': 8, 'scaling': {'factor': 8.0, 'original': 1000, 'fast': 20.0, 'slow': 1.0}}
    f, mag = O.blended_frequencies(rot)
    # the pair that makes t turns over 1000 positions: 8 ln(1000 / (2 pi t)) / (2 ln 10000) = 0.90 (t = 20), 2.20 (t = 1)
    lo, hi = 0, 3
    for i in range(4):
        plain, slow = 10000.0 ** (-2 * i / 8), min(max((i - lo) / (hi - lo), 0), 1)
        assert abs(f[i] - (plain / 8.0 * slow + plain * (1 - slow))) < 1e-15
    assert abs(mag - (1 + 0.1 * math.log(8.0))) < 1e-15
    assert O.blended_frequencies({'base': 100.0, 'dims': 4}) == ([1.0, 0.1], 1.0)


def test_oracle_rotation_pairs_halves_and_is_partial():
    rot = {'base': 100.0, 'dims': 4, 'scaling': {'factor': 3.0, 'original': 50, 'fast': 4.0, 'slow': 1.0}}
    f, mag = O.blended_frequencies(rot)
    v = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0, 6.0]]], dtype=F64).repeat(2, 1, 1)
    out = O.rotate_halves(v, torch.tensor([0, 3]), rot)
    assert torch.allclose(out[0, 0], torch.tensor([mag, 2 * mag, 3 * mag, 4 * mag, 5, 6], dtype=F64))
    a0, a1 = 3 * f[0], 3 * f[1]                               # number 0 turns with 2, number 1 with 3; 4 and 5 pass
    want = [mag * (1 * math.cos(a0) - 3 * math.sin(a0)), mag * (2 * math.cos(a1) - 4 * math.sin(a1)),
            mag * (3 * math.cos(a0) + 1 * math.sin(a0)), mag * (4 * math.cos(a1) + 2 * math.sin(a1)), 5.0, 6.0]
    assert torch.allclose(out[1, 0], torch.tensor(want, dtype=F64))


def test_oracle_chunks_and_sink():
    vis = O.same_chunk(7, 3)
    assert vis[2].tolist() == [True, True, True, False, False, False, False] and vis[3].tolist() == [False] * 3 + [True] + [False] * 3
    assert vis[5].tolist() == [False] * 3 + [True] * 3 + [False] and vis[6].tolist() == [False] * 6 + [True]
    assert O.same_chunk(4, 0).tolist() == torch.ones(4, 4).tril().bool().tolist() and O.same_chunk(3, 1).tolist() == torch.eye(3).bool().tolist()
    s = torch.tensor([[0.3, -1.0, 2.0]], dtype=F64)
    p = O.softmax_with_sink(s, torch.tensor([[True, False, True]]), 0.7)
    den = math.exp(0.3) + math.exp(2.0) + math.exp(0.7)       # the sink counts once, unscaled, and has no value
    assert torch.allclose(p, torch.tensor([[math.exp(0.3) / den, 0.0, math.exp(2.0) / den]], dtype=F64))


def test_oracle_attention_against_a_token_loop():
    torch.manual_seed(1)
    T, W, H, G, d, dv, size = 11, 8, 4, 2, 6, 5, 4
    mc = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=0.7, mask={'size': size},
              rot={'base': 50.0, 'dims': 4, 'scaling': {'factor': 2.0, 'original': 30, 'fast': 3.0, 'slow': 0.5}})
    w = {'p.' + n: torch.randn(s, dtype=F64) for n, s in dict(q=(H * d, W), k=(G * d, W), v=(G * dv, W), o=(W, H * dv)).items()}
    for n, s in (('q.b', H * d), ('k.b', G * d), ('v.b', G * dv), ('sink', H)):
        w['p.' + n] = torch.randn(s, dtype=F64)
    h = torch.randn(T, W, dtype=F64)
    got = O.chunked_attention(h, w, 'p.', mc, 1e-2)
    q, k = (h @ w['p.q'].T + w['p.q.b']).view(T, H, d), (h @ w['p.k'].T + w['p.k.b']).view(T, G, d)
    v = (h @ w['p.v'].T + w['p.v.b']).view(T, G, dv)
    pos = torch.arange(T)
    q, k = O.rotate_halves(q, pos, mc['rot']), O.rotate_halves(k, pos, mc['rot'])
    unit = lambda x: x / torch.sqrt((x * x).mean() + 1e-2)    # eps inside the root, no weight, after the rotation
    heads = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        for t in range(T):
            js = [j for j in range(t + 1) if j // size == t // size]
            e = torch.exp(torch.stack([unit(q[t, hh]) @ unit(k[j, hh // 2]) * 0.7 for j in js]))
            heads[t, hh] = sum(e[n] / (e.sum() + torch.exp(w['p.sink'][hh])) * v[j, hh // 2] for n, j in enumerate(js))
    assert torch.allclose(got, heads.reshape(T, H * dv) @ w['p.o'].T, atol=1e-10)


def test_oracle_short_convolution():
    z = torch.arange(1.0, 7.0, dtype=F64)[:, None] * torch.tensor([[1.0, 10.0]], dtype=F64)
    cw = torch.tensor([[1.0, 2.0, 3.0], [0.0, 0.0, 1.0]], dtype=F64)
    out = O.short_conv(z, cw)                                 # the last tap meets the current token, zeros before the start
    assert out[0].tolist() == [3.0, 10.0] and out[1].tolist() == [2.0 * 1 + 3.0 * 2, 20.0] and out[4].tolist() == [1 * 3 + 2 * 4 + 3 * 5.0, 50.0]
    assert torch.equal(O.short_conv(z, torch.tensor([[2.0], [1.0]], dtype=F64)), z * torch.tensor([2.0, 1.0], dtype=F64))


def test_oracle_delta_rule_against_its_closed_forms():
    torch.manual_seed(2)
    T, H, d, dv = 7, 2, 4, 3
    q, k, v = torch.randn(T, H, d, dtype=F64), O.unit(torch.randn(T, H, d, dtype=F64)), torch.randn(T, H, dv, dtype=F64)
    decay, beta = torch.rand(T, H, dtype=F64), torch.rand(T, H, dtype=F64)
    o = O.delta_rule(q, k, v, decay, beta)
    # one matrix recurrence: S_t = g_t (I - b_t k_t k_t^T) S_(t-1) + b_t k_t v_t^T
    for hh in range(H):
        S = torch.zeros(d, dv, dtype=F64)
        for t in range(T):
            kk = k[t, hh][:, None]
            S = decay[t, hh] * (torch.eye(d, dtype=F64) - beta[t, hh] * kk @ kk.T) @ S + beta[t, hh] * kk @ v[t, hh][None, :]
            assert torch.allclose(o[t, hh], S.T @ q[t, hh], atol=1e-12)
    # beta 1, no decay, unit keys: the read-out at the key just written is the value just written
    o1 = O.delta_rule(k, k, v, torch.ones(T, H, dtype=F64), torch.ones(T, H, dtype=F64))
    assert torch.allclose(o1, v, atol=1e-5)


def test_oracle_delta_mixer_shares_heads_and_gates():
    torch.manual_seed(3)
    T, W, H, G, d, dv, taps = 5, 6, 4, 2, 3, 2, 2
    mc = dict(heads=H, kv_heads=G, dim=d, vdim=dv, conv=taps)
    w = {'p.' + n: torch.randn(s, dtype=F64) for n, s in dict(q=(G * d, W), k=(G * d, W), v=(H * dv, W), g=(H * dv, W), b=(H, W), a=(H, W),
                                                               o=(W, H * dv)).items()}
    w.update({'p.q.conv': torch.randn(G * d, taps, dtype=F64), 'p.k.conv': torch.randn(G * d, taps, dtype=F64),
              'p.v.conv': torch.randn(H * dv, taps, dtype=F64), 'p.A_log': torch.randn(H, dtype=F64), 'p.dt_bias': torch.randn(H, dtype=F64),
              'p.norm': torch.rand(dv, dtype=F64) + 0.5})
    h = torch.randn(T, W, dtype=F64)
    got = O.gated_delta(h, w, 'p.', mc, 1e-3)
    silu = lambda x: x / (1 + torch.exp(-x))
    out = torch.zeros(T, H * dv, dtype=F64)
    for hh in range(H):
        S = torch.zeros(d, dv, dtype=F64)
        g = hh // 2                                            # heads 0 and 1 use query / key head 0, heads 2 and 3 head 1
        for t in range(T):
            def conv(n, rows):
                x = w['p.' + n][rows] @ h.T
                c = w[f'p.{n}.conv'][rows]
                return silu(c[:, 1] * x[:, t] + (c[:, 0] * x[:, t - 1] if t else 0))
            q, k, v = conv('q', slice(g * d, g * d + d)), conv('k', slice(g * d, g * d + d)), conv('v', slice(hh * dv, hh * dv + dv))
            q, k = q / math.sqrt(float(q @ q) + 1e-6) / math.sqrt(d), k / math.sqrt(float(k @ k) + 1e-6)
            z = float(w['p.a'][hh] @ h[t] + w['p.dt_bias'][hh])
            S = S * math.exp(-math.exp(float(w['p.A_log'][hh])) * math.log1p(math.exp(z)))
            u = (v - S.T @ k) / (1 + math.exp(-float(w['p.b'][hh] @ h[t])))
            S = S + k[:, None] * u[None, :]
            o = S.T @ q
            o = o / math.sqrt(float((o * o).mean()) + 1e-3) * w['p.norm']
            out[t, hh * dv:hh * dv + dv] = o * silu(w['p.g'][hh * dv:hh * dv + dv] @ h[t])
    assert torch.allclose(got, out @ w['p.o'].T, atol=1e-10)


def test_oracle_layer_runs_and_the_start_of_the_stream():
    assert O.layer_runs({'layers': [0] * 4, 'loop': {'start': 1, 'stop': 3, 'times': 3}}) == [
        (0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert O.layer_runs({'layers': [0] * 2, 'loop': {'start': 0, 'stop': 1, 'times': 2}}) == [(0, False), (0, True), (1, False)]
    assert O.layer_runs({'layers': [0] * 2}) == [(0, False), (1, False)]
    d = configs.tiny_lupusun()
    w = weights.random_lupusun_weights(d, 3)
    toks = [5, 17, 3, 250, 17, 17, 9]
    trace = []
    lg = O.forward(d, w, toks, F64, trace)
    assert lg.shape == (7, 300) and len(trace) == 6 and all(t.shape == (7, 96) for t in trace)
    assert torch.allclose(O.forward(d, w, toks[:4], F64), lg[:4], atol=1e-10)          # causal
    # the second pass of layer 1 starts from the stream behind layer 2 plus the normed embedding rows
    wd = {k: v.double() for k, v in w.items()}
    e = O.embed(toks, wd, 1e-5, F64)
    x = trace[2] + e
    x = x + 0.8 * O.chunked_attention(O.rms_norm(x, wd['l1.norm1'], 1e-5), wd, 'l1.mix.', d['layers'][1]['mixer'], 1e-5)
    x = x + 0.8 * O.dense_ff(O.rms_norm(x, wd['l1.norm2'], 1e-5), wd, 'l1.mlp.')
    assert torch.allclose(x, trace[3], atol=1e-10)


# ------------------------------------------------------------------------------------------------ planted mistakes
def _shift(fn):
    """a chunk mask one position off"""
    def wrong(T, size):
        i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
        return (j <= i) & ((i + 1) // size == (j + 1) // size) if size else j <= i
    return wrong


MISTAKES = {
    'chunk one off': ('same_chunk', _shift),
    'no sink': ('softmax_with_sink', lambda f: lambda s, vis, sink: torch.softmax(s.masked_fill(~vis, float('-inf')), -1)),
    'no magnitude': ('blended_frequencies', lambda f: lambda rot: (f(rot)[0], 1.0)),
    'plain frequencies': ('blended_frequencies', lambda f: lambda rot: (f({k: v for k, v in rot.items() if k != 'scaling'})[0], f(rot)[1])),
    'reversed taps': ('short_conv', lambda f: lambda z, cw: f(z, cw.flip(-1))),
    'read before write': ('delta_rule', lambda f: lambda q, k, v, g, b: f(q, k, v, g, b) - b[..., None] * (q * k).sum(-1, keepdim=True) * v),
    'no decay': ('delta_rule', lambda f: lambda q, k, v, g, b: f(q, k, v, torch.ones_like(g), b)),
    'no unit length': ('unit', lambda f: lambda v: v),
    'start not added': ('layer_runs', lambda f: lambda cfg: [(i, False) for i, _ in f(cfg)]),
}


@pytest.mark.parametrize('name', list(MISTAKES))
def test_a_mistake_in_any_mechanism_shows_in_the_logits(monkeypatch, name):
    """the weights the GPU tests use decide the logits through every mechanism: a mistake is far above the tolerance of 2e-4"""
    d = configs.tiny_lupusun()
    w = weights.random_lupusun_weights(d, 0)
    toks = torch.randint(0, 300, (70,), generator=torch.Generator().manual_seed(1)).tolist()
    right = O.forward(d, w, toks, F64)
    attr, make = MISTAKES[name]
    monkeypatch.setattr(O, attr, make(getattr(O, attr)))
    wrong = O.forward(d, w, toks, F64)
    diff = wrong - right
    diff = diff - diff.mean(-1, keepdim=True)
    assert float((diff.pow(2).mean(-1).sqrt() / right.std()).max()) > 0.02
