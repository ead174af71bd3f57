"""Lupusun on the continuous-batching engine against the plain CPU restatement (oracle/lupusun_oracle.py).

Small random checkpoints of several shapes; the CUDA path (model, page pool with its state rows, engine, scheduler, public API,
trace runner) must give the oracle's logits whatever the schedule: whole prompts, token-by-token decoding, portions down to two
tokens, mixed batches, reused pages and slots. Each mechanism is also probed alone at the kernel level, with inputs made so that a
fault shows (one dominant key far back, at a page border, on either side of a chunk's edge; a sink that takes most of the weight;
decays and step sizes at both ends of their range; a slot's stale state and stale convolution inputs).
"""
import json
import math
import os
import random
import subprocess

import pytest
import torch

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, B16 = torch.float32, torch.bfloat16
TOL = {F32: 2e-4, B16: 8e-2}


@pytest.fixture(scope='module')
def lib(dev):
    import phi3_b200  # noqa: F401
    from phi3_b200 import _lib
    _lib.lib()
    return _lib


def _mods():
    import phi3_b200  # noqa: F401
    from phi3_b200 import configs, weights, engine, lupusun, paged
    from oracle import lupusun_oracle as O
    return configs, weights, engine, lupusun, paged, O


def row_err(got, ref):
    """per row: rms of the mean-free difference, relative to the spread of the reference"""
    got, ref = got.double().cpu(), ref.double().cpu()
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / ref.std()


def rel_err(got, ref):
    return float(row_err(got, ref).max())


def assert_close(got, ref, dtype, what='', loose=False):
    """fp32: every row within 2e-4. bf16: every row within the rounding bound and the median well inside it. loose (random
    configurations in bf16): nine rows in ten. The read-out of a recurrent head is divided by its own root mean square, so where a
    sequence's first tokens happen to give q . k near zero the rounding of the inputs decides the sign of the whole head, and such a
    row differs by a head's output however exact the kernels are."""
    e = row_err(got, ref)
    if dtype == F32:
        assert float(e.max()) < TOL[F32], (what, float(e.max()))
    elif loose:
        q = torch.quantile(e, torch.tensor([0.5, 0.9], dtype=e.dtype))
        assert float(q[0]) < 0.03 and float(q[1]) < TOL[B16], (what, q.tolist(), float(e.max()))
    else:
        assert float(e.median()) < 0.03 and float(e.max()) < TOL[B16], (what, float(e.median()), float(e.max()))


def make(cfg_dict, dtype, seed=0):
    configs, weights, engine, lupusun, paged, O = _mods()
    w = weights.random_lupusun_weights(cfg_dict, seed)
    return lupusun.LupusunB200(cfg_dict, w, dtype=dtype), w


def tokens(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def poison(eng):
    """whatever an earlier owner left must never be read: finite junk in the cache pages (a masked key is multiplied by a zero
    weight), NaN in the matrix states and in the convolution inputs (a new sequence must not even load them)"""
    for t in eng.pool.k + eng.pool.v:
        t.fill_(300.0)
    for s in eng.pool.state:
        s.fill_(float('nan'))


def run_schedule(model, toks, cuts, max_tokens=None, engine=None, rid='r'):
    """feed `toks` in portions of the given sizes (the rest one by one); logits of every position, in order"""
    configs, weights, eng_mod, *_ = _mods()
    eng = engine or eng_mod.Engine(model, max_tokens or len(toks) + 64, 4)
    if engine is None:
        poison(eng)
    out, at = [], 0
    sizes = list(cuts)
    while at < len(toks):
        n = sizes.pop(0) if sizes else 1
        n = min(n, len(toks) - at)
        out.append(eng.step([(rid, toks[at:at + n], list(range(n)))]))
        at += n
    eng.finish(rid)
    return torch.cat(out, 0)


# ------------------------------------------------------------------------------------------------ whole model, schedules
@pytest.mark.parametrize('dtype', [F32, B16])
def test_whole_prompt_and_every_layer_match_the_oracle(lib, dtype):
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, dtype)
    toks = tokens(150, cfg['vocab'], 1)                       # more than two pages, several chunks
    ref_trace = []
    ref = O.forward(cfg, w, toks, torch.float64, ref_trace)
    eng = engine.Engine(model, 256, 4)
    poison(eng)
    trace = []
    got = eng.step([('a', toks, list(range(len(toks))))], ['a'], trace=trace)
    assert_close(got, ref, dtype)
    assert len(trace) == len(ref_trace) == 6                  # a looped layer counts once per pass
    if dtype == F32:
        for i, (g, r) in enumerate(zip(trace, ref_trace)):
            assert (g.cpu().double() - r).abs().max() < 2e-4 * float(r.abs().max()), f'residual stream after layer run {i}'
    assert len(eng.pool.free_pages) == eng.pool.n_pages and len(eng.pool.free_slots) == 4
    assert len(eng.pool.state) == 6 and len(eng.pool.k) == 6   # matrix states and convolution inputs of three recurrent runs


@pytest.mark.parametrize('dtype', [F32, B16])
def test_prefill_then_token_by_token_decoding(lib, dtype):
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, dtype, seed=2)
    toks = tokens(140, cfg['vocab'], 3)
    ref = O.forward(cfg, w, toks, torch.float64)
    got = run_schedule(model, toks, [30])                     # 110 decoded tokens: chunk edges and page borders pass by
    assert_close(got, ref, dtype)
    whole = run_schedule(model, toks, [len(toks)])
    if dtype == F32:
        assert rel_err(got, whole) < 1e-5
    else:
        assert_close(got, whole, dtype)


@pytest.mark.parametrize('cuts', [[2, 2, 3, 31, 33, 2, 64, 1, 2], [63, 2, 63, 2], [1, 1, 64, 65], [100, 2, 2], [5, 32, 37, 3]])
def test_prompt_portions_of_any_size(lib, cuts):
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, F32, seed=4)
    toks = tokens(sum(cuts) + 5, cfg['vocab'], 5)
    ref = O.forward(cfg, w, toks, torch.float64)
    assert rel_err(run_schedule(model, toks, cuts), ref) < TOL[F32]


@pytest.mark.parametrize('dtype', [F32, B16])
def test_mixed_batch_of_unequal_requests_equals_each_alone(lib, dtype):
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, dtype, seed=6)
    lens = {'a': 150, 'b': 37, 'c': 2, 'd': 90}
    toks = {k: tokens(n, cfg['vocab'], 10 + i) for i, (k, n) in enumerate(lens.items())}
    alone = {k: run_schedule(model, t, [len(t)]) for k, t in toks.items()}
    eng = engine.Engine(model, 64 * 8, 4)
    poison(eng)
    plan = {'a': [40, 1, 1, 33, 1, 2, 72], 'b': [1, 30, 1, 1, 1, 3], 'c': [1, 1], 'd': [64, 1, 25]}   # sizes per step
    at = {k: 0 for k in toks}
    got = {k: [] for k in toks}
    for s in range(max(len(v) for v in plan.values())):
        entries = []
        for k in toks:
            if s < len(plan[k]) and at[k] < lens[k]:
                n = min(plan[k][s], lens[k] - at[k])
                entries.append((k, toks[k][at[k]:at[k] + n], list(range(n))))
                at[k] += n
        lg = eng.step(entries)
        o = 0
        for k, t, wnt in entries:
            got[k].append(lg[o:o + len(wnt)])
            o += len(wnt)
    for k in toks:
        assert at[k] == lens[k]
        if dtype == F32:
            assert rel_err(torch.cat(got[k], 0), alone[k]) < 1e-5, k
        else:
            assert_close(torch.cat(got[k], 0), alone[k], dtype, k)
        assert_close(torch.cat(got[k], 0), O.forward(cfg, w, toks[k], torch.float64), dtype, k)


def test_pages_slots_and_state_rows_are_given_back_and_used_again(lib):
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, F32, seed=7)
    eng = engine.Engine(model, 64 * 4, 2)                     # four pages, two slots
    poison(eng)
    seen = []
    for r in range(5):
        n = [130, 200, 70, 256, 129][r]
        toks = tokens(n, cfg['vocab'], 20 + r)
        got = run_schedule(model, toks, [50, 3, 70], engine=eng, rid=f'r{r}')   # the slot's state is the previous request's
        assert rel_err(got, O.forward(cfg, w, toks, torch.float64)) < TOL[F32], r
        seen.append(len(eng.pool.free_pages))
    assert seen == [4] * 5 and sorted(eng.pool.free_slots) == [0, 1]
    # two live requests interleaved, one leaves, a third takes its slot, pages and state rows while the other goes on
    ta, tb, tc = tokens(100, cfg['vocab'], 31), tokens(60, cfg['vocab'], 32), tokens(120, cfg['vocab'], 33)
    la = [eng.step([('a', ta[:50], list(range(50))), ('b', tb, list(range(60)))], ['b'])]
    la.append(eng.step([('a', ta[50:], list(range(50))), ('c', tc[:64], list(range(64)))]))
    lc = [la[1][50:], eng.step([('c', tc[64:], list(range(56)))], ['a', 'c'])]
    with pytest.raises(paged.PoolExhausted):
        eng.step([('x', tokens(64 * 5, cfg['vocab'], 1), [])])
    assert rel_err(torch.cat([la[0][:50], la[1][:50]], 0), O.forward(cfg, w, ta, torch.float64)) < TOL[F32]
    assert rel_err(torch.cat(lc, 0), O.forward(cfg, w, tc, torch.float64)) < TOL[F32]


def test_first_tokens_and_long_decoding(lib):
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, F32, seed=8)
    for n in (1, 2, 3):
        toks = tokens(n, cfg['vocab'], 40 + n)
        assert rel_err(run_schedule(model, toks, [n]), O.forward(cfg, w, toks, torch.float64)) < TOL[F32]
    toks = tokens(230, cfg['vocab'], 44)
    assert rel_err(run_schedule(model, toks, [1]), O.forward(cfg, w, toks, torch.float64)) < TOL[F32]   # all decoded one by one


def test_a_request_that_sits_out_steps_keeps_its_state(lib):
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, F32, seed=3)
    ta, tb = tokens(90, cfg['vocab'], 81), tokens(80, cfg['vocab'], 82)
    eng = engine.Engine(model, 64 * 4, 4)
    poison(eng)
    ga = [eng.step([('a', ta[:40], list(range(40)))])]
    gb = [eng.step([('b', tb[:33], list(range(33)))])]        # a is left out ...
    gb.append(eng.step([('b', tb[33:34], [0])]))
    lg = eng.step([('b', tb[34:], list(range(46))), ('a', ta[40:], list(range(50)))])   # ... and goes on behind b
    gb.append(lg[:46])
    ga.append(lg[46:])
    assert rel_err(torch.cat(ga, 0), O.forward(cfg, w, ta, torch.float64)) < TOL[F32]
    assert rel_err(torch.cat(gb, 0), O.forward(cfg, w, tb, torch.float64)) < TOL[F32]


@pytest.mark.parametrize('dtype', [F32, B16])
def test_captured_decode_steps_equal_eager_steps(lib, dtype):
    """decode-only steps replay a CUDA graph from their third occurrence on; the logits must be those of eager launches, bit for
    bit, while requests sit out steps, leave and hand their slot, pages and state rows to a newcomer"""
    configs, weights, engine, lupusun, paged, O = _mods()
    cfg = configs.tiny_lupusun()
    model, w = make(cfg, dtype, seed=9)
    n_prompt = {'a': 120, 'b': 5, 'c': 70, 'd': 66}
    seqs = {k: tokens(n + 24, cfg['vocab'], 50 + i) for i, (k, n) in enumerate(n_prompt.items())}

    def run(graphs):
        eng = engine.Engine(model, 64 * 10, 4)
        eng.use_graphs = graphs
        poison(eng)
        got = {k: [] for k in seqs}
        at = dict(n_prompt)

        def step(names, end=()):
            entries = []
            for k in names:
                n = n_prompt[k] if not got[k] else 1
                lo = 0 if not got[k] else at[k]
                entries.append((k, seqs[k][lo:lo + n], [n - 1]))
                at[k] = lo + n
            lg = eng.step(entries, end)
            for i, k in enumerate(names):
                got[k].append(lg[i:i + 1])

        step(['a', 'b', 'c'])
        for s in range(20):
            live = ['a', 'c'] if 8 <= s < 12 else ['a', 'b', 'c']                  # b sits out four steps
            if s < 15:
                step(live)
            elif s == 15:
                step(live, ['c'])                                                # c leaves ...
                step(['d'])                                                      # ... and d takes its slot and pages
            else:
                step(['a', 'b', 'd'])
        return {k: torch.cat(v, 0) for k, v in got.items()}, eng

    eager, _ = run(False)
    replay, eng = run(True)
    assert any('graph' in g for g in eng._graphs.values()), 'no step was captured'
    for k in seqs:
        assert torch.equal(eager[k], replay[k]), k
        n = eager[k].shape[0]
        ref = O.forward(cfg, w, seqs[k][:n_prompt[k] + n - 1], torch.float64)[n_prompt[k] - 1:]
        assert_close(replay[k], ref, dtype, k)


# ------------------------------------------------------------------------------------------------ other sizes
def _att(heads, kv, dim, vdim, chunk, rd=None, scaling=(4.0, 64, 16.0, 1.5), base=10000.0, scale=None):
    rd = dim if rd is None else rd
    sc = {'scaling': dict(zip(('factor', 'original', 'fast', 'slow'), scaling))} if scaling else {}
    return {'type': 'attention',
            'mixer': dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or 2.0 * dim ** -0.5,
                          **({'mask': {'size': chunk}} if chunk else {}), **({'rot': {'base': base, 'dims': rd, **sc}} if rd else {}))}


def _delta(heads, kv, dim, vdim, taps):
    return {'type': 'delta', 'mixer': dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=taps)}


def _dense(ff):
    return {'kind': 'dense', 'ff': ff}


OTHER = {
    # every head count 1, chunks of one token (a token sees itself alone) and of two, one tap (no history at all), the whole stack runs
    # three times, no factor on the sublayers
    'ones': (64, dict(loop=(0, 4, 3), residual_mult=1.0),
             [dict(_att(1, 1, 16, 16, 1), mlp=_dense(64)), dict(_delta(1, 1, 16, 16, 1), mlp=_dense(64)),
              dict(_att(1, 1, 8, 8, 2, 2), mlp=None), dict(_delta(1, 1, 1, 8, 2), mlp=_dense(16))]),
    # sizes that tile the tensor-core kernels and equal each other; chunks of a page and of two pages less one token
    'tiled': (128, dict(loop=(2, 4, 2), residual_mult=0.6),
              [dict(_att(4, 4, 64, 64, 64), mlp=_dense(256)), dict(_delta(4, 4, 64, 64, 4), mlp=_dense(256)),
               dict(_att(8, 2, 128, 128, 127, 64, (8.0, 4096, 32.0, 1.0), 500000.0), mlp=_dense(256)), dict(_delta(4, 2, 128, 128, 4), mlp=_dense(128)),
               dict(_att(8, 8, 32, 64, 128), mlp=None)]),
    # nothing is a multiple of 8: every product goes through the any-shape kernel, every attention through the fp32 kernels
    'ragged': (50, dict(loop=(1, 2, 3), residual_mult=1.3),
               [dict(_delta(6, 3, 7, 9, 5), mlp=_dense(33)), dict(_att(3, 1, 10, 7, 63, 6), mlp=_dense(21)), dict(_delta(5, 1, 13, 3, 3), mlp=None),
                dict(_att(6, 2, 11, 14, 65, 2, (3.0, 30, 2.0, 0.3)), mlp=_dense(19)), dict(_delta(2, 2, 130, 5, 4), mlp=_dense(10))]),
    # a history longer than the shortest portions, wide recurrent keys, many heads on one key head, a chunk longer than anything fed, heads
    # without a rotation, value heads of 200 numbers, no loop
    'wide': (96, dict(loop=None, residual_mult=0.9),
             [dict(_delta(6, 2, 260, 40, 9), mlp=_dense(96)), dict(_att(12, 1, 24, 200, 1000), mlp=None),
              dict(_delta(2, 1, 48, 136, 4), mlp=_dense(48)), dict(_att(2, 2, 160, 96, 40, 0), mlp=_dense(40)), dict(_delta(3, 1, 66, 24, 6), mlp=None)]),
}


@pytest.mark.parametrize('name', list(OTHER))
@pytest.mark.parametrize('dtype', [F32, B16])
def test_other_sizes(lib, name, dtype):
    configs, weights, engine, lupusun, paged, O = _mods()
    width, kw, layers = OTHER[name]
    cfg = configs.tiny_lupusun(width=width, vocab=211 if name != 'ragged' else 101, layers=layers, **kw)
    model, w = make(cfg, dtype, seed=11)
    toks = tokens(150, cfg['vocab'], 12)
    ref = O.forward(cfg, w, toks, torch.float64)
    # (bf16, one value of one key number per head: the sign of q . k is all a read-out keeps, see assert_close)
    assert_close(run_schedule(model, toks, [70, 2, 40]), ref, dtype, name, loose=name == 'ones')


def test_only_recurrent_and_only_attention_stacks(lib):
    configs, weights, engine, lupusun, paged, O = _mods()
    for layers in ([dict(_delta(2, 1, 24, 16, 4), mlp=_dense(40))] * 2, [dict(_att(4, 2, 24, 16, 20), mlp=None)] * 2):
        cfg = configs.tiny_lupusun(width=48, vocab=90, layers=layers, loop=(0, 1, 2))
        model, w = make(cfg, F32, seed=5)
        toks = tokens(100, 90, 6)
        assert rel_err(run_schedule(model, toks, [50, 2, 3, 30]), O.forward(cfg, w, toks, torch.float64)) < TOL[F32]


def test_small_batches_take_the_weight_streaming_products(lib):
    configs, weights, engine, lupusun, paged, O = _mods()
    width, kw, layers = OTHER['tiled']
    cfg = configs.tiny_lupusun(width=width, vocab=256, layers=layers, **kw)
    model, w = make(cfg, B16, seed=15)
    toks = tokens(40, cfg['vocab'], 16)
    ref = O.forward(cfg, w, toks, torch.float64)
    a = run_schedule(model, toks, [20])
    model.use_skinny = False
    b = run_schedule(model, toks, [20])
    assert_close(a, ref, B16)
    assert_close(b, ref, B16)


def _random_config(rng):
    """a random order of the two mixers with random sizes, and now and then a looped block"""
    layers = []
    for i in range(rng.randint(2, 5)):
        mlp = _dense(rng.choice([24, 40, 64])) if rng.random() < 0.8 else None
        kv = rng.randint(1, 3)
        if rng.random() < 0.5:
            dim = rng.choice([8, 16, 24, 40])
            lay = _att(kv * rng.randint(1, 3), kv, dim, rng.choice([8, 24, 32]), rng.choice([0, 1, 5, 33, 64, 100]),
                       rng.choice([r for r in (0, 2, 4, 8, 16, dim) if r <= dim]),
                       rng.choice([None, (4.0, 64, 16.0, 1.5), (16.0, 512, 32.0, 1.0), (1.5, 10, 1.0, 0.2)]), rng.choice([100.0, 10000.0, 1000000.0]))
        else:
            lay = _delta(kv * rng.randint(1, 3), kv, rng.choice([8, 24, 40, 72]), rng.choice([8, 24, 40, 70]), rng.choice([1, 2, 3, 4, 4, 6]))
        layers.append(dict(lay, mlp=mlp))
    lo = rng.randrange(len(layers))
    loop = (lo, rng.randint(lo + 1, len(layers)), rng.randint(1, 3)) if rng.random() < 0.7 else None
    return _mods()[0].tiny_lupusun(width=rng.choice([48, 64, 72, 96]), vocab=rng.choice([77, 128, 300]), layers=layers, loop=loop,
                                   residual_mult=rng.choice([0.3, 0.7, 1.0]))


@pytest.mark.parametrize('seed', [21, 22, 23, 24, 25, 26])
def test_random_configurations_under_random_schedules(lib, seed):
    """random layer orders and sizes, random requests fed in random portions beside each other through a pool that forces pages,
    slots and state rows to change hands"""
    configs, weights, engine, lupusun, paged, O = _mods()
    rng = random.Random(seed)
    cfg = _random_config(rng)
    dtype = F32 if seed % 2 else B16
    model, w = make(cfg, dtype, seed=seed)
    lens = [rng.choice([1, 2, 3, 30, 64, 65, 100, 129, 190]) for _ in range(6)]
    toks = [tokens(n, cfg['vocab'], seed * 10 + i) for i, n in enumerate(lens)]
    ref = [O.forward(cfg, w, t, torch.float64) for t in toks]
    eng = engine.Engine(model, 64 * 8, 3)
    poison(eng)
    fed, got = [0] * 6, [[] for _ in range(6)]
    live, nxt = [], 0
    while nxt < 6 or live:
        while nxt < 6 and len(live) < 3 and eng.can_take(f'r{nxt}', min(lens[nxt], 64)) and \
                sum(-(-lens[i] // 64) for i in live) + -(-lens[nxt] // 64) <= 8:
            live.append(nxt)
            nxt += 1
        entries, end = [], []
        for i in live:
            if rng.random() < 0.2 and len(live) > 1 and entries:
                continue                                       # sits this step out
            n = min(lens[i] - fed[i], rng.choice([1, 1, 2, 3, 17, 64, 100]))
            entries.append((f'r{i}', toks[i][fed[i]:fed[i] + n], list(range(n))))
            fed[i] += n
            if fed[i] == lens[i]:
                end.append(f'r{i}')
        lg = eng.step(entries, end)
        o = 0
        for rid, t, _ in entries:
            got[int(rid[1:])].append(lg[o:o + len(t)])
            o += len(t)
        live = [i for i in live if fed[i] < lens[i]]
    if dtype == F32:
        for i in range(6):
            assert_close(torch.cat(got[i], 0), ref[i], dtype, (seed, i))
    else:
        assert_close(torch.cat([torch.cat(g, 0) for g in got], 0), torch.cat(ref, 0), dtype, seed, loose=True)


# ------------------------------------------------------------------------------------------------ mechanisms alone
def _attention_case(dtype, H, G, d, dv, n_ctx, chunk, hot, *, scale=1.0, seed=0, tile_rows=32, n_splits=1, sink=None, window=0, keep=0,
                    first_row=0):
    """random queries, keys and values with a few dominant (query, key) pairs `hot` = [(i, j)]: both rows get a large common
    component, so that the weight of that pair dwarfs the rest when it is visible and a lost, misplaced or wrongly masked key
    changes the output completely. sink: per-head numbers in the softmax denominator. first_row: the prefill tiles begin there (a
    prompt's portion). Returns (prefill result, decode result, plain reference) of the rows from first_row on."""
    from phi3_b200._lib import AttnWindowArgs, call_struct, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(seed)
    q = torch.randn(n_ctx, H, d, generator=g) * 0.5
    k = torch.randn(n_ctx, G, d, generator=g) * 0.5
    v = torch.randn(n_ctx, G, dv, generator=g)
    for n, (i, j) in enumerate(hot):
        u = torch.zeros(d)
        u[n % d] = 6.0
        q[i] += u
        k[j] += u
    if dtype == B16:
        q, k, v = q.bfloat16().float(), k.bfloat16().float(), v.bfloat16().float()
    ii, jj = torch.arange(n_ctx)[:, None], torch.arange(n_ctx)[None, :]
    vis = jj <= ii
    if window:
        vis = vis & ((ii - jj < window) | (jj < keep))
    if chunk:
        vis = vis & ((ii // chunk == jj // chunk) | ((jj < keep) & (jj <= ii)))
    ref = torch.zeros(n_ctx, H, dv, dtype=torch.float64)
    for h in range(H):
        sc = ((q[:, h].double() @ k[:, h // (H // G)].double().T) * scale).masked_fill(~vis, float('-inf'))
        if sink is None:
            wgt = torch.softmax(sc, -1)
        else:
            m = torch.clamp(sc.max(-1, keepdim=True).values, min=float(sink[h]))
            e = torch.exp(sc - m)
            wgt = e / (e.sum(-1, keepdim=True) + torch.exp(sink[h].double() - m))
        ref[:, h] = wgt @ v[:, h // (H // G)].double()
    n_pg = -(-n_ctx // 64)
    perm = torch.randperm(n_pg + 3, generator=g)[:n_pg]
    kp, vp = torch.full((n_pg + 3, G, 64, d), 50.0), torch.full((n_pg + 3, G, 64, dv), -70.0)
    for p in range(n_pg):
        n = min(64, n_ctx - 64 * p)
        kp[perm[p], :, :n] = k[64 * p:64 * p + n].transpose(0, 1)
        vp[perm[p], :, :n] = v[64 * p:64 * p + n].transpose(0, 1)
    bt = torch.zeros(2, n_pg + 3, dtype=torch.int32)
    bt[1, :n_pg] = perm.int()
    kp, vp, bt = kp.to(dev, dtype), vp.to(dev, dtype), bt.to(dev)
    qd = q.reshape(n_ctx, H * d).to(dev, dtype).contiguous()
    sd = None if sink is None else sink.float().to(dev)
    outs = []
    for kind in ('prefill', 'decode'):
        step = tile_rows if kind == 'prefill' else 1
        tiles = [(r0, min(step, n_ctx - r0), 1, r0) for r0 in range(first_row, n_ctx, step)]
        td = torch.tensor(tiles, dtype=torch.int32, device=dev).reshape(-1)
        out = torch.zeros(n_ctx, H * dv, dtype=dtype, device=dev)
        a_ = AttnWindowArgs()
        a_.q, a_.ld_q, a_.k_pool, a_.v_pool, a_.block_table, a_.bt_stride = ptr(qd), H * d, ptr(kp), ptr(vp), ptr(bt), bt.stride(0)
        a_.out, a_.ld_out, a_.sink = ptr(out), H * dv, ptr(sd)
        a_.n_heads, a_.n_kv, a_.dim, a_.vdim, a_.scale, a_.chunk, a_.window, a_.keep_first = H, G, d, dv, scale, chunk, window, keep
        a_.act_f32 = a_.cache_f32 = int(dtype == F32)
        a_.tiles, a_.n_tiles = ptr(td), len(tiles)
        if kind == 'decode' and n_splits > 1:
            ws = torch.empty(len(tiles) * H * n_splits * (dv + 2), device=dev)
            a_.n_splits, a_.ws = n_splits, ptr(ws)
        call_struct('p3_attn_window_' + kind, a_, 0)
        torch.cuda.synchronize()
        outs.append(out.float().cpu().reshape(n_ctx, H, dv)[first_row:])
    return outs[0], outs[1], ref[first_row:]


def _tile_rows(lib, dtype, H, G, d, dv):
    import ctypes as C
    a = lib.AttnWindowArgs()
    a.q = a.out = a.k_pool = a.v_pool = a.block_table = a.tiles = 256
    a.ld_q, a.ld_out, a.n_heads, a.n_kv, a.dim, a.vdim = H * d, H * dv, H, G, d, dv
    a.act_f32 = a.cache_f32 = int(dtype == F32)
    return int(lib.lib().p3_attn_window_tile_rows(C.byref(a)))


@pytest.mark.parametrize('shape', [(3, 3, 28, 20), (6, 2, 64, 64), (8, 1, 48, 40), (4, 2, 128, 96), (2, 1, 264, 200), (2, 2, 160, 128)])
@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('n_splits', [1, 3])
@pytest.mark.parametrize('chunk', [36, 64, 100, 0])
def test_chunk_edges_sinks_far_keys_and_page_borders(lib, shape, dtype, n_splits, chunk):
    """dominant pairs sit just inside and just outside a chunk (its first key from its last query, the key before its first from any of
    its queries), at page borders, at the query's own position and at the first positions; one head's sink outweighs every ordinary
    key, another's is negligible; the tiles start in the middle of a chunk, too."""
    H, G, d, dv = shape
    n, c = 300, chunk or 90
    hot = [(299, 0), (299, 299 // c * c), (299, 299 // c * c - 1), (2 * c - 1, c), (2 * c - 1, c - 1), (2 * c, c), (2 * c, 2 * c), (c, c - 1),
           (c, 0), (c - 1, 0), (c + 1, c), (1, 0), (0, 0), (64, 63), (64, 64), (128, 127), (130, 128), (131, 66), (192, 191), (200, 150),
           (255, 250), (256, 255), (256, 192), (290, 64)]
    sink = torch.linspace(-6.0, 5.0, H)
    tile = _tile_rows(lib, dtype, H, G, d, dv)
    tol = 1e-4 if dtype == F32 else 3e-2
    for first in (0, 77):
        pf, dc, ref = _attention_case(dtype, H, G, d, dv, n, chunk, hot, scale=0.7, tile_rows=tile, n_splits=n_splits, sink=sink, first_row=first)
        assert (pf.double() - ref).abs().max() < tol * max(1.0, float(ref.abs().max()))
        assert (dc.double() - ref).abs().max() < tol * max(1.0, float(ref.abs().max()))
    if chunk:                                                  # a chunk that begins one position earlier gives something else entirely
        _, _, other = _attention_case(dtype, H, G, d, dv, n, chunk + 1, hot, scale=0.7, sink=sink, first_row=77)
        assert (other - ref).abs().max() > 0.3


@pytest.mark.parametrize('dtype', [F32, B16])
def test_chunks_together_with_a_window_and_kept_first_tokens(lib, dtype):
    for chunk, window, keep in ((50, 20, 0), (50, 20, 3), (70, 0, 66), (0, 40, 5), (30, 200, 0)):
        hot = [(60, 50), (69, 50), (70, 50), (70, 51), (199, 150), (199, 180), (199, 179), (149, 2), (149, 3), (140, 65), (140, 66)]
        pf, dc, ref = _attention_case(dtype, 4, 2, 32, 48, 200, chunk, hot, window=window, keep=keep, tile_rows=_tile_rows(lib, dtype, 4, 2, 32, 48),
                                      n_splits=2, sink=torch.linspace(-2.0, 2.0, 4))
        tol = (1e-4 if dtype == F32 else 3e-2) * float(ref.abs().max())
        assert (pf.double() - ref).abs().max() < tol and (dc.double() - ref).abs().max() < tol, (chunk, window, keep)


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('shape', [(4, 2, 24, 40, 16), (3, 3, 7, 5, 2), (2, 1, 128, 64, 128), (2, 1, 300, 20, 130), (5, 5, 64, 64, 0)])
def test_rotation_magnitude_and_unit_heads(lib, dtype, shape):
    """biases, the partial rotation with a factor on cos and sin, then heads divided by their root mean square (small numbers, so that
    eps counts), and the plain form without the norm"""
    configs, weights, engine, lupusun, paged, O = _mods()
    from phi3_b200._lib import QkvRopePostArgs, call_struct, ptr
    dev = torch.device('cuda')
    H, G, d, dv, rn = shape
    g = torch.Generator().manual_seed(3)
    T, eps = 9, 1e-3
    rot = {'base': 10000.0, 'dims': rn, 'scaling': {'factor': 6.0, 'original': 64, 'fast': 16.0, 'slow': 1.5}}
    cols = (H + G) * d + G * dv
    proj, bias = torch.randn(T, cols, generator=g) * 0.05, torch.randn(cols, generator=g) * 0.05
    pos = torch.tensor([0, 1, 2, 63, 64, 65, 126, 127, 128])
    bt = torch.tensor([[2, 0, 3]], dtype=torch.int32)
    freq, mag = O.blended_frequencies(rot) if rn else ([], 1.0)
    x = (proj + bias).double()
    q, k, v = x[:, :H * d].view(T, H, d), x[:, H * d:(H + G) * d].view(T, G, d), x[:, (H + G) * d:].view(T, G, dv)
    if rn:
        q, k = O.rotate_halves(q, pos, rot), O.rotate_halves(k, pos, rot)
    for unit in (1, 0):
        q_ref, k_ref = (O.rms_norm(q, None, eps), O.rms_norm(k, None, eps)) if unit else (q, k)
        qd = torch.empty(T, H * d, dtype=dtype, device=dev)
        kp, vp = torch.zeros(4, G, 64, d, dtype=dtype, device=dev), torch.zeros(4, G, 64, dv, dtype=dtype, device=dev)
        dd = [proj.to(dev), bias.to(dev), torch.tensor(freq, dtype=torch.float32, device=dev), bt.to(dev),
              torch.zeros(T, dtype=torch.int32, device=dev), pos.int().to(dev)]
        a = QkvRopePostArgs()
        a.proj, a.ld_proj, a.q_off, a.k_off, a.v_off, a.bias = ptr(dd[0]), cols, 0, H * d, (H + G) * d, ptr(dd[1])
        a.n_heads, a.n_kv, a.dim, a.vdim, a.rot_n, a.freq, a.rot_mag, a.unit_norm, a.eps = H, G, d, dv, rn, ptr(dd[2]), mag, unit, eps
        a.q_out, a.ld_q, a.k_pool, a.v_pool, a.block_table, a.bt_stride = ptr(qd), H * d, ptr(kp), ptr(vp), ptr(dd[3]), 3
        a.tok_slot, a.tok_pos, a.T, a.act_f32, a.cache_f32 = ptr(dd[4]), ptr(dd[5]), T, int(dtype == F32), int(dtype == F32)
        call_struct('p3_qkv_rope_post', a, 0)
        torch.cuda.synchronize()
        tol = 2e-5 if dtype == F32 else 2e-2
        assert (qd.double().cpu().view(T, H, d) - q_ref).abs().max() < tol
        for t in range(T):
            pg, off = int(bt[0, int(pos[t]) // 64]), int(pos[t]) % 64
            assert (kp[pg, :, off].double().cpu() - k_ref[t]).abs().max() < tol
            assert (vp[pg, :, off].double().cpu() - v[t]).abs().max() < tol


@pytest.mark.parametrize('shape', [(4, 2, 24, 40, 4), (1, 1, 7, 5, 4), (3, 1, 20, 64, 3), (3, 3, 64, 64, 4), (4, 2, 128, 96, 4), (2, 1, 200, 33, 2),
                                   (5, 5, 136, 70, 1), (2, 2, 300, 40, 4), (6, 2, 34, 22, 7), (2, 1, 1, 8, 4), (2, 2, 66, 12, 40)])
@pytest.mark.parametrize('rs', [0, 2, 4, 8])
def test_convolutions_and_delta_rule_in_portions(lib, shape, rs):
    """the mixer's recurrent part alone (convolutions, unit heads, gates, state): whole sequences against the oracle, then the same
    sequences in portions (states and convolution inputs carry on, portions shorter than the taps among them) with a second sequence in
    the batch, bit for bit equal to the whole run. Some tokens make a head forget everything, some keep everything, some write in full
    and some not at all. rs: the shape of a warp (0: the launch's own choice)"""
    configs, weights, engine, lupusun, paged, O = _mods()
    from phi3_b200._lib import ShortConvArgs, DeltaScanArgs, call_struct, ptr
    dev = torch.device('cuda')
    H, G, d, dv, taps = shape
    g = torch.Generator().manual_seed(7)
    T = {0: 83, 1: 37}
    C = 2 * G * d + H * dv
    cols = C + 2 * H + 3
    proj = {s: torch.randn(n, cols, generator=g) for s, n in T.items()}
    for s in proj:
        a_, b_ = proj[s][:, C + H:C + 2 * H], proj[s][:, C:C + H]
        a_[20:22] = 60.0                                       # forget everything ...
        a_[24:34] = -60.0                                      # ... keep everything
        b_[26:28], b_[30:32] = 50.0, -50.0                     # replace the value at the key, leave it alone
    cw, a_log, dt = torch.randn(C, taps, generator=g) * 0.6, torch.randn(H, generator=g) * 0.5, torch.randn(H, generator=g) - 2.0
    ref = {}
    for s, p in proj.items():
        x = p.double()
        z = torch.nn.functional.silu(O.short_conv(x[:, :C], cw.double()))
        of = [h // (H // G) for h in range(H)]
        q = (O.unit(z[:, :G * d].view(-1, G, d)) * d ** -0.5)[:, of]
        k = O.unit(z[:, G * d:2 * G * d].view(-1, G, d))[:, of]
        rate = torch.nn.functional.softplus(x[:, C + H:C + 2 * H] + dt.double(), threshold=1e9)
        ref[s] = O.delta_rule(q, k, z[:, 2 * G * d:].reshape(-1, H, dv), torch.exp(-torch.exp(a_log.double()) * rate),
                              torch.sigmoid(x[:, C:C + H])).reshape(-1, H * dv)
    n_state = int(lib.lib().p3_delta_state_floats(H, d, dv))
    assert n_state == H * d * dv
    cwd, ald, dtd = cw.t().contiguous().to(dev), a_log.to(dev), dt.to(dev)

    def run(plans):
        state = torch.full((3, n_state), float('nan'), device=dev)
        hist = torch.full((3, max(taps - 1, 1) * C), float('nan'), device=dev)
        got = {s: [] for s in T}
        for plan in plans:
            seqs, rows, slots = [], [], []
            slot_seq = [0] * 3
            r0 = 0
            for slot, p0, n in plan:
                slot_seq[slot] = len(seqs)
                seqs.append((r0, n, slot, p0))
                rows.append(proj[slot - 1][p0:p0 + n])
                slots += [slot] * n
                r0 += n
            pd = torch.cat(rows, 0).to(dev)
            qkv, gates, out = torch.empty(r0, C, device=dev), torch.empty(r0, H, 2, device=dev), torch.empty(r0, H * dv, device=dev)
            i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev).reshape(-1)
            sq, sl, ss = i32(seqs), i32(slots), i32(slot_seq)
            c = ShortConvArgs()
            c.proj, c.ld_proj, c.n_unit, c.dim, c.n_scaled, c.n_plain = ptr(pd), cols, 2 * G, d, G, H * dv
            c.w, c.taps, c.conv_state, c.scale, c.unit_eps = ptr(cwd), taps, ptr(hist), d ** -0.5, 1e-6
            c.seqs, c.slot_seq, c.tok_slot, c.n_rows, c.out, c.ld_out = ptr(sq), ptr(ss), ptr(sl), r0, ptr(qkv), C
            c.b_off, c.a_off, c.n_gates, c.a_log, c.dt_bias, c.gates = C, C + H, H, ptr(ald), ptr(dtd), ptr(gates)
            call_struct('p3_short_conv', c, 0)
            a = DeltaScanArgs()
            a.qkv, a.ld_qkv, a.q_off, a.k_off, a.v_off, a.gates = ptr(qkv), C, 0, G * d, 2 * G * d, ptr(gates)
            a.n_heads, a.n_kv, a.dim, a.vdim, a.state, a.seqs, a.n_seqs = H, G, d, dv, ptr(state), ptr(sq), len(seqs)
            a.out, a.ld_out, a.rs_force = ptr(out), H * dv, rs
            a.conv_in, a.ld_conv_in, a.channels, a.taps, a.conv_state = ptr(pd), cols, C, taps, ptr(hist)
            call_struct('p3_delta_scan', a, 0)
            torch.cuda.synchronize()
            o = 0
            for slot, p0, n in plan:
                got[slot - 1].append(out[o:o + n].cpu())
                o += n
        return {s: torch.cat(v, 0) for s, v in got.items()}

    whole = run([[(1, 0, 83), (2, 0, 37)]])                    # sequence s lives in slot s + 1
    parts = run([[(1, 0, 17)], [(2, 0, 2), (1, 17, 1)], [(1, 18, 16), (2, 2, 33)], [(1, 34, 1)], [(2, 35, 2), (1, 35, 2)], [(1, 37, 46)]])
    for s in T:
        assert (whole[s].double() - ref[s]).abs().max() < 1e-4 * max(1.0, float(ref[s].abs().max())), s
        assert torch.equal(whole[s], parts[s]), s


def test_convolutions_of_many_rows_equal_those_of_few(lib):
    """long steps walk several rows per warp, with unequal sequences that begin and end inside a warp's rows"""
    configs, weights, engine, lupusun, paged, O = _mods()
    from phi3_b200._lib import ShortConvArgs, call_struct, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(8)
    lens = [1, 2, 3, 130, 1, 5, 250, 16, 15, 300, 2]
    for G, d, plain, taps in ((2, 128, 300, 4), (1, 40, 22, 4), (3, 64, 64, 4), (1, 33, 7, 3)):
        C = 2 * G * d + plain
        x = torch.randn(sum(lens), C, generator=g)
        cw = torch.randn(C, taps, generator=g)
        seqs, slots, r0, ref = [], [], 0, []
        for s, n in enumerate(lens):
            seqs.append((r0, n, s, 0))
            slots += [s] * n
            z = torch.nn.functional.silu(O.short_conv(x[r0:r0 + n].double(), cw.double()))
            ref.append(torch.cat([(O.unit(z[:, :G * d].view(n, G, d)) * 0.25).reshape(n, G * d), O.unit(z[:, G * d:2 * G * d].view(n, G, d)).reshape(n, G * d),
                                  z[:, 2 * G * d:]], 1))
            r0 += n
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev).reshape(-1)
        xd, wd, sq, sl, ss = x.to(dev), cw.t().contiguous().to(dev), i32(seqs), i32(slots), i32(list(range(len(lens))))
        hist, out = torch.full((len(lens), (taps - 1) * C), float('nan'), device=dev), torch.empty(r0, C, device=dev)
        c = ShortConvArgs()
        c.proj, c.ld_proj, c.n_unit, c.dim, c.n_scaled, c.n_plain = ptr(xd), C, 2 * G, d, G, plain
        c.w, c.taps, c.conv_state, c.scale, c.unit_eps = ptr(wd), taps, ptr(hist), 0.25, 1e-6
        c.seqs, c.slot_seq, c.tok_slot, c.n_rows, c.out, c.ld_out = ptr(sq), ptr(ss), ptr(sl), r0, ptr(out), C
        call_struct('p3_short_conv', c, 0)
        torch.cuda.synchronize()
        assert (out.cpu().double() - torch.cat(ref, 0)).abs().max() < 2e-5 * float(torch.cat(ref, 0).abs().max())


@pytest.mark.parametrize('W', [50, 96, 1030, 2048, 4100, 8200, 9001])
@pytest.mark.parametrize('dtype', [F32, B16])
def test_normed_embedding_and_residual_norm(lib, W, dtype):
    configs, weights, engine, lupusun, paged, O = _mods()
    from phi3_b200._lib import call, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(2)
    T, V, eps, f32 = 5, 11, 1e-2, int(dtype == F32)
    table = (torch.randn(V, W, generator=g) * 0.1).bfloat16()
    ids = torch.tensor([3, 0, 10, 3, 7], dtype=torch.int32)
    ge, gp = torch.rand(W, generator=g) + 0.5, torch.rand(W, generator=g) + 0.5
    x, copy, h = torch.empty(T, W, device=dev), torch.empty(T, W, device=dev), torch.empty(T, W, dtype=dtype, device=dev)
    td, idd, ged, gpd = table.to(dev), ids.to(dev), ge.to(dev), gp.to(dev)
    tol = 2e-5 if dtype == F32 else 3e-2
    call('p3_embed_norm_rows_f32', ptr(td), ptr(idd), ptr(ged), ptr(x), ptr(copy), ptr(gpd), ptr(h), f32, T, W, V, eps, 0)
    want = O.rms_norm(table[ids.long()].double(), ge.double(), eps)
    assert (x.cpu().double() - want).abs().max() < 2e-5 and torch.equal(x, copy)
    assert (h.cpu().double() - O.rms_norm(want, gp.double(), eps)).abs().max() < tol
    x2 = torch.empty_like(x)
    call('p3_embed_norm_rows_f32', ptr(td), ptr(idd), ptr(ged), ptr(x2), None, None, None, f32, T, W, V, eps, 0)
    assert torch.equal(x2, x)
    y, add = torch.randn(T, W + 4, generator=g), torch.randn(T, W, generator=g)
    yd, ad = y.to(dev), add.to(dev)
    rows = torch.tensor([4, 0, 2], dtype=torch.int32, device=dev)
    for use_y, use_add, use_gain, use_rows in ((1, 0, 1, 0), (1, 1, 1, 0), (0, 1, 1, 0), (0, 0, 1, 0), (1, 0, 0, 0), (1, 0, 1, 1), (0, 0, 1, 1)):
        xs = x.clone()
        R = 3 if use_rows else T
        h = torch.full((R, W), float('nan'), dtype=dtype, device=dev)
        call('p3_residual_rmsnorm', ptr(xs), ptr(yd) if use_y else None, W + 4, 0.7, ptr(ad) if use_add else None, ptr(rows) if use_rows else None,
             ptr(gpd) if use_gain else None, ptr(h) if use_gain else None, f32, R, W, eps, 0)
        torch.cuda.synchronize()
        new = want + (0.7 * y[:, :W].double() if use_y else 0) + (add.double() if use_add else 0)
        if use_rows:
            assert torch.equal(xs, x)
        else:
            assert (xs.cpu().double() - new).abs().max() < 2e-5
        if use_gain:
            hw = O.rms_norm(new, gp.double(), eps)
            assert (h.cpu().double() - (hw[[4, 0, 2]] if use_rows else hw)).abs().max() < tol


def test_gated_units_with_both_activations(lib):
    from phi3_b200 import _lib
    from phi3_b200._lib import call, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(4)
    for F in (24, 33):
        gu = torch.randn(7, 2 * F, generator=g)
        gd = gu.to(dev)
        for act, fn in ((_lib.GLU_SILU, torch.nn.functional.silu), (_lib.GLU_RELU, torch.relu)):
            for dt in (F32, B16):
                out = torch.empty(7, F, dtype=dt, device=dev)
                call('p3_glu_act', ptr(gd), ptr(gd[:, F:]), 2 * F, ptr(out), F, int(dt == F32), 7, F, act, 0)
                torch.cuda.synchronize()
                assert (out.float().cpu() - fn(gu[:, :F]) * gu[:, F:]).abs().max() < (1e-5 if dt == F32 else 3e-2)
    with pytest.raises(RuntimeError):
        call('p3_glu_act', ptr(gd), ptr(gd), 33, ptr(gd), 33, 1, 1, 33, 9, 0)


# ------------------------------------------------------------------------------------------------ entry points
def test_greedy_generation_through_load_generate_and_the_scheduler(lib, tmp_path):
    configs, weights, engine, lupusun, paged, O = _mods()
    from phi3_b200 import api
    from safetensors.torch import save_file
    cfg = configs.tiny_lupusun()
    w = weights.random_lupusun_weights(cfg, 13)
    json.dump(cfg, open(tmp_path / 'config.json', 'w'))
    save_file(w, str(tmp_path / 'model.safetensors'))
    model, proc = api.load(model_path=str(tmp_path), dtype=F32)
    assert type(model).__name__ == 'LupusunB200'
    prompts = [tokens(n, cfg['vocab'], 60 + n) for n in (70, 3, 130, 20, 65)]
    n_new = 12
    # five requests through two slots and a pool of 8 pages: queueing, portions, slot, page and state reuse
    from phi3_b200.engine import generate_tokens
    outs = generate_tokens(model, prompts, max_new=n_new, max_tokens=64 * 8, n_slots=2, token_budget=96, chunk=40)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(n_new):
            seq.append(int(O.forward(cfg, w, seq, torch.float64)[-1].argmax()))
        assert o == seq[len(p):]
    assert api.generate_batch(prompts[:2], preload=(model, proc), max_tokens=n_new, return_tokens=True) == outs[:2]
    text = api.generate('hello there', preload=(model, proc), max_tokens=5, verbose=False)
    assert isinstance(text, str)


def test_trace_runner_replays_steps(lib, tmp_path):
    configs, weights, engine, lupusun, paged, O = _mods()
    from safetensors.torch import save_file
    import numpy as np
    cfg = configs.tiny_lupusun()
    w = weights.random_lupusun_weights(cfg, 14)
    mdir, out = tmp_path / 'm', tmp_path / 'out'
    mdir.mkdir()
    json.dump(cfg, open(mdir / 'config.json', 'w'))
    save_file(w, str(mdir / 'model.safetensors'))
    a, b = tokens(80, cfg['vocab'], 70), tokens(9, cfg['vocab'], 71)
    steps = [{'step': 0, 'entries': [{'id': 'a', 'tokens': a[:70], 'want': [0, 69]}, {'id': 'b', 'tokens': b[:2], 'want': []}], 'end': []},
             {'step': 1, 'entries': [{'id': 'b', 'tokens': b[2:], 'want': [6]}], 'end': ['b']},
             {'step': 2, 'entries': [{'id': 'a', 'tokens': a[70:71], 'want': []}], 'end': []},
             {'step': 3, 'entries': [{'id': 'a', 'tokens': a[71:], 'want': [8]}], 'end': ['a']}]
    for dt, tol in (('float32', TOL[F32]), ('bfloat16', TOL[B16])):
        r = subprocess.run([os.path.join(ROOT, 'bin', 'trace_run'), '--model', str(mdir), '--dtype', dt, '--out', str(out),
                            '--max-tokens', '192'], input='\n'.join(json.dumps(s) for s in steps) + '\n', capture_output=True,
                           text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith('done')] == ['done 0', 'done 1', 'done 2', 'done 3']
        ra, rb = O.forward(cfg, w, a, torch.float64), O.forward(cfg, w, b, torch.float64)
        rd = lambda n: torch.from_numpy(np.fromfile(out / f'{n}.f32', dtype='<f4').reshape(-1, cfg['vocab']))
        assert not (out / '2.f32').exists()
        assert rel_err(rd(0), ra[[0, 69]]) < tol and rel_err(rd(1), rb[[8]]) < tol and rel_err(rd(3), ra[[79]]) < tol
        for f in out.iterdir():
            f.unlink()
