"""Gugezen on the continuous-batching engine against the plain CPU restatement (oracle/gugezen_oracle.py).

Small random checkpoints of several shapes; the CUDA path (model, page pool with its state rows, engine, scheduler, public API,
trace runner) must give the oracle's logits whatever the schedule: whole prompts, token-by-token decoding, portions down to two
tokens, mixed batches, reused pages and slots. Each mechanism is also probed alone at the kernel level, with inputs made so that a
fault shows (one dominant key far back, at a page border or at the query itself; a sink that takes most of the weight; decays and
steps at both ends of their range; a slot's stale state and stale convolution inputs; streams that differ by orders of magnitude).
"""
import ctypes
import json
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
    from phi3_b200 import configs, weights, engine, gugezen, paged
    from oracle import gugezen_oracle as O
    return configs, weights, engine, gugezen, paged, O


def row_err(got, ref):
    """per row: rms of the mean-free difference, relative to the spread of the reference"""
    got, ref = got.double().cpu(), ref.double().cpu()
    d = got - ref
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / ref.std()


def rel_err(got, ref):
    return float(row_err(got, ref).max())


def assert_close(got, ref, dtype, what=''):
    """fp32: every row within 2e-4. bf16: the median row well inside the rounding bound and nine rows in ten within it. (A few may lie
    outside for reasons that are not the kernels': where two experts' scores are nearly equal, rounding decides which one a token
    takes; where a sequence's first tokens give a read-out near zero, the norm behind it enlarges the rounding of its inputs.)"""
    e = row_err(got, ref)
    if dtype == F32:
        assert float(e.max()) < TOL[F32], (what, float(e.max()))
    else:
        q = torch.quantile(e, torch.tensor([0.5, 0.9], dtype=e.dtype))
        assert float(q[0]) < 0.03 and float(q[1]) < TOL[B16], (what, q.tolist(), float(e.max()))


def make(cfg_dict, dtype, seed=0):
    configs, weights, engine, gugezen, paged, O = _mods()
    w = weights.random_gugezen_weights(cfg_dict, seed)
    return gugezen.GugezenB200(cfg_dict, w, dtype=dtype), w


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
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
    model, w = make(cfg, dtype)
    toks = tokens(150, cfg['vocab'], 1)                       # more than two pages
    ref_trace = []
    ref = O.forward(cfg, w, toks, torch.float64, ref_trace)
    eng = engine.Engine(model, 256, 4)
    poison(eng)
    trace = []
    got = eng.step([('a', toks, list(range(len(toks))))], ['a'], trace=trace)
    assert_close(got, ref, dtype)
    assert len(trace) == len(ref_trace) == 6                  # layers that share tensors count each time
    if dtype == F32:
        for i, (g, r) in enumerate(zip(trace, ref_trace)):
            assert (g.cpu().double() - r).abs().max() < 2e-4 * float(r.abs().max()), f'residual streams after layer {i}'
    assert len(eng.pool.free_pages) == eng.pool.n_pages and len(eng.pool.free_slots) == 4
    assert len(eng.pool.state) == 9 and len(eng.pool.k) == 6   # a state per linear memory, a state and convolution inputs per state-space layer


@pytest.mark.parametrize('dtype', [F32, B16])
def test_prefill_then_token_by_token_decoding(lib, dtype):
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
    model, w = make(cfg, dtype, seed=2)
    toks = tokens(140, cfg['vocab'], 3)
    ref = O.forward(cfg, w, toks, torch.float64)
    got = run_schedule(model, toks, [30])                     # 110 decoded tokens: page borders pass by
    assert_close(got, ref, dtype)
    whole = run_schedule(model, toks, [len(toks)])
    if dtype == F32:
        assert rel_err(got, whole) < 1e-5
    else:
        assert_close(got, whole, dtype)


@pytest.mark.parametrize('cuts', [[2, 2, 3, 31, 33, 2, 64, 1, 2], [63, 2, 63, 2], [1, 1, 64, 65], [100, 2, 2], [5, 32, 37, 3]])
def test_prompt_portions_of_any_size(lib, cuts):
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
    model, w = make(cfg, F32, seed=4)
    toks = tokens(sum(cuts) + 5, cfg['vocab'], 5)
    ref = O.forward(cfg, w, toks, torch.float64)
    assert rel_err(run_schedule(model, toks, cuts), ref) < TOL[F32]


@pytest.mark.parametrize('dtype', [F32, B16])
def test_mixed_batch_of_unequal_requests_equals_each_alone(lib, dtype):
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
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
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
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
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
    model, w = make(cfg, F32, seed=8)
    for n in (1, 2, 3):
        toks = tokens(n, cfg['vocab'], 40 + n)
        assert rel_err(run_schedule(model, toks, [n]), O.forward(cfg, w, toks, torch.float64)) < TOL[F32]
    toks = tokens(230, cfg['vocab'], 44)
    assert rel_err(run_schedule(model, toks, [1]), O.forward(cfg, w, toks, torch.float64)) < TOL[F32]   # all decoded one by one


def test_a_request_that_sits_out_steps_keeps_its_state(lib):
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
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
    configs, weights, engine, gugezen, paged, O = _mods()
    cfg = configs.tiny_gugezen()
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
def _par(heads, kv, dim, vdim, mh, mdim, mvdim, rd=None, scaling=(4.0, 1.0, 4.0, 64), base=10000.0, scale=None, ls=0.8, rs=1.1, decay=None):
    rd = dim if rd is None else rd
    sc = {'scaling': dict(zip(('factor', 'low', 'high', 'original'), scaling))} if scaling else {}
    return {'type': 'parallel',
            'mixer': {'left': dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or 2.0 * dim ** -0.5,
                                   **({'rot': {'base': base, 'dims': rd, **sc}} if rd else {})),
                      'right': dict(heads=mh, dim=mdim, vdim=mvdim, decay=decay or [1.0 - 2.0 ** -(1 + 1.5 * h) for h in range(mh)]),
                      'left_scale': ls, 'right_scale': rs}}


def _ssm(heads, vdim, state, groups, taps, parts):
    return {'type': 'mamba2', 'mixer': dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=taps, norm_groups=parts)}


def _dense(ff):
    return {'kind': 'dense', 'ff': ff}


def _moe(ff, e, top, shared=None):
    return {'kind': 'moe', 'expert': {'ff': ff}, 'router': dict(experts=e, top=top), **({'shared': {'ff': shared}} if shared else {})}


OTHER = {
    # every count 1: one stream, one head, one group, one tap (no history at all), one expert; factors of one
    'ones': (64, dict(streams=1, embed_scale=1.0, logit_scale=1.0),
             [dict(_par(1, 1, 16, 16, 1, 16, 16, ls=1.0, rs=1.0), mlp=_moe(16, 1, 1)), dict(_ssm(1, 16, 16, 1, 1, 1), mlp=_dense(64)),
              dict(_par(1, 1, 8, 8, 1, 1, 8, 2, ls=0.0), mlp=None), dict(_ssm(1, 8, 1, 1, 2, 1), mlp=_moe(8, 2, 1, 16))]),
    # sizes that tile the tensor-core kernels and equal each other
    'tiled': (128, dict(streams=2, embed_scale=0.5, logit_scale=0.25),
              [dict(_par(4, 4, 64, 64, 4, 64, 64), mlp=_dense(256)), dict(_ssm(4, 64, 64, 4, 4, 4), mlp=_moe(128, 4, 2, 128)),
               dict(_par(8, 2, 128, 128, 2, 128, 128, 64, (8.0, 1.0, 4.0, 100)), mlp=_moe(64, 8, 8)), dict(_ssm(8, 32, 128, 2, 4, 1), mlp=None),
               dict(_ssm(4, 64, 64, 4, 4, 4), weights_of=1, mlp=_moe(128, 4, 2, 128))]),
    # nothing is a multiple of 8: every product goes through the any-shape kernel, every attention through the fp32 kernels
    'ragged': (50, dict(streams=5, embed_scale=2.0, logit_scale=3.0),
               [dict(_ssm(6, 7, 9, 3, 5, 2), mlp=_dense(33)), dict(_par(3, 1, 10, 7, 5, 13, 3, 6), mlp=_moe(21, 3, 2, 11)), dict(_ssm(5, 3, 13, 1, 3, 5), mlp=None),
                dict(_par(6, 2, 11, 14, 3, 6, 9, 2, (3.0, 0.5, 2.0, 30)), mlp=_dense(19)), dict(_ssm(6, 7, 9, 3, 5, 2), weights_of=0, mlp=_dense(33))]),
    # a history longer than the shortest portions, wide states, many heads on one group, heads without a rotation, value heads of 200 numbers,
    # parts longer than a warp's registers, a memory that keeps everything and one that keeps nothing
    'wide': (96, dict(streams=9),
             [dict(_ssm(12, 24, 260, 1, 9, 1), mlp=_dense(96)), dict(_par(12, 1, 24, 200, 2, 260, 40, decay=[1.0, 0.0]), mlp=None),
              dict(_ssm(2, 136, 48, 2, 4, 2), mlp=_moe(24, 12, 5)), dict(_par(2, 2, 160, 96, 3, 24, 136, 0), mlp=_dense(40))]),
}


@pytest.mark.parametrize('name', list(OTHER))
@pytest.mark.parametrize('dtype', [F32, B16])
def test_other_sizes(lib, name, dtype):
    configs, weights, engine, gugezen, paged, O = _mods()
    width, kw, layers = OTHER[name]
    cfg = configs.tiny_gugezen(width=width, vocab=211 if name != 'ragged' else 101, layers=layers, **kw)
    model, w = make(cfg, dtype, seed=11)
    toks = tokens(150, cfg['vocab'], 12)
    assert_close(run_schedule(model, toks, [70, 2, 40]), O.forward(cfg, w, toks, torch.float64), dtype, name)


def test_stacks_of_one_kind_and_layers_that_share_tensors(lib):
    """a borrowed layer keeps a cache and a state of its own: the same tensors three times in a row, fed in portions"""
    configs, weights, engine, gugezen, paged, O = _mods()
    for lay in (dict(_ssm(2, 16, 24, 1, 4, 1), mlp=_dense(40)), dict(_par(4, 2, 24, 16, 2, 16, 24), mlp=None)):
        cfg = configs.tiny_gugezen(width=48, vocab=90, layers=[lay, dict(lay, weights_of=0), dict(lay, weights_of=1)], streams=2)
        model, w = make(cfg, F32, seed=5)
        assert len(set(k.split('.')[0] for k in w if k[0] == 'l')) == 1 and model.layers[2] is model.layers[0]
        toks = tokens(100, 90, 6)
        assert rel_err(run_schedule(model, toks, [50, 2, 3, 30]), O.forward(cfg, w, toks, torch.float64)) < TOL[F32]


def test_large_steps_take_the_dense_expert_products_and_the_second_stream(lib):
    """prompt steps of several hundred rows: experts as per-expert products (segment offsets read back), the two halves of a parallel mixer
    on two streams; the same rows through the small-batch paths"""
    configs, weights, engine, gugezen, paged, O = _mods()
    width, kw, layers = OTHER['tiled']
    cfg = configs.tiny_gugezen(width=width, vocab=256, layers=layers, **kw)
    model, w = make(cfg, B16, seed=15)
    lens = {'a': 410, 'b': 300, 'c': 1, 'd': 90}
    toks = {k: tokens(n, 256, 16 + i) for i, (k, n) in enumerate(lens.items())}
    model.moe_dense_rows = 256
    assert model.experts_dense(model.cfg.layers[1].ff, 801) and sum(lens.values()) > model.SIDE_ROWS
    eng = engine.Engine(model, 64 * 20, 4)
    poison(eng)
    for rnd in range(2):
        big = eng.step([(k, t, list(range(len(t)))) for k, t in toks.items()], list(toks))
        o = 0
        for k, t in toks.items():
            ref = O.forward(cfg, w, t, torch.float64) if k != 'a' or rnd == 0 else None
            if ref is not None:
                assert_close(big[o:o + len(t)], ref, B16, k)
            o += len(t)
    model.moe_dense_rows, model.SIDE_ROWS = 1 << 30, 1 << 30
    assert_close(big[:410], run_schedule(model, toks['a'], [410], max_tokens=512), B16)
    m32, _ = make(cfg, F32, seed=15)                          # fp32: the second stream alone
    assert rel_err(run_schedule(m32, toks['b'], [300], max_tokens=320), O.forward(cfg, w, toks['b'], torch.float64)) < TOL[F32]


def test_small_batches_take_the_weight_streaming_products(lib):
    """the tiled stack with dense units only (no close calls between experts, which rounding alone would decide)"""
    configs, weights, engine, gugezen, paged, O = _mods()
    width, kw, layers = OTHER['tiled']
    cfg = configs.tiny_gugezen(width=width, vocab=256, layers=[dict(l, mlp=_dense(192)) for l in layers], **kw)
    model, w = make(cfg, B16, seed=15)
    toks = tokens(40, cfg['vocab'], 16)
    ref = O.forward(cfg, w, toks, torch.float64)
    a = run_schedule(model, toks, [20])
    model.use_skinny = False
    b = run_schedule(model, toks, [20])
    assert_close(a, ref, B16)
    assert_close(b, ref, B16)


def _random_config(rng):
    """a random order of the two mixers with random sizes, and now and then a layer that borrows an earlier one's tensors"""
    layers = []
    for i in range(rng.randint(2, 5)):
        own = [j for j, l in enumerate(layers) if 'weights_of' not in l]
        if own and rng.random() < 0.3:
            j = rng.choice(own)
            layers.append(dict(layers[j], weights_of=j))
            continue
        mlp = rng.choice([None, _dense(rng.choice([24, 40, 64])), _dense(40), _moe(rng.choice([16, 24]), 4, rng.randint(1, 4), rng.choice([None, 24, 32]))])
        n = rng.randint(1, 3)
        if rng.random() < 0.5:
            dim = rng.choice([8, 16, 24, 40])
            lay = _par(n * rng.randint(1, 3), n, dim, rng.choice([8, 24, 32]), rng.randint(1, 3), rng.choice([8, 24, 40]), rng.choice([8, 24, 70]),
                       rng.choice([r for r in (0, 2, 4, 8, 16, dim) if r <= dim]), rng.choice([None, (4.0, 1.0, 4.0, 64), (16.0, 0.5, 2.0, 512)]),
                       rng.choice([100.0, 10000.0, 1000000.0]), ls=rng.choice([0.5, 1.0]), rs=rng.choice([0.7, 1.0]))
        else:
            heads, vdim = n * rng.randint(1, 3), rng.choice([8, 24, 40])
            lay = _ssm(heads, vdim, rng.choice([8, 24, 40, 72]), n, rng.choice([1, 2, 3, 4, 4, 6]), rng.choice([1, 2, heads]))
        layers.append(dict(lay, mlp=mlp))
    return _mods()[0].tiny_gugezen(width=rng.choice([48, 64, 72, 96]), vocab=rng.choice([77, 128, 300]), layers=layers, streams=rng.choice([1, 2, 3, 4]),
                                   embed_scale=rng.choice([0.3, 1.0]), logit_scale=rng.choice([0.5, 1.0, 2.0]))


@pytest.mark.parametrize('seed', [21, 22, 23, 24, 25, 26])
def test_random_configurations_under_random_schedules(lib, seed):
    """random layer orders and sizes, random requests fed in random portions beside each other through a pool that forces pages,
    slots and state rows to change hands"""
    configs, weights, engine, gugezen, paged, O = _mods()
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
        assert_close(torch.cat([torch.cat(g, 0) for g in got], 0), torch.cat(ref, 0), dtype, seed)


# ------------------------------------------------------------------------------------------------ mechanisms alone
def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device='cuda').reshape(-1)


@pytest.mark.parametrize('shape', [(3, 3, 28, 20), (6, 2, 64, 64), (8, 1, 48, 40), (4, 2, 128, 96), (2, 1, 264, 200)])
@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('n_splits', [1, 3])
def test_sinks_gates_and_far_keys(lib, shape, dtype, n_splits):
    """dominant pairs far back (the first key from the last query), on both sides of page borders, at the query's own position and at the
    first positions; one head's sink outweighs every ordinary key, another's is negligible; every output number has a gate of its own
    and the heads leave through a factor into rows that are wider than they are; tiles begin inside a page, too"""
    from phi3_b200._lib import AttnWindowArgs, call_struct, ptr
    dev = torch.device('cuda')
    H, G, d, dv = shape
    n, scale, factor, pad = 300, 0.7, 0.6, 6
    g = torch.Generator().manual_seed(1)
    q, k, v = torch.randn(n, H, d, generator=g) * 0.5, torch.randn(n, G, d, generator=g) * 0.5, torch.randn(n, G, dv, generator=g)
    for m, (i, j) in enumerate([(299, 0), (298, 63), (297, 64), (1, 0), (0, 0), (64, 63), (64, 64), (128, 127), (130, 128), (131, 66), (192, 191),
                                (200, 150), (255, 250), (256, 255), (256, 192), (290, 64), (77, 76), (77, 0)]):
        u = torch.zeros(d)
        u[m % d] = 6.0
        q[i] += u
        k[j] += u
    if dtype == B16:
        q, k, v = q.bfloat16().float(), k.bfloat16().float(), v.bfloat16().float()
    sink, gate = torch.linspace(-6.0, 5.0, H), torch.randn(n, H * dv + 3, generator=g) * 3
    vis = torch.ones(n, n).tril().bool()
    ref = torch.zeros(n, H, dv, dtype=torch.float64)
    for h in range(H):
        sc = ((q[:, h].double() @ k[:, h // (H // G)].double().T) * scale).masked_fill(~vis, float('-inf'))
        m = torch.clamp(sc.max(-1, keepdim=True).values, min=float(sink[h]))
        e = torch.exp(sc - m)
        ref[:, h] = e / (e.sum(-1, keepdim=True) + torch.exp(sink[h].double() - m)) @ v[:, h // (H // G)].double()
    ref = ref.reshape(n, H * dv) * torch.sigmoid(gate[:, 3:].double()) * factor
    n_pg = -(-n // 64)
    perm = torch.randperm(n_pg + 3, generator=g)[:n_pg]
    kp, vp = torch.full((n_pg + 3, G, 64, d), 50.0), torch.full((n_pg + 3, G, 64, dv), -70.0)
    for p in range(n_pg):
        c = min(64, n - 64 * p)
        kp[perm[p], :, :c], vp[perm[p], :, :c] = k[64 * p:64 * p + c].transpose(0, 1), v[64 * p:64 * p + c].transpose(0, 1)
    bt = torch.zeros(2, n_pg + 3, dtype=torch.int32)
    bt[1, :n_pg] = perm.int()
    kp, vp, bt, sd, gd = kp.to(dev, dtype), vp.to(dev, dtype), bt.to(dev), sink.to(dev), gate.to(dev)
    qd = q.reshape(n, H * d).to(dev, dtype).contiguous()
    a = AttnWindowArgs()
    a.q, a.ld_q, a.k_pool, a.v_pool, a.block_table, a.bt_stride = ptr(qd), H * d, ptr(kp), ptr(vp), ptr(bt), bt.stride(0)
    a.ld_out, a.sink, a.elem_gate, a.ld_elem_gate, a.out_scale = H * dv + pad, ptr(sd), ptr(gd[:, 3:]), H * dv + 3, factor
    a.n_heads, a.n_kv, a.dim, a.vdim, a.scale, a.act_f32, a.cache_f32 = H, G, d, dv, scale, int(dtype == F32), int(dtype == F32)
    for kind, first in (('prefill', 0), ('prefill', 77), ('decode', 0)):
        out = torch.full((n, H * dv + pad), 7.0, dtype=dtype, device=dev)
        a.out = ptr(out)
        step = int(lib.lib().p3_attn_window_tile_rows(ctypes.byref(a))) if kind == 'prefill' else 1
        tiles = [(r0, min(step, n - r0), 1, r0) for r0 in range(first, n, step)]
        td = _i32(tiles)
        a.tiles, a.n_tiles = ptr(td), len(tiles)
        ws = torch.empty(len(tiles) * H * n_splits * (dv + 2), device=dev)
        a.n_splits, a.ws = n_splits, ptr(ws)
        call_struct('p3_attn_window_' + kind, a, 0)
        torch.cuda.synchronize()
        tol = (1e-4 if dtype == F32 else 3e-2) * max(1.0, float(ref.abs().max()))
        assert (out[first:, :H * dv].double().cpu() - ref[first:]).abs().max() < tol, (kind, first)
        assert (out[:, H * dv:] == 7.0).all()


@pytest.mark.parametrize('dtype', [F32, B16])
@pytest.mark.parametrize('shape', [(4, 2, 24, 40, 16), (3, 3, 7, 5, 2), (2, 1, 128, 64, 128), (2, 1, 300, 20, 130), (5, 5, 64, 64, 0)])
def test_neighbour_pairs_turn_and_memory_columns_pass_silu(lib, dtype, shape):
    """biases, the partial rotation of neighbours at positions on both sides of page borders and far out, the paged write; silu in place on
    the columns behind q, k, v alone; with few rows and with so many that a CTA takes a whole row"""
    configs, weights, engine, gugezen, paged, O = _mods()
    from phi3_b200._lib import QkvRopePostArgs, call_struct, ptr
    dev = torch.device('cuda')
    H, G, d, dv, rn = shape
    g = torch.Generator().manual_seed(3)
    rot = {'base': 10000.0, 'dims': rn, 'scaling': {'factor': 6.0, 'low': 1.0, 'high': 4.0, 'original': 64}}
    n_qkv = (H + G) * d + G * dv
    for T, n_act in ((9, 20), (9, 7), (1030, 132)):
        cols = n_qkv + 5 + n_act + 3
        proj, bias = torch.randn(T, cols, generator=g), torch.randn(n_qkv, generator=g)
        some = torch.tensor([0, 1, 2, 63, 64, 65, 126, 127, 128])
        pos = some.repeat(-(-T // 9))[:T]
        slot = torch.arange(-(-T // 9)).repeat_interleave(9)[:T]
        bt = torch.arange(3 * (int(slot.max()) + 1)).flip(0).view(-1, 3).int()
        x = proj[:, :n_qkv].double() + bias.double()
        q, k, v = x[:, :H * d].view(T, H, d), x[:, H * d:(H + G) * d].view(T, G, d), x[:, (H + G) * d:].view(T, G, dv)
        if rn:
            q, k = O.rotate_neighbours(q, pos, rot), O.rotate_neighbours(k, pos, rot)
        qd = torch.empty(T, H * d, dtype=dtype, device=dev)
        kp, vp = torch.zeros(bt.numel(), G, 64, d, dtype=dtype, device=dev), torch.zeros(bt.numel(), G, 64, dv, dtype=dtype, device=dev)
        freq = O.stretched_frequencies(rot) if rn else []
        dd = [proj.to(dev), bias.to(dev), torch.tensor(freq, dtype=torch.float32, device=dev), bt.to(dev), slot.int().to(dev), pos.int().to(dev)]
        a = QkvRopePostArgs()
        a.proj, a.ld_proj, a.q_off, a.k_off, a.v_off, a.bias = ptr(dd[0]), cols, 0, H * d, (H + G) * d, ptr(dd[1])
        a.n_heads, a.n_kv, a.dim, a.vdim, a.rot_n, a.freq, a.pair_mode = H, G, d, dv, rn, ptr(dd[2]), 1
        a.act_cols, a.n_act = ptr(dd[0][:, n_qkv + 5:]), n_act
        a.q_out, a.ld_q, a.k_pool, a.v_pool, a.block_table, a.bt_stride = ptr(qd), H * d, ptr(kp), ptr(vp), ptr(dd[3]), 3
        a.tok_slot, a.tok_pos, a.T, a.act_f32, a.cache_f32 = ptr(dd[4]), ptr(dd[5]), T, int(dtype == F32), int(dtype == F32)
        call_struct('p3_qkv_rope_post', a, 0)
        torch.cuda.synchronize()
        tol = 4e-5 if dtype == F32 else 3e-2
        assert (qd.double().cpu().view(T, H, d) - q).abs().max() < tol
        page = bt[slot, pos // 64].long()
        assert (kp.cpu()[page, :, pos % 64].double() - k).abs().max() < tol and (vp.cpu()[page, :, pos % 64].double() - v).abs().max() < tol
        after = dd[0].cpu()
        want = proj.clone()
        want[:, n_qkv + 5:n_qkv + 5 + n_act] = O.silu(proj[:, n_qkv + 5:n_qkv + 5 + n_act].double()).float()
        assert (after - want).abs().max() < 1e-6 and torch.equal(after[:, :n_qkv + 5], proj[:, :n_qkv + 5]) and torch.equal(after[:, -3:], proj[:, -3:])


@pytest.mark.parametrize('shape', [(4, 2, 24, 40, 4), (1, 1, 7, 5, 4), (3, 1, 20, 64, 3), (3, 3, 64, 64, 4), (4, 2, 128, 96, 4), (2, 1, 200, 33, 2),
                                   (5, 5, 136, 70, 1), (2, 2, 300, 40, 4), (6, 2, 34, 22, 7), (2, 1, 1, 8, 4), (2, 2, 66, 12, 40)])
@pytest.mark.parametrize('rs', [0, 2, 4, 8])
def test_convolution_and_scan_in_portions(lib, shape, rs):
    """the recurrent part of the state-space mixer alone (convolution with bias, gates, state, skip), and the same scan with fixed decays:
    whole sequences against the oracle, then the same sequences in portions (states and convolution inputs carry on, portions shorter
    than the taps among them) with a second sequence in the batch, bit for bit equal to the whole run. Some tokens make a head forget
    everything, some keep everything and write next to nothing. rs: the shape of a warp (0: the launch's own choice)"""
    configs, weights, engine, gugezen, paged, O = _mods()
    from phi3_b200._lib import ShortConvArgs, DeltaScanArgs, call_struct, ptr
    dev = torch.device('cuda')
    H, G, N, dv, taps = shape
    g = torch.Generator().manual_seed(7)
    T = {0: 83, 1: 37}
    inner, C = H * dv, H * dv + 2 * G * N
    cols = C + H + 3
    proj = {s: torch.randn(n, cols, generator=g) for s, n in T.items()}
    for s in proj:
        proj[s][20:22, C:C + H] = 60.0                         # forget everything ...
        proj[s][24:34, C:C + H] = -60.0                        # ... keep everything
    cw, cb = torch.randn(C, taps, generator=g) * 0.6, torch.randn(C, generator=g) * 0.5
    a_log, dt, skip = torch.randn(H, generator=g) * 0.5, torch.randn(H, generator=g) - 2.0, torch.randn(H, generator=g)
    fixed = torch.tensor([1.0, 0.0, 0.5, 0.9, 0.99, 0.999])[:H]
    of, ref, ref_fixed = [h // (H // G) for h in range(H)], {}, {}
    for s, p in proj.items():
        x = p.double()
        z = O.silu(O.short_conv(x[:, :C], cw.double(), cb.double()))
        xs, B, Cc = z[:, :inner].view(-1, H, dv), z[:, inner:inner + G * N].view(-1, G, N)[:, of], z[:, inner + G * N:].view(-1, G, N)[:, of]
        step = torch.nn.functional.softplus(x[:, C:C + H] + dt.double(), threshold=1e9)
        y = O.decayed_memory(Cc, B, step[..., None] * xs, torch.exp(-torch.exp(a_log.double()) * step))
        ref[s] = (y + skip.double()[:, None] * xs).reshape(-1, inner)
        ref_fixed[s] = O.decayed_memory(Cc, B, xs, fixed.double().expand(len(x), H)).reshape(-1, inner)
    n_state = int(lib.lib().p3_delta_state_floats(H, N, dv))
    cwd, cbd, ald, dtd, skd, fxd = (t.contiguous().to(dev) for t in (cw.t(), cb, a_log, dt, skip, fixed))

    def run(plans, constant):
        state = torch.full((3, n_state), float('nan'), device=dev)
        hist = torch.full((3, max(taps - 1, 1) * C), float('nan'), device=dev)
        got = {s: [] for s in T}
        for plan in plans:
            seqs, rows, slots, slot_seq, r0 = [], [], [], [0] * 3, 0
            for slot, p0, n in plan:
                slot_seq[slot] = len(seqs)
                seqs.append((r0, n, slot, p0))
                rows.append(proj[slot - 1][p0:p0 + n])
                slots += [slot] * n
                r0 += n
            pd = torch.cat(rows, 0).to(dev)
            xbc, gates, out = torch.empty(r0, C, device=dev), torch.empty(r0, H, 2, device=dev), torch.empty(r0, inner, device=dev)
            sq, sl, ss = _i32(seqs), _i32(slots), _i32(slot_seq)
            c = ShortConvArgs()
            c.proj, c.ld_proj, c.n_plain, c.w, c.bias, c.taps, c.conv_state = ptr(pd), cols, C, ptr(cwd), ptr(cbd), taps, ptr(hist)
            c.seqs, c.slot_seq, c.tok_slot, c.n_rows, c.out, c.ld_out = ptr(sq), ptr(ss), ptr(sl), r0, ptr(xbc), C
            c.a_off, c.n_gates, c.a_log, c.dt_bias, c.gates, c.gate_mode = C, H, ptr(ald), ptr(dtd), ptr(gates), 1
            call_struct('p3_short_conv', c, 0)
            a = DeltaScanArgs()
            a.qkv, a.ld_qkv, a.v_off, a.k_off, a.q_off = ptr(xbc), C, 0, inner, inner + G * N
            a.n_heads, a.n_kv, a.dim, a.vdim, a.state, a.seqs, a.n_seqs = H, G, N, dv, ptr(state), ptr(sq), len(seqs)
            if constant:
                a.decay = ptr(fxd)
            else:
                a.gates, a.skip = ptr(gates), ptr(skd)
            a.out, a.ld_out, a.rs_force = ptr(out), inner, rs
            a.conv_in, a.ld_conv_in, a.channels, a.taps, a.conv_state = ptr(pd), cols, C, taps, ptr(hist)
            call_struct('p3_decay_scan', a, 0)
            torch.cuda.synchronize()
            o = 0
            for slot, p0, n in plan:
                got[slot - 1].append(out[o:o + n].cpu())
                o += n
        return {s: torch.cat(v, 0) for s, v in got.items()}

    for constant, want in ((False, ref), (True, ref_fixed)):
        whole = run([[(1, 0, 83), (2, 0, 37)]], constant)      # sequence s lives in slot s + 1
        parts = run([[(1, 0, 17)], [(2, 0, 2), (1, 17, 1)], [(1, 18, 16), (2, 2, 33)], [(1, 34, 1)], [(2, 35, 2), (1, 35, 2)], [(1, 37, 46)]], constant)
        for s in T:
            assert (whole[s].double() - want[s]).abs().max() < 1e-4 * max(1.0, float(want[s].abs().max())), (s, constant)
            assert torch.equal(whole[s], parts[s]), (s, constant)


def test_convolution_of_many_rows_equals_that_of_few(lib):
    """long steps walk several rows per warp, with unequal sequences that begin and end inside a warp's rows"""
    configs, weights, engine, gugezen, paged, O = _mods()
    from phi3_b200._lib import ShortConvArgs, call_struct, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(8)
    lens = [1, 2, 3, 130, 1, 5, 250, 16, 15, 300, 2]
    for C, taps, H in ((812, 4, 40), (22, 4, 1), (64, 4, 3), (33, 3, 5)):
        x = torch.randn(sum(lens), 5 + C + H, generator=g)
        cw, cb, a_log, dt = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g)
        seqs, slots, r0, ref = [], [], 0, []
        for s, n in enumerate(lens):
            seqs.append((r0, n, s, 0))
            slots += [s] * n
            ref.append(O.silu(O.short_conv(x[r0:r0 + n, 5:5 + C].double(), cw.double(), cb.double())))
            r0 += n
        xd, wd, bd, ad, td, sq, sl, ss = (x.to(dev), cw.t().contiguous().to(dev), cb.to(dev), a_log.to(dev), dt.to(dev), _i32(seqs), _i32(slots),
                                          _i32(list(range(len(lens)))))
        hist, out, gates = torch.full((len(lens), (taps - 1) * C), float('nan'), device=dev), torch.empty(r0, C, device=dev), torch.empty(r0, H, 2, device=dev)
        c = ShortConvArgs()
        c.proj, c.ld_proj, c.c_off, c.n_plain, c.w, c.bias, c.taps, c.conv_state = ptr(xd), 5 + C + H, 5, C, ptr(wd), ptr(bd), taps, ptr(hist)
        c.seqs, c.slot_seq, c.tok_slot, c.n_rows, c.out, c.ld_out = ptr(sq), ptr(ss), ptr(sl), r0, ptr(out), C
        c.a_off, c.n_gates, c.a_log, c.dt_bias, c.gates, c.gate_mode = 5 + C, H, ptr(ad), ptr(td), ptr(gates), 1
        call_struct('p3_short_conv', c, 0)
        torch.cuda.synchronize()
        assert (out.cpu().double() - torch.cat(ref, 0)).abs().max() < 2e-5 * float(torch.cat(ref, 0).abs().max())
        step = torch.nn.functional.softplus(x[:, 5 + C:].double() + dt.double(), threshold=1e9)
        want = torch.stack([torch.exp(-torch.exp(a_log.double()) * step), step], -1)
        assert (gates.cpu().double() - want).abs().max() < 2e-6 * float(want.max())


@pytest.mark.parametrize('S,W', [(1, 96), (2, 96), (3, 50), (4, 1030), (5, 64), (16, 50), (2, 2048), (4, 4100), (3, 8200), (2, 9001), (1, 9001), (8, 9000)])
@pytest.mark.parametrize('dtype', [F32, B16])
def test_streams_and_their_start(lib, S, W, dtype):
    """streams of very different sizes, transfer matrices without symmetry, rows longer than the registers hold"""
    configs, weights, engine, gugezen, paged, O = _mods()
    from phi3_b200._lib import call, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(2)
    T, V, eps, f32 = 5, 11, 1e-2, int(dtype == F32)
    table = (torch.randn(V, W, generator=g) * 0.1).bfloat16()
    ids = torch.tensor([3, 0, 10, 3, 7], dtype=torch.int32)
    gain, a, b, M = (torch.rand(W, generator=g) + 0.5, torch.randn(S, generator=g), torch.randn(S, generator=g), torch.randn(S, S, generator=g))
    x, h = torch.full((T, S, W), float('nan'), device=dev), torch.full((T, W), float('nan'), dtype=dtype, device=dev)
    d = [t.to(dev) for t in (table, ids, gain, a, b, M)]
    tol = 2e-5 if dtype == F32 else 3e-2
    call('p3_embed_streams', ptr(d[0]), ptr(d[1]), 0.3, ptr(x), S, ptr(d[3]), ptr(d[2]), ptr(h), f32, T, W, V, eps, 0)
    e = table[ids.long()].double() * 0.3
    assert (x.cpu().double() - e[:, None]).abs().max() < 1e-6
    assert (h.cpu().double() - O.rms_norm(e * a.double().sum(), gain.double(), eps)).abs().max() < tol * 4
    X0 = torch.randn(T, S, W, generator=g) * torch.logspace(0, 2, S)[None, :, None] if S > 1 else torch.randn(T, S, W, generator=g)
    y = torch.randn(T, W + 4, generator=g)
    yd, rows = y.to(dev), torch.tensor([4, 0, 2], dtype=torch.int32, device=dev)
    new = O.write_streams(X0.double().transpose(0, 1), M.double(), b.double(), y[:, :W].double())
    old = X0.double().transpose(0, 1)
    for use_y, use_gain, use_rows in ((1, 1, 0), (0, 1, 0), (1, 0, 0), (1, 1, 1), (0, 1, 1)):
        xs = X0.to(dev).contiguous()
        R = 3 if use_rows else T
        h = torch.full((R, W), float('nan'), dtype=dtype, device=dev)
        call('p3_streams_rmsnorm', ptr(xs), S, ptr(yd) if use_y else None, W + 4, ptr(d[5]) if use_y else None, ptr(d[4]) if use_y else None,
             ptr(d[3]) if use_gain else None, ptr(rows) if use_rows else None, ptr(d[2]) if use_gain else None, ptr(h) if use_gain else None,
             f32, R, W, eps, 0)
        torch.cuda.synchronize()
        want = new if use_y else old
        if use_rows or not use_y:
            assert torch.equal(xs.cpu(), X0)
        else:
            assert (xs.cpu().double().transpose(0, 1) - want).abs().max() < 1e-6 * float(want.abs().max())
        if use_gain:
            hw = O.rms_norm(O.read_streams(want, a.double()), gain.double(), eps)
            assert (h.cpu().double() - (hw[[4, 0, 2]] if use_rows else hw)).abs().max() < tol * 4


@pytest.mark.parametrize('parts,n', [(1, 24), (3, 40), (2, 7), (1, 256), (4, 260), (1, 2048), (2, 1030), (1, 9001), (8, 64)])
@pytest.mark.parametrize('dtype', [F32, B16])
def test_norm_in_parts_with_the_gate_on_either_side(lib, parts, n, dtype):
    configs, weights, engine, gugezen, paged, O = _mods()
    from phi3_b200._lib import call, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(6)
    T, C, eps = 7, parts * n, 1e-2
    y = torch.randn(T, C + 4, generator=g) * 0.3
    y[:, :n] *= 0.01                                           # eps counts in the first part
    gate, gain = torch.randn(T, C + 8, generator=g) * 2, torch.rand(C, generator=g) + 0.5
    yd, gd, wd = y.to(dev), gate.to(dev), gain.to(dev)
    for use_gate, silu, first in ((1, 1, 1), (1, 0, 0), (1, 1, 0), (1, 0, 1), (0, 0, 0)):
        out = torch.full((T, C + 4), 7.0, dtype=dtype, device=dev)
        call('p3_part_norm_gate', ptr(yd), C + 4, parts, n, ptr(wd), ptr(gd) if use_gate else None, C + 8, silu, first, 0.7, eps, ptr(out), C + 4,
             int(dtype == F32), T, 0)
        torch.cuda.synchronize()
        yy, gg = y[:, :C].double(), gate[:, :C].double()
        f = (O.silu(gg) if silu else torch.sigmoid(gg)) if use_gate else torch.ones_like(gg)
        want = O.parts_norm(yy * f, parts, gain.double(), eps) if first else O.parts_norm(yy, parts, gain.double(), eps) * f
        assert (out[:, :C].double().cpu() - want * 0.7).abs().max() < (2e-5 if dtype == F32 else 3e-2) * max(1.0, float(want.abs().max()))
        assert (out[:, C:] == 7.0).all()


def test_gelus_with_and_without_a_gate(lib):
    configs, weights, engine, gugezen, paged, O = _mods()
    from phi3_b200 import _lib
    from phi3_b200._lib import call, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(4)
    for F in (24, 33):
        gu = torch.randn(7, 2 * F, generator=g) * 3
        gu[0] = torch.linspace(-12, 12, 2 * F)
        gd, z = gu.to(dev), gu.double()
        for dt in (F32, B16):
            tol = 4e-6 if dt == F32 else 4e-2
            out = torch.empty(7, F, dtype=dt, device=dev)
            call('p3_glu_act', ptr(gd), ptr(gd[:, F:]), 2 * F, ptr(out), F, int(dt == F32), 7, F, _lib.GLU_GELU_TANH, 0)
            want = O.gelu_tanh(z[:, :F]) * z[:, F:]
            assert (out.double().cpu() - want).abs().max() < tol * float(want.abs().max())
            for act, fn in ((_lib.UNIT_GELU, O.gelu_erf), (_lib.UNIT_GELU_TANH, O.gelu_tanh)):
                out = torch.empty(7, F, dtype=dt, device=dev)
                call('p3_unit_act', ptr(gd), 2 * F, ptr(out), F, int(dt == F32), 7, F, act, 0)
                assert (out.double().cpu() - fn(z[:, :F])).abs().max() < tol * 12
    with pytest.raises(RuntimeError):
        call('p3_unit_act', ptr(gd), 66, ptr(gd), 33, 1, 1, 33, 2, 0)
    with pytest.raises(RuntimeError):
        call('p3_glu_act', ptr(gd), ptr(gd), 33, ptr(gd), 33, 1, 1, 33, 3, 0)


@pytest.mark.parametrize('E,top,W', [(8, 2, 64), (5, 5, 33), (1, 1, 48), (300, 7, 130), (40, 3, 2048)])
def test_softmax_shares_and_the_weighted_sum(lib, E, top, W):
    """router shares of the chosen, among them a token whose first choice takes nearly everything; the sum with and without a shared unit"""
    from phi3_b200 import _lib
    from phi3_b200._lib import call, ptr
    dev = torch.device('cuda')
    g = torch.Generator().manual_seed(9)
    T = 17
    z = torch.randn(T, E + 2, generator=g) * 2
    z[3, 0] += 40.0
    zd = z.to(dev)
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=dev), torch.empty(T, top, device=dev)
    call('p3_router_groups', ptr(zd), E + 2, None, T, E, top, 1, 1, 1.0, _lib.ROUTER_SOFTMAX, ptr(ids), ptr(wts), 0)
    s, order = torch.softmax(z[:, :E].double(), -1).sort(-1, descending=True)
    assert torch.equal(ids.cpu().long(), order[:, :top])
    share = s[:, :top] / (s[:, :top].sum(-1, keepdim=True) + 1e-20)
    assert (wts.cpu().double() - share).abs().max() < 1e-6
    y, add = torch.randn(T * top, W, generator=g), torch.randn(T, W + 4, generator=g)
    where = torch.randperm(T * top, generator=g).int()
    yd, ad, wd, out = y.to(dev), add.to(dev), where.to(dev), torch.empty(T, W, device=dev)
    for shared in (0, 1):
        call('p3_moe_combine_identity', ptr(yd), W, ptr(wd), None, ptr(wts), top, E, None, ptr(ad) if shared else None, W + 4, ptr(out), T, W, 0)
        want = (share[..., None] * y[where.long()].view(T, top, W).double()).sum(1) + (add[:, :W].double() if shared else 0)
        assert (out.cpu().double() - want).abs().max() < 1e-5
    rows = torch.randint(0, T * top, (23,), generator=g).int().to(dev)
    for dt in (F32, B16):
        src, dst = y.to(dev, dt), torch.empty(23, W, dtype=dt, device=dev)
        call('p3_gather_rows', ptr(src), W, int(dt == F32), ptr(rows), top, ptr(dst), 23, W, 0)
        assert torch.equal(dst, src[rows.long() // top])


# ------------------------------------------------------------------------------------------------ entry points
def test_greedy_generation_through_load_generate_and_the_scheduler(lib, tmp_path):
    configs, weights, engine, gugezen, paged, O = _mods()
    from phi3_b200 import api
    from safetensors.torch import save_file
    cfg = configs.tiny_gugezen()
    w = weights.random_gugezen_weights(cfg, 13)
    json.dump(cfg, open(tmp_path / 'config.json', 'w'))
    save_file(w, str(tmp_path / 'model.safetensors'))
    model, proc = api.load(model_path=str(tmp_path), dtype=F32)
    assert type(model).__name__ == 'GugezenB200'
    prompts = [tokens(n, cfg['vocab'], 60 + n) for n in (70, 3, 130, 20, 65)]
    n_new = 12
    # five requests through two slots and a pool of 8 pages: queueing, portions, slot, page and state reuse
    from phi3_b200.engine import generate_tokens
    outs = generate_tokens(model, prompts, max_new=n_new, max_tokens=64 * 8, n_slots=2, token_budget=96, chunk=40)
    for p, o in zip(prompts, outs):
        assert O.forward(cfg, w, p + o[:-1], torch.float64)[len(p) - 1:].argmax(-1).tolist() == o
    assert api.generate_batch(prompts[:2], preload=(model, proc), max_tokens=n_new, return_tokens=True) == outs[:2]
    text = api.generate('hello there', preload=(model, proc), max_tokens=5, verbose=False)
    assert isinstance(text, str)


def test_trace_runner_replays_steps(lib, tmp_path):
    configs, weights, engine, gugezen, paged, O = _mods()
    from safetensors.torch import save_file
    import numpy as np
    cfg = configs.tiny_gugezen()
    w = weights.random_gugezen_weights(cfg, 14)
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
