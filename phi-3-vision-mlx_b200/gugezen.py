"""Gugezen on B200: a decoder-only language model with several fp32 residual streams per token. A sublayer reads a weighted sum of the
streams through an RMS norm (gain stored around zero) and writes its output back while the streams are mixed, all from the old ones
(hyper-connections): X_t <- sum_s M[s][t] X_s + b_t f(N(sum_s a_s X_s)). Two kinds of mixers, in any order; a layer may use another
layer's tensors with a cache and a state of its own:

  'parallel'  two mixers read the same input and their outputs are added with fixed factors: grouped-query attention over the whole
              context with projection biases, neighbour pairs turned by wavelength-dependent frequencies, a learned per-head sink and an
              element-wise sigmoid gate; and a linear memory whose matrix state decays by one fixed factor per head, with silu on queries,
              keys and values, one RMS norm over all heads together and a sigmoid gate;
  'mamba2'    a state-space mixer: a short convolution with bias and silu, a matrix state per head that decays by a token-dependent
              step, read and write vectors shared by groups of heads, a skip term, a silu gate in front of a norm in equal parts.
Feed-forwards are gated units (tanh form of gelu), or a mixture of gelu units without a gate behind a softmax router plus a shared one.
The output matrix is the embedding table.

The model owns weights and launches kernels; it has no cache, no state and no loop of its own. `forward(batch, pool)` runs ONE step
of the engine (engine.py): a ragged batch of new tokens of several sequences against the shared page pool (paged.py). A parallel layer
has K/V pools and one state row per sequence slot there (the matrix states), a state-space layer two state rows (the matrix states
and the last inputs of the convolution).

Kernels per layer (csrc/): p3_embed_streams (first layer: embedding rows into all streams, the first sublayer's normed input) ->
  parallel: ONE product [q | k | v | gate | memory q | k | v | memory gate] -> p3_qkv_rope_post (biases, rotation, paged K/V write; silu on
            the memory's columns) -> p3_attn_window_prefill / _decode (sink, element-wise gate, factor) and, in prompt steps beside it
            on a second stream, p3_decay_scan -> p3_part_norm_gate -> ONE output product over [attention heads | memory heads]
  mamba2:   ONE product [z | x | B | C | dt] -> p3_short_conv (convolution, silu; decay and step per head) -> p3_decay_scan ->
            p3_part_norm_gate -> output product
-> p3_streams_rmsnorm (streams mixed with the sublayer's output, norm in front of the next sublayer) -> dense: ONE product [gate | up] ->
p3_glu_act -> down product; mixture: ONE product [shared up | router logits] -> p3_unit_act -> shared down product, p3_router_groups ->
p3_moe_sort -> grouped up product -> p3_unit_act -> grouped down product -> p3_moe_combine_identity (the shared unit joins the sum) ->
p3_streams_rmsnorm (behind the last layer: the final norm of the wanted rows alone, the logit factor folded into its gain).

Precision. dtype=bfloat16 (serving): matrices, activations that feed a matrix product and the K/V cache are bf16, accumulation is
fp32; positions, angles, scores, softmax, norms, router, the residual streams, convolutions and their history, decays and their
logarithms, step sizes, the recurrent states and their sums are fp32. dtype=float32: everything is fp32 on the FMA pipes (no TF32).
"""
import os

import torch
from . import _lib
from ._lib import call_struct, ptr
from .configs import GugezenConfig, wavelength_frequencies
from .lm_base import PagedLM, _stream


class GugezenB200(PagedLM):
    arch = 'Gugezen'
    SIDE_ROWS = int(os.environ.get('P3_LM_SIDE_ROWS', '256'))    # rows of a step from which the two halves of a parallel mixer overlap

    def __init__(self, cfg, weights, device='cuda', dtype=torch.bfloat16):
        if not torch.cuda.is_available():
            raise RuntimeError('GugezenB200 needs a CUDA device (sm_100a); there is no CPU fallback')
        _lib.lib()
        if isinstance(cfg, dict):
            cfg = GugezenConfig(cfg)
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError('dtype must be torch.bfloat16 or torch.float32')
        self.cfg, self.dev, self.dtype = cfg, torch.device(device), dtype
        self.W, self.V, self.S, self.eps = cfg.width, cfg.vocab_size, cfg.streams, cfg.eps
        self._init_products()
        self._side = None
        w, W, S = weights, self.W, self.S
        mat = lambda t: t.to(self.dev, dtype).contiguous()                     # matrices: the compute type
        f32 = lambda t: t.to(self.dev, torch.float32).contiguous()            # everything that enters fp32 arithmetic
        gain = lambda t, k=1.0: ((1.0 + t.to(self.dev, torch.float32)) * k).contiguous()   # weights stored around zero

        def expect(name, *shape):
            if name not in w:
                raise KeyError(f'the checkpoint has no tensor {name!r}')
            if tuple(w[name].shape) != shape:
                raise ValueError(f'{name}: shape {tuple(w[name].shape)}, the config gives {shape}')
            return w[name]

        self.embed = expect('embed', self.V, W).to(self.dev, torch.bfloat16).contiguous()      # bf16 values are exact in both modes
        self.head = self.embed if dtype == torch.bfloat16 else mat(w['embed'])
        self.final = dict(a=torch.ones(S, dtype=torch.float32, device=self.dev), gain=gain(expect('final.norm', W), cfg.logit_scale))
        own = {}
        for i in sorted(set(cfg.sources)):
            lc = cfg.layers[i]
            p, f = f'l{i}.', lc.ff
            L = dict(cfg=lc)
            (self._load_parallel if lc.mixer.kind == 'parallel' else self._load_mamba2)(L, lc.mixer, p + 'mix.', expect, mat, f32)
            for q in (1, 2) if f is not None else (1,):
                h = f'{p}hc{q}.'
                L[f'hc{q}'] = dict(a=f32(expect(h + 'in', S)), b=f32(expect(h + 'out', S)), mix=f32(expect(h + 'mix', S, S)),
                                   gain=gain(expect(f'{p}norm{q}', W)))
            if f is not None:
                q = p + 'mlp.'
                if f.kind == 'dense':
                    L['gu'] = mat(torch.cat([expect(q + 'gate', f.ff, W), expect(q + 'up', f.ff, W)], 0))
                    L['down'] = mat(expect(q + 'down', W, f.ff))
                else:
                    # the shared unit's up rows and the router's rows are one product (fp32 accumulation of exact bf16 products; all-fp32
                    # in the fp32 mode)
                    sff = f.shared_ff
                    L['in2_w'] = self.stacked_rows(([expect(q + 'shared.up', sff, W)] if sff else []) + [expect(q + 'router', f.experts, W)])
                    L['sh_down'] = mat(expect(q + 'shared.down', W, sff)) if sff else None
                    L['up'] = mat(torch.stack([expect(f'{q}e{e}.up', f.ff, W) for e in range(f.experts)], 0))
                    L['down'] = mat(torch.stack([expect(f'{q}e{e}.down', W, f.ff) for e in range(f.experts)], 0))
            own[i] = L
        self.layers = [own[j] for j in cfg.sources]
        # query rows per attention tile the engine cuts prompt portions into: 64 when every attention takes the tensor-core prefill
        # kernel (csrc/attention_window.cu), else 32
        self.q_tile = min(L['tile_rows'] for L in self.layers)
        # state buffers of the page pool: the matrix states of every layer, then (state-space layers) the inputs of the convolution
        self._state_layout, self._state_of = [], []
        for lc in cfg.layers:
            m = lc.mixer
            self._state_of.append(len(self._state_layout))
            if m.kind == 'parallel':
                self._state_layout.append(int(_lib.lib().p3_delta_state_floats(m.mem.heads, m.mem.dim, m.mem.vdim)))
            else:
                self._state_layout += [int(_lib.lib().p3_delta_state_floats(m.heads, m.state, m.vdim)), (m.taps - 1) * m.channels]

    def _load_parallel(self, L, m, a, expect, mat, f32):
        W, at, mem = self.W, m.att, m.mem
        H, G, d, dv, Hm, dm, dvm = at.heads, at.kv_heads, at.dim, at.vdim, mem.heads, mem.dim, mem.vdim
        b, c = a + 'left.', a + 'right.'
        qkv = [('q', H * d), ('k', G * d), ('v', G * dv)]
        # all input projections of the layer are one product; the output projections of both halves read one concatenated row
        parts = [(b + n, rows) for n, rows in qkv + [('g', H * dv)]] + [(c + n, rows) for n, rows in
                                                                        (('q', Hm * dm), ('k', Hm * dm), ('v', Hm * dvm), ('g', Hm * dvm))]
        L['in_w'] = self.stacked_rows([expect(n, rows, W) for n, rows in parts])
        L['g_off'] = H * d + G * (d + dv)
        L['m_off'] = L['g_off'] + H * dv                                       # memory q | k | v
        L['mg_off'] = L['m_off'] + 2 * Hm * dm + Hm * dvm
        L['in_b'] = torch.cat([f32(expect(f'{b}{n}.b', rows)) for n, rows in qkv])
        L['sink'], L['m_gain'] = f32(expect(b + 'sink', H)), f32(expect(c + 'norm', Hm * dvm))
        wo = expect(b + 'o', W, H * dv)
        # the kernels read a factor of zero as one
        L['out_w'] = mat(torch.cat([wo if m.att_scale != 0.0 else torch.zeros_like(wo), expect(c + 'o', W, Hm * dvm)], 1))
        L['decay'] = torch.tensor(mem.decay, dtype=torch.float64).to(self.dev, torch.float32)
        if at.rot is not None:
            L['freq'], L['rot_n'] = torch.tensor(wavelength_frequencies(at.rot), dtype=torch.float64).to(self.dev, torch.float32), at.rot.dims
        else:
            L['freq'], L['rot_n'] = None, 0
        L['tile_rows'] = self.attention_tile_rows(H, G, d, dv, 0, ld_out=L['out_w'].shape[1])

    def _load_mamba2(self, L, m, a, expect, mat, f32):
        W, H, C = self.W, m.heads, m.channels
        L['in_w'] = self.stacked_rows([expect(a + 'in', m.inner + C + H, W)])
        L['conv_w'], L['conv_b'] = f32(expect(a + 'conv', C, m.taps)).t().contiguous(), f32(expect(a + 'conv.b', C))    # [taps, channels]
        L['dt_bias'], L['a_log'], L['skip'] = (f32(expect(a + n, H)) for n in ('dt_bias', 'A_log', 'D'))
        L['m_gain'], L['out_w'] = f32(expect(a + 'norm', m.inner)), mat(expect(a + 'o', W, m.inner))
        L['tile_rows'] = 64

    # ------------------------------------------------------------------ what the engine asks of a model
    def kv_layout(self):
        return self.cfg.kv_layout()

    def state_layout(self):
        """fp32 numbers per sequence slot and state buffer (self._state_of[layer] indexes a layer's first)"""
        return list(self._state_layout)

    def prepare(self, max_context):
        """nothing depends on the longest context: angles are formed from the positions in the kernels"""

    def graph_safe(self, b):
        """may this step be captured as a CUDA graph? Not when a mixture layer would read its segment offsets back."""
        return not any(l.ff is not None and l.ff.kind == 'moe' and self.experts_dense(l.ff, b.T) for l in self.cfg.layers)

    # ------------------------------------------------------------------ one engine step
    def _streams(self, x, y, cur, nxt, T, rows=None):
        """the streams take the output y of sublayer `cur` (None: they stay); -> the normed input of sublayer `nxt` in the activation type
        (None: not wanted). With `rows` only those rows are normed (T of them) and the streams stay."""
        h = torch.empty((T, self.W), dtype=self.dtype, device=self.dev) if nxt is not None else None
        nb = T * self.W * (4 * self.S * (1 if y is None or rows is not None else 2) + (4 if y is not None else 0)
                           + (0 if nxt is None else (4 if self.f32 else 2)))
        c, n = cur or {}, nxt or {}
        self.rows('norm', nb, 'p3_streams_rmsnorm', ptr(x), self.S, ptr(y), y.stride(0) if y is not None else 0, ptr(c.get('mix')),
                  ptr(c.get('b')), ptr(n.get('a')), ptr(rows), ptr(n.get('gain')), ptr(h), self.f32, T, self.W, self.eps, _stream())
        return h

    def forward(self, b, pool, trace=None):
        """b: StepBatch, pool: paged.PagePool -> fp32 logits [b.R, vocab] (None when no row is wanted).
        `trace` (a list) receives the sum of the residual streams after every layer."""
        T, W, S = b.T, self.W, self.S
        e = lambda *s, dt=torch.float32: torch.empty(s, dtype=dt, device=self.dev)
        x, h = e(T, S, W), e(T, W, dt=self.dtype)
        first = self.layers[0]['hc1']
        self.rows('embed', T * W * (2 + 4 * S + (4 if self.f32 else 2)), 'p3_embed_streams', ptr(self.embed), ptr(b.ids), self.cfg.embed_scale,
                  ptr(x), S, ptr(first['a']), ptr(first['gain']), ptr(h), self.f32, T, W, self.V, self.eps, _stream())
        for li, L in enumerate(self.layers):
            f = L['cfg'].ff
            y = (self._parallel if L['cfg'].mixer.kind == 'parallel' else self._mamba2)(L, li, h, b, pool)
            cur = L['hc1']
            if f is not None:
                h = self._streams(x, y, cur, L['hc2'], T)
                y = self._dense(L, f, h, T) if f.kind == 'dense' else self._moe(L, f, h, T)
                cur = L['hc2']
            if trace is not None:
                self._streams(x, y, cur, None, T)
                y = None
                trace.append(x.sum(1))
            if li + 1 < len(self.layers):
                h = self._streams(x, y, cur, self.layers[li + 1]['hc1'], T)
        if not b.R:
            return None
        xn = self._streams(x, y, cur, self.final, b.R, rows=b.want_rows)
        logits = e(b.R, self.V)
        self.linear(xn, self.head, logits)
        return logits

    def _after(self, L):
        """the matrix of the product behind a mixer's output product"""
        f = L['cfg'].ff
        return None if f is None else L['gu'] if f.kind == 'dense' else L['in2_w']

    def _scan(self, kind, s, state, b, T, H, d, dv, nbytes):
        s.n_heads, s.dim, s.vdim, s.state, s.seqs, s.n_seqs = H, d, dv, ptr(state), ptr(b.seqs), b.n_seq
        ev = self._ev()
        call_struct('p3_decay_scan', s, _stream())
        self._ev(ev, kind, 4 * T * H * d * dv, b.n_seq * H * d * dv * 8 + nbytes)

    def _parallel(self, L, li, h, b, pool):
        """normed input h (act [T, W]) -> mixer output, fp32 [T, W]"""
        T, W, act = b.T, self.W, self.dtype
        e = lambda *s, dt=torch.float32: torch.empty(s, dtype=dt, device=self.dev)
        m = L['cfg'].mixer
        at, mem = m.att, m.mem
        H, G, d, dv, Hm, dm, dvm = at.heads, at.kv_heads, at.dim, at.vdim, mem.heads, mem.dim, mem.vdim
        nq, nk, nv, n_att, n_mem = H * d, G * d, G * dv, H * dv, Hm * dvm
        esz = 4 if self.f32 else 2
        proj = e(T, L['in_w'].shape[0])
        self.linear(h, L['in_w'], proj, nxt=L['out_w'])
        q, cat, o = e(T, nq, dt=act), e(T, n_att + n_mem, dt=act), e(T, n_mem)
        a = _lib.QkvRopePostArgs()
        a.proj, a.ld_proj, a.q_off, a.k_off, a.v_off, a.bias = ptr(proj), proj.stride(0), 0, nq, nq + nk, ptr(L['in_b'])
        a.n_heads, a.n_kv, a.dim, a.vdim, a.rot_n, a.freq, a.pair_mode = H, G, d, dv, L['rot_n'], ptr(L['freq']), 1
        a.act_cols, a.n_act = ptr(proj[:, L['m_off']:]), 2 * Hm * dm + n_mem
        a.q_out, a.ld_q = ptr(q), q.stride(0)
        a.k_pool, a.v_pool = ptr(pool.k[li]), ptr(pool.v[li])
        a.block_table, a.bt_stride = ptr(pool.block_table), pool.block_table.stride(0)
        a.tok_slot, a.tok_pos, a.T, a.act_f32, a.cache_f32 = ptr(b.tok_slot), ptr(b.tok_pos), T, self.f32, self.f32
        self.rows('qkv_post', T * ((nq + nk + nv) * (4 + esz) + a.n_act * 8), 'p3_qkv_rope_post', a)

        def memory():
            s = _lib.DeltaScanArgs()
            s.qkv, s.ld_qkv, s.n_kv, s.decay = ptr(proj), proj.stride(0), Hm, ptr(L['decay'])
            s.q_off, s.k_off, s.v_off = L['m_off'], L['m_off'] + Hm * dm, L['m_off'] + 2 * Hm * dm
            s.out, s.ld_out = ptr(o), o.stride(0)
            self._scan('memory_scan', s, pool.state[self._state_of[li]], b, T, Hm, dm, dvm, T * (2 * Hm * dm + 2 * n_mem) * 4)
            self.rows('headnorm', T * n_mem * (8 + esz), 'p3_part_norm_gate', ptr(o), o.stride(0), 1, n_mem, ptr(L['m_gain']),
                      ptr(proj[:, L['mg_off']:]), proj.stride(0), 0, 0, m.mem_scale, self.eps, ptr(cat[:, n_att:]), cat.stride(0), self.f32, T, _stream())

        # prompt steps: the recurrence (few CTAs, FP32 pipes) runs beside the attention (tensor cores) on a second stream
        side = T >= self.SIDE_ROWS and self.profile is None and not torch.cuda.is_current_stream_capturing()
        if side:
            if self._side is None:
                self._side = torch.cuda.Stream(self.dev)
            main = torch.cuda.current_stream()
            self._side.wait_stream(main)
            with torch.cuda.stream(self._side):
                memory()
        w = _lib.AttnWindowArgs()
        w.q, w.ld_q, w.k_pool, w.v_pool = ptr(q), q.stride(0), ptr(pool.k[li]), ptr(pool.v[li])
        w.block_table, w.bt_stride = ptr(pool.block_table), pool.block_table.stride(0)
        w.sink, w.out, w.ld_out = ptr(L['sink']), ptr(cat), cat.stride(0)
        w.elem_gate, w.ld_elem_gate = ptr(proj[:, L['g_off']:]), proj.stride(0)
        w.n_heads, w.n_kv, w.dim, w.vdim, w.scale, w.out_scale = H, G, d, dv, at.scale, m.att_scale
        w.act_f32, w.cache_f32 = self.f32, self.f32
        self.attend(w, L['tile_rows'], b, G, d, dv, lambda n: n, G * (d + dv))
        if side:
            main.wait_stream(self._side)
        else:
            memory()
        y = e(T, W)
        self.linear(cat, L['out_w'], y, nxt=self._after(L))
        return y

    def _mamba2(self, L, li, h, b, pool):
        """normed input h (act [T, W]) -> mixer output, fp32 [T, W]"""
        T, W, st = b.T, self.W, _stream()
        e = lambda *s, dt=torch.float32: torch.empty(s, dtype=dt, device=self.dev)
        m = L['cfg'].mixer
        H, dv, N, G, C, inner = m.heads, m.vdim, m.state, m.groups, m.channels, m.inner
        state, history = pool.state[self._state_of[li]], pool.state[self._state_of[li] + 1]
        proj = e(T, L['in_w'].shape[0])
        self.linear(h, L['in_w'], proj, nxt=L['out_w'])
        xbc, gates, o = e(T, C), e(T, H, 2), e(T, inner)
        c = _lib.ShortConvArgs()
        c.proj, c.ld_proj, c.c_off, c.n_plain = ptr(proj), proj.stride(0), inner, C
        c.w, c.bias, c.taps, c.conv_state = ptr(L['conv_w']), ptr(L['conv_b']), m.taps, ptr(history)
        c.seqs, c.slot_seq, c.tok_slot, c.n_rows = ptr(b.seqs), ptr(b.slot_seq), ptr(b.tok_slot), T
        c.out, c.ld_out = ptr(xbc), xbc.stride(0)
        c.a_off, c.n_gates, c.a_log, c.dt_bias, c.gates, c.gate_mode = inner + C, H, ptr(L['a_log']), ptr(L['dt_bias']), ptr(gates), 1
        self.rows('conv', T * (C * 8 + H * 12), 'p3_short_conv', c)
        s = _lib.DeltaScanArgs()
        s.qkv, s.ld_qkv, s.v_off, s.k_off, s.q_off = ptr(xbc), xbc.stride(0), 0, inner, inner + G * N
        s.n_kv, s.gates, s.skip, s.out, s.ld_out = G, ptr(gates), ptr(L['skip']), ptr(o), o.stride(0)
        s.conv_in, s.ld_conv_in, s.channels, s.taps, s.conv_state = ptr(proj[:, inner:]), proj.stride(0), C, m.taps, ptr(history)
        self._scan('ssm_scan', s, state, b, T, H, N, dv, T * (C + inner) * 4)
        cat = e(T, inner, dt=self.dtype)
        self.rows('headnorm', T * inner * (8 + (4 if self.f32 else 2)), 'p3_part_norm_gate', ptr(o), o.stride(0), m.norm_groups,
                  inner // m.norm_groups, ptr(L['m_gain']), ptr(proj), proj.stride(0), 1, 1, 1.0, self.eps, ptr(cat), cat.stride(0), self.f32, T, st)
        y = e(T, W)
        self.linear(cat, L['out_w'], y, nxt=self._after(L))
        return y

    def _dense(self, L, f, h, T):
        ff = f.ff
        gu = torch.empty((T, 2 * ff), dtype=torch.float32, device=self.dev)
        hid = torch.empty((T, ff), dtype=self.dtype, device=self.dev)
        y = torch.empty((T, self.W), dtype=torch.float32, device=self.dev)
        self.linear(h, L['gu'], gu, nxt=L['down'])
        self.rows('activation', T * ff * (8 + (4 if self.f32 else 2)), 'p3_glu_act', ptr(gu), ptr(gu[:, ff:]), gu.stride(0), ptr(hid),
                  hid.stride(0), self.f32, T, ff, _lib.GLU_GELU_TANH, _stream())
        self.linear(hid, L['down'], y)
        return y

    def _gelu(self, up, hid, n, ff):
        self.rows('activation', n * ff * (4 + (4 if self.f32 else 2)), 'p3_unit_act', ptr(up), up.stride(0), ptr(hid), hid.stride(0),
                  self.f32, n, ff, _lib.UNIT_GELU, _stream())

    def _moe(self, L, f, h, T):
        """mixture: the shared unit for every token, plus the chosen experts weighted by their shares of the router's softmax"""
        st, W = _stream(), self.W
        e = lambda *s, dt=torch.float32: torch.empty(s, dtype=dt, device=self.dev)
        p2 = e(T, L['in2_w'].shape[0])
        self.linear(h, L['in2_w'], p2, nxt=L['sh_down'])
        shid, ysh = (e(T, f.shared_ff, dt=self.dtype), e(T, W)) if f.shared_ff else (None, None)

        def shared():
            self._gelu(p2, shid, T, f.shared_ff)
            self.linear(shid, L['sh_down'], ysh)

        ids, wts, y = e(T, f.top, dt=torch.int32), e(T, f.top), e(T, W)
        self.rows('route', T * (f.experts * 4 + f.top * 8), 'p3_router_groups', ptr(p2[:, f.shared_ff:]), p2.stride(0), None, T, f.experts,
                  f.top, 1, 1, 1.0, _lib.ROUTER_SOFTMAX, ptr(ids), ptr(wts), st)
        nb = T * W * 4 * (f.top + (1 if ysh is None else 2))
        combine = lambda dn, where: self.rows('combine', nb, 'p3_moe_combine_identity', ptr(dn), dn.stride(0), ptr(where), None, ptr(wts), f.top,
                                              f.experts, None, ptr(ysh), ysh.stride(0) if ysh is not None else 0, ptr(y), T, W, st)
        self.experts(L['up'], L['down'], f, h, y, T, ids, wts, lambda up, hid, n: self._gelu(up, hid, n, f.ff), combine=combine,
                     meanwhile=shared if f.shared_ff else None)
        return y
