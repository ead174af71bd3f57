"""Lupusun on B200: a decoder-only language model with ONE RMS norm in front of every sublayer, x <- x + m mixer(N(x)),
x <- x + m ff(N(x)), an fp32 residual stream that starts as the normed embedding row, and a block of layers that runs several times
with the same weights; the stream's start is added again ahead of every further pass. Two kinds of mixers, in any order:

  'delta'      gated delta rule: short causal convolutions with silu on queries, keys and values, unit-length queries and keys shared by
               groups of heads, a matrix state per head that decays, is corrected at the current key and read by the query, a head norm
               and a silu gate;
  'attention'  grouped-query attention with projection biases, a partial rotation with blended frequencies, unit query and key heads
               after it, keys limited to the query's own chunk of positions, a learned per-head sink in the softmax denominator.
Feed-forwards are gated relu units.

The model owns weights and launches kernels; it has no cache, no state and no loop of its own. `forward(batch, pool)` runs ONE step
of the engine (engine.py): a ragged batch of new tokens of several sequences against the shared page pool (paged.py). Every layer RUN
(a looped layer once per pass) has its own K/V pools there, or its own two state rows per sequence slot: the matrix states and the last
inputs of the convolutions.

Kernels per layer run (csrc/): p3_embed_norm_rows_f32 (first run: embedding row, its norm, the first layer's norm) ->
  delta:     ONE product [q | k | v | gate | b | a] -> p3_short_conv (convolutions, silu, unit heads; decay and step size per head) ->
             p3_delta_scan -> p3_headnorm_gate_x -> output product
  attention: ONE product [q | k | v] -> p3_qkv_rope_post (biases, rotation, unit norm, paged K/V write) -> p3_attn_window_prefill /
             _decode (chunk, sink) -> output product
-> p3_residual_rmsnorm (residual add, norm in front of the feed-forward) -> ONE product [gate | up] -> p3_glu_act -> down product ->
p3_residual_rmsnorm (residual add, the stream's start where a pass begins, norm in front of the next run; behind the last run the final
norm of the wanted rows alone).

Precision. dtype=bfloat16 (serving): matrices, activations that feed a matrix product and the K/V cache are bf16, accumulation is
fp32; positions, angles, scores, softmax, norms, the residual sum, convolutions and their history, decays and their logarithms, step
sizes, the recurrent state and its sums are fp32. dtype=float32: everything is fp32 on the FMA pipes (no TF32).
"""
import torch
from . import _lib
from ._lib import call_struct, ptr
from .configs import LupusunConfig, yarn_frequencies
from .lm_base import PagedLM, _stream


class LupusunB200(PagedLM):
    arch = 'Lupusun'

    def __init__(self, cfg, weights, device='cuda', dtype=torch.bfloat16):
        if not torch.cuda.is_available():
            raise RuntimeError('LupusunB200 needs a CUDA device (sm_100a); there is no CPU fallback')
        _lib.lib()
        if isinstance(cfg, dict):
            cfg = LupusunConfig(cfg)
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError('dtype must be torch.bfloat16 or torch.float32')
        self.cfg, self.dev, self.dtype = cfg, torch.device(device), dtype
        self.W, self.V, self.eps, self.mult = cfg.width, cfg.vocab_size, cfg.eps, cfg.residual_mult
        self._init_products()
        w, W = weights, self.W
        mat = lambda t: t.to(self.dev, dtype).contiguous()                     # matrices: the compute type
        f32 = lambda t: t.to(self.dev, torch.float32).contiguous()            # everything that enters fp32 arithmetic

        def expect(name, *shape):
            if name not in w:
                raise KeyError(f'the checkpoint has no tensor {name!r}')
            if tuple(w[name].shape) != shape:
                raise ValueError(f'{name}: shape {tuple(w[name].shape)}, the config gives {shape}')
            return w[name]

        self.embed = expect('embed', self.V, W).to(self.dev, torch.bfloat16).contiguous()      # bf16 values are exact in both modes
        self.embed_gain = f32(expect('embed.norm', W))
        self.final_gain, self.head = f32(expect('final.norm', W)), mat(expect('head', self.V, W))
        self.layers = []
        for i, lc in enumerate(cfg.layers):
            p, m, f = f'l{i}.', lc.mixer, lc.ff
            a = p + 'mix.'
            H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
            L = dict(cfg=lc, pre1=f32(expect(p + 'norm1', W)), out_w=mat(expect(a + 'o', W, H * dv)))
            if m.kind == 'attention':
                qkv = [(n, rows) for n, rows in (('q', H * d), ('k', G * d), ('v', G * dv))]
                L['in_w'] = self.stacked_rows([expect(a + n, rows, W) for n, rows in qkv])
                L['in_b'] = torch.cat([f32(expect(f'{a}{n}.b', rows)) for n, rows in qkv])
                L['sink'] = f32(expect(a + 'sink', H))
                if m.rot is not None:
                    fr, mag = yarn_frequencies(m.rot)
                    L['freq'], L['rot_mag'], L['rot_n'] = torch.tensor(fr, dtype=torch.float64).to(self.dev, torch.float32), float(mag), m.rot.dims
                else:
                    L['freq'], L['rot_mag'], L['rot_n'] = None, 1.0, 0
                L['tile_rows'] = self.attention_tile_rows(H, G, d, dv, 0)
            else:
                C = 2 * G * d + H * dv                                         # channels of the convolutions: q | k | v
                qkv = [(n, rows) for n, rows in (('q', G * d), ('k', G * d), ('v', H * dv))]
                # all input projections of the layer are one product: q | k | v | output gate | step size | decay
                L['in_w'] = self.stacked_rows([expect(a + n, rows, W) for n, rows in qkv] +
                                              [expect(a + 'g', H * dv, W), expect(a + 'b', H, W), expect(a + 'a', H, W)])
                L['channels'], L['g_off'], L['b_off'], L['a_off'] = C, C, C + H * dv, C + H * dv + H
                L['conv_w'] = torch.cat([f32(expect(f'{a}{n}.conv', rows, m.taps)) for n, rows in qkv], 0).t().contiguous()   # [taps, channels]
                L['a_log'], L['dt_bias'], L['gain'] = f32(expect(a + 'A_log', H)), f32(expect(a + 'dt_bias', H)), f32(expect(a + 'norm', dv))
                L['tile_rows'] = 64
            if f is not None:
                q = p + 'mlp.'
                L['pre2'] = f32(expect(p + 'norm2', W))
                L['gu'] = mat(torch.cat([expect(q + 'gate', f.ff, W), expect(q + 'up', f.ff, W)], 0))
                L['down'] = mat(expect(q + 'down', W, f.ff))
            self.layers.append(L)
        # query rows per attention tile the engine cuts prompt portions into: 64 when every attention takes the tensor-core prefill
        # kernel (csrc/attention_window.cu), else 32
        self.q_tile = min(L['tile_rows'] for L in self.layers)
        # state buffers of the page pool: per recurrent layer run the matrix states, then the inputs of the convolutions
        self._state_layout, self._run_state = [], {}
        for ri, (li, _) in enumerate(cfg.runs):
            m = cfg.layers[li].mixer
            if m.kind == 'delta':
                self._run_state[ri] = len(self._state_layout)
                self._state_layout += [int(_lib.lib().p3_delta_state_floats(m.heads, m.dim, m.vdim)), (m.taps - 1) * self.layers[li]['channels']]

    # ------------------------------------------------------------------ what the engine asks of a model
    def kv_layout(self):
        return self.cfg.kv_layout()

    def state_layout(self):
        """fp32 numbers per sequence slot and state buffer: two buffers per recurrent layer run (self._run_state indexes the first)"""
        return list(self._state_layout)

    def prepare(self, max_context):
        """nothing depends on the longest context: angles are formed from the positions in the kernels"""

    def graph_safe(self, b):
        """may this step be captured as a CUDA graph? Always: no kernel of this design needs a host read."""
        return True

    # ------------------------------------------------------------------ one engine step
    def _residual(self, y, x, gain, T, add=None, rows=None):
        """x += mult * y (+ add); -> N(x) * gain in the activation type (None without gain). With `rows` only those rows are normed
        (T of them) and x stays."""
        h = torch.empty((T, self.W), dtype=self.dtype, device=self.dev) if gain is not None else None
        nb = T * self.W * (4 + (8 if y is not None else 0) + (4 if add is not None else 0) + (0 if gain is None else (4 if self.f32 else 2)))
        self.rows('norm', nb, 'p3_residual_rmsnorm', ptr(x), ptr(y), y.stride(0) if y is not None else 0, self.mult, ptr(add), ptr(rows),
                  ptr(gain), ptr(h), self.f32, T, self.W, self.eps, _stream())
        return h

    def forward(self, b, pool, trace=None):
        """b: StepBatch, pool: paged.PagePool -> fp32 logits [b.R, vocab] (None when no row is wanted).
        `trace` (a list) receives a copy of the residual stream after every layer run."""
        T, W, cfg = b.T, self.W, self.cfg
        e = lambda *s, dt=torch.float32: torch.empty(s, dtype=dt, device=self.dev)
        x, h = e(T, W), e(T, W, dt=self.dtype)
        start = e(T, W) if cfg.loop is not None and cfg.loop.times > 1 else None      # the embedding output, for the further passes
        runs = cfg.runs
        self.rows('embed', T * W * (6 + (4 if start is not None else 0) + (4 if self.f32 else 2)), 'p3_embed_norm_rows_f32', ptr(self.embed),
                  ptr(b.ids), ptr(self.embed_gain), ptr(x), ptr(start), ptr(self.layers[runs[0][0]]['pre1']), ptr(h), self.f32, T, W, self.V,
                  self.eps, _stream())
        seen = False                                                           # has a pass of the looped block begun?
        for ri, (li, pass_start) in enumerate(runs):
            L = self.layers[li]
            seen |= pass_start
            y = (self._attention if L['cfg'].mixer.kind == 'attention' else self._delta)(L, ri, h, b, pool)
            if L['cfg'].ff is not None:
                h = self._residual(y, x, L['pre2'], T)
                y = self._feed_forward(L, h, T)
            last = ri + 1 == len(runs)
            if trace is not None:
                self._residual(y, x, None, T)
                y = None
                trace.append(x.clone())
            if not last:
                nli, again = runs[ri + 1]
                h = self._residual(y, x, self.layers[nli]['pre1'], T, add=start if again and seen else None)
        if not b.R:
            return None
        xn = self._residual(y, x, self.final_gain, b.R, rows=b.want_rows)
        logits = e(b.R, self.V)
        self.linear(xn, self.head, logits)
        return logits

    def _attention(self, L, ri, h, b, pool):
        """normed input h (act [T, W]) -> mixer output, fp32 [T, W]"""
        T, W, act = b.T, self.W, self.dtype
        e = lambda *s, dt=torch.float32: torch.empty(s, dtype=dt, device=self.dev)
        m = L['cfg'].mixer
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        nq, nk, nv = H * d, G * d, G * dv
        proj = e(T, L['in_w'].shape[0])
        self.linear(h, L['in_w'], proj, nxt=L['out_w'])
        q, att = e(T, nq, dt=act), e(T, H * dv, dt=act)
        a = _lib.QkvRopePostArgs()
        a.proj, a.ld_proj, a.q_off, a.k_off, a.v_off, a.bias = ptr(proj), proj.stride(0), 0, nq, nq + nk, ptr(L['in_b'])
        a.n_heads, a.n_kv, a.dim, a.vdim, a.rot_n, a.freq, a.rot_mag = H, G, d, dv, L['rot_n'], ptr(L['freq']), L['rot_mag']
        a.unit_norm, a.eps = 1, self.eps
        a.q_out, a.ld_q = ptr(q), q.stride(0)
        a.k_pool, a.v_pool = ptr(pool.k[ri]), ptr(pool.v[ri])
        a.block_table, a.bt_stride = ptr(pool.block_table), pool.block_table.stride(0)
        a.tok_slot, a.tok_pos, a.T, a.act_f32, a.cache_f32 = ptr(b.tok_slot), ptr(b.tok_pos), T, self.f32, self.f32
        esz = 4 if self.f32 else 2
        self.rows('qkv_post', T * (nq + nk + nv) * (4 + esz), 'p3_qkv_rope_post', a)
        w = _lib.AttnWindowArgs()
        w.q, w.ld_q, w.k_pool, w.v_pool = ptr(q), q.stride(0), ptr(pool.k[ri]), ptr(pool.v[ri])
        w.block_table, w.bt_stride = ptr(pool.block_table), pool.block_table.stride(0)
        w.sink, w.out, w.ld_out = ptr(L['sink']), ptr(att), att.stride(0)
        w.n_heads, w.n_kv, w.dim, w.vdim, w.scale, w.chunk = H, G, d, dv, m.scale, m.chunk
        w.act_f32, w.cache_f32 = self.f32, self.f32
        seen = (lambda n: min(m.chunk, n)) if m.chunk else (lambda n: n)
        self.attend(w, L['tile_rows'], b, G, d, dv, seen, G * (d + dv), pf_span=-(-seen(b.max_pos + 1) // 2))
        y = e(T, W)
        self.linear(att, L['out_w'], y, nxt=L.get('gu'))
        return y

    def _delta(self, L, ri, h, b, pool):
        """normed input h (act [T, W]) -> mixer output, fp32 [T, W]"""
        T, W, act, st = b.T, self.W, self.dtype, _stream()
        e = lambda *s, dt=torch.float32: torch.empty(s, dtype=dt, device=self.dev)
        m = L['cfg'].mixer
        H, G, d, dv, C = m.heads, m.kv_heads, m.dim, m.vdim, L['channels']
        state, history = pool.state[self._run_state[ri]], pool.state[self._run_state[ri] + 1]
        proj = e(T, L['in_w'].shape[0])
        self.linear(h, L['in_w'], proj, nxt=L['out_w'])
        qkv, gates, o = e(T, C), e(T, H, 2), e(T, H * dv)
        c = _lib.ShortConvArgs()
        c.proj, c.ld_proj, c.c_off = ptr(proj), proj.stride(0), 0
        c.n_unit, c.dim, c.n_scaled, c.n_plain = 2 * G, d, G, H * dv           # query and key heads are unit vectors, queries scaled
        c.w, c.taps, c.conv_state, c.scale, c.unit_eps = ptr(L['conv_w']), m.taps, ptr(history), d ** -0.5, self.cfg.UNIT_EPS
        c.seqs, c.slot_seq, c.tok_slot, c.n_rows = ptr(b.seqs), ptr(b.slot_seq), ptr(b.tok_slot), T
        c.out, c.ld_out = ptr(qkv), qkv.stride(0)
        c.a_off, c.b_off, c.n_gates, c.a_log, c.dt_bias, c.gates = L['a_off'], L['b_off'], H, ptr(L['a_log']), ptr(L['dt_bias']), ptr(gates)
        self.rows('conv', T * (C * 8 + H * 16), 'p3_short_conv', c)
        s = _lib.DeltaScanArgs()
        s.qkv, s.ld_qkv, s.q_off, s.k_off, s.v_off = ptr(qkv), qkv.stride(0), 0, G * d, 2 * G * d
        s.gates, s.n_heads, s.n_kv, s.dim, s.vdim = ptr(gates), H, G, d, dv
        s.state, s.seqs, s.n_seqs, s.out, s.ld_out = ptr(state), ptr(b.seqs), b.n_seq, ptr(o), o.stride(0)
        s.conv_in, s.ld_conv_in, s.channels, s.taps, s.conv_state = ptr(proj), proj.stride(0), C, m.taps, ptr(history)
        ev = self._ev()
        call_struct('p3_delta_scan', s, st)
        self._ev(ev, 'delta_scan', 6 * T * H * d * dv, b.n_seq * H * d * dv * 8 + T * (C + H * dv) * 4)
        cat = e(T, H * dv, dt=act)
        self.rows('headnorm', T * H * dv * (8 + (4 if self.f32 else 2)), 'p3_headnorm_gate_x', ptr(o), o.stride(0), None, H, dv, ptr(L['gain']),
                  1, ptr(proj[:, L['g_off']:]), proj.stride(0), 1, 1.0, self.eps, ptr(cat), cat.stride(0), self.f32, T, st)
        y = e(T, W)
        self.linear(cat, L['out_w'], y, nxt=L.get('gu'))
        return y

    def _feed_forward(self, L, h, T):
        ff = L['cfg'].ff.ff
        gu = torch.empty((T, 2 * ff), dtype=torch.float32, device=self.dev)
        hid = torch.empty((T, ff), dtype=self.dtype, device=self.dev)
        y = torch.empty((T, self.W), dtype=torch.float32, device=self.dev)
        self.linear(h, L['gu'], gu, nxt=L['down'])
        self.rows('activation', T * ff * (8 + (4 if self.f32 else 2)), 'p3_glu_act', ptr(gu), ptr(gu[:, ff:]), gu.stride(0), ptr(hid),
                  hid.stride(0), self.f32, T, ff, _lib.GLU_RELU, _stream())
        self.linear(hid, L['down'], y)
        return y
