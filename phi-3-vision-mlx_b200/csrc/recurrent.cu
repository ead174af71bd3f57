// Recurrent mixers that carry a state per sequence slot instead of a key/value cache.
//
// Matrix memory (the mLSTM cell of xLSTM: Beck et al., "xLSTM: Extended Long Short-Term Memory"). Per head a memory S [dim][vdim],
// a normaliser n [dim] and a stabiliser m (0 at the start of a sequence). With log gates a_t (input) and b_t (forget):
//     m_t = max(b_t + m_(t-1), a_t)
//     S_t = e^(b_t + m_(t-1) - m_t) S_(t-1) + e^(a_t - m_t) k_t v_t^T        n_t alike with k_t alone
//     y_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
// Both exponents are <= 0 by the choice of m_t. Everything here is fp32: the gates and their logarithms, the state and the sums.
//
//   matrix_memory_scan_kernel   token by token. One CTA = one sequence of the step x one head x a block of value columns. A thread of
//                               the four main warps owns one or two columns and a slice of the dim rows of S, in registers for the
//                               whole step; a warp is RS row slices x 32 / RS lanes, so a column's sum over the rows is one or two
//                               shuffles and no barrier separates two tokens. q, k, v of 32 tokens are staged in shared memory at
//                               a time by async copies, one round ahead of the arithmetic (k and q rows are read as 16-byte
//                               broadcasts). A fifth warp turns the gate pre-activations of the next round into log gates, walks
//                               the stabiliser through them (the only serial part: one add and one max per token) and leaves
//                               e^(b + m' - m), e^(a - m) and e^(-m) of every token in shared memory; in the CTA of the first
//                               column block a sixth warp carries the normaliser n and writes the denominators
//                               max(|n . q|, e^(-m)) + 1e-6. The main warps write numerators S^T q; headnorm_gate_kernel divides.
//                               The shape of a warp (row slices, columns per lane) trades parallelism against shared-memory
//                               traffic and is chosen per launch; the arithmetic of a token is the same for every choice and does
//                               not depend on how the sequence was cut into steps, so a prompt fed in portions, or token by token,
//                               leaves bit-identical states and outputs. State of a head: S [dim][vdim], n [dim], then one copy of
//                               m per 32 value columns: every CTA needs m at its start and the first CTA to finish must not
//                               overwrite what another still has to read, so a CTA reads the copy of its first 32 columns and
//                               rewrites those of all its columns.
//   headnorm_gate_kernel        y / rms(y over the head) * gain * sigmoid(gate logits) * scale -> activation type (the gate may also
//                               be silu, the gain one vector shared by the heads)
//
// Gated linear attention (Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training"). Per head a state
// S [dim][vdim] that starts at zero, with one decay per key channel and token:
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T        y_t = S_t^T q_t        a_t = sigmoid(z_t)^(1/tau) = exp(logsigmoid(z_t) / tau)
//   gla_decay_kernel            decay logits of all rows of the step -> decays, in place (one pass at memory speed)
//   gla_scan_kernel             the matrix-memory scan's layout (columns of S in registers, rounds of staged tokens, async copies one
//                               round ahead) with a staged row of decays beside every k and q row. There is no normaliser and no
//                               stabiliser (every factor is in (0, 1]), so all four warps own columns. As there, a token's
//                               arithmetic does not depend on how the sequence was cut into steps.
//
// Gated delta rule (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"). Per head a state S [dim][vdim]
// that starts at zero, one decay g and one step size b per head and token:
//     S <- g_t S        u_t = b_t (v_t - S^T k_t)        S <- S + k_t u_t^T        y_t = S^T q_t
//   short_conv_kernel           what precedes the recurrence, over all rows of the step at once: a causal convolution of a few taps per
//                               channel, silu, unit length per query / key head, and the gates g and b of every head. A warp owns the
//                               channels of one head (or a block of value channels) and walks a few rows with its last inputs in
//                               registers; inputs of earlier steps come from the slot's history, which it only reads
//   delta_scan_kernel           the layout of the linear-attention scan; two passes over the state columns per token, the sums S^T k
//                               (a shuffle reduction closes them, on the critical path) and then update and read-out. It also moves the
//                               convolution history on: by then no kernel of the step reads the old one.
//
// Memory with one decay per head and token, without the correction: S <- g_t S + b_t k_t v_t^T, y_t = S^T q_t + c v_t. This is the
// recurrence of Mamba-2 (Dao, Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space
// Duality": q = C, k = B, v = x, g = exp(-exp(A) dt), b = dt, heads in groups that share B and C, a skip factor c) and, with a constant
// g per head, b = 1 and c = 0, linear attention with fixed decays.
//   short_conv_kernel           as above, with a bias per channel; the gates are then g and b = dt
//   delta_scan_kernel           with DELTA = false: one pass over the state columns per token, four tokens between two reductions
//   part_norm_gate_kernel       rows normed in equal parts (one part: all heads together), with the gate in front of the norm or behind it
#include "common.cuh"
#include "../../include/phi3_b200.h"
#include <cfloat>

namespace {
template <typename T> __device__ __forceinline__ void stv(T* p, float v);
template <> __device__ __forceinline__ void stv<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void stv<bf16>(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

constexpr int MM_TB = 32;        // tokens staged per round (16 for rows above 256 numbers, so that two rounds fit shared memory)
constexpr int MM_MAIN = 4;       // warps that own columns of S; one more warp for the gates, one for the normaliser
constexpr int MM_WARPS = MM_MAIN + 2;

__host__ __device__ inline int mm_m_copies(int vdim) { return (vdim + 31) / 32; }
// floats of one head's state: S [dim][vdim], n [dim], m per 32 value columns
__host__ __device__ inline int64_t mm_head_floats(int dim, int vdim) { return (int64_t)dim * vdim + dim + mm_m_copies(vdim); }

__device__ __forceinline__ float log_sigmoid(float z) {       // -softplus(-z), without overflow on either side
    return z >= 0.f ? -log1pf(expf(-z)) : z - log1pf(expf(z));
}

// 4-byte async copy global -> shared; src_bytes 0 writes zeros
__device__ __forceinline__ void cp_async4z(uint32_t dst, const void* src, int src_bytes) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(dst), "l"(src), "r"(src_bytes) : "memory");
}

template <int DS, int RS, int NC, int TB>
__global__ void __launch_bounds__(MM_WARPS * 32) matrix_memory_scan_kernel(p3_matrix_memory_args a) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    // a warp = RS row slices x CW lanes, every lane with NC columns (CW apart); DP: dim rounded up; NR: n rows per lane
    constexpr int CW = 32 / RS, WCOLS = CW * NC, COLS = MM_MAIN * WCOLS, DP = DS * RS, NR = (DP + 31) / 32;
    constexpr int NT = MM_WARPS * 32;
    // a staged q / k row keeps its RS slices 4 floats apart (pitch DPP): the 16-byte reads of a warp's slices then fall into
    // different banks and one read serves all of them
    constexpr int DPP = DP + 4 * RS;
    constexpr int ROUND = TB * (2 * DPP + COLS + 3);      // floats of one staged round
    auto at_row = [](int c) { return c + 4 * (c / DS); };    // where number c of a row lives
    extern __shared__ __align__(16) float sm[];
    const int d = a.dim, dv = a.vdim, H = a.n_heads;
    // two rounds in flight: [q [TB][DP] (zeros beyond dim) | k alike | v [TB][COLS] | e^(a - m) | e^(b + m' - m) | e^(-m)]
    const int4 rec = reinterpret_cast<const int4*>(a.seqs)[blockIdx.x];
    const int row0 = rec.x, n_tok = rec.y, slot = rec.z, pos0 = rec.w;
    const int hd = blockIdx.y, vb = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const bool fresh = pos0 == 0, main = warp < MM_MAIN, gate_warp = warp == MM_MAIN, first_block = vb == 0;
    float* Sg = a.state + ((size_t)slot * H + hd) * mm_head_floats(d, dv);
    float* ng = Sg + (size_t)d * dv;
    float* mg = ng + d;
    const int col = vb * COLS + warp * WCOLS + lane % CW, d0 = (lane / CW) * DS;   // first of this lane's columns
    float S[NC][DS], nr[NR];
    float m = 0.f;
    if (main) {
#pragma unroll
        for (int c = 0; c < NC; c++)
#pragma unroll
            for (int j = 0; j < DS; j++)
                S[c][j] = (!fresh && col + c * CW < dv && d0 + j < d) ? Sg[(size_t)(d0 + j) * dv + col + c * CW] : 0.f;
    } else if (gate_warp) {
        if (!fresh) m = mg[vb * (COLS / 32)];
    } else {
#pragma unroll
        for (int r = 0; r < NR; r++) nr[r] = (!fresh && first_block && lane * NR + r < d) ? ng[lane * NR + r] : 0.f;
    }
    const float inv_cap = 1.0f / a.gate_cap;
    const bool vec = d % 4 == 0 && a.ld_proj % 4 == 0 && a.q_off % 4 == 0 && a.k_off % 4 == 0 && ((uintptr_t)a.proj & 15) == 0;

    // all threads: start the copies of the round that begins at token t0 into buffer `buf` (q, k, v as projected; q is scaled when
    // the sums are written)
    auto stage = [&](int t0, int buf) {
        const int nb = min(TB, n_tok - t0);
        float* qs = sm + buf * ROUND;
        float* ks = qs + TB * DPP;
        float* vs = ks + TB * DPP;
        if (vec) {
            for (int i = tid; i < nb * (DP / 4); i += NT) {
                const int tt = i / (DP / 4), c = (i - tt * (DP / 4)) * 4;
                const float* pr = a.proj + (size_t)(row0 + t0 + tt) * a.ld_proj + (size_t)hd * d + (c < d ? c : 0);
                cp_async16(smem_u32(qs + tt * DPP + at_row(c)), pr + a.q_off, c < d ? 16 : 0);
                cp_async16(smem_u32(ks + tt * DPP + at_row(c)), pr + a.k_off, c < d ? 16 : 0);
            }
        } else {
            for (int i = tid; i < nb * DP; i += NT) {
                const int tt = i / DP, c = i - tt * DP;
                const float* pr = a.proj + (size_t)(row0 + t0 + tt) * a.ld_proj + (size_t)hd * d + (c < d ? c : 0);
                cp_async4z(smem_u32(qs + tt * DPP + at_row(c)), pr + a.q_off, c < d ? 4 : 0);
                cp_async4z(smem_u32(ks + tt * DPP + at_row(c)), pr + a.k_off, c < d ? 4 : 0);
            }
        }
        for (int i = tid; i < nb * COLS; i += NT) {
            const int tt = i / COLS, c = vb * COLS + (i - tt * COLS);
            cp_async4z(smem_u32(vs + i), a.proj + (size_t)(row0 + t0 + tt) * a.ld_proj + a.v_off + (size_t)hd * dv + (c < dv ? c : 0), c < dv ? 4 : 0);
        }
    };
    // gate warp: the log gates of the round (one token per lane), the walk of the stabiliser through them (every lane walks, the
    // gates come by shuffle: one add and one max per token on the critical path), and the three factors of every token
    auto gates = [&](int t0, int buf) {
        const int nb = min(TB, n_tok - t0);
        float* ga = sm + buf * ROUND + TB * (2 * DPP + COLS);
        float* gb = ga + TB;
        float* gm = gb + TB;
        float at = 0.f, bt = 0.f;
        if (lane < nb) {
            const float* pr = a.proj + (size_t)(row0 + t0 + lane) * a.ld_proj + hd;
            at = a.gate_cap * tanhf((pr[a.i_off] + a.i_bias[hd]) * inv_cap);
            bt = log_sigmoid(a.gate_cap * tanhf((pr[a.f_off] + a.f_bias[hd]) * inv_cap));
        }
        float m_before = 0.f, m_after = 0.f;
#pragma unroll
        for (int tt = 0; tt < TB; tt++) {
            const float as = __shfl_sync(0xffffffffu, at, tt), bs = __shfl_sync(0xffffffffu, bt, tt);
            if (tt < nb) {
                const float mn = fmaxf(bs + m, as);
                if (lane == tt) { m_before = m; m_after = mn; }
                m = mn;
            }
        }
        if (lane < nb) {
            gb[lane] = expf(bt + m_before - m_after);
            ga[lane] = expf(at - m_after);
            gm[lane] = expf(-m_after);
        }
    };

    stage(0, 0);
    cp_async_commit();
    if (gate_warp) gates(0, 0);
    for (int t0 = 0, r = 0; t0 < n_tok; t0 += TB, r++) {
        const int nb = min(TB, n_tok - t0), buf = r & 1;
        cp_async_wait<0>();                                  // this thread's copies of round r have landed ...
        __syncthreads();                                     // ... and everyone's, with the round's factors; round r - 1 is consumed
        if (t0 + TB < n_tok) stage(t0 + TB, buf ^ 1);
        cp_async_commit();
        const float* qs = sm + buf * ROUND;
        const float* ks = qs + TB * DPP;
        const float* vs = ks + TB * DPP;
        const float* ga = vs + TB * COLS;
        const float* gb = ga + TB;
        const float* gm = gb + TB;
        if (main) {
#pragma unroll 2
            for (int tt = 0; tt < nb; tt++) {
                const float keep = gb[tt], take = ga[tt];
                float tv[NC], acc[NC][4];
#pragma unroll
                for (int c = 0; c < NC; c++) {
                    tv[c] = take * vs[tt * COLS + warp * WCOLS + lane % CW + c * CW];
                    acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
                }
                const float4* kq = reinterpret_cast<const float4*>(ks + tt * DPP + at_row(d0));
                const float4* qq = reinterpret_cast<const float4*>(qs + tt * DPP + at_row(d0));
#pragma unroll
                for (int j = 0; j < DS; j += 4) {
                    const float4 kk = kq[j / 4], qv = qq[j / 4];
#pragma unroll
                    for (int c = 0; c < NC; c++) {
                        S[c][j] = fmaf(kk.x, tv[c], keep * S[c][j]);         acc[c][0] = fmaf(S[c][j], qv.x, acc[c][0]);
                        S[c][j + 1] = fmaf(kk.y, tv[c], keep * S[c][j + 1]); acc[c][1] = fmaf(S[c][j + 1], qv.y, acc[c][1]);
                        S[c][j + 2] = fmaf(kk.z, tv[c], keep * S[c][j + 2]); acc[c][2] = fmaf(S[c][j + 2], qv.z, acc[c][2]);
                        S[c][j + 3] = fmaf(kk.w, tv[c], keep * S[c][j + 3]); acc[c][3] = fmaf(S[c][j + 3], qv.w, acc[c][3]);
                    }
                }
#pragma unroll
                for (int c = 0; c < NC; c++) {
                    float y = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
                    if (RS >= 2) y += __shfl_xor_sync(0xffffffffu, y, CW);
                    if (RS >= 4) y += __shfl_xor_sync(0xffffffffu, y, 2 * CW);
                    if (lane < CW && col + c * CW < dv)
                        a.out[(size_t)(row0 + t0 + tt) * a.ld_out + (size_t)hd * dv + col + c * CW] = y * a.q_scale;
                }
            }
        } else if (gate_warp) {
            if (t0 + TB < n_tok) gates(t0 + TB, buf ^ 1);      // the next round's factors, while the main warps work on this one
        } else {
            if (first_block) {
#pragma unroll 4
                for (int tt = 0; tt < nb; tt++) {
                    const float keep = gb[tt], take = ga[tt];
                    float nq = 0.f;
#pragma unroll
                    for (int rr = 0; rr < NR; rr++) {
                        if (lane * NR + rr < d) {
                            nr[rr] = fmaf(take, ks[tt * DPP + at_row(lane * NR + rr)], keep * nr[rr]);
                            nq = fmaf(nr[rr], qs[tt * DPP + at_row(lane * NR + rr)], nq);
                        }
                    }
                    nq = warp_sum(nq);
                    if (lane == 0) a.den[(size_t)(row0 + t0 + tt) * H + hd] = fmaxf(fabsf(nq * a.q_scale), gm[tt]) + 1e-6f;
                }
            }
        }
    }
    if (main) {
#pragma unroll
        for (int c = 0; c < NC; c++)
#pragma unroll
            for (int j = 0; j < DS; j++)
                if (col + c * CW < dv && d0 + j < d) Sg[(size_t)(d0 + j) * dv + col + c * CW] = S[c][j];
    } else if (gate_warp) {
        if (lane == 0)
            for (int c = vb * (COLS / 32); c < min((vb + 1) * (COLS / 32), mm_m_copies(dv)); c++) mg[c] = m;
    } else if (first_block) {
#pragma unroll
        for (int r = 0; r < NR; r++) if (lane * NR + r < d) ng[lane * NR + r] = nr[r];
    }
}

__host__ __device__ inline int64_t gla_head_floats(int dim, int vdim) { return (int64_t)dim * vdim; }

// decay logits -> decays, in place: z <- exp(logsigmoid(z + bias) * inv_tau), n numbers per row
__global__ void gla_decay_kernel(float* __restrict__ z, int64_t ld_z, const float* __restrict__ bias, int64_t T, int n, float inv_tau, int vec) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    const int64_t step = (int64_t)gridDim.x * blockDim.x, me = blockIdx.x * (int64_t)blockDim.x + threadIdx.x;
    if (vec) {
        const int nq = n / 4;
        for (int64_t i = me; i < T * nq; i += step) {
            const int64_t t = i / nq;
            const int c = (int)(i - t * nq) * 4;
            float4 v = *reinterpret_cast<float4*>(z + t * ld_z + c);
            const float4 b = bias ? *reinterpret_cast<const float4*>(bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            v.x = expf(log_sigmoid(v.x + b.x) * inv_tau); v.y = expf(log_sigmoid(v.y + b.y) * inv_tau);
            v.z = expf(log_sigmoid(v.z + b.z) * inv_tau); v.w = expf(log_sigmoid(v.w + b.w) * inv_tau);
            *reinterpret_cast<float4*>(z + t * ld_z + c) = v;
        }
    } else {
        for (int64_t i = me; i < T * n; i += step) {
            const int64_t t = i / n;
            const int c = (int)(i - t * n);
            z[t * ld_z + c] = expf(log_sigmoid(z[t * ld_z + c] + (bias ? bias[c] : 0.f)) * inv_tau);
        }
    }
}

// the same with the logits formed on the way: z[t][c] = exp(logsigmoid(bias[c] + sum_r lr[t][r] a2[c][r]) * inv_tau). A thread owns
// one column with its a2 row in registers and walks the tokens of its CTA's chunk, whose low-rank vectors are staged in shared
// memory 32 tokens at a time (every thread reads the same number: a broadcast); the FMA chain runs in ascending r.
constexpr int GD_TOK = 32;
template <int RMAX>
__global__ void __launch_bounds__(256) gla_decay_lowrank_kernel(float* __restrict__ z, int64_t ld_z, const float* __restrict__ bias,
                                                                const float* __restrict__ lr, int64_t ld_lr, const float* __restrict__ a2,
                                                                int rank, int64_t T, int n, float inv_tau, int tok_per_cta) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    __shared__ float lrs[GD_TOK][RMAX];
    const int c = blockIdx.x * 256 + threadIdx.x;
    float w[RMAX];
#pragma unroll
    for (int r = 0; r < RMAX; r++) w[r] = (c < n && r < rank) ? a2[(size_t)c * rank + r] : 0.f;
    const float b = (c < n && bias) ? bias[c] : 0.f;
    const int64_t t_end = min(T, (int64_t)(blockIdx.y + 1) * tok_per_cta);
    for (int64_t t0 = (int64_t)blockIdx.y * tok_per_cta; t0 < t_end; t0 += GD_TOK) {
        const int nb = (int)min((int64_t)GD_TOK, t_end - t0);
        __syncthreads();                                     // the round before is consumed
        for (int i = threadIdx.x; i < nb * RMAX; i += 256) {
            const int tt = i / RMAX, r = i - tt * RMAX;
            lrs[tt][r] = r < rank ? lr[(t0 + tt) * ld_lr + r] : 0.f;
        }
        __syncthreads();
        if (c < n) {
            for (int tt = 0; tt < nb; tt++) {
                float acc = b;
#pragma unroll
                for (int r = 0; r < RMAX; r++) acc = fmaf(lrs[tt][r], w[r], acc);
                z[(t0 + tt) * ld_z + c] = expf(log_sigmoid(acc) * inv_tau);
            }
        }
    }
}

constexpr int GLA_WARPS = 4;     // every warp owns columns of S

template <int DS, int RS, int NC, int TB>
__global__ void __launch_bounds__(GLA_WARPS * 32) gla_scan_kernel(p3_gla_args a) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    // a warp = RS row slices x CW lanes, every lane with NC columns (CW apart); DP: dim rounded up
    constexpr int CW = 32 / RS, WCOLS = CW * NC, COLS = GLA_WARPS * WCOLS, DP = DS * RS;
    constexpr int NT = GLA_WARPS * 32;
    constexpr int DPP = DP + 4 * RS;                         // pitch of a staged row: its RS slices 4 floats apart (bank spread)
    constexpr int ROUND = TB * (3 * DPP + COLS);             // floats of one staged round
    auto at_row = [](int c) { return c + 4 * (c / DS); };    // where number c of a row lives
    extern __shared__ __align__(16) float sm[];
    const int d = a.dim, dv = a.vdim, H = a.n_heads;
    // two rounds in flight: [q [TB][DPP] (zeros beyond dim) | k alike | decays alike | v [TB][COLS]]
    const int4 rec = reinterpret_cast<const int4*>(a.seqs)[blockIdx.x];
    const int row0 = rec.x, n_tok = rec.y, slot = rec.z, pos0 = rec.w;
    const int hd = blockIdx.y, vb = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const bool fresh = pos0 == 0;
    float* Sg = a.state + ((size_t)slot * H + hd) * gla_head_floats(d, dv);
    const int col = vb * COLS + warp * WCOLS + lane % CW, d0 = (lane / CW) * DS;   // first of this lane's columns
    float S[NC][DS];
#pragma unroll
    for (int c = 0; c < NC; c++)
#pragma unroll
        for (int j = 0; j < DS; j++)
            S[c][j] = (!fresh && col + c * CW < dv && d0 + j < d) ? Sg[(size_t)(d0 + j) * dv + col + c * CW] : 0.f;
    const bool vec = d % 4 == 0 && a.ld_proj % 4 == 0 && a.q_off % 4 == 0 && a.k_off % 4 == 0 && ((uintptr_t)a.proj & 15) == 0 &&
                     a.ld_z % 4 == 0 && ((uintptr_t)a.z & 15) == 0;

    // all threads: start the copies of the round that begins at token t0 into buffer `buf` (q is scaled when the sums are written)
    auto stage = [&](int t0, int buf) {
        const int nb = min(TB, n_tok - t0);
        float* qs = sm + buf * ROUND;
        float* ks = qs + TB * DPP;
        float* as = ks + TB * DPP;
        float* vs = as + TB * DPP;
        if (vec) {
            for (int i = tid; i < nb * (DP / 4); i += NT) {
                const int tt = i / (DP / 4), c = (i - tt * (DP / 4)) * 4;
                const float* pr = a.proj + (size_t)(row0 + t0 + tt) * a.ld_proj + (size_t)hd * d + (c < d ? c : 0);
                cp_async16(smem_u32(qs + tt * DPP + at_row(c)), pr + a.q_off, c < d ? 16 : 0);
                cp_async16(smem_u32(ks + tt * DPP + at_row(c)), pr + a.k_off, c < d ? 16 : 0);
                cp_async16(smem_u32(as + tt * DPP + at_row(c)), a.z + (size_t)(row0 + t0 + tt) * a.ld_z + (size_t)hd * d + (c < d ? c : 0), c < d ? 16 : 0);
            }
        } else {
            for (int i = tid; i < nb * DP; i += NT) {
                const int tt = i / DP, c = i - tt * DP;
                const float* pr = a.proj + (size_t)(row0 + t0 + tt) * a.ld_proj + (size_t)hd * d + (c < d ? c : 0);
                cp_async4z(smem_u32(qs + tt * DPP + at_row(c)), pr + a.q_off, c < d ? 4 : 0);
                cp_async4z(smem_u32(ks + tt * DPP + at_row(c)), pr + a.k_off, c < d ? 4 : 0);
                cp_async4z(smem_u32(as + tt * DPP + at_row(c)), a.z + (size_t)(row0 + t0 + tt) * a.ld_z + (size_t)hd * d + (c < d ? c : 0), c < d ? 4 : 0);
            }
        }
        for (int i = tid; i < nb * COLS; i += NT) {
            const int tt = i / COLS, c = vb * COLS + (i - tt * COLS);
            cp_async4z(smem_u32(vs + i), a.proj + (size_t)(row0 + t0 + tt) * a.ld_proj + a.v_off + (size_t)hd * dv + (c < dv ? c : 0), c < dv ? 4 : 0);
        }
    };

    stage(0, 0);
    cp_async_commit();
    for (int t0 = 0, r = 0; t0 < n_tok; t0 += TB, r++) {
        const int nb = min(TB, n_tok - t0), buf = r & 1;
        cp_async_wait<0>();                                  // this thread's copies of round r have landed ...
        __syncthreads();                                     // ... and everyone's; round r - 1 is consumed
        if (t0 + TB < n_tok) stage(t0 + TB, buf ^ 1);
        cp_async_commit();
        const float* qs = sm + buf * ROUND;
        const float* ks = qs + TB * DPP;
        const float* as = ks + TB * DPP;
        const float* vs = as + TB * DPP;
#pragma unroll(DS >= 128 ? 1 : 2)
        for (int tt = 0; tt < nb; tt++) {
            float tv[NC], acc[NC][4];
#pragma unroll
            for (int c = 0; c < NC; c++) {
                tv[c] = vs[tt * COLS + warp * WCOLS + lane % CW + c * CW];
                acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
            }
            const float4* kq = reinterpret_cast<const float4*>(ks + tt * DPP + at_row(d0));
            const float4* qq = reinterpret_cast<const float4*>(qs + tt * DPP + at_row(d0));
            const float4* aq = reinterpret_cast<const float4*>(as + tt * DPP + at_row(d0));
#pragma unroll
            for (int j = 0; j < DS; j += 4) {
                const float4 kk = kq[j / 4], qv = qq[j / 4], al = aq[j / 4];
#pragma unroll
                for (int c = 0; c < NC; c++) {
                    S[c][j] = fmaf(kk.x, tv[c], al.x * S[c][j]);         acc[c][0] = fmaf(S[c][j], qv.x, acc[c][0]);
                    S[c][j + 1] = fmaf(kk.y, tv[c], al.y * S[c][j + 1]); acc[c][1] = fmaf(S[c][j + 1], qv.y, acc[c][1]);
                    S[c][j + 2] = fmaf(kk.z, tv[c], al.z * S[c][j + 2]); acc[c][2] = fmaf(S[c][j + 2], qv.z, acc[c][2]);
                    S[c][j + 3] = fmaf(kk.w, tv[c], al.w * S[c][j + 3]); acc[c][3] = fmaf(S[c][j + 3], qv.w, acc[c][3]);
                }
            }
#pragma unroll
            for (int c = 0; c < NC; c++) {
                float y = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
                if (RS >= 2) y += __shfl_xor_sync(0xffffffffu, y, CW);
                if (RS >= 4) y += __shfl_xor_sync(0xffffffffu, y, 2 * CW);
                if (lane < CW && col + c * CW < dv)
                    a.out[(size_t)(row0 + t0 + tt) * a.ld_out + (size_t)hd * dv + col + c * CW] = y * a.q_scale;
            }
        }
    }
#pragma unroll
    for (int c = 0; c < NC; c++)
#pragma unroll
        for (int j = 0; j < DS; j++)
            if (col + c * CW < dv && d0 + j < d) Sg[(size_t)(d0 + j) * dv + col + c * CW] = S[c][j];
}

// ---------------------------------------------------------------- short convolutions, unit heads, gates of the scan behind them
template <int VEC> __device__ __forceinline__ void ldvec(const float* p, float* v) {
    if constexpr (VEC == 4) { const float4 u = *reinterpret_cast<const float4*>(p); v[0] = u.x; v[1] = u.y; v[2] = u.z; v[3] = u.w; }
    else if constexpr (VEC == 2) { const float2 u = *reinterpret_cast<const float2*>(p); v[0] = u.x; v[1] = u.y; }
    else v[0] = *p;
}
template <int VEC> __device__ __forceinline__ void stvec(float* p, const float* v) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else if constexpr (VEC == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
    else *p = v[0];
}

// A lane owns NV vectors of VEC neighbouring channels, 32 VEC apart. TAPS > 0: the last TAPS - 1 inputs stay in registers from row
// to row; TAPS 0: any number of taps, every row reads its inputs again.
template <int VEC, int NV, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(p3_short_conv_args a, int rows_per, int n_conv_jobs) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    constexpr int N = VEC * NV, WB = 32 * N, WIN = TAPS > 1 ? TAPS - 1 : 1;
    const int lane = threadIdx.x & 31, job = blockIdx.y * 4 + (threadIdx.x >> 5);
    const int taps = TAPS > 0 ? TAPS : a.taps;
    const int C = a.n_unit * a.dim + a.n_plain;
    const int r_lo = blockIdx.x * rows_per, r_hi = min(a.n_rows, r_lo + rows_per);
    if (job >= n_conv_jobs) {                                // gates: {decay, beta or step} of every head
        if (job > n_conv_jobs || !a.gates) return;
        for (int i = lane; i < (r_hi - r_lo) * a.n_gates; i += 32) {
            const int r = r_lo + i / a.n_gates, h = i % a.n_gates;
            const float* pr = a.proj + (size_t)r * a.ld_proj;
            const float z = pr[a.a_off + h] + a.dt_bias[h];
            const float soft = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));              // softplus without overflow
            float* g = a.gates + ((size_t)r * a.n_gates + h) * 2;
            g[0] = expf(-expf(a.a_log[h]) * soft);
            g[1] = a.gate_mode == 1 ? soft : 1.0f / (1.0f + expf(-pr[a.b_off + h]));
        }
        return;
    }
    const bool unit = job < a.n_unit;
    const int c0 = unit ? job * a.dim : a.n_unit * a.dim + (job - a.n_unit) * WB;
    const int width = unit ? a.dim : min(WB, C - c0);
    const float scale = unit && job < a.n_scaled ? a.scale : 1.f;
    const float* in = a.proj + a.c_off + c0;
    auto load = [&](const float* p, float* v) {              // the lane's channels of one row (zeros beyond the width)
#pragma unroll
        for (int k = 0; k < NV; k++) {
            const int i = (k * 32 + lane) * VEC;
            if (i < width) ldvec<VEC>(p + i, v + k * VEC);
            else
#pragma unroll
                for (int e = 0; e < VEC; e++) v[k * VEC + e] = 0.f;
        }
    };
    float w[TAPS > 0 ? TAPS : 1][N], win[WIN][N], cur[N], nxt[N], bias[N];
#pragma unroll
    for (int e = 0; e < N; e++) bias[e] = 0.f;
    if (a.bias) load(a.bias + c0, bias);
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS; j++) load(a.w + (size_t)j * C + c0, w[j]);
    }
    int seq_lo = 0, seq_hi = 0, slot = 0, pos0 = 0;          // the sequence the row belongs to: its rows of this step, slot, first position
    // the input `back` rows before row r of the batch: from the step's rows, from the slot's history, or zero before the start
    auto load_back = [&](int r, int back, float* v) {
        const int rel = r - seq_lo - back;                   // row of the sequence in this step; negative: an earlier step
        if (rel >= 0) load(in + (size_t)(r - back) * a.ld_proj, v);
        else if (pos0 + rel >= 0) load(a.conv_state + ((size_t)slot * (taps - 1) + (taps - 1 + rel)) * C + c0, v);
        else
#pragma unroll
            for (int e = 0; e < N; e++) v[e] = 0.f;
    };
    if (r_lo < r_hi) load(in + (size_t)r_lo * a.ld_proj, cur);
    for (int r = r_lo; r < r_hi; r++) {
        if (r + 1 < r_hi) load(in + (size_t)(r + 1) * a.ld_proj, nxt);
        if (r >= seq_hi) {                                   // another sequence begins (or this warp's first row)
            const int4 rec = reinterpret_cast<const int4*>(a.seqs)[a.slot_seq[a.tok_slot[r]]];   // {first row, rows, slot, first position}
            seq_lo = rec.x; seq_hi = rec.x + rec.y; slot = rec.z; pos0 = rec.w;
            if (TAPS > 1) {
#pragma unroll
                for (int j = 0; j < TAPS - 1; j++) load_back(r, TAPS - 1 - j, win[j]);
            }
        }
        float z[N];
#pragma unroll
        for (int e = 0; e < N; e++) z[e] = bias[e];
        if (TAPS > 0) {
#pragma unroll
            for (int j = 0; j < TAPS - 1; j++)
#pragma unroll
                for (int e = 0; e < N; e++) z[e] = fmaf(w[j][e], win[j][e], z[e]);
#pragma unroll
            for (int e = 0; e < N; e++) z[e] = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][e], cur[e], z[e]);
#pragma unroll
            for (int j = 0; j < TAPS - 1; j++)
#pragma unroll
                for (int e = 0; e < N; e++) win[j][e] = j + 2 < TAPS ? win[j + 1 < WIN ? j + 1 : 0][e] : cur[e];
        } else {
            for (int j = 0; j < taps; j++) {
                float x[N], wj[N];
                load_back(r, taps - 1 - j, x);
                load(a.w + (size_t)j * C + c0, wj);
#pragma unroll
                for (int e = 0; e < N; e++) z[e] = fmaf(wj[e], x[e], z[e]);
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < N; e++) { z[e] = z[e] / (1.0f + expf(-z[e])); ss = fmaf(z[e], z[e], ss); }   // silu; channels beyond the width stay 0
        if (unit) {
            const float f = scale / sqrtf(warp_sum(ss) + a.unit_eps);
#pragma unroll
            for (int e = 0; e < N; e++) z[e] *= f;
        }
        float* o = a.out + (size_t)r * a.ld_out + c0;
#pragma unroll
        for (int k = 0; k < NV; k++) {
            const int i = (k * 32 + lane) * VEC;
            if (i < width) stvec<VEC>(o + i, z + k * VEC);
        }
#pragma unroll
        for (int e = 0; e < N; e++) cur[e] = nxt[e];
    }
}

// ---------------------------------------------------------------- gated delta rule, and the same memory without the correction
// a 16-byte shared load that the compiler does not merge with an earlier one of the same address
__device__ __forceinline__ float4 lds_again(const float4* p) {
    float4 v;
    asm volatile("ld.shared.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(smem_u32(p)));
    return v;
}

__host__ __device__ inline int64_t delta_head_floats(int dim, int vdim) { return (int64_t)dim * vdim; }

template <int DS, int RS, int NC, int TB, bool DELTA>
__global__ void __launch_bounds__(GLA_WARPS * 32) delta_scan_kernel(p3_delta_scan_args a) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    // a warp = RS row slices x CW lanes, every lane with NC columns (CW apart); DP: dim rounded up
    constexpr int CW = 32 / RS, WCOLS = CW * NC, COLS = GLA_WARPS * WCOLS, DP = DS * RS;
    constexpr int NT = GLA_WARPS * 32;
    constexpr int DPP = DP + 4 * RS;                         // pitch of a staged row: its RS slices 4 floats apart (bank spread)
    constexpr int ROUND = TB * (2 * DPP + COLS + 2);         // floats of one staged round
    auto at_row = [](int c) { return c + 4 * (c / DS); };    // where number c of a row lives
    extern __shared__ __align__(16) float sm[];
    const int d = a.dim, dv = a.vdim, H = a.n_heads;
    // two rounds in flight: [q [TB][DPP] (zeros beyond dim) | k alike | v [TB][COLS] | {decay, beta} [TB]]
    const int4 rec = reinterpret_cast<const int4*>(a.seqs)[blockIdx.x];
    const int row0 = rec.x, n_tok = rec.y, slot = rec.z, pos0 = rec.w;
    const int hd = blockIdx.y, hk = hd / (H / a.n_kv), vb = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const bool fresh = pos0 == 0;
    float* Sg = a.state + ((size_t)slot * H + hd) * delta_head_floats(d, dv);
    const int col = vb * COLS + warp * WCOLS + lane % CW, d0 = (lane / CW) * DS;   // first of this lane's columns
    const bool vec = d % 4 == 0 && a.ld_qkv % 4 == 0 && a.q_off % 4 == 0 && a.k_off % 4 == 0 && ((uintptr_t)a.qkv & 15) == 0;

    // all threads: start the copies of the round that begins at token t0 into buffer `buf`
    auto stage = [&](int t0, int buf) {
        const int nb = min(TB, n_tok - t0);
        float* qs = sm + buf * ROUND;
        float* ks = qs + TB * DPP;
        float* vs = ks + TB * DPP;
        float* gs = vs + TB * COLS;
        if (vec) {
            for (int i = tid; i < nb * (DP / 4); i += NT) {
                const int tt = i / (DP / 4), c = (i - tt * (DP / 4)) * 4;
                const float* pr = a.qkv + (size_t)(row0 + t0 + tt) * a.ld_qkv + (size_t)hk * d + (c < d ? c : 0);
                cp_async16(smem_u32(qs + tt * DPP + at_row(c)), pr + a.q_off, c < d ? 16 : 0);
                cp_async16(smem_u32(ks + tt * DPP + at_row(c)), pr + a.k_off, c < d ? 16 : 0);
            }
        } else {
            for (int i = tid; i < nb * DP; i += NT) {
                const int tt = i / DP, c = i - tt * DP;
                const float* pr = a.qkv + (size_t)(row0 + t0 + tt) * a.ld_qkv + (size_t)hk * d + (c < d ? c : 0);
                cp_async4z(smem_u32(qs + tt * DPP + at_row(c)), pr + a.q_off, c < d ? 4 : 0);
                cp_async4z(smem_u32(ks + tt * DPP + at_row(c)), pr + a.k_off, c < d ? 4 : 0);
            }
        }
        for (int i = tid; i < nb * COLS; i += NT) {
            const int tt = i / COLS, c = vb * COLS + (i - tt * COLS);
            cp_async4z(smem_u32(vs + i), a.qkv + (size_t)(row0 + t0 + tt) * a.ld_qkv + a.v_off + (size_t)hd * dv + (c < dv ? c : 0), c < dv ? 4 : 0);
        }
        if (DELTA || a.gates)
            for (int i = tid; i < nb * 2; i += NT) cp_async4z(smem_u32(gs + i), a.gates + ((size_t)(row0 + t0 + i / 2) * H + hd) * 2 + (i & 1), 4);
    };

    stage(0, 0);
    cp_async_commit();
    // the convolution history moves on by this sequence's rows: channel by channel in order of time, so that a history longer than
    // the step's rows can shift in place
    if (a.taps > 1) {
        const int keep = a.taps - 1, n_thr = NT * gridDim.y * gridDim.z;
        float* hist = a.conv_state + (size_t)slot * keep * a.channels;
        for (int c = (blockIdx.z * gridDim.y + blockIdx.y) * NT + tid; c < a.channels; c += n_thr)
            for (int j = 0; j < keep; j++) {
                const int rel = n_tok - keep + j;            // row of the step; negative: an entry of the old history
                hist[(size_t)j * a.channels + c] = rel >= 0 ? a.conv_in[(size_t)(row0 + rel) * a.ld_conv_in + c]
                                                            : pos0 + rel >= 0 ? hist[(size_t)(j + n_tok) * a.channels + c] : 0.f;
            }
    }
    const float fixed = DELTA || a.gates ? 0.f : a.decay[hd], skip = DELTA || !a.skip ? 0.f : a.skip[hd];
    float S[NC][DS];
#pragma unroll
    for (int c = 0; c < NC; c++)
#pragma unroll
        for (int j = 0; j < DS; j++)
            S[c][j] = (!fresh && col + c * CW < dv && d0 + j < d) ? Sg[(size_t)(d0 + j) * dv + col + c * CW] : 0.f;
    for (int t0 = 0, r = 0; t0 < n_tok; t0 += TB, r++) {
        const int nb = min(TB, n_tok - t0), buf = r & 1;
        cp_async_wait<0>();                                  // this thread's copies of round r have landed ...
        __syncthreads();                                     // ... and everyone's; round r - 1 is consumed
        if (t0 + TB < n_tok) stage(t0 + TB, buf ^ 1);
        cp_async_commit();
        const float* qs = sm + buf * ROUND;
        const float* ks = qs + TB * DPP;
        const float* vs = ks + TB * DPP;
        const float* gs = vs + TB * COLS;
        int tt = 0;
        if constexpr (!DELTA && DS <= 64) {
            // four tokens at a time: no sum of one of them waits for another's shuffles, and the row slices share the reduction out, so
            // that slice s ends with the whole sums of token s (RS = 4; of tokens s and s + 2 with RS = 2) and writes them
            for (; tt + 4 <= nb; tt += 4) {
                float p[4][NC];
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const float keep = a.gates ? gs[2 * (tt + i)] : fixed, beta = a.gates ? gs[2 * (tt + i) + 1] : 1.f;
                    const float4* kq = reinterpret_cast<const float4*>(ks + (tt + i) * DPP + at_row(d0));
                    const float4* qq = reinterpret_cast<const float4*>(qs + (tt + i) * DPP + at_row(d0));
                    float acc[NC][4], u[NC];
#pragma unroll
                    for (int c = 0; c < NC; c++) {
                        acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
                        u[c] = beta * vs[(tt + i) * COLS + warp * WCOLS + lane % CW + c * CW];
                    }
#pragma unroll
                    for (int j = 0; j < DS; j += 4) {
                        const float4 kk = kq[j / 4], qv = qq[j / 4];
#pragma unroll
                        for (int c = 0; c < NC; c++) {
                            S[c][j] = fmaf(kk.x, u[c], keep * S[c][j]);         acc[c][0] = fmaf(S[c][j], qv.x, acc[c][0]);
                            S[c][j + 1] = fmaf(kk.y, u[c], keep * S[c][j + 1]); acc[c][1] = fmaf(S[c][j + 1], qv.y, acc[c][1]);
                            S[c][j + 2] = fmaf(kk.z, u[c], keep * S[c][j + 2]); acc[c][2] = fmaf(S[c][j + 2], qv.z, acc[c][2]);
                            S[c][j + 3] = fmaf(kk.w, u[c], keep * S[c][j + 3]); acc[c][3] = fmaf(S[c][j + 3], qv.w, acc[c][3]);
                        }
                    }
#pragma unroll
                    for (int c = 0; c < NC; c++) p[i][c] = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
                }
                const int sl = lane / CW;
                float r[2][NC];
#pragma unroll
                for (int h = 0; h < 2; h++)
#pragma unroll
                    for (int c = 0; c < NC; c++)
                        r[h][c] = (sl & 1 ? p[2 * h + 1][c] : p[2 * h][c]) + __shfl_xor_sync(0xffffffffu, sl & 1 ? p[2 * h][c] : p[2 * h + 1][c], CW);
                auto write = [&](int t, int c, float y) {
                    y = fmaf(skip, vs[t * COLS + warp * WCOLS + lane % CW + c * CW], y);
                    if (col + c * CW < dv) a.out[(size_t)(row0 + t0 + t) * a.ld_out + (size_t)hd * dv + col + c * CW] = y;
                };
#pragma unroll
                for (int c = 0; c < NC; c++) {
                    if (RS == 4) write(tt + sl, c, (sl & 2 ? r[1][c] : r[0][c]) + __shfl_xor_sync(0xffffffffu, sl & 2 ? r[0][c] : r[1][c], 2 * CW));
                    else { write(tt + sl, c, r[0][c]); write(tt + 2 + sl, c, r[1][c]); }
                }
            }
        }
#pragma unroll(DS >= (DELTA ? 64 : 128) ? 1 : 2)
        for (; tt < nb; tt++) {
            const float keep = DELTA || a.gates ? gs[2 * tt] : fixed, beta = DELTA || a.gates ? gs[2 * tt + 1] : 1.f;
            const float4* kq = reinterpret_cast<const float4*>(ks + tt * DPP + at_row(d0));
            const float4* qq = reinterpret_cast<const float4*>(qs + tt * DPP + at_row(d0));
            float acc[NC][4], u[NC];
#pragma unroll
            for (int c = 0; c < NC; c++) acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
            if constexpr (DELTA) {
#pragma unroll
                for (int j = 0; j < DS; j += 4) {
                    const float4 kk = kq[j / 4];
#pragma unroll
                    for (int c = 0; c < NC; c++) {
                        acc[c][0] = fmaf(S[c][j], kk.x, acc[c][0]);         acc[c][1] = fmaf(S[c][j + 1], kk.y, acc[c][1]);
                        acc[c][2] = fmaf(S[c][j + 2], kk.z, acc[c][2]);     acc[c][3] = fmaf(S[c][j + 3], kk.w, acc[c][3]);
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < NC; c++) {
                const float vv = vs[tt * COLS + warp * WCOLS + lane % CW + c * CW];
                if constexpr (!DELTA) { u[c] = beta * vv; continue; }
                float p = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
                if (RS >= 2) p += __shfl_xor_sync(0xffffffffu, p, CW);
                if (RS >= 4) p += __shfl_xor_sync(0xffffffffu, p, 2 * CW);
                u[c] = beta * (vv - keep * p);             // (decay S)^T k = decay (S^T k)
                acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
            }
#pragma unroll
            for (int j = 0; j < DS; j += 4) {
                // up to 32 rows per lane the k row stays in registers between the passes
                const float4 kk = DS <= 32 || !DELTA ? kq[j / 4] : lds_again(kq + j / 4), qv = qq[j / 4];
#pragma unroll
                for (int c = 0; c < NC; c++) {
                    S[c][j] = fmaf(kk.x, u[c], keep * S[c][j]);         acc[c][0] = fmaf(S[c][j], qv.x, acc[c][0]);
                    S[c][j + 1] = fmaf(kk.y, u[c], keep * S[c][j + 1]); acc[c][1] = fmaf(S[c][j + 1], qv.y, acc[c][1]);
                    S[c][j + 2] = fmaf(kk.z, u[c], keep * S[c][j + 2]); acc[c][2] = fmaf(S[c][j + 2], qv.z, acc[c][2]);
                    S[c][j + 3] = fmaf(kk.w, u[c], keep * S[c][j + 3]); acc[c][3] = fmaf(S[c][j + 3], qv.w, acc[c][3]);
                }
            }
#pragma unroll
            for (int c = 0; c < NC; c++) {
                float y = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
                if (RS >= 2) y += __shfl_xor_sync(0xffffffffu, y, CW);
                if (RS >= 4) y += __shfl_xor_sync(0xffffffffu, y, 2 * CW);
                if (!DELTA) y = fmaf(skip, vs[tt * COLS + warp * WCOLS + lane % CW + c * CW], y);
                if (lane < CW && col + c * CW < dv)
                    a.out[(size_t)(row0 + t0 + tt) * a.ld_out + (size_t)hd * dv + col + c * CW] = y;
            }
        }
    }
#pragma unroll
    for (int c = 0; c < NC; c++)
#pragma unroll
        for (int j = 0; j < DS; j++)
            if (col + c * CW < dv && d0 + j < d) Sg[(size_t)(d0 + j) * dv + col + c * CW] = S[c][j];
}

// one warp per (token, head)
template <typename AT>
__global__ void headnorm_gate_kernel(const float* __restrict__ y, int64_t ldy, const float* __restrict__ den, int H, int dv,
                                     const float* __restrict__ gain, int gain_shared,
                                     const float* __restrict__ gate, int64_t ld_gate, int gate_silu, float scale, float eps,
                                     AT* __restrict__ out, int64_t ldo, int64_t T) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    const int lane = threadIdx.x & 31;
    const int64_t job = blockIdx.x * (int64_t)(blockDim.x >> 5) + (threadIdx.x >> 5);
    if (job >= T * H) return;
    const int64_t t = job / H;
    const int h = (int)(job - t * H);
    const float* yr = y + t * ldy + (size_t)h * dv;
    const float dn = den ? den[t * H + h] : 1.f;             // the read-out's denominator, when the producer left numerators
    // up to 8 numbers per lane stay in registers between the statistic and the write (heads of up to 256 numbers)
    float v[8];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 8; k++) { const int i = lane + 32 * k; v[k] = i < dv ? yr[i] / dn : 0.f; ss = fmaf(v[k], v[k], ss); }
    for (int i = lane + 256; i < dv; i += 32) { const float u = yr[i] / dn; ss = fmaf(u, u, ss); }
    ss = warp_sum(ss);
    const float r = scale / sqrtf(ss / (float)dv + eps);
    auto gated = [&](int c) {                                // the gate of output column c: sigmoid(g), or silu(g) = g sigmoid(g)
        if (!gate) return 1.f;
        const float g = gate[t * ld_gate + c], sg = 1.0f / (1.0f + expf(-g));
        return gate_silu ? g * sg : sg;
    };
#pragma unroll
    for (int k = 0; k < 8; k++) {
        const int i = lane + 32 * k, c = h * dv + i;
        if (i < dv) stv(out + t * ldo + c, v[k] * r * gain[gain_shared ? i : c] * gated(c));
    }
    for (int i = lane + 256; i < dv; i += 32) {
        const int c = h * dv + i;
        stv(out + t * ldo + c, yr[i] / dn * r * gain[gain_shared ? i : c] * gated(c));
    }
}

// One job = one part (n numbers) of a row: a warp (WARP, four jobs per CTA) or a whole CTA. Up to PN numbers per thread stay in registers,
// VEC neighbours loaded and stored together.
constexpr int PN = 8;
template <typename AT, int VEC, bool WARP>
__global__ void part_norm_gate_kernel(const float* __restrict__ y, int64_t ldy, int parts, int n, const float* __restrict__ gain,
                                      const float* __restrict__ gate, int64_t ld_gate, int gate_silu, int gate_first, float scale, float eps,
                                      AT* __restrict__ out, int64_t ldo, int64_t T) {
    pdl_trigger();                                           // the next kernel may set up while this one runs ...
    pdl_wait();                                              // ... and this one touches memory only after its predecessors are done
    __shared__ float sh[32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nt = WARP ? 32 : blockDim.x, me = WARP ? lane : threadIdx.x;
    const int64_t job = WARP ? blockIdx.x * (int64_t)(blockDim.x >> 5) + warp : blockIdx.x;
    if (WARP && job >= T * parts) return;
    const int64_t t = job / parts;
    const int c0 = (int)(job - t * parts) * n;
    const float* yr = y + t * ldy + c0;
    const float* gr = gate ? gate + t * ld_gate + c0 : nullptr;
    const float* wr = gain + c0;
    AT* o = out + t * ldo + c0;
    auto at = [&](int k) { return ((k / VEC) * nt + me) * VEC + k % VEC; };
    auto act = [&](float g) { const float s = 1.0f / (1.0f + expf(-g)); return gate_silu ? g * s : s; };
    float v[PN], g[PN];
#pragma unroll
    for (int k = 0; k < PN; k += VEC) {
#pragma unroll
        for (int e = 0; e < VEC; e++) { v[k + e] = 0.f; g[k + e] = 0.f; }
        const int i = at(k);
        if (i < n) { ldvec<VEC>(yr + i, v + k); if (gr) ldvec<VEC>(gr + i, g + k); }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < PN; k++) {
        g[k] = gr ? act(g[k]) : 1.f;
        if (gate_first) v[k] *= g[k];
        ss = fmaf(v[k], v[k], ss);
    }
    auto first = [&](int i) { return gate_first && gr ? yr[i] * act(gr[i]) : yr[i]; };
    for (int i = me + PN * nt; i < n; i += nt) { const float u = first(i); ss = fmaf(u, u, ss); }
    ss = warp_sum(ss);
    if (!WARP) {
        if (lane == 0) sh[warp] = ss;
        __syncthreads();
        ss = 0.f;
        for (int w = 0; w < (int)(blockDim.x >> 5); w++) ss += sh[w];
    }
    const float r = scale / sqrtf(ss / (float)n + eps);
#pragma unroll
    for (int k = 0; k < PN; k += VEC) {
        const int i = at(k);
        if (i >= n) continue;
        float w[VEC];
        ldvec<VEC>(wr + i, w);
#pragma unroll
        for (int e = 0; e < VEC; e++) w[e] = v[k + e] * r * w[e] * (gate_first ? 1.f : g[k + e]);
        if constexpr (VEC == 4 && sizeof(AT) == 2) *reinterpret_cast<uint2*>(o + i) = make_uint2(pack_bf16(w[0], w[1]), pack_bf16(w[2], w[3]));
        else if constexpr (VEC == 4) stvec<4>((float*)o + i, w);
        else stv(o + i, w[0]);
    }
    for (int i = me + PN * nt; i < n; i += nt) stv(o + i, first(i) * r * wr[i] * (gr && !gate_first ? act(gr[i]) : 1.f));
}
template <typename K>
int set_smem_attr(K kernel, size_t bytes) {
    if (bytes > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
        P3_CHECK_ARG(e == cudaSuccess, "matrix_memory_scan: shared memory attribute: %s", cudaGetErrorString(e));
    }
    return 0;
}
}  // namespace

extern "C" int64_t p3_matrix_memory_state_floats(int n_heads, int dim, int vdim) { return (int64_t)n_heads * mm_head_floats(dim, vdim); }

extern "C" int p3_matrix_memory_scan(const p3_matrix_memory_args* a, cudaStream_t st) {
    P3_CHECK_ARG(a && a->proj && a->i_bias && a->f_bias && a->state && a->seqs && a->out && a->den, "matrix_memory_scan: null argument");
    P3_CHECK_ARG(a->n_heads >= 1 && a->dim >= 1 && a->dim <= 512 && a->vdim >= 1, "matrix_memory_scan: need heads >= 1, 1 <= dim <= 512, vdim >= 1");
    P3_CHECK_ARG(a->gate_cap > 0.f, "matrix_memory_scan: the gate cap must be positive");
    P3_CHECK_ARG(((uintptr_t)a->seqs & 15) == 0, "matrix_memory_scan: the sequence records must be 16-byte aligned");
    if (a->n_seqs == 0) return 0;
    // A warp is four row slices x eight lanes; a lane owns two columns (each k / q read from shared memory, the limit of this
    // kernel, then serves two columns) when that still leaves a CTA for every SM, else one. rs_force (tests): 2 or 4 row slices
    // with one column per lane, 8 = four slices with two columns.
    int rs = 4, nc = (int64_t)a->n_seqs * a->n_heads * ((a->vdim + 63) / 64) >= 148 ? 2 : 1;
    if (a->rs_force == 2 || a->rs_force == 4) { rs = a->rs_force; nc = 1; }
    if (a->rs_force == 8) { rs = 4; nc = 2; }
    if (a->dim > 256) { rs = 4; nc = 1; }                    // 128 rows per thread, 16 tokens per round
    const int per = (a->dim + rs - 1) / rs, ds = per <= 16 ? 16 : per <= 32 ? 32 : per <= 64 ? 64 : 128;
    const int cols = MM_MAIN * 32 / rs * nc, tb = a->dim > 256 ? 16 : MM_TB;
    const dim3 grid((unsigned)a->n_seqs, (unsigned)a->n_heads, (unsigned)((a->vdim + cols - 1) / cols));
    const size_t bytes = sizeof(float) * (size_t)2 * tb * (2 * (ds * rs + 4 * rs) + cols + 3);   // two staged rounds
#define GO(DS, RS, NC)                                                                                              \
    do { if (set_smem_attr(matrix_memory_scan_kernel<DS, RS, NC, MM_TB>, bytes)) return -1;                           \
         p3_launch_pdl(matrix_memory_scan_kernel<DS, RS, NC, MM_TB>, dim3(grid), dim3(MM_WARPS * 32), (size_t)(bytes), st, *a); } while (0)
    if (a->dim > 256) {
        if (set_smem_attr(matrix_memory_scan_kernel<128, 4, 1, 16>, bytes)) return -1;
        p3_launch_pdl(matrix_memory_scan_kernel<128, 4, 1, 16>, dim3(grid), dim3(MM_WARPS * 32), (size_t)(bytes), st, *a);
    } else if (rs == 2) { if (ds == 16) GO(16, 2, 1); else if (ds == 32) GO(32, 2, 1); else if (ds == 64) GO(64, 2, 1); else GO(128, 2, 1); }
    else if (nc == 1) { if (ds == 16) GO(16, 4, 1); else if (ds == 32) GO(32, 4, 1); else GO(64, 4, 1); }
    else { if (ds == 16) GO(16, 4, 2); else if (ds == 32) GO(32, 4, 2); else GO(64, 4, 2); }
#undef GO
    P3_CHECK_LAUNCH("matrix_memory_scan");
    return 0;
}

extern "C" int p3_headnorm_gate_x(const float* y, int64_t ldy, const float* den, int n_heads, int vdim, const float* gain, int gain_shared,
                                  const float* gate, int64_t ld_gate, int gate_silu, float scale, float eps, void* out, int64_t ldo,
                                  int out_f32, int64_t T, cudaStream_t st) {
    P3_CHECK_ARG(y && gain && out && n_heads >= 1 && vdim >= 1, "headnorm_gate: null argument");
    if (T == 0) return 0;
    const int64_t jobs = T * n_heads;
    const unsigned grid = (unsigned)((jobs + 3) / 4);
    if (out_f32) p3_launch_pdl(headnorm_gate_kernel<float>, dim3(grid), dim3(128), (size_t)(0), st, y, ldy, den, n_heads, vdim, gain, gain_shared, gate, ld_gate, gate_silu, scale, eps, (float*)out, ldo, T);
    else p3_launch_pdl(headnorm_gate_kernel<bf16>, dim3(grid), dim3(128), (size_t)(0), st, y, ldy, den, n_heads, vdim, gain, gain_shared, gate, ld_gate, gate_silu, scale, eps, (bf16*)out, ldo, T);
    P3_CHECK_LAUNCH("headnorm_gate");
    return 0;
}

extern "C" int p3_headnorm_gate(const float* y, int64_t ldy, const float* den, int n_heads, int vdim, const float* gain, const float* gate,
                                int64_t ld_gate, float scale, float eps, void* out, int64_t ldo, int out_f32, int64_t T, cudaStream_t st) {
    return p3_headnorm_gate_x(y, ldy, den, n_heads, vdim, gain, 0, gate, ld_gate, 0, scale, eps, out, ldo, out_f32, T, st);
}

extern "C" int p3_part_norm_gate(const float* y, int64_t ldy, int parts, int n, const float* gain, const float* gate, int64_t ld_gate,
                                 int gate_silu, int gate_first, float scale, float eps, void* out, int64_t ldo, int out_f32, int64_t T,
                                 cudaStream_t st) {
    P3_CHECK_ARG(y && gain && out && parts >= 1 && n >= 1, "part_norm_gate: null argument");
    if (T == 0) return 0;
    const bool vec = n % 4 == 0 && ldy % 4 == 0 && (!gate || ld_gate % 4 == 0) && ldo % 4 == 0 &&
                     (((uintptr_t)y | (uintptr_t)gain | (uintptr_t)gate) & 15) == 0 && ((uintptr_t)out & (out_f32 ? 15 : 7)) == 0;
    const int64_t jobs = T * parts;
    const bool warp = n <= 32 * PN;
    int th = (n + PN * 32 - 1) / (PN * 32) * 32;             // threads whose registers hold a part of n numbers (up to 8192)
    th = warp ? 128 : th > 1024 ? 1024 : th;
    const unsigned grid = (unsigned)(warp ? (jobs + 3) / 4 : jobs);
#define GO(AT, V, WP) p3_launch_pdl(part_norm_gate_kernel<AT, V, WP>, dim3(grid), dim3(th), (size_t)(0), st, y, ldy, parts, n, gain, gate, ld_gate, \
                                    gate_silu, gate_first, scale, eps, (AT*)out, ldo, T)
#define GV(AT) do { if (vec) { if (warp) GO(AT, 4, true); else GO(AT, 4, false); } else { if (warp) GO(AT, 1, true); else GO(AT, 1, false); } } while (0)
    if (out_f32) GV(float); else GV(bf16);
#undef GV
#undef GO
    P3_CHECK_LAUNCH("part_norm_gate");
    return 0;
}

extern "C" int64_t p3_gla_state_floats(int n_heads, int dim, int vdim) { return (int64_t)n_heads * gla_head_floats(dim, vdim); }

extern "C" int p3_gla_scan(const p3_gla_args* a, cudaStream_t st) {
    P3_CHECK_ARG(a && a->proj && a->z && a->state && a->seqs && a->out, "gla_scan: null argument");
    P3_CHECK_ARG(a->n_heads >= 1 && a->dim >= 1 && a->dim <= 512 && a->vdim >= 1, "gla_scan: need heads >= 1, 1 <= dim <= 512, vdim >= 1");
    P3_CHECK_ARG(((uintptr_t)a->seqs & 15) == 0, "gla_scan: the sequence records must be 16-byte aligned");
    P3_CHECK_ARG(a->n_rows >= 0, "gla_scan: the number of rows must not be negative");
    if (a->n_seqs == 0 || a->n_rows == 0) return 0;
    P3_CHECK_ARG(!a->lr || (a->a2 && a->rank >= 1 && a->rank <= 64), "gla_scan: the low-rank decay projection needs a2 and 1 <= rank <= 64");
    if (a->lr) {   // decays first, over all rows of the step at once, logits formed on the way: the scan then stages them like k and q
        const int n = a->n_heads * a->dim;
        const unsigned gx = (unsigned)((n + 255) / 256);
        // enough CTAs for four per SM, at least one staged round of tokens each
        int64_t per = (a->n_rows + (148 * 4 / gx)) / (148 * 4 / gx + 1);
        per = (per + GD_TOK - 1) / GD_TOK * GD_TOK;
        if (per < GD_TOK) per = GD_TOK;
        const dim3 dgrid(gx, (unsigned)((a->n_rows + per - 1) / per));
#define GD(R) p3_launch_pdl(gla_decay_lowrank_kernel<R>, dim3(dgrid), dim3(256), (size_t)(0), st, a->z, a->ld_z, a->z_bias, a->lr, a->ld_lr, \
                            a->a2, a->rank, (int64_t)a->n_rows, n, a->inv_tau, (int)per)
        if (a->rank <= 16) GD(16); else if (a->rank <= 32) GD(32); else GD(64);
#undef GD
    } else {       // decays first, over all rows of the step at once and in place
        const int n = a->n_heads * a->dim;
        const int vec = n % 4 == 0 && a->ld_z % 4 == 0 && ((uintptr_t)a->z & 15) == 0 && (!a->z_bias || ((uintptr_t)a->z_bias & 15) == 0);
        const int64_t work = (int64_t)a->n_rows * (vec ? n / 4 : n);
        const unsigned blocks = (unsigned)(work + 255) / 256 < 148u * 8 ? (unsigned)((work + 255) / 256) : 148u * 8;
        p3_launch_pdl(gla_decay_kernel, dim3(blocks ? blocks : 1), dim3(256), (size_t)(0), st, a->z, a->ld_z, a->z_bias, (int64_t)a->n_rows, n, a->inv_tau, vec);
    }
    // A warp is four row slices x eight lanes. Two columns per lane halve the shared-memory reads per FMA, which is what bounds
    // this kernel (three staged rows per token against two of the matrix memory): a CTA then takes 1.14 times as long for twice
    // the columns, so that shape wins as soon as one column per lane would need more CTAs than there are SMs.
    int rs = 4, nc = (int64_t)a->n_seqs * a->n_heads * ((a->vdim + 31) / 32) > 148 ? 2 : 1;
    if (a->rs_force == 2 || a->rs_force == 4) { rs = a->rs_force; nc = 1; }
    if (a->rs_force == 8) { rs = 4; nc = 2; }
    if (a->dim > 256) { rs = 4; nc = 1; }                    // 128 rows per thread, 16 tokens per round
    const int per = (a->dim + rs - 1) / rs, ds = per <= 16 ? 16 : per <= 32 ? 32 : per <= 64 ? 64 : 128;
    const int cols = GLA_WARPS * 32 / rs * nc, tb = a->dim > 256 ? 16 : MM_TB;
    const dim3 grid((unsigned)a->n_seqs, (unsigned)a->n_heads, (unsigned)((a->vdim + cols - 1) / cols));
    const size_t bytes = sizeof(float) * (size_t)2 * tb * (3 * (ds * rs + 4 * rs) + cols);   // two staged rounds
#define GO(DS, RS, NC)                                                                                              \
    do { if (set_smem_attr(gla_scan_kernel<DS, RS, NC, MM_TB>, bytes)) return -1;                                     \
         p3_launch_pdl(gla_scan_kernel<DS, RS, NC, MM_TB>, dim3(grid), dim3(GLA_WARPS * 32), (size_t)(bytes), st, *a); } while (0)
    if (a->dim > 256) {
        if (set_smem_attr(gla_scan_kernel<128, 4, 1, 16>, bytes)) return -1;
        p3_launch_pdl(gla_scan_kernel<128, 4, 1, 16>, dim3(grid), dim3(GLA_WARPS * 32), (size_t)(bytes), st, *a);
    } else if (rs == 2) { if (ds == 16) GO(16, 2, 1); else if (ds == 32) GO(32, 2, 1); else if (ds == 64) GO(64, 2, 1); else GO(128, 2, 1); }
    else if (nc == 1) { if (ds == 16) GO(16, 4, 1); else if (ds == 32) GO(32, 4, 1); else GO(64, 4, 1); }
    else { if (ds == 16) GO(16, 4, 2); else if (ds == 32) GO(32, 4, 2); else GO(64, 4, 2); }
#undef GO
    P3_CHECK_LAUNCH("gla_scan");
    return 0;
}

extern "C" int p3_short_conv(const p3_short_conv_args* a, cudaStream_t st) {
    P3_CHECK_ARG(a && a->proj && a->w && a->seqs && a->slot_seq && a->tok_slot && a->out, "short_conv: null argument");
    P3_CHECK_ARG(a->taps >= 1 && (a->taps == 1 || a->conv_state), "short_conv: several taps need the history");
    P3_CHECK_ARG(a->n_unit >= 0 && a->n_plain >= 0 && a->n_scaled <= a->n_unit && (a->n_unit == 0 || (a->dim >= 1 && a->dim <= 512)),
                 "short_conv: need 1 <= dim <= 512 and n_scaled <= n_unit");
    P3_CHECK_ARG(!a->gates || (a->n_gates >= 1 && a->a_log && a->dt_bias), "short_conv: the gates need a_log and dt_bias");
    P3_CHECK_ARG(a->gate_mode == 0 || a->gate_mode == 1, "short_conv: gate_mode is 0 (decay, beta) or 1 (decay, step)");
    P3_CHECK_ARG(((uintptr_t)a->seqs & 15) == 0, "short_conv: the sequence records must be 16-byte aligned");
    if (a->n_rows == 0) return 0;
    const int d = a->n_unit ? a->dim : 128, C = a->n_unit * a->dim + a->n_plain;
    auto fits = [&](int v) {                                 // may a lane take v neighbouring channels at once?
        const uintptr_t m = (uintptr_t)v * 4 - 1;
        return d % v == 0 && C % v == 0 && a->c_off % v == 0 && a->ld_proj % v == 0 && a->ld_out % v == 0 &&
               (((uintptr_t)a->proj | (uintptr_t)a->w | (uintptr_t)a->bias | (uintptr_t)a->out | (uintptr_t)a->conv_state) & m) == 0;
    };
    const int vec = d > 64 && fits(4) ? 4 : d > 32 && fits(2) ? 2 : 1;
    const int need = (d + 32 * vec - 1) / (32 * vec), nv = need <= 1 ? 1 : need <= 2 ? 2 : need <= 4 ? 4 : need <= 8 ? 8 : 16;
    const int wb = 32 * vec * nv, conv_jobs = a->n_unit + (a->n_plain + wb - 1) / wb, jobs = conv_jobs + (a->gates ? 1 : 0);
    const int rows_per = a->n_rows >= 512 ? 16 : a->n_rows >= 128 ? 4 : 1;
    const dim3 grid((unsigned)((a->n_rows + rows_per - 1) / rows_per), (unsigned)((jobs + 3) / 4));
#define GO(V, N)                                                                                                               \
    do { if (a->taps == 4) p3_launch_pdl(short_conv_kernel<V, N, 4>, dim3(grid), dim3(128), (size_t)(0), st, *a, rows_per, conv_jobs); \
         else p3_launch_pdl(short_conv_kernel<V, N, 0>, dim3(grid), dim3(128), (size_t)(0), st, *a, rows_per, conv_jobs); } while (0)
    if (vec == 4) { if (nv == 1) GO(4, 1); else if (nv == 2) GO(4, 2); else GO(4, 4); }
    else if (vec == 2) { if (nv == 1) GO(2, 1); else if (nv == 2) GO(2, 2); else if (nv == 4) GO(2, 4); else GO(2, 8); }
    else { if (nv == 1) GO(1, 1); else if (nv == 2) GO(1, 2); else if (nv == 4) GO(1, 4); else if (nv == 8) GO(1, 8); else GO(1, 16); }
#undef GO
    P3_CHECK_LAUNCH("short_conv");
    return 0;
}

extern "C" int64_t p3_delta_state_floats(int n_heads, int dim, int vdim) { return (int64_t)n_heads * delta_head_floats(dim, vdim); }

namespace {
template <bool DELTA>
int launch_scan(const p3_delta_scan_args* a, cudaStream_t st, const char* who) {
    P3_CHECK_ARG(a && a->qkv && a->state && a->seqs && a->out, "%s: null argument", who);
    P3_CHECK_ARG(a->n_heads >= 1 && a->n_kv >= 1 && a->n_heads % a->n_kv == 0, "%s: heads must be a multiple of kv heads", who);
    P3_CHECK_ARG(a->dim >= 1 && a->dim <= 512 && a->vdim >= 1, "%s: need 1 <= dim <= 512, vdim >= 1", who);
    P3_CHECK_ARG(a->taps <= 1 || (a->conv_in && a->conv_state && a->channels >= 1), "%s: the convolution history needs its inputs", who);
    P3_CHECK_ARG(((uintptr_t)a->seqs & 15) == 0, "%s: the sequence records must be 16-byte aligned", who);
    if (a->n_seqs == 0) return 0;
    // A warp is four row slices x eight lanes, a lane owns one or two columns: the choice of the linear-attention scan. Without the
    // correction a CTA with one column per lane takes about 0.6 of the time of one with two; the busiest SM decides.
    const int64_t c1 = (int64_t)a->n_seqs * a->n_heads * ((a->vdim + 31) / 32), c2 = (int64_t)a->n_seqs * a->n_heads * ((a->vdim + 63) / 64);
    int rs = 4, nc = (DELTA ? c1 > 148 : 10 * ((c2 + 147) / 148) <= 6 * ((c1 + 147) / 148)) ? 2 : 1;
    if (a->rs_force == 2 || a->rs_force == 4) { rs = a->rs_force; nc = 1; }
    if (a->rs_force == 8) { rs = 4; nc = 2; }
    if (a->dim > 256) { rs = 4; nc = 1; }                    // 128 rows per thread, 16 tokens per round
    const int per = (a->dim + rs - 1) / rs, ds = per <= 16 ? 16 : per <= 32 ? 32 : per <= 64 ? 64 : 128;
    const int cols = GLA_WARPS * 32 / rs * nc, tb = a->dim > 256 ? 16 : MM_TB;
    const dim3 grid((unsigned)a->n_seqs, (unsigned)a->n_heads, (unsigned)((a->vdim + cols - 1) / cols));
    const size_t bytes = sizeof(float) * (size_t)2 * tb * (2 * (ds * rs + 4 * rs) + cols + 2);   // two staged rounds
#define GO(DS, RS, NC, TB)                                                                                             \
    do { if (set_smem_attr(delta_scan_kernel<DS, RS, NC, TB, DELTA>, bytes)) return -1;                                  \
         p3_launch_pdl(delta_scan_kernel<DS, RS, NC, TB, DELTA>, dim3(grid), dim3(GLA_WARPS * 32), (size_t)(bytes), st, *a); } while (0)
    if (a->dim > 256) GO(128, 4, 1, 16);
    else if (rs == 2) { if (ds == 16) GO(16, 2, 1, MM_TB); else if (ds == 32) GO(32, 2, 1, MM_TB); else if (ds == 64) GO(64, 2, 1, MM_TB); else GO(128, 2, 1, MM_TB); }
    else if (nc == 1) { if (ds == 16) GO(16, 4, 1, MM_TB); else if (ds == 32) GO(32, 4, 1, MM_TB); else GO(64, 4, 1, MM_TB); }
    else { if (ds == 16) GO(16, 4, 2, MM_TB); else if (ds == 32) GO(32, 4, 2, MM_TB); else GO(64, 4, 2, MM_TB); }
#undef GO
    P3_CHECK_LAUNCH(who);
    return 0;
}
}  // namespace

extern "C" int p3_delta_scan(const p3_delta_scan_args* a, cudaStream_t st) {
    P3_CHECK_ARG(a && a->gates, "delta_scan: null argument");
    return launch_scan<true>(a, st, "delta_scan");
}

extern "C" int p3_decay_scan(const p3_delta_scan_args* a, cudaStream_t st) {
    P3_CHECK_ARG(a && (a->gates || a->decay), "decay_scan: needs gates, or one decay per head");
    return launch_scan<false>(a, st, "decay_scan");
}
