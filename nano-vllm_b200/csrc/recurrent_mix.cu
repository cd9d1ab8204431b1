// Linear recurrences with per-sequence state slots: a gated diagonal recurrence and the gated delta rule.
//
// Everything that enters a recurrence (gates, decays, step sizes, unit norms, the state) is fp32 in both element types; the
// activation type T only names what the projections and convolutions in front left in memory and what the result is rounded to.
// A step whose sequence has no tokens behind it starts from zeros whatever the slot holds, so a slot needs no clearing when
// it changes hands.
//
// Gated diagonal recurrence (one scalar state per channel):
//     r = sigmoid(gr + br), i = sigmoid(gi + bi)          gr, gi: block-diagonal maps of u, computed by the caller (fp32)
//     a = exp(rate * r)                                   rate = -c softplus(lambda) <= 0, per channel
//     S <- a S + sqrt(1 - a^2) (i u)                      out = S * gelu_tanh(y)
//   diag_scan_kernel<MODE 0>  whole portions, one thread per channel walking the tokens (single-token steps included)
//   diag_scan_kernel<MODE 1>, diag_carry_kernel, diag_scan_kernel<MODE 3>: long portions as chunks in parallel -- every chunk from
//   zero keeping (product of a, end state), a serial pass over the chunk summaries that leaves every chunk's start state, and
//   every chunk again from its start state writing the output.
//
// Matrix states (per head S [dim, vdim]; query/key head h / (H / G)); one kernel, four rules:
//   gated delta rule            q <- q / sqrt(|q|^2 + 1e-6) * q_scale,  k <- k / sqrt(|k|^2 + 1e-6)
//                               g = exp(rate_h softplus(a_t + dt_bias_h)),  beta = sigmoid(b_t)
//                               S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   delta rule, channel decays  the same with g per (head, key channel) on the rows of S
//   gated linear attention      S <- diag(g) S + k (q_scale q, k as they are) v^T;  o = S^T q;  g per (head, key channel)
//   scalar linear attention     S <- g S + w k v^T  (q_scale q, k as they are);  o = S^T q;  g and w one number per head: either
//                               w = softplus(a_t + bias_h), g = exp(rate_h w) (a state-space step), or log g and w ready-made (a
//                               matrix memory with exponential gates, mlstm_gates_kernel).  `ones`: one more state column whose
//                               value is always 1, the running sum of weighted keys that normalises the read-out
//   Channel decays are g = exp(rate_h softplus(sign (a + bias))): sign 1 is the softplus form; sigmoid(z)^(1 / tau) is rate
//   -1 / tau with sign -1.  Columns of S are independent: a lane group owns one or two of them and walks the tokens.
#include "state_common.cuh"

namespace {

__device__ __forceinline__ float gelu_tanh1_(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

// gates: fp32 [blocks, rows, 2 * cb]: for block b and token row t the cb pre-activations of r, then those of i.
template <typename T, int MODE>
__global__ void __launch_bounds__(128) diag_scan_kernel(const T* __restrict__ u, int64_t u_stride, const float* __restrict__ gates, int64_t rows,
                                                        const float* __restrict__ gate_bias, const float* __restrict__ rate,
                                                        const T* __restrict__ y, int64_t y_stride, float* __restrict__ state,
                                                        const int32_t* __restrict__ state_slots, const int32_t* __restrict__ cu_q,
                                                        const int32_t* __restrict__ cu_k, const int32_t* __restrict__ ctx_lens,
                                                        T* __restrict__ out, int channels, int cb, int chunk_len, int nchunks,
                                                        float* __restrict__ ws) {
    B200_PDL_SYNC();
    const int s = blockIdx.y;
    const SeqSpan sp = seq_span(cu_q, cu_k, ctx_lens, s);
    if (sp.qlen <= 0) return;
    const int i_begin = MODE == 0 ? 0 : blockIdx.z * chunk_len;
    if (i_begin >= sp.qlen) return;
    const int i_end = MODE == 0 ? sp.qlen : min(sp.qlen, i_begin + chunk_len);
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int b = c / cb, j = c - b * cb;
    const float br = gate_bias[(int64_t)b * 2 * cb + j], bi = gate_bias[(int64_t)b * 2 * cb + cb + j], rt = rate[c];
    const float* gb = gates + (int64_t)b * rows * 2 * cb + j;
    float* st = state + (int64_t)state_slots[s] * channels + c;
    float* wsp = ws ? ws + (((int64_t)s * nchunks + blockIdx.z) * channels + c) * 2 : nullptr;
    float S = 0.f, P = 1.f;
    if (MODE == 0) S = (sp.klen - sp.qlen > 0) ? *st : 0.f;
    if (MODE == 3) S = wsp[0];
    constexpr int TB = 4;                                    // tokens whose operands are fetched before their (serial) arithmetic
    for (int i0 = i_begin; i0 < i_end; i0 += TB) {
        float uu[TB], gr[TB], gi[TB], yy[TB];
#pragma unroll
        for (int k = 0; k < TB; ++k) {
            const int64_t row = sp.q0 + min(i0 + k, i_end - 1);
            uu[k] = ldf(u + row * u_stride + c);
            gr[k] = gb[row * 2 * cb];
            gi[k] = gb[row * 2 * cb + cb];
            yy[k] = MODE == 1 ? 0.f : ldf(y + row * y_stride + c);
        }
#pragma unroll
        for (int k = 0; k < TB; ++k) {
            if (i0 + k >= i_end) break;
            const float la = rt * sigmoidf_(gr[k] + br);     // log a <= 0
            const float a = expf(la);
            const float drive = sqrtf(-expm1f(2.0f * la)) * sigmoidf_(gi[k] + bi) * uu[k];
            S = fmaf(a, S, drive);
            if (MODE == 1) P *= a;
            else stf(out + (int64_t)(sp.q0 + i0 + k) * channels + c, S * gelu_tanh1_(yy[k]));
        }
    }
    if (MODE == 0) *st = S;
    if (MODE == 1) {
        wsp[0] = P;
        wsp[1] = S;
    }
}

// ws[s, z, c] = (product of a over chunk z, end state of chunk z from zero) -> ws[s, z, c, 0] = state at the start of chunk z
__global__ void __launch_bounds__(128) diag_carry_kernel(float* __restrict__ ws, float* __restrict__ state, const int32_t* __restrict__ state_slots,
                                                         const int32_t* __restrict__ cu_q, const int32_t* __restrict__ cu_k,
                                                         const int32_t* __restrict__ ctx_lens, int channels, int chunk_len, int nchunks) {
    B200_PDL_SYNC();
    const int s = blockIdx.y;
    const SeqSpan sp = seq_span(cu_q, cu_k, ctx_lens, s);
    if (sp.qlen <= 0) return;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    float* st = state + (int64_t)state_slots[s] * channels + c;
    float S = (sp.klen - sp.qlen > 0) ? *st : 0.f;
    const int used = (sp.qlen + chunk_len - 1) / chunk_len;
    for (int z = 0; z < used; ++z) {
        float* w = ws + (((int64_t)s * nchunks + z) * channels + c) * 2;
        const float P = w[0], E = w[1];
        w[0] = S;
        S = fmaf(P, S, E);
    }
    *st = S;
}

// Matrix-state recurrences.  LANES lanes share COLS columns of a head's state: lane `sub` of a group owns rows sub * DPL ..
// sub * DPL + DPL - 1 of them (zero beyond dim) in registers; a CTA covers MS_THREADS / LANES * COLS columns of one (sequence, head).
// state: [slots, H, vdim, dim] (a column's rows are contiguous).
//   CH    : decays come per (head, key channel) as rows of decay_in instead of one number per (token, head)
//   DELTA : delta rule (unit-norm q and k, write strength, correction towards v); otherwise S <- g S + k v^T with q and k as they are
// Tokens are staged through shared memory TB at a time, as fp32: the chunk after the current one is fetched into registers
// before the current one is worked on and stored afterwards (two buffers), so the serial walk never waits for global memory.
// A staged row is LANES segments of DPL floats, each padded by four: 128-bit reads without bank conflicts.  After a chunk
// lands, MS_THREADS / TB threads per token form its unit-norm factors and k . q once for the CTA.  The delta rule reads out
// before it writes, o = (g S)^T q + u (k . q), so that both column sums of a token are reduced together.
constexpr int MS_THREADS = 128;
constexpr int MS_CHUNK_MIN = 16;       // longest portion up to which a step of scalar linear attention stays off the tensor cores

struct DecayIn {
    const float* in;          // pre-activations, CH: [n, >= H * dim], else one per head.  (The token-at-a-time kernel reads CH decays ready-made.)
    int64_t stride;
    const float* rate;        // [H]
    const float* bias;        // CH: [H * dim], else [H]
    float sign;               // g = exp(rate_h * softplus(sign * (in + bias)))
};
__device__ __forceinline__ float decay_of(float a, float rate, float bias, float sign) { return expf(rate * softplus_(sign * (a + bias))); }

template <typename T, int DPL, int LANES, int COLS, bool CH, bool DELTA>
__global__ void __launch_bounds__(MS_THREADS) matrix_state_kernel(
    const T* __restrict__ x, int64_t stride, int q_off, int k_off, int v_off,     // per token: q, k [G, dim], v [H, vdim]
    const float* __restrict__ write_in, const T* __restrict__ write_t, int64_t write_stride,      // DELTA: H write strengths (pre-activation), fp32 or T
    DecayIn dec, ScalarGate<T> sg, float* __restrict__ state, const int32_t* __restrict__ state_slots, const int32_t* __restrict__ cu_q,
    const int32_t* __restrict__ cu_k, const int32_t* __restrict__ ctx_lens, float* __restrict__ out,      // [n, H, vcols] fp32
    int H, int G, int dim, int vdim, int ones, float q_scale) {
    B200_PDL_SYNC();
    constexpr bool LIN = !CH && !DELTA;
    const int vcols = LIN ? vdim + ones : vdim;            // columns of the state
    constexpr int NT = MS_THREADS, GC = NT / LANES * COLS;  // columns of the CTA
    constexpr int DP = LANES * DPL, SEG = DPL + 4, ROW = LANES * SEG;
    constexpr int TB = DP >= 256 ? 4 : (DP >= 128 || CH) ? 8 : 16;
    constexpr int PF = (TB * DP + NT - 1) / NT;            // key (query, decay) elements a thread fetches per chunk
    constexpr int PV = (TB * GC + NT - 1) / NT;            // value elements a thread fetches per chunk
    constexpr int TPT = NT / TB < 32 ? NT / TB : 32;       // threads that share one token's factors
    __shared__ __align__(16) float ks[2][TB][ROW];
    __shared__ __align__(16) float qs[2][TB][ROW];
    __shared__ __align__(16) float gs[CH ? 2 : 1][CH ? TB : 1][CH ? ROW : 4];
    __shared__ __align__(16) float vs[2][TB][GC];
    __shared__ __align__(16) float sc[2][TB][4];           // key normaliser, query normaliser * scale, write strength, (k . q) of the unit keys and scaled queries
    __shared__ float sd[2][TB];                            // decay per token (not CH)
    const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
    const SeqSpan sp = seq_span(cu_q, cu_k, ctx_lens, s);
    if (sp.qlen <= 0) return;
    const int sub = tid % LANES, grp = tid / LANES;
    const int col0 = blockIdx.z * GC, mycol = col0 + grp * COLS;
    const int g = h / (H / G);
    float* st = state + ((int64_t)state_slots[s] * H + h) * vcols * dim + sub * DPL;     // + column * dim
    const bool has_hist = sp.klen - sp.qlen > 0;
    const bool vec_state = dim % 4 == 0;                    // 16-byte aligned segments: 128-bit state accesses
    float S[COLS][DPL];
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
        const bool have = has_hist && mycol + c < vcols;
        const float* sr = st + (int64_t)(mycol + c) * dim;
        if (vec_state) {
#pragma unroll
            for (int k = 0; k < DPL / 4; ++k) {
                float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
                if (have && sub * DPL + 4 * k < dim) f = reinterpret_cast<const float4*>(sr)[k];
                S[c][4 * k] = f.x, S[c][4 * k + 1] = f.y, S[c][4 * k + 2] = f.z, S[c][4 * k + 3] = f.w;
            }
        } else {
#pragma unroll
            for (int k = 0; k < DPL; ++k) S[c][k] = (have && sub * DPL + k < dim) ? sr[k] : 0.f;
        }
    }
    const float* rate = LIN ? sg.rate : dec.rate;
    const float rt = (CH || rate == nullptr) ? 0.f : rate[h], db = (CH || rate == nullptr) ? 0.f : (LIN ? sg.bias : dec.bias)[h];
    const T* qp = x + q_off + (int64_t)g * dim;
    const T* kp = x + k_off + (int64_t)g * dim;
    const T* vp = x + v_off + (int64_t)h * vdim + col0;
    const float* gp = CH ? dec.in + (int64_t)h * dim : dec.in + h;
    float fk[PF], fq[PF], fg[CH ? PF : 1], fv[PV], fb = 0.f, fa = 0.f;      // the next chunk, in flight
    auto fetch = [&](int i0) {
#pragma unroll
        for (int j = 0; j < PF; ++j) {
            const int e = tid + NT * j, t = e / DP, d = e - t * DP;
            const bool ok = t < TB && i0 + t < sp.qlen && d < dim;
            const int64_t row = sp.q0 + i0 + t;
            fk[j] = ok ? ldf(kp + row * stride + d) : 0.f;
            fq[j] = ok ? ldf(qp + row * stride + d) : 0.f;
            if constexpr (CH) fg[j] = ok ? gp[row * dec.stride + d] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < PV; ++j) {
            const int e = tid + NT * j, t = e / GC, c = e - t * GC;
            fv[j] = (t < TB && i0 + t < sp.qlen && col0 + c < vdim) ? ldf(vp + (int64_t)(sp.q0 + i0 + t) * stride + c) : 0.f;
            if (LIN && ones && col0 + c == vdim) fv[j] = 1.0f;
        }
        if (tid < TB && i0 + tid < sp.qlen) {
            const int64_t row = sp.q0 + i0 + tid;
            if constexpr (DELTA) fb = write_in ? write_in[row * write_stride + h] : ldf(write_t + row * write_stride + h);
            if constexpr (LIN) {
                const float2 f = sg.fetch(row, h);
                fa = f.x, fb = f.y;
            } else if constexpr (!CH) {
                fa = gp[row * dec.stride];
            }
        }
    };
    auto land = [&](int buf) {                             // registers -> shared memory
#pragma unroll
        for (int j = 0; j < PF; ++j) {
            const int e = tid + NT * j, t = e / DP, d = e - t * DP;
            if (t >= TB) break;
            const int at = (d / DPL) * SEG + (d % DPL);
            ks[buf][t][at] = fk[j];
            qs[buf][t][at] = DELTA ? fq[j] : fq[j] * q_scale;
            if constexpr (CH) gs[buf][t][at] = fg[j];      // zero beyond dim
        }
#pragma unroll
        for (int j = 0; j < PV; ++j) {
            const int e = tid + NT * j;
            if (e < TB * GC) vs[buf][e / GC][e % GC] = fv[j];
        }
        if (tid < TB) {
            if constexpr (DELTA) sc[buf][tid][2] = sigmoidf_(fb);
            if constexpr (LIN) {
                const float2 f = sg.gates(make_float2(fa, fb), rt, db);
                sd[buf][tid] = expf(f.x);
                sc[buf][tid][2] = f.y;
            } else if constexpr (!CH) {
                sd[buf][tid] = decay_of(fa, rt, db, dec.sign);
            }
        }
    };
    auto factors = [&](int buf) {                          // after a barrier: the unit-norm factors and k . q of the chunk's tokens
        if constexpr (DELTA) {
            const int t = tid / TPT, j = tid % TPT;
            float ssk = 0.f, ssq = 0.f, skq = 0.f;
            if (t < TB)
                for (int d = j; d < DP; d += TPT) {
                    const int at = (d / DPL) * SEG + (d % DPL);
                    const float a = ks[buf][t][at], b = qs[buf][t][at];
                    ssk = fmaf(a, a, ssk);
                    ssq = fmaf(b, b, ssq);
                    skq = fmaf(a, b, skq);
                }
#pragma unroll
            for (int o = 1; o < TPT; o <<= 1) {
                ssk += __shfl_xor_sync(0xffffffffu, ssk, o);
                ssq += __shfl_xor_sync(0xffffffffu, ssq, o);
                skq += __shfl_xor_sync(0xffffffffu, skq, o);
            }
            if (j == 0 && t < TB) {
                const float rk = 1.0f / sqrtf(ssk + 1e-6f), rq = q_scale / sqrtf(ssq + 1e-6f);
                sc[buf][t][0] = rk;
                sc[buf][t][1] = rq;
                sc[buf][t][3] = skq * rq;                  // times u (which carries the key's normaliser): what the token's own write adds to its read-out
            }
        }
    };
    // Column sums over the group's lanes.  COLS = 2: the first exchange sends one column each way, after which even lanes carry
    // column 0 and odd lanes column 1.
    auto reduce = [&](float (&v)[COLS]) -> float {
        if constexpr (COLS == 2) {
            const bool odd = sub & 1;
            float r = (odd ? v[1] : v[0]) + __shfl_xor_sync(0xffffffffu, odd ? v[0] : v[1], 1);
#pragma unroll
            for (int o = 2; o < LANES; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
            return r;
        } else {
            float r = v[0];
#pragma unroll
            for (int o = 1; o < LANES; o <<= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
            return r;
        }
    };
    const int ocol = mycol + (COLS == 2 ? (sub & 1) : 0);  // the column whose sum this lane holds after reduce()
    const bool writer = sub < COLS && ocol < vcols;
    fetch(0);
    land(0);
    __syncthreads();
    factors(0);
    __syncthreads();
    for (int i0 = 0, buf = 0; i0 < sp.qlen; i0 += TB, buf ^= 1) {
        const bool more = i0 + TB < sp.qlen;
        if (more) fetch(i0 + TB);
        const int nt = min(TB, sp.qlen - i0);
        for (int t = 0; t < nt; ++t) {
            const float4* kr = reinterpret_cast<const float4*>(&ks[buf][t][sub * SEG]);
            const float4* qr = reinterpret_cast<const float4*>(&qs[buf][t][sub * SEG]);
            const float4* gr = reinterpret_cast<const float4*>(&gs[CH ? buf : 0][CH ? t : 0][CH ? sub * SEG : 0]);
            const float gt = CH ? 0.f : sd[buf][t];
            float v[COLS], o[COLS];
#pragma unroll
            for (int c = 0; c < COLS; ++c) {
                v[c] = vs[buf][t][grp * COLS + c];
                if constexpr (LIN) v[c] *= sc[buf][t][2];
                o[c] = 0.f;
            }
            if constexpr (DELTA) {
                float4 kk[DPL / 4];
                float d[COLS];
#pragma unroll
                for (int c = 0; c < COLS; ++c) d[c] = 0.f;
#pragma unroll
                for (int k = 0; k < DPL / 4; ++k) {
                    kk[k] = kr[k];
                    const float4 qq = qr[k];
                    const float4 gg = CH ? gr[k] : make_float4(gt, gt, gt, gt);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        S[c][4 * k] *= gg.x, S[c][4 * k + 1] *= gg.y, S[c][4 * k + 2] *= gg.z, S[c][4 * k + 3] *= gg.w;
                        d[c] = fmaf(S[c][4 * k], kk[k].x, d[c]), o[c] = fmaf(S[c][4 * k], qq.x, o[c]);
                        d[c] = fmaf(S[c][4 * k + 1], kk[k].y, d[c]), o[c] = fmaf(S[c][4 * k + 1], qq.y, o[c]);
                        d[c] = fmaf(S[c][4 * k + 2], kk[k].z, d[c]), o[c] = fmaf(S[c][4 * k + 2], qq.z, o[c]);
                        d[c] = fmaf(S[c][4 * k + 3], kk[k].w, d[c]), o[c] = fmaf(S[c][4 * k + 3], qq.w, o[c]);
                    }
                }
                const float dk = reduce(d), oq = reduce(o);
                const float4 f = *reinterpret_cast<const float4*>(sc[buf][t]);
                const float vo = COLS == 2 ? ((sub & 1) ? v[COLS - 1] : v[0]) : v[0];
                const float ub = f.z * (vo - dk * f.x) * f.x;             // u times the key's normaliser: S += (k rk) u
                if (writer) out[((int64_t)(sp.q0 + i0 + t) * H + h) * vcols + ocol] = fmaf(ub, f.w, oq * f.y);
                float u[COLS];
                if constexpr (COLS == 2) {
                    const float other = __shfl_xor_sync(0xffffffffu, ub, 1);
                    u[0] = (sub & 1) ? other : ub;
                    u[COLS - 1] = (sub & 1) ? ub : other;
                } else {
                    u[0] = ub;
                }
#pragma unroll
                for (int k = 0; k < DPL / 4; ++k)
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        S[c][4 * k] = fmaf(kk[k].x, u[c], S[c][4 * k]);
                        S[c][4 * k + 1] = fmaf(kk[k].y, u[c], S[c][4 * k + 1]);
                        S[c][4 * k + 2] = fmaf(kk[k].z, u[c], S[c][4 * k + 2]);
                        S[c][4 * k + 3] = fmaf(kk[k].w, u[c], S[c][4 * k + 3]);
                    }
            } else {
#pragma unroll
                for (int k = 0; k < DPL / 4; ++k) {
                    const float4 kk = kr[k], qq = qr[k];
                    const float4 gg = CH ? gr[k] : make_float4(gt, gt, gt, gt);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        S[c][4 * k] = fmaf(kk.x, v[c], gg.x * S[c][4 * k]), o[c] = fmaf(S[c][4 * k], qq.x, o[c]);
                        S[c][4 * k + 1] = fmaf(kk.y, v[c], gg.y * S[c][4 * k + 1]), o[c] = fmaf(S[c][4 * k + 1], qq.y, o[c]);
                        S[c][4 * k + 2] = fmaf(kk.z, v[c], gg.z * S[c][4 * k + 2]), o[c] = fmaf(S[c][4 * k + 2], qq.z, o[c]);
                        S[c][4 * k + 3] = fmaf(kk.w, v[c], gg.w * S[c][4 * k + 3]), o[c] = fmaf(S[c][4 * k + 3], qq.w, o[c]);
                    }
                }
                const float oq = reduce(o);
                if (writer) out[((int64_t)(sp.q0 + i0 + t) * H + h) * vcols + ocol] = oq;
            }
        }
        if (more) {
            land(buf ^ 1);                                 // its last readers passed the barrier that closed the previous chunk
            __syncthreads();
            factors(buf ^ 1);
            __syncthreads();
        }
    }
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
        if (mycol + c >= vcols) break;
        float* sr = st + (int64_t)(mycol + c) * dim;
        if (vec_state) {
#pragma unroll
            for (int k = 0; k < DPL / 4; ++k)
                if (sub * DPL + 4 * k < dim)
                    reinterpret_cast<float4*>(sr)[k] = make_float4(S[c][4 * k], S[c][4 * k + 1], S[c][4 * k + 2], S[c][4 * k + 3]);
        } else {
#pragma unroll
            for (int k = 0; k < DPL; ++k)
                if (sub * DPL + k < dim) sr[k] = S[c][k];
        }
    }
}

// Decay pre-activations -> decays, in place: a[t, h, c] <- exp(rate[h] * softplus(sign * (a + bias[h, c]))).  In front of the
// token-at-a-time kernel, whose column tiles would otherwise each form a head's decays on their critical path.
__global__ void __launch_bounds__(256) channel_decay_kernel(float* __restrict__ a, int64_t stride, const float* __restrict__ rate,
                                                            const float* __restrict__ bias, float sign, int cols, int dim) {
    B200_PDL_SYNC();
    const int64_t t = blockIdx.x;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < cols; c += gridDim.y * blockDim.x) {
        float* p = a + t * stride + c;
        *p = decay_of(*p, rate[c / dim], bias[c], sign);
    }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Prompt portions: the same rules four tokens at a time.  With P_t = g_1 ... g_t the products of a block's decays (per channel) and
// R_s = g_(s+1) ... g_4, and S the state before the block,
//     d_t = S^T (P_t k_t),  o'_t = S^T (P_t q_t),  A_ts = (R-weighted) k_s g_(s+1)..g_t . k_t,  B_ts likewise with q_t
//     u_t = beta_t (v_t - d_t - sum_(s<t) A_ts u_s)       (linear attention: u_t = v_t)
//     o_t = o'_t + sum_(s<=t) B_ts u_s,       S <- P_4 S + sum_s (R_s k_s) u_s
// which is the token-by-token recurrence regrouped: only products of decays (never quotients), everything in fp32.  Four producer
// warps form the scaled vectors and the small coefficient sets, a block each, up to two stages of sixteen tokens ahead; four consumer
// warps hold the state (eight lanes x COLS columns, packed pairs of fp32 in 64-bit registers for the two-wide FMA) and do the four
// tokens' column sums in one shuffle tree.  The two sides meet at named barriers (full / empty per stage).
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int MB_T = 4, MB_BLOCKS = 4, MB_STAGE = MB_T * MB_BLOCKS, MB_LANES = 8, MB_THREADS = 256;

__device__ __forceinline__ uint64_t fma2_(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul2_(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t pack2_(float lo, float hi) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 unpack2_(uint64_t v) {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
    return f;
}
template <int ID0>
__device__ __forceinline__ void named_sync(int s) {       // barrier ID0 or ID0 + 1 (as constants: a barrier number in a register reserves all sixteen)
    if (s == 0) asm volatile("bar.sync %0, %1;" ::"n"(ID0), "n"(MB_THREADS) : "memory");
    else asm volatile("bar.sync %0, %1;" ::"n"(ID0 + 1), "n"(MB_THREADS) : "memory");
}
template <int ID0>
__device__ __forceinline__ void named_arrive(int s) {
    if (s == 0) asm volatile("bar.arrive %0, %1;" ::"n"(ID0), "n"(MB_THREADS) : "memory");
    else asm volatile("bar.arrive %0, %1;" ::"n"(ID0 + 1), "n"(MB_THREADS) : "memory");
}

// N consecutive elements as 32-bit words (two bf16 or one float each), without conversion, so that a load stays in flight until its use
template <typename T, int N>
struct RawCols {
    static constexpr int W = (N * (int)sizeof(T) + 3) / 4;
    uint32_t w[W];
    __device__ __forceinline__ void zero() {
#pragma unroll
        for (int i = 0; i < W; ++i) w[i] = 0;
    }
    __device__ __forceinline__ void load(const T* p, int avail, bool vec) {      // the first `avail` elements; vec: all or none, aligned
        zero();
        if (vec) {
            if (avail <= 0) return;
            if constexpr (N * sizeof(T) == 4) w[0] = *reinterpret_cast<const uint32_t*>(p);
            else if constexpr (N * sizeof(T) == 8) *reinterpret_cast<uint2*>(w) = *reinterpret_cast<const uint2*>(p);
            else if constexpr (N * sizeof(T) % 16 == 0) {
#pragma unroll
                for (int i = 0; i < W / 4; ++i) {
                    const uint4 v = reinterpret_cast<const uint4*>(p)[i];
                    w[4 * i] = v.x, w[4 * i + 1] = v.y, w[4 * i + 2] = v.z, w[4 * i + 3] = v.w;
                }
            } else {
                w[0] = *reinterpret_cast<const unsigned short*>(p);
            }
            return;
        }
#pragma unroll
        for (int e = 0; e < N; ++e)
            if (e < avail) {
                if constexpr (sizeof(T) == 4) w[e] = reinterpret_cast<const uint32_t*>(p)[e];
                else w[e / 2] |= (uint32_t)reinterpret_cast<const unsigned short*>(p)[e] << (16 * (e & 1));
            }
    }
    __device__ __forceinline__ float at(int e) const {
        if constexpr (sizeof(T) == 4) return __uint_as_float(w[e]);
        else return (e & 1) ? bf16hi(w[e / 2]) : bf16lo(w[e / 2]);
    }
};

template <int DPL, int COLS>
struct BlockShape {
    static constexpr int DP = MB_LANES * DPL, SEG = DPL + 4, ROW = MB_LANES * SEG, GC = 16 * COLS;
    // one stage: P k, P q, R k rows of its tokens, the blocks' whole decays, values, coefficients (32 per block)
    static constexpr int KD = 0, QD = MB_STAGE * ROW, KR = 2 * MB_STAGE * ROW, PE = 3 * MB_STAGE * ROW, VS = PE + MB_BLOCKS * ROW,
                         CF = VS + MB_STAGE * GC, FLOATS = CF + MB_BLOCKS * 32;
};
// coefficient places of a block: key normalisers, query normalisers (* scale), A (t, s < t), B (t, s <= t), write strengths * key normaliser
constexpr int CF_RK = 0, CF_RQ = 4, CF_A = 8, CF_B = 14, CF_W = 24;

template <typename T, int DPL, int COLS, bool CH, bool DELTA>
__global__ void __launch_bounds__(MB_THREADS, DPL <= 16 ? 2 : 1) matrix_state_block_kernel(
    const T* __restrict__ x, int64_t stride, int q_off, int k_off, int v_off, const float* __restrict__ write_in,
    const T* __restrict__ write_t, int64_t write_stride, DecayIn dec, ScalarGate<T> sg, float* __restrict__ state,
    const int32_t* __restrict__ state_slots, const int32_t* __restrict__ cu_q, const int32_t* __restrict__ cu_k,
    const int32_t* __restrict__ ctx_lens, float* __restrict__ out, int H, int G, int dim, int vdim, int ones, float q_scale, int vec_x, int vec_g) {
    B200_PDL_SYNC();
    constexpr bool LIN = !CH && !DELTA;
    const int vcols = LIN ? vdim + ones : vdim;            // columns of the state
    using SH = BlockShape<DPL, COLS>;
    constexpr int FULL = 1, EMPTY = 3;
    extern __shared__ __align__(16) float mb_smem[];       // two stages
    const int h = blockIdx.x, s = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const SeqSpan sp = seq_span(cu_q, cu_k, ctx_lens, s);
    if (sp.qlen <= 0) return;
    const int nst = (sp.qlen + MB_STAGE - 1) / MB_STAGE;
    const int col0 = blockIdx.z * SH::GC;
    if (warp >= 4) {
        // ---- producers: warp - 4 is the block of a stage, a lane owns CPL consecutive channels ----
        constexpr int CPL = SH::DP / 32;
        const int b = warp - 4, c0 = lane * CPL, avail = dim - c0;
        const int at = (c0 / DPL) * SH::SEG + c0 % DPL;     // CPL <= DPL: a lane's channels stay inside one segment
        const T* qp = x + q_off + (int64_t)(h / (H / G)) * dim + c0;
        const T* kp = x + k_off + (int64_t)(h / (H / G)) * dim + c0;
        const T* vp = x + v_off + (int64_t)h * vdim + col0;
        const float* gp = CH ? dec.in + (int64_t)h * dim + c0 : dec.in + h;
        const float* rate = LIN ? sg.rate : dec.rate;
        const float rt = rate ? rate[h] : 0.f;
        float gb[CH ? CPL : 1];
#pragma unroll
        for (int e = 0; e < (CH ? CPL : 1); ++e)
            gb[e] = CH ? (e < avail ? dec.bias[(int64_t)h * dim + c0 + e] : 0.f) : rate ? (LIN ? sg.bias : dec.bias)[h] : 0.f;
        constexpr int VPL = MB_T * SH::GC / 32;             // value elements of a block per lane
        RawCols<T, CPL> rk[MB_T], rq[MB_T];
        RawCols<float, CH ? CPL : 1> rg[MB_T];
        float2 rs[MB_T];                                    // LIN: the tokens' gate inputs
        RawCols<T, 1> rv[VPL], rw;
        float rwf = 0.f;
        auto fetch = [&](int it) {
            const int i0 = it * MB_STAGE + b * MB_T;
#pragma unroll
            for (int t = 0; t < MB_T; ++t) {
                const int64_t row = sp.q0 + i0 + t;
                const int have = i0 + t < sp.qlen ? avail : 0;
                rk[t].load(kp + row * stride, have, vec_x);
                rq[t].load(qp + row * stride, have, vec_x);
                if constexpr (CH) rg[t].load(gp + row * dec.stride, have, vec_g);
                else if constexpr (LIN) rs[t] = i0 + t < sp.qlen ? sg.fetch(row, h) : make_float2(0.f, 0.f);
                else rg[t].load(gp + row * dec.stride, i0 + t < sp.qlen, false);
            }
#pragma unroll
            for (int j = 0; j < VPL; ++j) {
                const int e = lane + 32 * j, t = e / SH::GC, c = e % SH::GC;
                rv[j].load(vp + (int64_t)(sp.q0 + i0 + t) * stride + c, i0 + t < sp.qlen && col0 + c < vdim, false);
            }
            if constexpr (DELTA) {
                const bool have = lane < MB_T && i0 + lane < sp.qlen;
                const int64_t row = sp.q0 + i0 + lane;
                if (write_in) rwf = have ? write_in[row * write_stride + h] : 0.f;
                else rw.load(write_t + row * write_stride + h, have, false);
            }
        };
        fetch(0);
        for (int it = 0; it < nst; ++it) {
            const int i0 = it * MB_STAGE + b * MB_T, st = it & 1;
            float* sm = mb_smem + st * SH::FLOATS;
            if (it >= 2) named_sync<EMPTY>(st);
            if (i0 < sp.qlen) {
                float sum[32];
#pragma unroll
                for (int i = 0; i < 32; ++i) sum[i] = 0.f;
                float pe[CPL], kd[MB_T][CPL], qd[MB_T][CPL], kr[MB_T][CPL];
                float gt[MB_T], wt[MB_T];                   // LIN: decay and write weight of every token
                if constexpr (LIN) {
#pragma unroll
                    for (int t = 0; t < MB_T; ++t) {
                        const float2 f = sg.gates(rs[t], rt, gb[0]);
                        gt[t] = i0 + t < sp.qlen ? expf(f.x) : 1.f;
                        wt[t] = i0 + t < sp.qlen ? f.y : 0.f;
                    }
                }
#pragma unroll
                for (int e = 0; e < CPL; ++e) {
                    float g[MB_T], k[MB_T], q[MB_T];
#pragma unroll
                    for (int t = 0; t < MB_T; ++t) {
                        k[t] = rk[t].at(e);
                        q[t] = rq[t].at(e);
                        if constexpr (LIN) g[t] = gt[t];
                        else g[t] = i0 + t < sp.qlen ? decay_of(rg[t].at(CH ? e : 0), rt, gb[CH ? e : 0], dec.sign) : 1.f;
                    }
                    float p = 1.f;
#pragma unroll
                    for (int t = 0; t < MB_T; ++t) {
                        p *= g[t];
                        kd[t][e] = p * k[t];
                        qd[t][e] = p * q[t];
                    }
                    pe[e] = p;
#pragma unroll
                    for (int a = 0; a < MB_T; ++a) {
                        float w = k[a];
                        if constexpr (DELTA) {
                            sum[CF_RK + a] = fmaf(k[a], k[a], sum[CF_RK + a]);
                            sum[CF_RQ + a] = fmaf(q[a], q[a], sum[CF_RQ + a]);
                        }
                        sum[CF_B + a * (a + 1) / 2 + a] = fmaf(w, q[a], sum[CF_B + a * (a + 1) / 2 + a]);
#pragma unroll
                        for (int t = a + 1; t < MB_T; ++t) {
                            w *= g[t];
                            if constexpr (DELTA) sum[CF_A + t * (t - 1) / 2 + a] = fmaf(w, k[t], sum[CF_A + t * (t - 1) / 2 + a]);
                            sum[CF_B + t * (t + 1) / 2 + a] = fmaf(w, q[t], sum[CF_B + t * (t + 1) / 2 + a]);
                        }
                        kr[a][e] = w;
                    }
                }
                auto put = [&](float* dst, const float (&v)[CPL]) {
                    if constexpr (CPL % 4 == 0) {
#pragma unroll
                        for (int e = 0; e < CPL; e += 4) *reinterpret_cast<float4*>(dst + e) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
                    } else if constexpr (CPL == 2) {
                        *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
                    } else {
                        dst[0] = v[0];
                    }
                };
#pragma unroll
                for (int t = 0; t < MB_T; ++t) {
                    const int r = (b * MB_T + t) * SH::ROW + at;
                    if constexpr (DELTA) put(sm + SH::KD + r, kd[t]);
                    put(sm + SH::QD + r, qd[t]);
                    put(sm + SH::KR + r, kr[t]);
                }
                put(sm + SH::PE + b * SH::ROW + at, pe);
#pragma unroll
                for (int j = 0; j < VPL; ++j) {
                    const int e = lane + 32 * j;
                    float v = rv[j].at(0);
                    if constexpr (LIN) {
                        if (ones && col0 + e % SH::GC == vdim) v = 1.0f;
                        v *= wt[(32 * j) / SH::GC];             // a warp's 32 values belong to one token
                    }
                    sm[SH::VS + b * MB_T * SH::GC + e] = v;
                }
                // lane i ends with the warp's sum number i
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
                    const bool hi = lane & o;
#pragma unroll
                    for (int i = 0; i < o; ++i) {
                        const float send = hi ? sum[i] : sum[i + o], keep = hi ? sum[i + o] : sum[i];
                        sum[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                    }
                }
                float* cf = sm + SH::CF + b * 32;
                if constexpr (DELTA) {
                    const float r = 1.0f / sqrtf(sum[0] + 1e-6f);
                    if (lane < 4) {
                        const float beta = i0 + lane < sp.qlen ? sigmoidf_(write_in ? rwf : rw.at(0)) : 0.f;
                        cf[CF_RK + lane] = r;
                        cf[CF_W + lane] = beta * r;
                    } else if (lane < 8) {
                        cf[lane] = r * q_scale;
                    } else if (lane < 24) {
                        cf[lane] = sum[0];
                    }
                } else if (lane >= CF_B && lane < CF_B + 10) {
                    cf[lane] = sum[0] * q_scale;
                }
            }
            if (it + 1 < nst) fetch(it + 1);
            named_arrive<FULL>(st);
        }
        return;
    }
    // ---- consumers ----
    const int sub = lane & (MB_LANES - 1), grp = warp * 4 + (lane >> 3);
    const int mycol = col0 + grp * COLS;
    float* stp = state + ((int64_t)state_slots[s] * H + h) * vcols * dim + sub * DPL;
    const bool has_hist = sp.klen - sp.qlen > 0, vec_state = dim % 4 == 0;
    uint64_t S[COLS][DPL / 2];
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
        const bool have = has_hist && mycol + c < vcols;
        const float* sr = stp + (int64_t)(mycol + c) * dim;
#pragma unroll
        for (int k = 0; k < DPL / 4; ++k) {
            float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
            const int d = sub * DPL + 4 * k;
            if (have && vec_state) {
                if (d < dim) f = reinterpret_cast<const float4*>(sr)[k];
            } else if (have) {
                if (d < dim) f.x = sr[4 * k];
                if (d + 1 < dim) f.y = sr[4 * k + 1];
                if (d + 2 < dim) f.z = sr[4 * k + 2];
                if (d + 3 < dim) f.w = sr[4 * k + 3];
            }
            S[c][2 * k] = pack2_(f.x, f.y);
            S[c][2 * k + 1] = pack2_(f.z, f.w);
        }
    }
    // After the shuffle tree a lane holds, for one column, either all four d sums or all four o sums (delta rule), or the o sums
    // of some tokens (linear attention).
    constexpr int KINDS = DELTA ? 2 : 1, COMBOS = COLS * KINDS;          // 8, 4 or 2 sets of four sums
    constexpr int OT = DELTA ? 4 : COMBOS * 4 / 8;                        // linear attention: 16 or 8 sums spread over the eight lanes
    const int own = DELTA ? (sub & (COMBOS - 1)) / 2 : sub / (8 / COLS);   // this lane's column
    const int ocol = mycol + own;
    const bool odd = sub & 1;
    const bool idle = col0 + warp * 4 * COLS >= vcols;      // no column of this warp exists: it only keeps the barriers company
    for (int it = 0; it < nst; ++it) {
        const int st = it & 1, i0 = it * MB_STAGE;
        const float* sm = mb_smem + st * SH::FLOATS;
        named_sync<FULL>(st);
        for (int b = 0; b < MB_BLOCKS && i0 + b * MB_T < sp.qlen && !idle; ++b) {
            const float* cf = sm + SH::CF + b * 32;
            float w[COMBOS][MB_T];
#pragma unroll
            for (int t = 0; t < MB_T; ++t) {
                const float* kd = sm + SH::KD + (b * MB_T + t) * SH::ROW + sub * SH::SEG;
                const float* qd = sm + SH::QD + (b * MB_T + t) * SH::ROW + sub * SH::SEG;
                uint64_t a[COLS][KINDS];
#pragma unroll
                for (int k = 0; k < DPL / 4; ++k) {
                    const ulonglong2 q2 = *reinterpret_cast<const ulonglong2*>(qd + 4 * k);
                    ulonglong2 k2 = q2;
                    if constexpr (DELTA) k2 = *reinterpret_cast<const ulonglong2*>(kd + 4 * k);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        if constexpr (DELTA) {
                            a[c][0] = k == 0 ? mul2_(S[c][0], k2.x) : fma2_(S[c][2 * k], k2.x, a[c][0]);
                            a[c][0] = fma2_(S[c][2 * k + 1], k2.y, a[c][0]);
                        }
                        a[c][KINDS - 1] = k == 0 ? mul2_(S[c][0], q2.x) : fma2_(S[c][2 * k], q2.x, a[c][KINDS - 1]);
                        a[c][KINDS - 1] = fma2_(S[c][2 * k + 1], q2.y, a[c][KINDS - 1]);
                    }
                }
#pragma unroll
                for (int c = 0; c < COLS; ++c)
#pragma unroll
                    for (int n = 0; n < KINDS; ++n) {
                        const float2 f = unpack2_(a[c][n]);
                        w[c * KINDS + n][t] = f.x + f.y;
                    }
            }
            float u[COLS][MB_T];
            const float* vs = sm + SH::VS + b * MB_T * SH::GC + grp * COLS;
            if constexpr (DELTA) {
                if constexpr (COMBOS == 4) {
#pragma unroll
                    for (int i = 0; i < 4; ++i)
#pragma unroll
                        for (int t = 0; t < MB_T; ++t) w[i][t] += __shfl_xor_sync(0xffffffffu, w[i][t], 4);
                }
#pragma unroll
                for (int o = COMBOS / 2; o > 0; o >>= 1) {
                    const bool hi = sub & o;
#pragma unroll
                    for (int i = 0; i < o; ++i)
#pragma unroll
                        for (int t = 0; t < MB_T; ++t) {
                            const float send = hi ? w[i][t] : w[i + o][t], keep = hi ? w[i + o][t] : w[i][t];
                            w[i][t] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                        }
                }
                float mu[MB_T];                            // u times the key's normaliser (correct on the lanes with the d sums)
#pragma unroll
                for (int t = 0; t < MB_T; ++t) {
                    float acc = w[0][t];
#pragma unroll
                    for (int a = 0; a < t; ++a) acc = fmaf(cf[CF_A + t * (t - 1) / 2 + a], mu[a], acc);
                    mu[t] = cf[CF_W + t] * fmaf(-cf[CF_RK + t], acc, vs[t * SH::GC + own]);
                }
#pragma unroll
                for (int t = 0; t < MB_T; ++t)
#pragma unroll
                    for (int c = 0; c < COLS; ++c) u[c][t] = __shfl_sync(0xffffffffu, mu[t], (lane & ~7) | (2 * c));
#pragma unroll
                for (int t = 0; t < MB_T; ++t) {
                    const float e = __shfl_xor_sync(0xffffffffu, mu[t], 1);
                    mu[t] = odd ? e : mu[t];
                }
#pragma unroll
                for (int t = 0; t < MB_T; ++t) {
                    float acc = w[0][t];
#pragma unroll
                    for (int a = 0; a <= t; ++a) acc = fmaf(cf[CF_B + t * (t + 1) / 2 + a], mu[a], acc);
                    const int i = i0 + b * MB_T + t;
                    if (odd && sub < COMBOS && ocol < vcols && i < sp.qlen) out[((int64_t)(sp.q0 + i) * H + h) * vcols + ocol] = acc * cf[CF_RQ + t];
                }
            } else {
#pragma unroll
                for (int t = 0; t < MB_T; ++t)
#pragma unroll
                    for (int c = 0; c < COLS; ++c) u[c][t] = vs[t * SH::GC + c];
                // 4 * COLS sums as eight sets of OT: set number = column * (8 / COLS) + token / OT
                float r[8][OT];
#pragma unroll
                for (int i = 0; i < 8; ++i)
#pragma unroll
                    for (int j = 0; j < OT; ++j) r[i][j] = w[i / (8 / COLS)][(i % (8 / COLS)) * OT + j];
#pragma unroll
                for (int o = 4; o > 0; o >>= 1) {
                    const bool hi = sub & o;
#pragma unroll
                    for (int i = 0; i < o; ++i)
#pragma unroll
                        for (int j = 0; j < OT; ++j) {
                            const float send = hi ? r[i][j] : r[i + o][j], keep = hi ? r[i + o][j] : r[i][j];
                            r[i][j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                        }
                }
                float mv[MB_T];
#pragma unroll
                for (int t = 0; t < MB_T; ++t) mv[t] = vs[t * SH::GC + own];
#pragma unroll
                for (int j = 0; j < OT; ++j) {
                    const int t = (sub % (8 / COLS)) * OT + j, i = i0 + b * MB_T + t;
                    float acc = r[0][j] * q_scale;
#pragma unroll
                    for (int a = 0; a < MB_T; ++a)
                        if (a <= t) acc = fmaf(cf[CF_B + t * (t + 1) / 2 + a], mv[a], acc);
                    if (ocol < vcols && i < sp.qlen) out[((int64_t)(sp.q0 + i) * H + h) * vcols + ocol] = acc;
                }
            }
            const float* pe = sm + SH::PE + b * SH::ROW + sub * SH::SEG;
            const float* kr = sm + SH::KR + b * MB_T * SH::ROW + sub * SH::SEG;
#pragma unroll
            for (int k = 0; k < DPL / 4; ++k) {
                const ulonglong2 p2 = *reinterpret_cast<const ulonglong2*>(pe + 4 * k);
#pragma unroll
                for (int c = 0; c < COLS; ++c) {
                    S[c][2 * k] = mul2_(S[c][2 * k], p2.x);
                    S[c][2 * k + 1] = mul2_(S[c][2 * k + 1], p2.y);
                }
#pragma unroll
                for (int t = 0; t < MB_T; ++t) {
                    const ulonglong2 r2 = *reinterpret_cast<const ulonglong2*>(kr + t * SH::ROW + 4 * k);
#pragma unroll
                    for (int c = 0; c < COLS; ++c) {
                        const uint64_t uu = pack2_(u[c][t], u[c][t]);
                        S[c][2 * k] = fma2_(r2.x, uu, S[c][2 * k]);
                        S[c][2 * k + 1] = fma2_(r2.y, uu, S[c][2 * k + 1]);
                    }
                }
            }
        }
        if (it + 2 < nst) named_arrive<EMPTY>(st);
    }
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
        if (mycol + c >= vcols) break;
        float* sr = stp + (int64_t)(mycol + c) * dim;
#pragma unroll
        for (int k = 0; k < DPL / 4; ++k) {
            const float2 lo = unpack2_(S[c][2 * k]), hi = unpack2_(S[c][2 * k + 1]);
            const int d = sub * DPL + 4 * k;
            if (vec_state) {
                if (d < dim) reinterpret_cast<float4*>(sr)[k] = make_float4(lo.x, lo.y, hi.x, hi.y);
            } else {
                if (d < dim) sr[4 * k] = lo.x;
                if (d + 1 < dim) sr[4 * k + 1] = lo.y;
                if (d + 2 < dim) sr[4 * k + 2] = hi.x;
                if (d + 3 < dim) sr[4 * k + 3] = hi.y;
            }
        }
    }
}

// Scalar linear attention, single-token steps: the state streams through registers once.  LPC lanes share a column (VPL float4s of its dim
// rows each), a warp works on eight columns per lane group at a time, all of whose loads are in flight together; no shared memory.
constexpr int LD_COLS = 8;
template <typename T, int LPC, int VPL>
__global__ void __launch_bounds__(128) linear_state_token_kernel(const T* __restrict__ x, int64_t stride, int q_off, int k_off, int v_off, ScalarGate<T> sg,
                                                                 float* __restrict__ state, const int32_t* __restrict__ state_slots,
                                                                 const int32_t* __restrict__ ctx_lens, float* __restrict__ out, int H, int G, int dim,
                                                                 int vdim, int ones, float q_scale, int vec_x) {
    B200_PDL_SYNC();
    constexpr int GROUPS = 32 / LPC;
    const int h = blockIdx.x, s = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane % LPC;
    const int klen = ctx_lens[s];
    if (klen <= 0) return;                                  // padding row
    const int vcols = vdim + ones, col0 = (blockIdx.z * 4 + warp) * LD_COLS * GROUPS + lane / LPC;
    if ((blockIdx.z * 4 + warp) * LD_COLS * GROUPS >= vcols) return;
    float* st = state + ((int64_t)state_slots[s] * H + h) * vcols * dim;
    float4 S[LD_COLS][VPL];
#pragma unroll
    for (int i = 0; i < LD_COLS; ++i)
#pragma unroll
        for (int j = 0; j < VPL; ++j) {
            const int col = col0 + i * GROUPS, d = (j * LPC + sub) * 4;
            S[i][j] = klen > 1 && col < vcols && d < dim ? *reinterpret_cast<const float4*>(st + (int64_t)col * dim + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    const T* xr = x + (int64_t)s * stride;
    const float2 f = sg.gates(sg.fetch(s, h), sg.rate ? sg.rate[h] : 0.f, sg.rate ? sg.bias[h] : 0.f);
    const float g = expf(f.x), w = f.y;
    float k[VPL][4], q[VPL][4], v[LD_COLS], o[LD_COLS];
#pragma unroll
    for (int j = 0; j < VPL; ++j) {
        const int d = (j * LPC + sub) * 4;
        RawCols<T, 4> rk, rq;
        rk.load(xr + k_off + (int64_t)(h / (H / G)) * dim + d, dim - d, vec_x);
        rq.load(xr + q_off + (int64_t)(h / (H / G)) * dim + d, dim - d, vec_x);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            k[j][e] = rk.at(e);
            q[j][e] = rq.at(e) * q_scale;
        }
    }
#pragma unroll
    for (int i = 0; i < LD_COLS; ++i) {
        const int col = col0 + i * GROUPS;
        v[i] = w * (col < vdim ? ldf(xr + v_off + (int64_t)h * vdim + col) : 1.0f);        // the column behind the values holds ones
        o[i] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < LD_COLS; ++i)
#pragma unroll
        for (int j = 0; j < VPL; ++j) {
            const int col = col0 + i * GROUPS, d = (j * LPC + sub) * 4;
            float4& t = S[i][j];
            t.x = fmaf(k[j][0], v[i], g * t.x), t.y = fmaf(k[j][1], v[i], g * t.y), t.z = fmaf(k[j][2], v[i], g * t.z), t.w = fmaf(k[j][3], v[i], g * t.w);
            o[i] = fmaf(t.x, q[j][0], fmaf(t.y, q[j][1], fmaf(t.z, q[j][2], fmaf(t.w, q[j][3], o[i]))));
            if (col < vcols && d < dim) *reinterpret_cast<float4*>(st + (int64_t)col * dim + d) = t;
        }
    // eight sums over LPC lanes: three steps halve the sums a lane carries, the rest add up the one that is left
    int own = 0;
#pragma unroll
    for (int n = LD_COLS / 2, off = LPC / 2; off > 0; n >>= 1, off >>= 1) {
        if (n > 0) {
            const bool hi = sub & off;
            own += hi ? n : 0;
#pragma unroll
            for (int i = 0; i < LD_COLS / 2; ++i)
                if (i < n) {
                    const float send = hi ? o[i] : o[i + n], keep = hi ? o[i + n] : o[i];
                    o[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
                }
        } else {
            o[0] += __shfl_xor_sync(0xffffffffu, o[0], off);
        }
    }
    const int col = col0 + own * GROUPS;
    if ((sub & (LPC / LD_COLS - 1)) == 0 && col < vcols) out[((int64_t)s * H + h) * vcols + col] = o[0];
}

template <typename T, bool CH, bool DELTA>
int launch_matrix_state(const void* x, int64_t stride, int q_off, int k_off, int v_off, const float* write_in, const void* write_t,
                        int64_t write_stride, const DecayIn& dec, float* state, const int32_t* state_slots, const int32_t* cu_q,
                        const int32_t* cu_k, const int32_t* ctx_lens, float* out, int total_rows, int num_seqs, int max_q, int H, int G, int dim,
                        int vdim, float q_scale, cudaStream_t st, const ScalarGate<T>& sg = {}, int ones = 0) {
    if (dim > 256) return B200_EUNSUPPORTED;
    const int vcols = vdim + ones;
#define MB_GO(DPL, COLS)                                                                                                           \
    do {                                                                                                                           \
        using SH = BlockShape<DPL, COLS>;                                                                                          \
        constexpr int CPL = SH::DP / 32;                                                                                           \
        const size_t smem = sizeof(float) * 2 * SH::FLOATS;                                                                        \
        static B200SmemOptIn opt;                                                                                                  \
        if (opt.ensure(matrix_state_block_kernel<T, DPL, COLS, CH, DELTA>, smem) != cudaSuccess) return B200_ECUDA;                \
        const int vx = dim % CPL == 0 && stride % CPL == 0 && q_off % CPL == 0 && k_off % CPL == 0 &&                              \
                       reinterpret_cast<uintptr_t>(x) % 16 == 0;                                                                   \
        const int vg = CH && dim % CPL == 0 && dec.stride % (CPL < 4 ? CPL : 4) == 0 && reinterpret_cast<uintptr_t>(dec.in) % 16 == 0;  \
        B200_LAUNCH((matrix_state_block_kernel<T, DPL, COLS, CH, DELTA>), dim3(H, num_seqs, (vcols + SH::GC - 1) / SH::GC), MB_THREADS, \
                    smem, st, static_cast<const T*>(x), stride, q_off, k_off, v_off, write_in, static_cast<const T*>(write_t),     \
                    write_stride, dec, sg, state, state_slots, cu_q, cu_k, ctx_lens, out, H, G, dim, vdim, ones, q_scale, vx, vg); \
        return b200_launch_status(nullptr);                                                                                        \
    } while (0)
    if (cu_q != nullptr && max_q > MB_T) {                  // prompt portions: four tokens at a time
        if (dim <= 32) MB_GO(4, 4);
        if (dim <= 64) MB_GO(8, 4);
        if (dim <= 128) MB_GO(16, 4);
        MB_GO(32, 2);
    }
#undef MB_GO
    if constexpr (!CH && !DELTA) {
        if (cu_q == nullptr && dim % 4 == 0) {
            const int vx = (stride | q_off | k_off) % 4 == 0 && reinterpret_cast<uintptr_t>(x) % 16 == 0;
#define LS_GO(LPC, VPL)                                                                                                            \
    do {                                                                                                                           \
        constexpr int CC = 4 * LD_COLS * (32 / LPC);                                                                               \
        B200_LAUNCH((linear_state_token_kernel<T, LPC, VPL>), dim3(H, num_seqs, (vcols + CC - 1) / CC), 128, 0, st, static_cast<const T*>(x), stride, \
                    q_off, k_off, v_off, sg, state, state_slots, ctx_lens, out, H, G, dim, vdim, ones, q_scale, vx);                \
        return b200_launch_status(nullptr);                                                                                        \
    } while (0)
            if (dim <= 32) LS_GO(8, 1);
            if (dim <= 64) LS_GO(16, 1);
            if (dim <= 128) LS_GO(32, 1);
            LS_GO(32, 2);
#undef LS_GO
        }
    }
    if constexpr (CH) {
        const int cols = H * dim, rows = cu_q ? total_rows : num_seqs;
        B200_LAUNCH((channel_decay_kernel), dim3(rows, (unsigned)((cols + 1023) / 1024)), 256, 0, st, const_cast<float*>(dec.in), dec.stride,
                    dec.rate, dec.bias, dec.sign, cols, dim);
        const int rc = b200_launch_status(nullptr);
        if (rc != B200_OK) return rc;
    }
#define MS_GO(DPL, LANES, COLS)                                                                                                    \
    do {                                                                                                                           \
        constexpr int GC = MS_THREADS / LANES * COLS;                                                                              \
        B200_LAUNCH((matrix_state_kernel<T, DPL, LANES, COLS, CH, DELTA>), dim3(H, num_seqs, (vcols + GC - 1) / GC), MS_THREADS, 0, st, \
                    static_cast<const T*>(x), stride, q_off, k_off, v_off, write_in, static_cast<const T*>(write_t), write_stride, dec, \
                    sg, state, state_slots, cu_q, cu_k, ctx_lens, out, H, G, dim, vdim, ones, q_scale);                             \
        return b200_launch_status(nullptr);                                                                                        \
    } while (0)
    if (dim <= 16) MS_GO(4, 4, 1);
    if (dim <= 32) MS_GO(4, 8, 2);
    if (dim <= 64) MS_GO(8, 8, 2);
    if (dim <= 128) MS_GO(16, 8, 2);
    if (dim <= 256) MS_GO(32, 8, 2);
#undef MS_GO
    return B200_EUNSUPPORTED;
}

// Exponential gates of a matrix memory: from pre-activations (i | f) of H heads each, i <- cap tanh((i + b) / cap), f <- logsigmoid(cap
// tanh((f + b) / cap)), the running maximum m_t = max(f_t + m_(t-1), i_t) (from 0 for a new sequence), and with it
//     log_decay = f_t + m_(t-1) - m_t,   write = exp(i_t - m_t),   floor = exp(-m_t)                        (all fp32)
// One CTA of NW warps per (sequence, head), a token per thread and step: (f, i) pairs compose as (f1 + f2, max(i1 + f2, i2)), a scan over
// the lanes and then over the warps.
template <int NW>
__global__ void __launch_bounds__(NW * 32) mlstm_gates_kernel(const float* __restrict__ in, int64_t stride, const float* __restrict__ bias, float cap,
                                                              float* __restrict__ mstate, const int32_t* __restrict__ state_slots,
                                                              const int32_t* __restrict__ cu_q, const int32_t* __restrict__ cu_k,
                                                              const int32_t* __restrict__ ctx_lens, float* __restrict__ log_decay,
                                                              float* __restrict__ write, float* __restrict__ flr, int H) {
    B200_PDL_SYNC();
    __shared__ float2 part[2][NW];                          // (F, I) of every warp's tokens, double-buffered over the steps
    const int s = blockIdx.y, h = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const SeqSpan sp = seq_span(cu_q, cu_k, ctx_lens, s);
    if (sp.qlen <= 0) return;
    float* mp = mstate + (int64_t)state_slots[s] * H + h;
    float m = sp.klen - sp.qlen > 0 ? *mp : 0.f;
    const float bi = bias[h], bf = bias[H + h];
    float ri = 0.f, rf = 0.f;
    auto fetch = [&](int i) {
        if (i < sp.qlen) {
            const float* row = in + (int64_t)(sp.q0 + i) * stride + h;
            ri = row[0], rf = row[H];
        }
    };
    fetch(threadIdx.x);
    for (int i0 = 0, buf = 0; i0 < sp.qlen; i0 += NW * 32, buf ^= 1) {
        const int i = i0 + threadIdx.x;
        const bool ok = i < sp.qlen;                         // past the end: nothing is added and the maximum stays
        const float gi = ok ? cap * tanhf((ri + bi) / cap) : -INFINITY, gf = ok ? -softplus_(-cap * tanhf((rf + bf) / cap)) : 0.f;
        fetch(i + NW * 32);
        float F = gf, I = gi;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pf = __shfl_up_sync(0xffffffffu, F, o), pi = __shfl_up_sync(0xffffffffu, I, o);
            if (lane >= o) {
                I = fmaxf(pi + F, I);
                F += pf;
            }
        }
        if constexpr (NW > 1) {
            if (lane == 31) part[buf][warp] = make_float2(F, I);
            __syncthreads();
        }
        float prev = m;                                      // maximum before this warp's tokens
        if constexpr (NW > 1) {
#pragma unroll
            for (int w = 0; w < NW; ++w) {
                const float2 p = part[buf][w];
                m = fmaxf(p.x + m, p.y);
                if (w + 1 == warp) prev = m;
            }
        }
        const float mt = fmaxf(F + prev, I);
        const float up = __shfl_up_sync(0xffffffffu, mt, 1);
        if (lane > 0) prev = up;
        if constexpr (NW == 1) m = __shfl_sync(0xffffffffu, mt, 31);
        if (ok) {
            const int64_t at = (int64_t)(sp.q0 + i) * H + h;
            log_decay[at] = gf + prev - mt;
            write[at] = expf(gi - mt);
            flr[at] = expf(-mt);
        }
    }
    if (threadIdx.x == 0) *mp = m;
}

// out[t, h, :] = c * o / sqrt(mean(o^2) + eps) * w * act(gate[t, h, :]) for o = x[t, h, :] (fp32), one warp per (token, head).
// act 0: sigmoid, 1: silu.  w (optional): [vdim], shared by the heads, or (w_heads) [H * vdim].  flr (optional, [n, H]): rows of x have one
// more element z, and o is first divided by max(|z|, flr) + 1e-6.
template <typename T, int PER>
__global__ void __launch_bounds__(128) head_rmsnorm_gate_kernel(const float* __restrict__ x, const float* __restrict__ flr, const T* __restrict__ w,
                                                                int w_heads, const T* __restrict__ gate, int64_t gate_stride, int act,
                                                                T* __restrict__ out, int64_t out_stride, float out_scale, int64_t rows, int H,
                                                                int vdim, float eps) {
    B200_PDL_SYNC();
    const int64_t r = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (r >= rows) return;
    const int lane = threadIdx.x & 31;
    const int64_t t = r / H;
    const int h = (int)(r - t * H);
    const float* o = x + r * (vdim + (flr ? 1 : 0));
    const float inv = flr ? 1.0f / (fmaxf(fabsf(o[vdim]), flr[r]) + 1e-6f) : 1.0f;
    if (w && w_heads) w += (int64_t)h * vdim;
    const T* gr = gate ? gate + t * gate_stride + (int64_t)h * vdim : nullptr;
    T* dst = out + t * out_stride + (int64_t)h * vdim;
    if constexpr (PER > 0) {                                // the whole head in registers, every operand in flight at once
        float v[PER], g[PER], wv[PER];
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int c = lane + 32 * k;
            const bool in = c < vdim;
            v[k] = in ? o[c] : 0.f;
            g[k] = in && gr ? ldf(gr + c) : 0.f;
            wv[k] = in && w ? ldf(w + c) : 1.f;
        }
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            v[k] *= inv;
            ss = fmaf(v[k], v[k], ss);
        }
        const float rstd = out_scale / sqrtf(warp_sum(ss) / (float)vdim + eps);
#pragma unroll
        for (int k = 0; k < PER; ++k) {
            const int c = lane + 32 * k;
            if (c < vdim) stf(dst + c, v[k] * rstd * wv[k] * (gr ? (act ? siluf_(g[k]) : sigmoidf_(g[k])) : 1.f));
        }
        return;
    }
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) {
        const float v = o[c] * inv;
        ss = fmaf(v, v, ss);
    }
    const float rstd = inv / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int c = lane; c < vdim; c += 32) {
        float v = o[c] * rstd;
        if (w) v *= ldf(w + c);
        if (gr) {
            const float z = ldf(gr + c);
            v *= act ? siluf_(z) : sigmoidf_(z);
        }
        stf(dst + c, v * out_scale);
    }
}

// The close of a state-space mixer: t = (y[r, h, :] + D_h x[r, h, :]) * silu(z[r, :]), then every one of `groups` equal parts of the row
// divided by its own root mean square, times w.  One CTA per (row, part); V columns per access, PER such groups per thread stay
// in registers (wider parts are formed again).
template <typename T, int V, int PER>
__global__ void __launch_bounds__(128) skip_gate_groupnorm_kernel(const float* __restrict__ y, const T* __restrict__ x, int64_t x_stride,
                                                                  const float* __restrict__ D, const T* __restrict__ z, int64_t z_stride,
                                                                  const T* __restrict__ w, T* __restrict__ out, int64_t out_stride,
                                                                  int inner, int vdim, int part, float eps) {
    B200_PDL_SYNC();
    __shared__ float red[4];
    const int64_t row = blockIdx.x;
    const int p0 = blockIdx.y * part;
    auto ld = [](const auto* p, float (&f)[V]) {
        if constexpr (V == 1) {
            f[0] = ldf(p);
        } else if constexpr (sizeof(*p) == 4) {
            const float4 v = *reinterpret_cast<const float4*>(p);
            f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
        } else {
            const uint2 v = *reinterpret_cast<const uint2*>(p);
            f[0] = bf16lo(v.x), f[1] = bf16hi(v.x), f[2] = bf16lo(v.y), f[3] = bf16hi(v.y);
        }
    };
    auto gated = [&](int c, float (&f)[V]) {
        float a[V], b[V];
        ld(y + row * inner + c, f);
        ld(x + row * x_stride + c, a);
        ld(z + row * z_stride + c, b);
        const float d = D[c / vdim];                         // V columns never straddle two heads
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] = fmaf(d, a[e], f[e]) * siluf_(b[e]);
    };
    const int step = 128 * V;
    float r[PER][V];
    float q = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x * V + k * step;
#pragma unroll
        for (int e = 0; e < V; ++e) r[k][e] = 0.f;
        if (c < part) gated(p0 + c, r[k]);
#pragma unroll
        for (int e = 0; e < V; ++e) q = fmaf(r[k][e], r[k][e], q);
    }
    for (int c = threadIdx.x * V + PER * step; c < part; c += step) {
        float f[V];
        gated(p0 + c, f);
#pragma unroll
        for (int e = 0; e < V; ++e) q = fmaf(f[e], f[e], q);
    }
    const float rstd = 1.0f / sqrtf(block_sum(q, red) / (float)part + eps);
    auto emit = [&](int c, const float (&f)[V]) {
        float g[V];
        ld(w + c, g);
#pragma unroll
        for (int e = 0; e < V; ++e) g[e] *= f[e] * rstd;
        T* o = out + row * out_stride + c;
        if constexpr (V == 1) stf(o, g[0]);
        else if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(o) = make_float4(g[0], g[1], g[2], g[3]);
        else *reinterpret_cast<uint2*>(o) = make_uint2(pack_bf16x2(g[0], g[1]), pack_bf16x2(g[2], g[3]));
    };
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x * V + k * step;
        if (c < part) emit(p0 + c, r[k]);
    }
    for (int c = threadIdx.x * V + PER * step; c < part; c += step) {
        float f[V];
        gated(p0 + c, f);
        emit(p0 + c, f);
    }
}

}  // namespace

extern "C" int b200m_diag_scan(const void* u, int64_t u_stride, const float* gates, int64_t rows, const float* gate_bias, const float* rate,
                               const void* y, int64_t y_stride, float* state, const int32_t* state_slots, const int32_t* cu_q,
                               const int32_t* cu_k, const int32_t* ctx_lens, void* out, int num_seqs, int max_q, int channels,
                               int block_channels, int chunk_len, float* ws, int is32, void* stream) {
    if (!u || !gates || !gate_bias || !rate || !y || !state || !state_slots || !out) return B200_EINVAL;
    if ((cu_q == nullptr) != (cu_k == nullptr) || (cu_q == nullptr && ctx_lens == nullptr)) return B200_EINVAL;
    if (channels <= 0 || block_channels <= 0 || channels % block_channels) return B200_EINVAL;
    if (num_seqs <= 0 || max_q <= 0) return B200_OK;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const bool chunked = ws != nullptr && chunk_len > 0 && max_q > chunk_len;
    const int nchunks = chunked ? (max_q + chunk_len - 1) / chunk_len : 1;
    const int bx = (channels + 127) / 128;
#define DIAG_GO(MODE, GZ)                                                                                                          \
    B200M_DISPATCH(is32, B200_LAUNCH((diag_scan_kernel<T, MODE>), dim3(bx, num_seqs, GZ), 128, 0, st, static_cast<const T*>(u), u_stride, \
                                     gates, rows, gate_bias, rate, static_cast<const T*>(y), y_stride, state, state_slots, cu_q, cu_k,    \
                                     ctx_lens, static_cast<T*>(out), channels, block_channels, chunk_len, nchunks, ws))
    if (!chunked) {
        DIAG_GO(0, 1);
        return b200_launch_status(nullptr);
    }
    DIAG_GO(1, nchunks);
    int rc = b200_launch_status(nullptr);
    if (rc != B200_OK) return rc;
    B200_LAUNCH((diag_carry_kernel), dim3(bx, num_seqs), 128, 0, st, ws, state, state_slots, cu_q, cu_k, ctx_lens, channels, chunk_len, nchunks);
    rc = b200_launch_status(nullptr);
    if (rc != B200_OK) return rc;
    DIAG_GO(3, nchunks);
#undef DIAG_GO
    return b200_launch_status(nullptr);
}

extern "C" int b200m_gated_delta(const void* x, int64_t stride, int q_off, int k_off, int v_off, const float* ba, int64_t ba_stride,
                                 const float* rate, const float* dt_bias, float* state, const int32_t* state_slots, const int32_t* cu_q,
                                 const int32_t* cu_k, const int32_t* ctx_lens, float* out, int num_seqs, int max_q, int num_heads, int num_kv_heads,
                                 int dim, int vdim, float q_scale, int is32, void* stream) {
    if (!x || !ba || !rate || !dt_bias || !state || !state_slots || !out) return B200_EINVAL;
    if ((cu_q == nullptr) != (cu_k == nullptr) || (cu_q == nullptr && ctx_lens == nullptr)) return B200_EINVAL;
    if (num_heads <= 0 || num_kv_heads <= 0 || num_heads % num_kv_heads || dim <= 0 || vdim <= 0) return B200_EINVAL;
    if (num_seqs <= 0) return B200_OK;
    const DecayIn dec{ba + num_heads, ba_stride, rate, dt_bias, 1.0f};
    B200M_DISPATCH(is32, return (launch_matrix_state<T, false, true>(x, stride, q_off, k_off, v_off, ba, nullptr, ba_stride, dec, state,
                                                                     state_slots, cu_q, cu_k, ctx_lens, out, 0, num_seqs, max_q, num_heads,
                                                                     num_kv_heads, dim, vdim, q_scale, static_cast<cudaStream_t>(stream))));
    return B200_EUNSUPPORTED;
}

extern "C" int b200m_channel_state(const void* x, int64_t stride, int q_off, int k_off, int v_off, const void* write_in,
                                   int64_t write_stride, float* decay_in, int64_t decay_stride, const float* rate,
                                   const float* decay_bias, float decay_sign, float* state, const int32_t* state_slots,
                                   const int32_t* cu_q, const int32_t* cu_k, const int32_t* ctx_lens, float* out, int n, int num_seqs,
                                   int max_q, int num_heads, int num_kv_heads, int dim, int vdim, float q_scale, int is32,
                                   void* stream) {
    if (!x || !decay_in || !state || !state_slots || !out || !rate || !decay_bias) return B200_EINVAL;
    if ((cu_q == nullptr) != (cu_k == nullptr) || (cu_q == nullptr && ctx_lens == nullptr)) return B200_EINVAL;
    if (num_heads <= 0 || num_kv_heads <= 0 || num_heads % num_kv_heads || dim <= 0 || vdim <= 0) return B200_EINVAL;
    if (decay_stride < (int64_t)num_heads * dim || n < 0) return B200_EINVAL;
    if (num_seqs <= 0 || n == 0) return B200_OK;
    const DecayIn dec{decay_in, decay_stride, rate, decay_bias, decay_sign};
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    if (write_in) {
        B200M_DISPATCH(is32, return (launch_matrix_state<T, true, true>(x, stride, q_off, k_off, v_off, nullptr, write_in, write_stride, dec,
                                                                        state, state_slots, cu_q, cu_k, ctx_lens, out, n, num_seqs, max_q, num_heads,
                                                                        num_kv_heads, dim, vdim, q_scale, st)));
    } else {
        B200M_DISPATCH(is32, return (launch_matrix_state<T, true, false>(x, stride, q_off, k_off, v_off, nullptr, nullptr, 0, dec, state,
                                                                         state_slots, cu_q, cu_k, ctx_lens, out, n, num_seqs, max_q, num_heads,
                                                                         num_kv_heads, dim, vdim, q_scale, st)));
    }
    return B200_EUNSUPPORTED;
}

extern "C" int b200m_mlstm_gates(const float* in, int64_t stride, const float* bias, float cap, float* m_state, const int32_t* state_slots,
                                 const int32_t* cu_q, const int32_t* cu_k, const int32_t* ctx_lens, float* log_decay, float* write, float* floor,
                                 int num_seqs, int max_q, int num_heads, void* stream) {
    if (!in || !bias || !m_state || !state_slots || !log_decay || !write || !floor || num_heads <= 0 || !(cap > 0.f) || stride < 2 * num_heads)
        return B200_EINVAL;
    if ((cu_q == nullptr) != (cu_k == nullptr) || (cu_q == nullptr && ctx_lens == nullptr)) return B200_EINVAL;
    if (num_seqs <= 0) return B200_OK;
#define MG_GO(NW)                                                                                                                  \
    B200_LAUNCH((mlstm_gates_kernel<NW>), dim3(num_heads, num_seqs), NW * 32, 0, static_cast<cudaStream_t>(stream), in, stride, bias, cap, m_state, \
                state_slots, cu_q, cu_k, ctx_lens, log_decay, write, floor, num_heads)
    if (cu_q == nullptr || max_q <= 32) MG_GO(1);
    else MG_GO(8);
#undef MG_GO
    return b200_launch_status(nullptr);
}

extern "C" int b200m_linear_state(const void* x, int64_t stride, int q_off, int k_off, int v_off, const void* step_in, const float* log_decay,
                                  const float* write, int64_t gate_stride, const float* rate, const float* bias, float* state,
                                  const int32_t* state_slots, const int32_t* cu_q, const int32_t* cu_k, const int32_t* ctx_lens, float* out,
                                  int num_seqs, int max_q, int num_heads, int num_kv_heads, int dim, int vdim, int ones, float q_scale,
                                  int is32, int flags, void* stream) {
    if (!x || !state || !state_slots || !out || (step_in ? (!rate || !bias) : (!log_decay || !write))) return B200_EINVAL;
    if ((cu_q == nullptr) != (cu_k == nullptr) || (cu_q == nullptr && ctx_lens == nullptr)) return B200_EINVAL;
    if (num_heads <= 0 || num_kv_heads <= 0 || num_heads % num_kv_heads || dim <= 0 || vdim <= 0 || ones < 0 || ones > 1) return B200_EINVAL;
    if (num_seqs <= 0) return B200_OK;
    if (!is32 && max_q > MS_CHUNK_MIN && !(flags & 1)) {                    // prompt portions on the tensor cores
        using bf = __nv_bfloat16;
        const ScalarGate<bf> sg{static_cast<const bf*>(step_in), log_decay, write, gate_stride, step_in ? rate : nullptr, bias};
        const int rc = chunk_state_launch(static_cast<const bf*>(x), stride, q_off, k_off, v_off, sg, state, state_slots, cu_q, cu_k, out, num_seqs,
                                          num_heads, num_kv_heads, dim, vdim, ones, q_scale, static_cast<cudaStream_t>(stream));
        if (rc != B200_EUNSUPPORTED) return rc;
    }
    B200M_DISPATCH(is32, const ScalarGate<T> sg = (ScalarGate<T>{static_cast<const T*>(step_in), log_decay, write, gate_stride, step_in ? rate : nullptr, bias});
                   return (launch_matrix_state<T, false, false>(x, stride, q_off, k_off, v_off, nullptr, nullptr, 0, DecayIn{}, state, state_slots,
                                                                cu_q, cu_k, ctx_lens, out, 0, num_seqs, max_q, num_heads, num_kv_heads, dim, vdim,
                                                                q_scale, static_cast<cudaStream_t>(stream), sg, ones)));
    return B200_EUNSUPPORTED;
}

extern "C" int b200m_skip_gate_groupnorm(const float* y, const void* x, int64_t x_stride, const float* D, const void* z, int64_t z_stride,
                                         const void* w, void* out, int64_t out_stride, int n, int num_heads, int vdim, int groups, float eps,
                                         int is32, void* stream) {
    const int inner = num_heads * vdim;
    if (!y || !x || !D || !z || !w || !out || n < 0 || num_heads <= 0 || vdim <= 0 || groups <= 0 || inner % groups) return B200_EINVAL;
    if (n == 0) return B200_OK;
    const int part = inner / groups;
    cudaStream_t st = static_cast<cudaStream_t>(stream);
    const uintptr_t bits = reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(z) |
                           reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out);
    const bool vec = bits % 16 == 0 && vdim % 4 == 0 && part % 4 == 0 && x_stride % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0;
#define SGG_GO(V, PER)                                                                                                             \
    B200M_DISPATCH(is32, B200_LAUNCH((skip_gate_groupnorm_kernel<T, V, PER>), dim3(n, groups), 128, 0, st, y, static_cast<const T*>(x), x_stride, D, \
                                     static_cast<const T*>(z), z_stride, static_cast<const T*>(w), static_cast<T*>(out), out_stride, inner, vdim, part, eps))
    if (vec && part <= 512) SGG_GO(4, 1);
    else if (vec) SGG_GO(4, 4);
    else SGG_GO(1, 4);
#undef SGG_GO
    return b200_launch_status(nullptr);
}

extern "C" int b200m_head_rmsnorm_gate(const float* x, const float* floor, const void* w, int w_heads, const void* gate, int64_t gate_stride, int act,
                                       void* out, int64_t out_stride, float out_scale, int n, int num_heads, int vdim, float eps, int is32,
                                       void* stream) {
    if (!x || !out || n < 0 || num_heads <= 0 || vdim <= 0) return B200_EINVAL;
    if (n == 0) return B200_OK;
    const int64_t rows = (int64_t)n * num_heads;
#define HRG_GO(PER)                                                                                                                \
    B200M_DISPATCH(is32, B200_LAUNCH((head_rmsnorm_gate_kernel<T, PER>), (unsigned)((rows + 3) / 4), 128, 0, static_cast<cudaStream_t>(stream), x, floor, \
                                     static_cast<const T*>(w), w_heads, static_cast<const T*>(gate), gate_stride, act, static_cast<T*>(out), \
                                     out_stride, out_scale, rows, num_heads, vdim, eps))
    if (vdim <= 64) HRG_GO(2);
    else if (vdim <= 128) HRG_GO(4);
    else if (vdim <= 256) HRG_GO(8);
    else HRG_GO(0);
#undef HRG_GO
    return b200_launch_status(nullptr);
}
