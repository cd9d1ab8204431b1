// Scalar linear attention (one decay and one write weight per token and head) over prompt portions, 64 tokens at a time, on the tensor cores:
//     S <- g S + w k v^T,   o = q_scale * S^T q            per head S [dim, vdim], fp32
// With b_t = log g_1 + ... + log g_t inside a chunk and S the state before it,
//     o_t = e^(b_t) S^T q_t + sum_(s <= t) P_ts v_s,   P_ts = (q_t . k_s) e^(b_t - b_s) w_s        (q_scale folded into both terms)
//     S  <- e^(b_L) S + sum_s k_s (e^(b_L - b_s) w_s v_s)^T
// which is the token-by-token recurrence regrouped.  q, k and v are bf16 in memory and enter the products exactly.  What is fp32 by
// nature (P, S, the scaled values) enters as a sum of TERMS bf16 numbers, each the rounding of what the previous ones left, so that
// three of them carry all 24 bits; products accumulate in fp32, and a chunk's contribution to S is summed apart and added with one
// fused multiply-add per element, so the state itself only sees fp32 rounding.  Sums of log decays are kept as pairs of floats (from
// double), so that e^(b_t - b_s) is right also behind large decays.
//
// A CTA (four warps) owns 64 value columns of one (sequence, head).  A warp holds 16 rows of S^T [vdim, dim] as product accumulators in
// registers for the whole portion; read as the next product's left operand they need no shuffle (S^T Q^T).  Per chunk:
//     P          : 16 x 16 blocks of the lower triangle, two or three per warp, split into terms in shared memory
//     O^T = S^T Q^T, scaled by e^(b_t), += V^T P^T over the lower triangle        (V^T by transposing loads)
//     S^T <- e^(b_L) S^T + (V scaled)^T K
// The next chunk's q, k, v arrive by asynchronous copies into a second buffer meanwhile; warp 0 forms the next chunk's gates.
// `ones`: the running sum n of weighted keys and n . q, by the CTA of the first column tile on the FMA pipe: n . q_t = e^(b_t) n . q_t +
// sum_s P_ts.
#include "mma_common.cuh"
#include "state_common.cuh"

namespace {

constexpr int CS_L = 64, CS_VC = 64, CS_THREADS = 128, CS_TERMS = 3;

// byte offset of 16-byte piece `piece` of row `row`, COLS bf16 per row: pieces are permuted so that the same piece of eight neighbouring
// rows lies in eight different bank groups
template <int COLS>
__device__ __forceinline__ uint32_t swz(int row, int piece) {
    return row * (COLS * 2) + ((piece ^ (COLS >= 64 ? (row & 7) : ((row >> 1) & 3))) << 4);
}

template <int D>
struct ChunkSmem {
    static constexpr int Q = 0, QB = CS_L * D * 2, K = 2 * QB, V = K + 2 * QB, VB = CS_L * CS_VC * 2, P = V + 2 * VB, PB = CS_L * CS_L * 2,
                         GATE = P + CS_TERMS * PB, GB = 5 * CS_L * 4 + 16, NV = GATE + 2 * GB, RS = NV + D * 4, BYTES = RS + 4 * CS_L * 4;
};
// a chunk's gates: b * log2(e) as (high, low), write weight * q_scale, q_scale e^b, e^(b_L - b) w, then e^(b_L)
constexpr int CG_BH = 0, CG_BL = CS_L, CG_W = 2 * CS_L, CG_IN = 3 * CS_L, CG_OUT = 4 * CS_L, CG_ALL = 5 * CS_L;

// (a, b) -> packed bf16 pair of their roundings; a and b become what the rounding left
__device__ __forceinline__ uint32_t take_term(float& a, float& b) {
    const uint32_t r = pack_bf16x2(a, b);
    a -= bf16lo(r);
    b -= bf16hi(r);
    return r;
}

template <int D>
__global__ void __launch_bounds__(CS_THREADS, 2) chunk_state_kernel(
    const __nv_bfloat16* __restrict__ x, int64_t stride, int q_off, int k_off, int v_off, ScalarGate<__nv_bfloat16> sg,
    float* __restrict__ state, const int32_t* __restrict__ state_slots, const int32_t* __restrict__ cu_q, const int32_t* __restrict__ cu_k,
    float* __restrict__ out, int H, int G, int dim, int vdim, int ones, float q_scale) {
    B200_PDL_SYNC();
    using SM = ChunkSmem<D>;
    constexpr int NT = D / 8, KT = D / 16;                  // 8-column tiles of S^T, 16-deep steps over dim
    extern __shared__ __align__(128) unsigned char cs_smem[];
    const int h = blockIdx.x, s = blockIdx.y, col0 = blockIdx.z * CS_VC;
    const SeqSpan sp = seq_span(cu_q, cu_k, nullptr, s);
    if (sp.qlen <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, t4 = lane & 3;
    const int nch = (sp.qlen + CS_L - 1) / CS_L, vcols = vdim + ones;
    const bool with_n = ones && blockIdx.z == 0;
    const bool live = col0 + warp * 16 < vdim;              // this warp has value columns
    const bool has_hist = sp.klen - sp.qlen > 0;
    const uint32_t sbase = smem_u32(cs_smem);
    float* gates_s = reinterpret_cast<float*>(cs_smem + SM::GATE);
    float* nvec = reinterpret_cast<float*>(cs_smem + SM::NV);
    float* rsum = reinterpret_cast<float*>(cs_smem + SM::RS);
    float* st = state + ((int64_t)state_slots[s] * H + h) * vcols * dim;
    const __nv_bfloat16* xs = x + (int64_t)sp.q0 * stride;
    const __nv_bfloat16* qp = xs + q_off + (int64_t)(h / (H / G)) * dim;
    const __nv_bfloat16* kp = xs + k_off + (int64_t)(h / (H / G)) * dim;
    const __nv_bfloat16* vp = xs + v_off + (int64_t)h * vdim + col0;

    auto load_chunk = [&](int c, int buf) {                 // tokens past the end and columns past the sizes are zero
        constexpr int DP = D / 8;
#pragma unroll 4
        for (int e = tid; e < CS_L * DP; e += CS_THREADS) {
            const int r = e / DP, p = e % DP, t = c * CS_L + r;
            const bool in = t < sp.qlen && p * 8 < dim;
            wm_cp16(sbase + SM::Q + buf * SM::QB + swz<D>(r, p), in ? qp + (int64_t)t * stride + p * 8 : x, in ? 16 : 0);
            wm_cp16(sbase + SM::K + buf * SM::QB + swz<D>(r, p), in ? kp + (int64_t)t * stride + p * 8 : x, in ? 16 : 0);
        }
#pragma unroll
        for (int e = tid; e < CS_L * (CS_VC / 8); e += CS_THREADS) {
            const int r = e / (CS_VC / 8), p = e % (CS_VC / 8), t = c * CS_L + r;
            const bool in = t < sp.qlen && col0 + p * 8 < vdim;
            wm_cp16(sbase + SM::V + buf * SM::VB + swz<CS_VC>(r, p), in ? vp + (int64_t)t * stride + p * 8 : x, in ? 16 : 0);
        }
        wm_commit();
    };
    const float rt = sg.rate ? sg.rate[h] : 0.f, gb = sg.rate ? sg.bias[h] : 0.f;
    float2 graw[2];
    auto gate_fetch = [&](int c) {                          // warp 0: tokens 2 lane, 2 lane + 1
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = c * CS_L + 2 * lane + j;
            graw[j] = t < sp.qlen ? sg.fetch(sp.q0 + t, h) : make_float2(0.f, 0.f);
        }
    };
    auto gate_make = [&](int c, int buf) {
        float* gs = gates_s + buf * (SM::GB / 4);
        float2 g[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) g[j] = c * CS_L + 2 * lane + j < sp.qlen ? sg.gates(graw[j], rt, gb) : make_float2(0.f, 0.f);
        constexpr double LOG2E = 1.4426950408889634;
        double b0 = LOG2E * (double)g[0].x, b1 = b0 + LOG2E * (double)g[1].x, run = b1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += up;
        }
        const double before = run - b1, all = __shfl_sync(0xffffffffu, run, 31);
        b0 += before;
        b1 += before;
        const double bb[2] = {b0, b1};
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = 2 * lane + j;
            const float hi = (float)bb[j];
            gs[CG_BH + t] = hi;
            gs[CG_BL + t] = (float)(bb[j] - (double)hi);
            gs[CG_W + t] = g[j].y * q_scale;
            gs[CG_IN + t] = fast_exp2(hi) * q_scale;
            gs[CG_OUT + t] = fast_exp2((float)(all - bb[j])) * g[j].y;
        }
        if (lane == 0) gs[CG_ALL] = fast_exp2((float)all);
    };

    load_chunk(0, 0);
    float S[NT][4];                                         // rows gq, gq + 8 of the warp's 16 value columns, dim n * 8 + 2 t4 (+ 1)
    const int vr = col0 + warp * 16 + gq;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
            float2 f = make_float2(0.f, 0.f);
            if (has_hist && vr + 8 * hh < vdim && n * 8 < dim) f = *reinterpret_cast<const float2*>(st + (int64_t)(vr + 8 * hh) * dim + n * 8 + 2 * t4);
            S[n][2 * hh] = f.x;
            S[n][2 * hh + 1] = f.y;
        }
    float nn = (with_n && has_hist && tid < dim) ? st[(int64_t)vdim * dim + tid] : 0.f;     // thread c: channel c of n
    if (warp == 0) {
        gate_fetch(0);
        gate_make(0, 0);
    }

    for (int c = 0; c < nch; ++c) {
        const int buf = c & 1;
        const uint32_t qb = sbase + SM::Q + buf * SM::QB, kb = sbase + SM::K + buf * SM::QB, vb = sbase + SM::V + buf * SM::VB, pb = sbase + SM::P;
        const float* gs = gates_s + buf * (SM::GB / 4);
        wm_wait<0>();
        __syncthreads();                                    // the chunk and its gates are there; everyone is done with the previous one
        if (c + 1 < nch) {
            load_chunk(c + 1, buf ^ 1);
            if (warp == 0) gate_fetch(c + 1);
        }
        if (with_n && tid < D) nvec[tid] = nn;

        // ---- P: ten blocks of 16 tokens x 16 keys (keys up to the tokens), shared out over the warps ----
        {
            const int ar = lane & 15, br = (lane & 7) + ((lane >> 4) << 3);
            // warp 0: (0,0) (3,0)   1: (1,0) (1,1) (3,1)   2: (2,0) (2,1) (2,2)   3: (3,2) (3,3)      as (token block, key block)
            const int nblk = warp == 0 || warp == 3 ? 2 : 3;
            for (int i = 0; i < nblk; ++i) {
                const int tb = warp == 3 ? 3 : i == (warp == 0 ? 1 : 2) && warp < 2 ? 3 : warp;
                const int np = warp == 3 ? 2 + i : tb == warp ? i : warp;
                float sc[2][4], sd[2][4];                   // two sums each, over even and odd steps: more products in flight
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) sc[j][e] = sd[j][e] = 0.f;
#pragma unroll
                for (int kk = 0; kk < KT; kk += 2) {
                    uint32_t a[4], b[4], a2[4], b2[4];
                    wm_ldsm(qb + swz<D>(tb * 16 + ar, kk * 2 + (lane >> 4)), a[0], a[1], a[2], a[3]);
                    wm_ldsm(kb + swz<D>(np * 16 + br, kk * 2 + ((lane >> 3) & 1)), b[0], b[1], b[2], b[3]);
                    wm_ldsm(qb + swz<D>(tb * 16 + ar, kk * 2 + 2 + (lane >> 4)), a2[0], a2[1], a2[2], a2[3]);
                    wm_ldsm(kb + swz<D>(np * 16 + br, kk * 2 + 2 + ((lane >> 3) & 1)), b2[0], b2[1], b2[2], b2[3]);
                    wm_mma(sc[0], a[0], a[1], a[2], a[3], b[0], b[1]);
                    wm_mma(sc[1], a[0], a[1], a[2], a[3], b[2], b[3]);
                    wm_mma(sd[0], a2[0], a2[1], a2[2], a2[3], b2[0], b2[1]);
                    wm_mma(sd[1], a2[0], a2[1], a2[2], a2[3], b2[2], b2[3]);
                }
                const int t0 = tb * 16 + gq;
                const float bh0 = gs[CG_BH + t0], bl0 = gs[CG_BL + t0], bh1 = gs[CG_BH + t0 + 8], bl1 = gs[CG_BL + t0 + 8];
                float row0 = 0.f, row1 = 0.f;
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int s0 = np * 16 + j * 8 + 2 * t4;
                    const float2 bh = *reinterpret_cast<const float2*>(gs + CG_BH + s0), bl = *reinterpret_cast<const float2*>(gs + CG_BL + s0),
                                 w = *reinterpret_cast<const float2*>(gs + CG_W + s0);
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const float h_ = e ? bh.y : bh.x, l_ = e ? bl.y : bl.x, w_ = e ? w.y : w.x;
                        sc[j][e] = s0 + e <= t0 ? (sc[j][e] + sd[j][e]) * (fast_exp2((bh0 - h_) + (bl0 - l_)) * w_) : 0.f;
                        sc[j][2 + e] = s0 + e <= t0 + 8 ? (sc[j][2 + e] + sd[j][2 + e]) * (fast_exp2((bh1 - h_) + (bl1 - l_)) * w_) : 0.f;
                    }
                    row0 += sc[j][0] + sc[j][1];
                    row1 += sc[j][2] + sc[j][3];
#pragma unroll
                    for (int m = 0; m < CS_TERMS; ++m) {
                        unsigned char* dst = cs_smem + SM::P + m * SM::PB + t4 * 4;
                        *reinterpret_cast<uint32_t*>(dst + swz<CS_L>(t0, np * 2 + j)) = take_term(sc[j][0], sc[j][1]);
                        *reinterpret_cast<uint32_t*>(dst + swz<CS_L>(t0 + 8, np * 2 + j)) = take_term(sc[j][2], sc[j][3]);
                    }
                }
                if (with_n) {
                    row0 += __shfl_xor_sync(0xffffffffu, row0, 1), row1 += __shfl_xor_sync(0xffffffffu, row1, 1);
                    row0 += __shfl_xor_sync(0xffffffffu, row0, 2), row1 += __shfl_xor_sync(0xffffffffu, row1, 2);
                    if (t4 == 0) rsum[np * CS_L + t0] = row0, rsum[np * CS_L + t0 + 8] = row1;
                }
            }
        }
        // ---- O^T = S^T Q^T ----
        float o[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
        if (live) {
            const int br = (lane & 7) + ((lane >> 4) << 3);
#pragma unroll
            for (int kk = 0; kk < KT; ++kk) {
                uint32_t b[4][4];
#pragma unroll
                for (int np = 0; np < 4; ++np)
                    wm_ldsm(qb + swz<D>(np * 16 + br, kk * 2 + ((lane >> 3) & 1)), b[np][0], b[np][1], b[np][2], b[np][3]);
                float f[8] = {S[2 * kk][0], S[2 * kk][1], S[2 * kk][2], S[2 * kk][3], S[2 * kk + 1][0], S[2 * kk + 1][1], S[2 * kk + 1][2], S[2 * kk + 1][3]};
#pragma unroll
                for (int m = 0; m < CS_TERMS; ++m) {
                    const uint32_t a0 = take_term(f[0], f[1]), a1 = take_term(f[2], f[3]), a2 = take_term(f[4], f[5]), a3 = take_term(f[6], f[7]);
#pragma unroll
                    for (int np = 0; np < 4; ++np) {
                        wm_mma(o[2 * np], a0, a1, a2, a3, b[np][0], b[np][1]);
                        wm_mma(o[2 * np + 1], a0, a1, a2, a3, b[np][2], b[np][3]);
                    }
                }
            }
#pragma unroll
            for (int n = 0; n < 8; ++n) {
                const float2 g = *reinterpret_cast<const float2*>(gs + CG_IN + n * 8 + 2 * t4);
                o[n][0] *= g.x, o[n][1] *= g.y, o[n][2] *= g.x, o[n][3] *= g.y;
            }
        }
        __syncthreads();                                    // P is complete
        if (live) {
            uint32_t va[4][4];                              // V^T: the warp's 16 value columns x 64 tokens
#pragma unroll
            for (int ks = 0; ks < 4; ++ks)
                wm_ldsm_t(vb + swz<CS_VC>(ks * 16 + (lane & 7) + ((lane >> 4) << 3), warp * 2 + ((lane >> 3) & 1)), va[ks][0], va[ks][1], va[ks][2], va[ks][3]);
            const int br = (lane & 7) + ((lane >> 4) << 3);
#pragma unroll
            for (int m = 0; m < CS_TERMS; ++m)
#pragma unroll
                for (int ks = 0; ks < 4; ++ks)
#pragma unroll
                    for (int np = ks; np < 4; ++np) {       // keys ks * 16 .. are seen from token ks * 16 on
                        uint32_t b[4];
                        wm_ldsm(pb + m * SM::PB + swz<CS_L>(np * 16 + br, ks * 2 + ((lane >> 3) & 1)), b[0], b[1], b[2], b[3]);
                        wm_mma(o[2 * np], va[ks][0], va[ks][1], va[ks][2], va[ks][3], b[0], b[1]);
                        wm_mma(o[2 * np + 1], va[ks][0], va[ks][1], va[ks][2], va[ks][3], b[2], b[3]);
                    }
            const int nv = min(CS_L, sp.qlen - c * CS_L);
            float* op = out + ((int64_t)(sp.q0 + c * CS_L) * H + h) * vcols + vr;
            const int64_t ostr = (int64_t)H * vcols;
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int t = n * 8 + 2 * t4 + e;
                    if (t < nv) {
                        if (vr < vdim) op[t * ostr] = o[n][e];
                        if (vr + 8 < vdim) op[t * ostr + 8] = o[n][2 + e];
                    }
                }
            // ---- S^T <- e^(b_L) S^T + (scaled V)^T K ----
            float dS[NT][4];
#pragma unroll
            for (int n = 0; n < NT; ++n) dS[n][0] = dS[n][1] = dS[n][2] = dS[n][3] = 0.f;
            const int kr = (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                const float2 w0 = *reinterpret_cast<const float2*>(gs + CG_OUT + ks * 16 + 2 * t4);
                const float2 w1 = *reinterpret_cast<const float2*>(gs + CG_OUT + ks * 16 + 8 + 2 * t4);
                float f[8] = {bf16lo(va[ks][0]) * w0.x, bf16hi(va[ks][0]) * w0.y, bf16lo(va[ks][1]) * w0.x, bf16hi(va[ks][1]) * w0.y,
                              bf16lo(va[ks][2]) * w1.x, bf16hi(va[ks][2]) * w1.y, bf16lo(va[ks][3]) * w1.x, bf16hi(va[ks][3]) * w1.y};
                uint32_t a[CS_TERMS][4];
#pragma unroll
                for (int m = 0; m < CS_TERMS; ++m)
#pragma unroll
                    for (int i = 0; i < 4; ++i) a[m][i] = take_term(f[2 * i], f[2 * i + 1]);
                constexpr int NG = KT < 4 ? KT : 4;
#pragma unroll
                for (int n0 = 0; n0 < KT; n0 += NG) {
                    uint32_t b[NG][4];
#pragma unroll
                    for (int j = 0; j < NG; ++j) wm_ldsm_t(kb + swz<D>(ks * 16 + kr, (n0 + j) * 2 + (lane >> 4)), b[j][0], b[j][1], b[j][2], b[j][3]);
#pragma unroll
                    for (int m = 0; m < CS_TERMS; ++m)
#pragma unroll
                        for (int j = 0; j < NG; ++j) {
                            wm_mma(dS[2 * (n0 + j)], a[m][0], a[m][1], a[m][2], a[m][3], b[j][0], b[j][1]);
                            wm_mma(dS[2 * (n0 + j) + 1], a[m][0], a[m][1], a[m][2], a[m][3], b[j][2], b[j][3]);
                        }
                }
            }
            const float all = gs[CG_ALL];
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[n][e] = fmaf(all, S[n][e], dS[n][e]);
        }
        if (with_n) {                                       // CTA-uniform
            // n . q of token tid / 2, half of the channels per thread
            const int t = tid >> 1;
            float a = 0.f;
#pragma unroll
            for (int p = 0; p < D / 16; ++p) {
                const int piece = (tid & 1) * (D / 16) + p;
                float f[8];
                unpack8(*reinterpret_cast<const uint4*>(cs_smem + SM::Q + buf * SM::QB + swz<D>(t, piece)), f);
#pragma unroll
                for (int e = 0; e < 8; ++e) a = fmaf(nvec[piece * 8 + e], f[e], a);
            }
            a += __shfl_xor_sync(0xffffffffu, a, 1);
            if ((tid & 1) == 0 && c * CS_L + t < sp.qlen) {
                float r = 0.f;                              // sums of P over the key blocks up to the token's own
                for (int np = 0; np <= t >> 4; ++np) r += rsum[np * CS_L + t];
                out[((int64_t)(sp.q0 + c * CS_L + t) * H + h) * vcols + vdim] = fmaf(a, gs[CG_IN + t], r);
            }
            if (tid < D) {
                float b = 0.f;
#pragma unroll 8
                for (int j = 0; j < CS_L; ++j)
                    b = fmaf(gs[CG_OUT + j],
                             __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(cs_smem + SM::K + buf * SM::QB + swz<D>(j, tid >> 3) + (tid & 7) * 2)), b);
                nn = fmaf(gs[CG_ALL], nn, b);
            }
        }
        if (warp == 0 && c + 1 < nch) gate_make(c + 1, buf ^ 1);
    }
    if (live) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int hh = 0; hh < 2; ++hh)
                if (vr + 8 * hh < vdim && n * 8 < dim)
                    *reinterpret_cast<float2*>(st + (int64_t)(vr + 8 * hh) * dim + n * 8 + 2 * t4) = make_float2(S[n][2 * hh], S[n][2 * hh + 1]);
    }
    if (with_n && tid < dim) st[(int64_t)vdim * dim + tid] = nn;
}

template <int D>
int launch_chunk_state(const __nv_bfloat16* x, int64_t stride, int q_off, int k_off, int v_off, const ScalarGate<__nv_bfloat16>& sg, float* state,
                       const int32_t* state_slots, const int32_t* cu_q, const int32_t* cu_k, float* out, int num_seqs, int H, int G, int dim, int vdim,
                       int ones, float q_scale, cudaStream_t st) {
    static B200SmemOptIn opt;
    if (opt.ensure(chunk_state_kernel<D>, ChunkSmem<D>::BYTES) != cudaSuccess) return B200_ECUDA;
    B200_LAUNCH((chunk_state_kernel<D>), dim3(H, num_seqs, (vdim + CS_VC - 1) / CS_VC), CS_THREADS, ChunkSmem<D>::BYTES, st, x, stride, q_off, k_off, v_off,
                sg, state, state_slots, cu_q, cu_k, out, H, G, dim, vdim, ones, q_scale);
    return b200_launch_status(nullptr);
}

}  // namespace

int chunk_state_launch(const __nv_bfloat16* x, int64_t stride, int q_off, int k_off, int v_off, const ScalarGate<__nv_bfloat16>& sg, float* state,
                       const int32_t* state_slots, const int32_t* cu_q, const int32_t* cu_k, float* out, int num_seqs, int H, int G, int dim,
                       int vdim, int ones, float q_scale, cudaStream_t st) {
    if (cu_q == nullptr || dim > 128 || reinterpret_cast<uintptr_t>(x) % 16) return B200_EUNSUPPORTED;
    if (dim % 8 || vdim % 8 || stride % 8 || q_off % 8 || k_off % 8 || v_off % 8) return B200_EUNSUPPORTED;        // 16-byte copies
#define CS_GO(D) \
    return launch_chunk_state<D>(x, stride, q_off, k_off, v_off, sg, state, state_slots, cu_q, cu_k, out, num_seqs, H, G, dim, vdim, ones, q_scale, st)
    if (dim <= 32) CS_GO(32);
    if (dim <= 64) CS_GO(64);
    CS_GO(128);
#undef CS_GO
}
