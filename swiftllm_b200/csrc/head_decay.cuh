// Recurrences whose state is a MATRIX per head (dk x dv) with ONE decay per head and token, carried per SEQUENCE (row `seq` of a state
// tensor, the sequence's block-table row) in fp32.  Two rules:
//   DELTA (gated delta rule)     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//                                q, k divided by sqrt(sum of squares + 1e-6) over the head, q also times q_scale;
//                                g = exp(-rate_h softplus(ga + pa_h)),  beta = sigmoid(gb)
//   memory (mLSTM)               i = cap tanh((gb + pb_h) / cap),  f = log sigmoid(cap tanh((ga + pa_h) / cap)),  M = max(f + m, i);
//                                S <- e^(f + m - M) S + e^(i - M) k v^T,  n <- e^(f + m - M) n + e^(i - M) k,  m <- M;
//                                o = S^T q / (max(|n . q|, e^(-m)) + 1e-6),  q times q_scale
// Both end with out = o / sqrt(mean(o^2) + eps) * norm_w * act(gate), act = silu (DELTA) or sigmoid (memory).
// Query / key head of head h: h / (H / G).  A step brings SEGMENTS: rows seg_starts[b] .. seg_starts[b+1] - 1 of the packed batch are
// consecutive positions of sequence seq_ids[b].  A segment that starts at position 0 starts from the zero state (m = 0) whatever its row
// holds (rows are used again without being cleared).  Gates, decays, unit norms, the state, the read-out and the norm are fp32 for
// every storage type of q, k, v and the gate.
//
// Prompt portions (hd_prompt_kernel): tokens in batches of HD_TOKENS.  With S the state at the batch's start, D(l, j) the product of the
// decays of tokens l + 1 .. j and D(j) that of all tokens up to j:
//     u_j = beta_j (v_j - D(j) S^T k_j - sum_{l < j} D(l, j) (k_l . k_j) u_l),     o_j = D(j) S^T q_j + sum_{l <= j} D(l, j) (k_l . q_j) u_l,
//     S <- D(last) S + sum_l D(l, last) k_l u_l^T                                  (memory: u_l = e^(i_l - m_l) v_l)
// so S meets the batch's vectors in two dense products, the small triangular system is solved per column, and S is updated once.
// Every factor is a product of decays <= 1: nothing overflows, whatever the decays.  In floating point the result differs from the
// token-by-token rule by rounding only.  The columns of a head's state never mix: a CTA owns 32 CPT columns of one (segment, head), a
// warp 4 CPT of them with all their rows: lane (rg, cg) = (lane >> 2, lane & 3) holds rows 32 i + 4 rg + e (R of them) of CPT columns in
// registers for the whole segment (neighbouring lanes read the same shared-memory words: half the cost of the other order).  Eight warps
// own the columns, eight (CPT = 4: four) more HELPERS stage the next batch, make its small matrices and finish (norm, gate, store) the last one.
//
// Single decoded tokens (hd_decode_kernel): the state is read once into registers, both products with it are summed over the CTA, the
// update is applied and written back.
#pragma once

#include <type_traits>

#include "typed_io.cuh"

namespace sllm {

constexpr int HD_TOKENS = 8;               // tokens per batch, shared out among the helper warps
constexpr int HD_WARPS = 8;                // warps of the decode kernel; warps of the prompt kernel that own columns
constexpr float HD_UNIT_EPS = 1e-6f;       // unit queries and keys (DELTA)
constexpr float HD_DEN_EPS = 1e-6f;        // denominator (memory)

struct HeadDecayArgs {
    const void *q, *k, *v, *gate;
    int64_t q_stride, k_stride, v_stride, gate_stride;
    const float *ga, *gb;                  // gate logits [T, H] (row strides below)
    int64_t ga_stride, gb_stride;
    const float *pa, *pb;                  // [H]: DELTA: decay bias, rate; memory: forget bias, input bias
    float cap, q_scale, eps;
    const float* norm_w;                   // [dv] (norm_step 0) or [H, dv] (norm_step dv)
    int norm_step;
    float *state, *nstate, *mstate;        // [rows, H, dk, dv]; memory: [rows, H, dk], [rows, H]
    const int *seg_starts, *seq_ids, *tok_pos;
    float* o_raw;                          // [T, H, dv]: read-outs of heads whose columns several CTAs own
    float* carry;                          // [segments, H, dk + 1]: their n and m until every CTA has read the old ones
    void* out;                             // [T, H * dv]
    int64_t out_stride;
    int num_segs, H, G, dk, dv;
    int vec;                               // rows of q, k, v and the gate start on multiples of four entries
};

// N neighbouring storage elements as raw bits: loaded now, converted later (a prefetch must not wait for its conversion).  `vec`: their
// address is a multiple of their size.
template <typename T, int N> struct HdRaw {
    static constexpr int BYTES = N * (int)sizeof(T);
    static constexpr int WORDS = BYTES / 4 > 0 ? BYTES / 4 : 1;
    uint32_t w[WORDS];
    __device__ __forceinline__ void zero() {
#pragma unroll
        for (int i = 0; i < WORDS; i++) w[i] = 0u;
    }
    // entries i0 .. i0 + N - 1 of a row of `end` entries at p; those from `end` on are zero
    __device__ __forceinline__ void load(const T* p, int i0, int end, bool vec) {
        zero();
        if (vec && i0 + N <= end) {
            if constexpr (BYTES == 16) {
                const uint4 x = *reinterpret_cast<const uint4*>(p + i0);
                w[0] = x.x; w[1] = x.y; w[2] = x.z; w[3] = x.w;
            } else if constexpr (BYTES == 8) {
                const uint2 x = *reinterpret_cast<const uint2*>(p + i0);
                w[0] = x.x; w[1] = x.y;
            } else if constexpr (BYTES == 4) {
                w[0] = *reinterpret_cast<const uint32_t*>(p + i0);
            } else {
                w[0] = *reinterpret_cast<const unsigned short*>(p + i0);
            }
        } else {
#pragma unroll
            for (int i = 0; i < N; i++)
                if (i0 + i < end) {
                    if constexpr (sizeof(T) == 4) w[i] = reinterpret_cast<const uint32_t*>(p)[i0 + i];
                    else w[i / 2] |= (uint32_t) reinterpret_cast<const unsigned short*>(p)[i0 + i] << (16 * (i & 1));
                }
        }
    }
    __device__ __forceinline__ float get(int i) const {
        if constexpr (sizeof(T) == 4) return __uint_as_float(w[i]);
        else if constexpr (std::is_same<T, __nv_bfloat16>::value) return __uint_as_float((i & 1) ? w[i / 2] & 0xffff0000u : w[i / 2] << 16);
        else return __half2float(__ushort_as_half((unsigned short)((i & 1) ? w[i / 2] >> 16 : w[i / 2] & 0xffffu)));
    }
};

// v into entries i0 .. i0 + N - 1 of a row of `end` entries at p (from `end` on: dropped)
template <typename T, int N> __device__ __forceinline__ void hd_put(T* p, int i0, int end, bool vec, const float (&v)[N]) {
    if (vec && N > 1 && i0 + N <= end) {
        if constexpr (N > 1) {
            struct alignas(N * sizeof(T)) Pack { T e[N]; } x;
#pragma unroll
            for (int i = 0; i < N; i++) stf(x.e + i, v[i]);
            *reinterpret_cast<Pack*>(p + i0) = x;
        }
    } else {
#pragma unroll
        for (int i = 0; i < N; i++)
            if (i0 + i < end) stf(p + i0 + i, v[i]);
    }
}

// two fp32 multiply-adds in one instruction
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    unsigned long long d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)),
        "l"(*reinterpret_cast<unsigned long long*>(&c)));
    return *reinterpret_cast<float2*>(&d);
}

__device__ __forceinline__ float hd_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float hd_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// one token's gates from its logits and the head's parameters.  DELTA: a = log decay, b = beta.  memory: a = log forget gate, b = log
// input gate.
template <bool DELTA> __device__ __forceinline__ void hd_gates(float za, float zb, float pa, float pb, float cap, float& a, float& b) {
    if constexpr (DELTA) {
        a = -pb * hd_softplus(za + pa);
        b = hd_sigmoid(zb);
    } else {
        a = -hd_softplus(-cap * tanhf((za + pa) / cap));
        b = cap * tanhf((zb + pb) / cap);
    }
}

// silu or sigmoid of an output gate (relative error about 1e-6)
template <bool DELTA> __device__ __forceinline__ float hd_act(float z) {
    const float g = __fdividef(1.f, 1.f + __expf(-z));
    return DELTA ? z * g : g;
}

// Adds up v[8][N] over the eight row groups (bits BIT .. 2 of rg, lane bits 2 .. 4); columns are split between the lanes as long as there
// is more than one left.  `col`: which of the N columns this lane ends up with.
template <int BIT, int N> __device__ __forceinline__ void hd_reduce(float (&v)[HD_TOKENS][N], int lane, int& col, float (&r)[HD_TOKENS]) {
    if constexpr (BIT < 3 && N > 1) {
        constexpr int M = N / 2;
        const bool hi = (lane >> (BIT + 2)) & 1;
        float w[HD_TOKENS][M];
#pragma unroll
        for (int j = 0; j < HD_TOKENS; j++)
#pragma unroll
            for (int c = 0; c < M; c++) {
                const float give = hi ? v[j][c] : v[j][c + M], keep = hi ? v[j][c + M] : v[j][c];
                w[j][c] = keep + __shfl_xor_sync(0xffffffffu, give, 4 << BIT);
            }
        col += hi ? M : 0;
        hd_reduce<BIT + 1, M>(w, lane, col, r);
    } else if constexpr (BIT < 3) {
#pragma unroll
        for (int j = 0; j < HD_TOKENS; j++) v[j][0] += __shfl_xor_sync(0xffffffffu, v[j][0], 4 << BIT);
        hd_reduce<BIT + 1, N>(v, lane, col, r);
    } else {
        static_assert(N == 1, "at most eight columns per lane");
#pragma unroll
        for (int j = 0; j < HD_TOKENS; j++) r[j] = v[j][0];
    }
}

constexpr int HD_SMALL = 2 * HD_TOKENS * HD_TOKENS + 4 * HD_TOKENS;      // floats of a batch's small matrices and factors

template <bool DELTA, int R, int CPT> constexpr int hd_prompt_smem_floats() {
    constexpr int P = 8 * R + 4, COLS = 32 * CPT;
    return 2 * (2 * HD_TOKENS * P + HD_TOKENS * COLS + HD_TOKENS * COLS + 2 * HD_TOKENS + HD_SMALL)   // q, k, v, read-outs, gates (two batches)
           + (DELTA ? HD_TOKENS * COLS : 8 * R);                         // scaled u | n
}

constexpr int hd_helpers(int cpt) { return cpt == 4 ? 4 : 8; }            // helper warps: few where the owners need the registers
template <int THREADS> __device__ __forceinline__ void hd_barrier(int id) { asm volatile("bar.sync %0, %1;" ::"r"(id), "n"(THREADS) : "memory"); }

// eight neighbouring floats of shared memory (16-byte aligned)
__device__ __forceinline__ void hd_row(const float* p, float (&v)[HD_TOKENS]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}

// grid (segments, heads, ceil(dv / (32 CPT))), HD_WARPS + hd_helpers(CPT) warps
template <typename T, bool DELTA, int R, int CPT>
__global__ void __launch_bounds__((HD_WARPS + hd_helpers(CPT)) * 32) hd_prompt_kernel(const HeadDecayArgs p) {
    constexpr int DKP = 8 * R, P = DKP + 4, COLS = 32 * CPT, NQ = (DKP + 127) / 128;
    constexpr int HW = hd_helpers(CPT), TPW = HD_TOKENS / HW;             // helper warps; tokens each of them takes care of: warp + HW s
    constexpr int ALL = (HD_WARPS + HW) * 32, HELPERS = HW * 32;
    extern __shared__ __align__(16) float hd_smem[];
    float* qs = hd_smem;                                                 // [2][HD_TOKENS][P]
    float* ks = qs + 2 * HD_TOKENS * P;                                  // [2][HD_TOKENS][P]
    float* vs = ks + 2 * HD_TOKENS * P;                                  // [2][HD_TOKENS][COLS]
    float* os = vs + 2 * HD_TOKENS * COLS;                               // [2][HD_TOKENS][COLS] read-outs
    float* small = os + 2 * HD_TOKENS * COLS;                            // [2][HD_SMALL], see M1 .. below
    float* gates = small + 2 * HD_SMALL;                                 // [2][2][HD_TOKENS]
    float* us = gates + 4 * HD_TOKENS;                                   // DELTA: [HD_TOKENS][COLS] u_l D(l, last);  memory: n [DKP]
    // the small matrices and factors of a batch
    constexpr int M1 = 0;                                                // [l][j]: D(l, j) k_l . k_j
    constexpr int M2 = HD_TOKENS * HD_TOKENS;                            // [l][j]: D(l, j) k_l . q_j (memory: times e^(i_l - m_l))
    constexpr int DJ = 2 * HD_TOKENS * HD_TOKENS;                        // [j]: D(j)
    constexpr int TAIL = DJ + HD_TOKENS;                                 // [l]: D(l, last) (memory: times e^(i_l - m_l))
    constexpr int BJ = TAIL + HD_TOKENS;                                 // [j]: beta | 1 / denominator
    const int h = blockIdx.y, b = blockIdx.x;
    const int t0 = p.seg_starts[b], n = p.seg_starts[b + 1] - t0;
    if (n <= 0) return;
    const int seq = p.seq_ids[b], dk = p.dk, dv = p.dv, g = h / (p.H / p.G);
    const bool fresh = p.tok_pos[t0] == 0, vec = p.vec;
    const bool helper = threadIdx.x >= HD_WARPS * 32;
    const int tid = threadIdx.x - (helper ? HD_WARPS * 32 : 0), warp = tid >> 5, lane = tid & 31;      // among the warps of its kind
    const int cta_col = blockIdx.z * COLS;
    if (helper) {
        // ================ helpers
        const bool sliced = gridDim.z > 1;
        float m_run = 0.f;
        if constexpr (!DELTA) {
            const float* ns = p.nstate + ((int64_t)seq * p.H + h) * dk;
            for (int d = tid; d < DKP; d += HELPERS) us[d] = (!fresh && d < dk) ? ns[d] : 0.f;
            if (!fresh) m_run = p.mstate[(int64_t)seq * p.H + h];
        }
        // a token is staged by one warp: four neighbouring entries of q and k per lane and 128, CPT neighbouring columns of v and the gate
        const T* qp = (const T*)p.q + (int64_t)g * dk;
        const T* kp = (const T*)p.k + (int64_t)g * dk;
        const T* vp = (const T*)p.v + (int64_t)h * dv;
        const T* gp = (const T*)p.gate + (int64_t)h * dv;
        const int my_col = cta_col + lane * CPT;                             // this lane's columns while staging and finishing
        HdRaw<T, 4> rq[TPW][NQ], rk[TPW][NQ];
        HdRaw<T, CPT> rv[TPW], rgate[TPW];                                             // rgate: the output gate of the batch finished next
        float fa[TPW], fb[TPW], nw[CPT];
        const float pa = p.pa[h], pb = p.pb[h];
#pragma unroll
        for (int c = 0; c < CPT; c++) nw[c] = my_col + c < dv ? p.norm_w[h * p.norm_step + my_col + c] : 0.f;
        auto fetch = [&](int i0) {
#pragma unroll
            for (int s = 0; s < TPW; s++) {
                const int tok = i0 + warp + HW * s;
                const bool live = tok < n;
                const int64_t t = t0 + (live ? tok : 0);
#pragma unroll
                for (int e = 0; e < NQ; e++) {
                    rq[s][e].load(qp + t * p.q_stride, 4 * lane + 128 * e, live ? dk : 0, vec);
                    rk[s][e].load(kp + t * p.k_stride, 4 * lane + 128 * e, live ? dk : 0, vec);
                }
                rv[s].load(vp + t * p.v_stride, my_col, live ? dv : 0, vec);
                fa[s] = p.ga[t * p.ga_stride + h];
                fb[s] = p.gb[t * p.gb_stride + h];
            }
        };
        auto fetch_gate = [&](int i0) {
#pragma unroll
            for (int s = 0; s < TPW; s++) {
                const int tok = i0 + warp + HW * s;
                if (!sliced && i0 >= 0 && tok < n) rgate[s].load(gp + (int64_t)(t0 + tok) * p.gate_stride, my_col, dv, vec);
            }
        };
        // norm, gate and store of batch `i0`'s tokens (their read-outs are in `os`)
        auto finish = [&](int i0) {
#pragma unroll
            for (int s = 0; s < TPW; s++) {
                const int j = warp + HW * s;
                if (i0 + j >= n) return;
                const int64_t t = t0 + i0 + j;
                float o[CPT], ss = 0.f;
#pragma unroll
                for (int c = 0; c < CPT; c++) {
                    o[c] = os[((i0 / HD_TOKENS & 1) * HD_TOKENS + j) * COLS + lane * CPT + c];                   // columns past dv are zero
                    ss += o[c] * o[c];
                }
                if (sliced) {
                    hd_put<float, CPT>(p.o_raw + (t * p.H + h) * dv, my_col, dv, vec, o);
                    continue;
                }
                const float f = rsqrtf(warp_sum(ss) / (float)dv + p.eps);
#pragma unroll
                for (int c = 0; c < CPT; c++) o[c] *= f * nw[c] * hd_act<DELTA>(rgate[s].get(c));
                hd_put<T, CPT>((T*)p.out + t * p.out_stride + (int64_t)h * dv, my_col, dv, vec, o);
            }
        };
#pragma unroll
        for (int s = 0; s < TPW; s++) rgate[s].zero();
        auto prepare = [&](int i0) {                                     // stage batch i0 (fetched before), then everything but the state's part
            const int buf = (i0 / HD_TOKENS) & 1;
            float* qb = qs + buf * HD_TOKENS * P;
            float* kb = ks + buf * HD_TOKENS * P;
            float* vb = vs + buf * HD_TOKENS * COLS;
            float* sm = small + buf * HD_SMALL;
#pragma unroll
            for (int s = 0; s < TPW; s++) {
                const int tok = warp + HW * s;
                float fq = p.q_scale, fk = 1.f;
                if constexpr (DELTA) {
                    float sq = 0.f, sk = 0.f;
#pragma unroll
                    for (int e = 0; e < NQ; e++)
#pragma unroll
                        for (int i = 0; i < 4; i++) {
                            sq += rq[s][e].get(i) * rq[s][e].get(i);
                            sk += rk[s][e].get(i) * rk[s][e].get(i);
                        }
                    fq *= rsqrtf(warp_sum(sq) + HD_UNIT_EPS);
                    fk = rsqrtf(warp_sum(sk) + HD_UNIT_EPS);
                }
#pragma unroll
                for (int e = 0; e < NQ; e++) {
                    const int d = 4 * lane + 128 * e;
                    if (DKP % 128 != 0 && d >= DKP) break;
                    const HdRaw<T, 4>&x = rq[s][e], &y = rk[s][e];
                    *reinterpret_cast<float4*>(qb + tok * P + d) = make_float4(x.get(0) * fq, x.get(1) * fq, x.get(2) * fq, x.get(3) * fq);
                    *reinterpret_cast<float4*>(kb + tok * P + d) = make_float4(y.get(0) * fk, y.get(1) * fk, y.get(2) * fk, y.get(3) * fk);
                }
#pragma unroll
                for (int c = 0; c < CPT; c++) vb[tok * COLS + lane * CPT + c] = rv[s].get(c);
                float a = 0.f, bb = DELTA ? 0.f : -INFINITY;             // past the end: no decay, nothing written
                if (i0 + tok < n) hd_gates<DELTA>(fa[s], fb[s], pa, pb, p.cap, a, bb);
                if (lane == 0) { gates[buf * 2 * HD_TOKENS + tok] = a; gates[(buf * 2 + 1) * HD_TOKENS + tok] = bb; }
            }
            hd_barrier<HELPERS>(1);                                         // the batch is staged (memory: n is up to date)
            if (i0 + HD_TOKENS < n) fetch(i0 + HD_TOKENS);               // in flight while this batch is worked on
            // the small matrices, one column j after the other: lane = (l, quarter of the head)
            const int l = lane & 7, quarter = lane >> 3;
            float lg[HD_TOKENS], second[HD_TOKENS], own = 0.f;           // log decays; beta | running maximum; memory: log input weight of l
            hd_row(gates + buf * 2 * HD_TOKENS, lg);
            hd_row(gates + (buf * 2 + 1) * HD_TOKENS, second);
            if constexpr (!DELTA) {
#pragma unroll
                for (int i = 0; i < HD_TOKENS; i++) {
                    const float m_new = fmaxf(lg[i] + m_run, second[i]);
                    lg[i] += m_run - m_new;
                    if (i == l) own = second[i] - m_new;
                    second[i] = m_run = m_new;
                }
            }
#pragma unroll
            for (int s = 0; s < TPW; s++) {
                const int j = warp + HW * s;
                float sum = 0.f, upto = 0.f, at_j = 0.f;
#pragma unroll
                for (int i = 0; i < HD_TOKENS; i++) {
                    if (i > l && i <= j) sum += lg[i];
                    if (i <= j) upto += lg[i];
                    if (i == j) at_j = second[i];
                }
                float kk = 0.f, kq = 0.f;
                const float* kl = kb + l * P + quarter * (DKP / 4);
                const float* kj = kb + j * P + quarter * (DKP / 4);
                const float* qj = qb + j * P + quarter * (DKP / 4);
#pragma unroll 4
                for (int i = 0; i < DKP / 4; i += 4) {
                    const float4 a = *reinterpret_cast<const float4*>(kl + i), y = *reinterpret_cast<const float4*>(qj + i);
                    kq += a.x * y.x + a.y * y.y + a.z * y.z + a.w * y.w;
                    if constexpr (DELTA) {
                        const float4 x = *reinterpret_cast<const float4*>(kj + i);
                        kk += a.x * x.x + a.y * x.y + a.z * x.z + a.w * x.w;
                    }
                }
                kq += __shfl_xor_sync(0xffffffffu, kq, 8);
                kq += __shfl_xor_sync(0xffffffffu, kq, 16);
                if constexpr (DELTA) {
                    kk += __shfl_xor_sync(0xffffffffu, kk, 8);
                    kk += __shfl_xor_sync(0xffffffffu, kk, 16);
                }
                // memory: the input weight of l joins the decay (its log may be -inf: nothing was written)
                const float D = expf(DELTA ? sum : sum + own), d_upto = expf(upto);
                const float m2 = l <= j ? D * kq : 0.f;
                float nq = 0.f;
                if constexpr (!DELTA) {
                    for (int d = lane; d < DKP; d += 32) nq += us[d] * qb[j * P + d];
                    nq = warp_sum(nq) * d_upto;
                    float in = m2;                                       // every quarter holds the same eight entries
                    in += __shfl_xor_sync(0xffffffffu, in, 1);
                    in += __shfl_xor_sync(0xffffffffu, in, 2);
                    in += __shfl_xor_sync(0xffffffffu, in, 4);
                    nq += in;
                }
                if (quarter == 0) {
                    if constexpr (DELTA) sm[M1 + l * HD_TOKENS + j] = l < j ? D * kk : 0.f;
                    sm[M2 + l * HD_TOKENS + j] = m2;
                    if (j == HD_TOKENS - 1) sm[TAIL + l] = D;
                    if (l == 0) {
                        sm[DJ + j] = d_upto;
                        sm[BJ + j] = DELTA ? at_j : 1.f / (fmaxf(fabsf(nq), expf(-at_j)) + HD_DEN_EPS);
                    }
                }
            }
            if constexpr (!DELTA) {
                hd_barrier<HELPERS>(1);                                     // every warp has read n, D(l, last) is written
                for (int d = tid; d < DKP; d += HELPERS) {
                    float x = us[d] * sm[DJ + HD_TOKENS - 1];
#pragma unroll
                    for (int l = 0; l < HD_TOKENS; l++) x = fmaf(sm[TAIL + l], kb[l * P + d], x);
                    us[d] = x;
                }
            }
        };
        fetch(0);
        prepare(0);
        hd_barrier<ALL>(0);
        for (int i0 = 0; i0 < n; i0 += HD_TOKENS) {                      // while the other warps work on batch i0
            fetch_gate(i0 - HD_TOKENS);
            if (i0 + HD_TOKENS < n) prepare(i0 + HD_TOKENS);
            if (i0 > 0) finish(i0 - HD_TOKENS);
            hd_barrier<ALL>(0);
        }
        const int last = (n - 1) / HD_TOKENS * HD_TOKENS;
        fetch_gate(last);
        finish(last);
        if constexpr (!DELTA) {
            if (blockIdx.z != 0) return;
            // another CTA of this head may not have read the old n and m yet: they wait in `carry` for the head norm's launch
            float* ns = sliced ? p.carry + ((int64_t)b * p.H + h) * (dk + 1) : p.nstate + ((int64_t)seq * p.H + h) * dk;
            for (int d = tid; d < dk; d += HELPERS) ns[d] = us[d];
            if (tid == 0) *(sliced ? ns + dk : p.mstate + (int64_t)seq * p.H + h) = m_run;
        }
        return;
    }
    // ================ owners of the columns
    const int rg = lane >> 2, cg = lane & 3;
    const int col_l = warp * 4 * CPT + cg * CPT;                         // this lane's first column, in the CTA
    float* st = p.state + ((int64_t)seq * p.H + h) * dk * dv;
    float2 S[R / 2][CPT];                                                // rows 32 i + 4 rg + (0, 1), + (2, 3): entries 2 i, 2 i + 1
#pragma unroll
    for (int r = 0; r < R / 2; r++) {
        const int d = 32 * (r >> 1) + 4 * rg + 2 * (r & 1);
#pragma unroll
        for (int c = 0; c < CPT; c++) {
            const int col = cta_col + col_l + c;
            S[r][c].x = (!fresh && d < dk && col < dv) ? st[(int64_t)d * dv + col] : 0.f;
            S[r][c].y = (!fresh && d + 1 < dk && col < dv) ? st[(int64_t)(d + 1) * dv + col] : 0.f;
        }
    }
    hd_barrier<ALL>(0);
    for (int i0 = 0; i0 < n; i0 += HD_TOKENS) {
        const int buf = (i0 / HD_TOKENS) & 1;
        const float* qb = qs + buf * HD_TOKENS * P;
        const float* kb = ks + buf * HD_TOKENS * P;
        const float* vb = vs + buf * HD_TOKENS * COLS;
        const float* sm = small + buf * HD_SMALL;
        float* ob = os + buf * HD_TOKENS * COLS;
        // ---- the state against the batch's vectors
        float r[HD_TOKENS];
        int mine = 0;                                                    // which of the lane's columns r belongs to
        {
            constexpr int JH = CPT == 4 ? HD_TOKENS / 2 : HD_TOKENS;     // tokens at a time (registers)
            float z[HD_TOKENS][CPT];
#pragma unroll
            for (int j0 = 0; j0 < HD_TOKENS; j0 += JH) {
                auto against = [&](const float* x, float (&sum)[JH][CPT]) {
                    float2 acc[JH][CPT];
#pragma unroll
                    for (int j = 0; j < JH; j++)
#pragma unroll
                        for (int c = 0; c < CPT; c++) acc[j][c] = make_float2(0.f, 0.f);
#pragma unroll
                    for (int i = 0; i < R / 4; i++)
#pragma unroll
                        for (int j = 0; j < JH; j++) {
                            const float4 x4 = *reinterpret_cast<const float4*>(x + (j0 + j) * P + 32 * i + 4 * rg);
#pragma unroll
                            for (int c = 0; c < CPT; c++) {
                                acc[j][c] = fma2(S[2 * i][c], make_float2(x4.x, x4.y), acc[j][c]);
                                acc[j][c] = fma2(S[2 * i + 1][c], make_float2(x4.z, x4.w), acc[j][c]);
                            }
                        }
#pragma unroll
                    for (int j = 0; j < JH; j++)
#pragma unroll
                        for (int c = 0; c < CPT; c++) sum[j][c] = acc[j][c].x + acc[j][c].y;
                };
                float B[JH][CPT];
                against(qb, B);
                if constexpr (DELTA) {                                   // even row groups take S^T k, odd ones S^T q
                    float A[JH][CPT];
                    against(kb, A);
                    const bool odd = rg & 1;
#pragma unroll
                    for (int j = 0; j < JH; j++)
#pragma unroll
                        for (int c = 0; c < CPT; c++) {
                            const float give = odd ? A[j][c] : B[j][c], keep = odd ? B[j][c] : A[j][c];
                            z[j0 + j][c] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
                        }
                } else {
#pragma unroll
                    for (int j = 0; j < JH; j++)
#pragma unroll
                        for (int c = 0; c < CPT; c++) z[j0 + j][c] = B[j][c];
                }
            }
            hd_reduce<DELTA ? 1 : 0, CPT>(z, lane, mine, r);
        }
        // ---- one column per lane (several lanes hold the same one): the triangular system and the read-outs
        const int col = col_l + mine;
        float d8[HD_TOKENS], b8[HD_TOKENS];
        hd_row(sm + DJ, d8);
        hd_row(sm + BJ, b8);
#pragma unroll
        for (int j = 0; j < HD_TOKENS; j++) r[j] *= d8[j];
        if constexpr (DELTA) {
            float t8[HD_TOKENS], u[HD_TOKENS], o[HD_TOKENS];
            hd_row(sm + TAIL, t8);
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++) { u[j] = vb[j * COLS + col] - r[j]; o[j] = r[j]; }
#pragma unroll
            for (int l = 0; l < HD_TOKENS; l++) {
                float m8[HD_TOKENS];
                hd_row(sm + M1 + l * HD_TOKENS, m8);
                u[l] *= b8[l];
#pragma unroll
                for (int j = l + 1; j < HD_TOKENS; j++) u[j] = fmaf(-m8[j], u[l], u[j]);
            }
#pragma unroll
            for (int l = 0; l < HD_TOKENS; l++) u[l] = __shfl_sync(0xffffffffu, u[l], lane & ~4);
#pragma unroll
            for (int l = 0; l < HD_TOKENS; l++) {
                float m8[HD_TOKENS];
                hd_row(sm + M2 + l * HD_TOKENS, m8);
#pragma unroll
                for (int j = l; j < HD_TOKENS; j++) o[j] = fmaf(m8[j], u[l], o[j]);
            }
            float* to = (rg & 1 ? ob : us) + col;
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++) to[j * COLS] = rg & 1 ? o[j] : u[j] * t8[j];
            __syncwarp();
        } else {
#pragma unroll
            for (int l = 0; l < HD_TOKENS; l++) {
                float m8[HD_TOKENS];
                hd_row(sm + M2 + l * HD_TOKENS, m8);
                const float v = vb[l * COLS + col];
#pragma unroll
                for (int j = l; j < HD_TOKENS; j++) r[j] = fmaf(m8[j], v, r[j]);
            }
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++) ob[j * COLS + col] = r[j] * b8[j];
        }
        // ---- the state moves on
        const float keep = d8[HD_TOKENS - 1];
#pragma unroll
        for (int r_ = 0; r_ < R / 2; r_++)
#pragma unroll
            for (int c = 0; c < CPT; c++) { S[r_][c].x *= keep; S[r_][c].y *= keep; }
#pragma unroll
        for (int l = 0; l < HD_TOKENS; l++) {
            float w[CPT];
#pragma unroll
            for (int c = 0; c < CPT; c++) w[c] = DELTA ? us[l * COLS + col_l + c] : vb[l * COLS + col_l + c] * sm[TAIL + l];
#pragma unroll
            for (int i = 0; i < R / 4; i++) {
                const float4 k4 = *reinterpret_cast<const float4*>(kb + l * P + 32 * i + 4 * rg);
#pragma unroll
                for (int c = 0; c < CPT; c++) {
                    S[2 * i][c] = fma2(make_float2(k4.x, k4.y), make_float2(w[c], w[c]), S[2 * i][c]);
                    S[2 * i + 1][c] = fma2(make_float2(k4.z, k4.w), make_float2(w[c], w[c]), S[2 * i + 1][c]);
                }
            }
        }
        hd_barrier<ALL>(0);                                                // the next batch is prepared, `ob` is written
    }
#pragma unroll
    for (int r = 0; r < R / 2; r++) {
        const int d = 32 * (r >> 1) + 4 * rg + 2 * (r & 1);
#pragma unroll
        for (int c = 0; c < CPT; c++) {
            const int col = cta_col + col_l + c;
            if (d < dk && col < dv) st[(int64_t)d * dv + col] = S[r][c].x;
            if (d + 1 < dk && col < dv) st[(int64_t)(d + 1) * dv + col] = S[r][c].y;
        }
    }
}

// One warp per (row, head): the norm and the gate of a head whose columns several CTAs computed (prompt portions' rows are the first).
// VEC: four neighbouring columns per lane and turn (dv % 4 == 0, rows aligned).
template <typename T, bool DELTA, bool VEC>
__global__ void __launch_bounds__(256) hd_norm_kernel(const HeadDecayArgs p, int64_t units) {
    constexpr int N = VEC ? 4 : 1;
    const int lane = threadIdx.x & 31;
    const int64_t unit = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= units) return;
    const int64_t t = unit / p.H;
    const int h = (int)(unit - t * p.H);
    const float* o = p.o_raw + unit * p.dv;
    float ss = 0.f;
    for (int d = lane * N; d < p.dv; d += 32 * N) {
        if constexpr (VEC) {
            const float4 x = *reinterpret_cast<const float4*>(o + d);
            ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
        } else {
            ss += o[d] * o[d];
        }
    }
    const float f = rsqrtf(warp_sum(ss) / (float)p.dv + p.eps);
    const T* gr = (const T*)p.gate + t * p.gate_stride + (int64_t)h * p.dv;
    T* out = (T*)p.out + t * p.out_stride + (int64_t)h * p.dv;
    for (int d = lane * N; d < p.dv; d += 32 * N) {
        HdRaw<T, N> g;
        g.load(gr, d, p.dv, VEC);
#pragma unroll
        for (int i = 0; i < N; i++) stf(out + d + i, o[d + i] * f * p.norm_w[h * p.norm_step + d + i] * hd_act<DELTA>(g.get(i)));
    }
}

// grid (segments, heads): n and m of sliced heads into their rows
static __global__ void hd_carry_kernel(const HeadDecayArgs p) {
    const int b = blockIdx.x, h = blockIdx.y;
    if (p.seg_starts[b + 1] <= p.seg_starts[b]) return;
    const int64_t row = (int64_t)p.seq_ids[b] * p.H + h;
    const float* c = p.carry + ((int64_t)b * p.H + h) * (p.dk + 1);
    for (int d = threadIdx.x; d < p.dk; d += blockDim.x) p.nstate[row * p.dk + d] = c[d];
    if (threadIdx.x == 0) p.mstate[row] = c[p.dk];
}

// One single decoded token: grid (segments, heads), 8 warps.  Warp w takes state rows w, w + 8, .., a lane V neighbouring columns of each
// 32 V.  DELTA: RB rows stay in registers between the read (which the update needs a product with) and the write; memory: the update
// needs no product, rows stream through RB at a time.  Dynamic shared memory: (16 + 2) * 32 V + 2 dk + 2 dv floats.
template <typename T, bool DELTA, int V, int RB>
__global__ void __launch_bounds__(HD_WARPS * 32) hd_decode_kernel(const HeadDecayArgs p) {
    constexpr int CB = 32 * V;
    extern __shared__ __align__(16) float hd_smem[];
    float* red = hd_smem;                                               // [HD_WARPS][2][CB]
    float* tot = red + HD_WARPS * 2 * CB;                               // [2][CB]
    float* qv = tot + 2 * CB;                                           // [dk]
    float* kv = qv + p.dk;                                              // [dk]
    float* vv = kv + p.dk;                                              // [dv]
    float* ov = vv + p.dv;                                              // [dv]
    __shared__ float sums[3][HD_WARPS];
    __shared__ float bsum[32];
    const int b = blockIdx.x, h = blockIdx.y;
    const int64_t t = p.seg_starts[b];
    if (p.seg_starts[b + 1] <= t) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dk = p.dk, dv = p.dv, g = h / (p.H / p.G);
    const bool fresh = p.tok_pos[t] == 0;
    const int64_t row = (int64_t)p.seq_ids[b] * p.H + h;
    float* st = p.state + row * dk * dv;
    float S[RB][V];
    auto load_rows = [&](int d0, int c0) {
#pragma unroll
        for (int r = 0; r < RB; r++) {
            const int d = d0 + r * HD_WARPS;
#pragma unroll
            for (int c = 0; c < V; c++) S[r][c] = 0.f;
            if (!fresh && d < dk && c0 < dv) {
                const float* s = st + (int64_t)d * dv + c0;
                if constexpr (V == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(s);
                    S[r][0] = x.x; S[r][1] = x.y; S[r][2] = x.z; S[r][3] = x.w;
                } else {
                    S[r][0] = *s;
                }
            }
        }
    };
    load_rows(warp, lane * V);                                          // in flight while the vectors are staged
    float ga, gb;
    hd_gates<DELTA>(p.ga[t * p.ga_stride + h], p.gb[t * p.gb_stride + h], p.pa[h], p.pb[h], p.cap, ga, gb);
    float decay, take, m_new = 0.f;                                     // take: beta | e^(i - m)
    if constexpr (DELTA) {
        decay = expf(ga);
        take = gb;
    } else {
        const float m_old = fresh ? 0.f : p.mstate[row];
        m_new = fmaxf(ga + m_old, gb);
        decay = expf(ga + m_old - m_new);
        take = expf(gb - m_new);
    }
    const T* qp = (const T*)p.q + t * p.q_stride + (int64_t)g * dk;
    const T* kp = (const T*)p.k + t * p.k_stride + (int64_t)g * dk;
    const T* vp = (const T*)p.v + t * p.v_stride + (int64_t)h * dv;
    float s0 = 0.f, s1 = 0.f, s2 = 0.f;                                 // DELTA: q.q, k.k, k.q;  memory: n.q, -, k.q
    for (int d = tid; d < dk; d += HD_WARPS * 32) {
        const float x = ldf(qp + d), y = ldf(kp + d);
        qv[d] = x; kv[d] = y;
        s2 += x * y;
        if constexpr (DELTA) {
            s0 += x * x;
            s1 += y * y;
        } else {
            float* ns = p.nstate + row * dk + d;
            const float nn = decay * (fresh ? 0.f : *ns) + take * y;
            *ns = nn;
            s0 += nn * x;
        }
    }
    for (int d = tid; d < dv; d += HD_WARPS * 32) vv[d] = ldf(vp + d);
    s0 = warp_sum(s0); s1 = warp_sum(s1); s2 = warp_sum(s2);
    if (lane == 0) { sums[0][warp] = s0; sums[1][warp] = s1; sums[2][warp] = s2; }
    __syncthreads();                                                    // (memory: every thread has read m)
    s0 = s1 = s2 = 0.f;
#pragma unroll
    for (int w = 0; w < HD_WARPS; w++) { s0 += sums[0][w]; s1 += sums[1][w]; s2 += sums[2][w]; }
    float fq = p.q_scale, fk = 1.f, inv_den = 1.f;
    if constexpr (DELTA) {
        fq *= rsqrtf(s0 + HD_UNIT_EPS);
        fk = rsqrtf(s1 + HD_UNIT_EPS);
    } else {
        inv_den = 1.f / (fmaxf(fabsf(s0 * fq), expf(-m_new)) + HD_DEN_EPS);
        if (tid == 0) p.mstate[row] = m_new;
    }
    const float kq = s2 * fq * fk;
    auto store_row = [&](int r, int d, int c0, const float (&u)[V]) {   // S <- decay S + k u
        const float y = kv[d];
        float* s = st + (int64_t)d * dv + c0;
#pragma unroll
        for (int c = 0; c < V; c++) S[r][c] = fmaf(decay, S[r][c], y * u[c]);
        if constexpr (V == 4) *reinterpret_cast<float4*>(s) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
        else *s = S[r][0];
    };
    for (int cb = 0; cb < dv; cb += CB) {
        const int c0 = cb + lane * V;
        float A[V], B[V], u[V];
#pragma unroll
        for (int c = 0; c < V; c++) { A[c] = B[c] = 0.f; u[c] = c0 + c < dv ? take * vv[c0 + c] : 0.f; }
        for (int d0 = warp; d0 < dk; d0 += RB * HD_WARPS) {             // DELTA: one turn
            if (cb > 0 || d0 > warp) load_rows(d0, c0);
#pragma unroll
            for (int r = 0; r < RB; r++) {
                const int d = d0 + r * HD_WARPS;
                if (d >= dk) break;
#pragma unroll
                for (int c = 0; c < V; c++) {
                    if constexpr (DELTA) A[c] = fmaf(S[r][c], kv[d], A[c]);
                    B[c] = fmaf(S[r][c], qv[d], B[c]);
                }
                if constexpr (!DELTA) {
                    if (c0 < dv) store_row(r, d, c0, u);
                }
            }
        }
#pragma unroll
        for (int c = 0; c < V; c++) {
            if constexpr (DELTA) red[(warp * 2) * CB + lane * V + c] = A[c];
            red[(warp * 2 + 1) * CB + lane * V + c] = B[c];
        }
        __syncthreads();
        for (int i = tid + (DELTA ? 0 : CB); i < 2 * CB; i += HD_WARPS * 32) {
            float x = 0.f;
#pragma unroll
            for (int w = 0; w < HD_WARPS; w++) x += red[w * 2 * CB + i];
            tot[i] = x;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < V; c++) {
            if constexpr (DELTA) u[c] -= take * decay * fk * tot[lane * V + c];
            if (warp == 0 && c0 + c < dv) ov[c0 + c] = (decay * fq * tot[CB + lane * V + c] + kq * u[c]) * inv_den;
        }
        if constexpr (DELTA) {
#pragma unroll
            for (int c = 0; c < V; c++) u[c] *= fk;
            if (c0 < dv) {
#pragma unroll
                for (int r = 0; r < RB; r++) {
                    const int d = warp + r * HD_WARPS;
                    if (d < dk) store_row(r, d, c0, u);
                }
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int d = tid; d < dv; d += HD_WARPS * 32) ss += ov[d] * ov[d];
    const float f = rsqrtf(block_sum(ss, bsum) / (float)dv + p.eps);
    const T* gr = (const T*)p.gate + t * p.gate_stride + (int64_t)h * dv;
    for (int d = tid; d < dv; d += HD_WARPS * 32)
        stf((T*)p.out + t * p.out_stride + (int64_t)h * dv + d, ov[d] * f * p.norm_w[h * p.norm_step + d] * hd_act<DELTA>(ldf(gr + d)));
}

// ---------------------------------------------------------------- launchers
template <typename T, bool DELTA, int R, int CPT> static int hd_launch_prompt(const HeadDecayArgs& a, cudaStream_t stream) {
    static unsigned long long attr_mask = 0;
    auto kern = hd_prompt_kernel<T, DELTA, R, CPT>;
    const size_t smem = sizeof(float) * hd_prompt_smem_floats<DELTA, R, CPT>();
    if (first_use_on_this_device(attr_mask)) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    kern<<<dim3((unsigned)a.num_segs, (unsigned)a.H, (unsigned)cdiv(a.dv, 32 * CPT)), (HD_WARPS + hd_helpers(CPT)) * 32, smem, stream>>>(a);
    return cdiv(a.dv, 32 * CPT);
}

// -> CTAs per head.  want: columns per lane the caller would like (1, 2 or 4)
template <typename T, bool DELTA> static int hd_prompt(const HeadDecayArgs& a, int want, cudaStream_t s) {
    const int rows = cdiv(a.dk, 8);
    if (rows <= 8)
        return want >= 4 ? hd_launch_prompt<T, DELTA, 8, 4>(a, s) : want >= 2 ? hd_launch_prompt<T, DELTA, 8, 2>(a, s) : hd_launch_prompt<T, DELTA, 8, 1>(a, s);
    if (rows <= 16)
        return want >= 4 ? hd_launch_prompt<T, DELTA, 16, 4>(a, s) : want >= 2 ? hd_launch_prompt<T, DELTA, 16, 2>(a, s) : hd_launch_prompt<T, DELTA, 16, 1>(a, s);
    if (rows <= 32) return hd_launch_prompt<T, DELTA, 32, 1>(a, s);
    return hd_launch_prompt<T, DELTA, 64, 1>(a, s);
}

template <typename T, bool DELTA, int V, int RB> static void hd_launch_decode(const HeadDecayArgs& a, cudaStream_t s) {
    static unsigned long long attr_mask = 0;
    auto kern = hd_decode_kernel<T, DELTA, V, RB>;
    const size_t smem = sizeof(float) * (18 * 32 * V + 2 * (size_t)a.dk + 2 * (size_t)a.dv);
    if (first_use_on_this_device(attr_mask)) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
    kern<<<dim3((unsigned)a.num_segs, (unsigned)a.H), HD_WARPS * 32, smem, s>>>(a);
}

template <typename T, bool DELTA> static void hd_decode(const HeadDecayArgs& a, cudaStream_t s) {
    const bool wide = a.dv % 4 == 0 && ((uintptr_t)a.state & 15) == 0 && (!DELTA || a.dk <= 256);
    if constexpr (DELTA) {
        if (!wide) hd_launch_decode<T, DELTA, 1, 64>(a, s);
        else if (a.dk <= 64) hd_launch_decode<T, DELTA, 4, 8>(a, s);
        else if (a.dk <= 128) hd_launch_decode<T, DELTA, 4, 16>(a, s);
        else hd_launch_decode<T, DELTA, 4, 32>(a, s);
    } else {
        if (wide) hd_launch_decode<T, DELTA, 4, 8>(a, s);
        else hd_launch_decode<T, DELTA, 1, 8>(a, s);
    }
}

template <bool DELTA> static int hd_run(HeadDecayArgs a, sllm_dtype_t dtype, int64_t num_tokens, int64_t num_prefill_tokens,
                                        int num_prefill_segs, int64_t workspace_floats, cudaStream_t s) {
    const int total_segs = a.num_segs;
    SLLM_REQUIRE(num_tokens >= 0 && total_segs >= 0 && a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.dk > 0 && a.dv > 0 &&
                 a.dk <= 512 && a.dv <= 4096, "head decay: bad shape (heads %d / %d, dk %d <= 512, dv %d <= 4096)", a.H, a.G, a.dk, a.dv);
    SLLM_REQUIRE(num_prefill_segs >= 0 && num_prefill_segs <= total_segs && num_prefill_tokens >= 0 && num_prefill_tokens <= num_tokens &&
                 num_tokens - num_prefill_tokens == total_segs - num_prefill_segs,
                 "head decay: %d prompt segments of %d with %lld of %lld tokens: every other segment is one token", num_prefill_segs,
                 total_segs, (long long)num_prefill_tokens, (long long)num_tokens);
    if (num_tokens == 0 || total_segs == 0) return 0;
    SLLM_REQUIRE(a.q && a.k && a.v && a.gate && a.ga && a.gb && a.pa && a.pb && a.norm_w && a.state && a.seg_starts && a.seq_ids &&
                 a.tok_pos && a.out && (DELTA || (a.nstate && a.mstate)), "head decay: null pointer");
    // every head's row of q, k, v, the gate and the output starts on a multiple of four entries
    const int64_t item = dtype == SLLM_F32 ? 4 : 2;
    a.vec = a.dk % 4 == 0 && a.dv % 4 == 0 && ((a.q_stride | a.k_stride | a.v_stride | a.gate_stride | a.out_stride) & 3) == 0 &&
            (((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.gate | (uintptr_t)a.out) & (4 * item - 1)) == 0 &&
            ((uintptr_t)a.o_raw & 15) == 0;
    if (num_prefill_segs > 0 && num_prefill_tokens > 0) {
        const int64_t raw = num_prefill_tokens * a.H * a.dv, carry = DELTA ? 0 : (int64_t)num_prefill_segs * a.H * (a.dk + 1);
        SLLM_REQUIRE(a.o_raw && workspace_floats >= raw + carry, "head decay: workspace of %lld floats, need %lld",
                     (long long)workspace_floats, (long long)(raw + carry));
        a.carry = a.o_raw + raw;
        a.num_segs = num_prefill_segs;
        int num_sms = 0;
        cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, current_device());
        // columns per lane: a whole head per CTA where segments x heads nearly fill the GPU, else the widest slice that still does
        const int64_t units = (int64_t)num_prefill_segs * a.H;
        int want = 1;
        if (a.dv > 64 && 5 * units * cdiv(a.dv, 128) >= 3 * num_sms) want = 4;
        else if (a.dv > 32 && 5 * units * cdiv(a.dv, 64) >= 3 * num_sms) want = 2;
        int slices = 1;
        SLLM_DISPATCH_DTYPE_F32(dtype, (slices = hd_prompt<T, DELTA>(a, want, s)));
        if (check_launch("head decay (prompt portions)")) return 1;
        if (slices > 1) {
            const int64_t n = num_prefill_tokens * a.H;
            SLLM_DISPATCH_DTYPE_F32(dtype, {
                if (a.vec) hd_norm_kernel<T, DELTA, true><<<(unsigned)cdiv(n, 8), 256, 0, s>>>(a, n);
                else hd_norm_kernel<T, DELTA, false><<<(unsigned)cdiv(n, 8), 256, 0, s>>>(a, n);
            });
            if (check_launch("head decay (head norm)")) return 1;
            if (!DELTA) {
                hd_carry_kernel<<<dim3((unsigned)num_prefill_segs, (unsigned)a.H), 128, 0, s>>>(a);
                if (check_launch("head decay (carry)")) return 1;
            }
        }
    }
    if (total_segs > num_prefill_segs) {
        a.seg_starts += num_prefill_segs;
        a.seq_ids += num_prefill_segs;
        a.num_segs = total_segs - num_prefill_segs;
        SLLM_DISPATCH_DTYPE_F32(dtype, (hd_decode<T, DELTA>(a, s)));
        return check_launch("head decay (decode)");
    }
    return 0;
}

}  // namespace sllm
