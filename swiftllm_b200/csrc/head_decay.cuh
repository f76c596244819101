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
// warp 4 CPT of them with all their rows: lane (rg, cg) = (lane & 7, lane >> 3) holds rows 32 i + 4 rg + e (R of them) of CPT columns in
// registers for the whole segment.
//
// Single decoded tokens (hd_decode_kernel): the state is read once into registers, both products with it are summed over the CTA, the
// update is applied and written back.
#pragma once

#include "typed_io.cuh"

namespace sllm {

constexpr int HD_TOKENS = 8;               // tokens per batch, one staged by each warp
constexpr int HD_WARPS = 8;
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
    int dtype, num_segs, H, G, dk, dv;
};

// 16- or 32-bit storage element: raw bits now, value later (a prefetch must not wait for its conversion)
__device__ __forceinline__ uint32_t hd_raw(const void* p, int64_t i, int dtype) {
    return dtype == SLLM_F32 ? reinterpret_cast<const uint32_t*>(p)[i] : (uint32_t) reinterpret_cast<const unsigned short*>(p)[i];
}
__device__ __forceinline__ float hd_val(uint32_t raw, int dtype) {
    if (dtype == SLLM_F32) return __uint_as_float(raw);
    if (dtype == SLLM_BF16) return __uint_as_float(raw << 16);
    return __half2float(__ushort_as_half((unsigned short)raw));
}
__device__ __forceinline__ float hd_load(const void* p, int64_t i, int dtype) { return hd_val(hd_raw(p, i, dtype), dtype); }
__device__ __forceinline__ void hd_store(void* p, int64_t i, float v, int dtype) {
    if (dtype == SLLM_F32) reinterpret_cast<float*>(p)[i] = v;
    else if (dtype == SLLM_BF16) reinterpret_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16_rn(v);
    else reinterpret_cast<__half*>(p)[i] = __float2half_rn(v);
}

__device__ __forceinline__ float hd_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float hd_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// one token's gates.  DELTA: a = log decay, b = beta.  memory: a = log forget gate, b = log input gate.
template <bool DELTA> __device__ __forceinline__ void hd_gates(const HeadDecayArgs& p, int64_t t, int h, float& a, float& b) {
    const float za = p.ga[t * p.ga_stride + h], zb = p.gb[t * p.gb_stride + h];
    if constexpr (DELTA) {
        a = -p.pb[h] * hd_softplus(za + p.pa[h]);
        b = hd_sigmoid(zb);
    } else {
        a = -hd_softplus(-p.cap * tanhf((za + p.pa[h]) / p.cap));
        b = p.cap * tanhf((zb + p.pb[h]) / p.cap);
    }
}

template <bool DELTA> __device__ __forceinline__ float hd_out_gate(const HeadDecayArgs& p, int64_t t, int64_t col) {
    const float z = hd_load(p.gate, t * p.gate_stride + col, p.dtype);
    return DELTA ? z * hd_sigmoid(z) : hd_sigmoid(z);
}

// Adds up v[8][N] over the eight lanes of a row group (lane bits 0 .. 2 from bit FIRST on); columns are split between the lanes as long
// as there is more than one left.  `col`: which of the N columns this lane ends up with.
template <int BIT, int N> __device__ __forceinline__ void hd_reduce(float (&v)[HD_TOKENS][N], int lane, int& col, float (&r)[HD_TOKENS]) {
    if constexpr (BIT < 3 && N > 1) {
        constexpr int M = N / 2;
        const bool hi = (lane >> BIT) & 1;
        float w[HD_TOKENS][M];
#pragma unroll
        for (int j = 0; j < HD_TOKENS; j++)
#pragma unroll
            for (int c = 0; c < M; c++) {
                const float give = hi ? v[j][c] : v[j][c + M], keep = hi ? v[j][c + M] : v[j][c];
                w[j][c] = keep + __shfl_xor_sync(0xffffffffu, give, 1 << BIT);
            }
        col += hi ? M : 0;
        hd_reduce<BIT + 1, M>(w, lane, col, r);
    } else if constexpr (BIT < 3) {
#pragma unroll
        for (int j = 0; j < HD_TOKENS; j++) v[j][0] += __shfl_xor_sync(0xffffffffu, v[j][0], 1 << BIT);
        hd_reduce<BIT + 1, N>(v, lane, col, r);
    } else {
        static_assert(N == 1, "at most eight columns per lane");
#pragma unroll
        for (int j = 0; j < HD_TOKENS; j++) r[j] = v[j][0];
    }
}

template <bool DELTA, int R, int CPT> constexpr int hd_prompt_smem_floats() {
    constexpr int P = 8 * R + 4, COLS = 32 * CPT;
    return 2 * (2 * HD_TOKENS * P + HD_TOKENS * COLS + 2 * HD_TOKENS)   // q, k, v, gates (two batches)
           + HD_TOKENS * COLS                                            // read-outs
           + (DELTA ? HD_TOKENS * COLS : 8 * R)                          // scaled u | n
           + 2 * HD_TOKENS * HD_TOKENS + 4 * HD_TOKENS;                  // the small matrices, D(j), D(l, last), beta | 1 / denominator, m
}

// grid (segments, heads, ceil(dv / (32 CPT))), 256 threads
template <bool DELTA, int R, int CPT>
__global__ void __launch_bounds__(HD_WARPS * 32) hd_prompt_kernel(const HeadDecayArgs p) {
    constexpr int DKP = 8 * R, P = DKP + 4, COLS = 32 * CPT, NQ = DKP / 32;
    extern __shared__ __align__(16) float hd_smem[];
    float* qs = hd_smem;                                                 // [2][HD_TOKENS][P]
    float* ks = qs + 2 * HD_TOKENS * P;                                  // [2][HD_TOKENS][P]
    float* vs = ks + 2 * HD_TOKENS * P;                                  // [2][HD_TOKENS][COLS]
    float* ga = vs + 2 * HD_TOKENS * COLS;                               // [2][HD_TOKENS]
    float* gb = ga + 2 * HD_TOKENS;                                      // [2][HD_TOKENS]
    float* os = gb + 2 * HD_TOKENS;                                      // [HD_TOKENS][COLS]
    float* M1 = os + HD_TOKENS * COLS;                                   // [j][l]: D(l, j) k_l . k_j
    float* M2 = M1 + HD_TOKENS * HD_TOKENS;                              // [j][l]: D(l, j) k_l . q_j (memory: times e^(i_l - m_l))
    float* dj = M2 + HD_TOKENS * HD_TOKENS;                              // [j]: D(j)
    float* tail = dj + HD_TOKENS;                                        // [l]: D(l, last) (memory: times e^(i_l - m_l))
    float* bj = tail + HD_TOKENS;                                        // [j]: beta | 1 / denominator
    float* us = bj + 2 * HD_TOKENS;                                      // DELTA: [HD_TOKENS][COLS] u_l D(l, last);  memory: n [DKP]
    const int h = blockIdx.y, b = blockIdx.x;
    const int t0 = p.seg_starts[b], n = p.seg_starts[b + 1] - t0;
    if (n <= 0) return;
    const int seq = p.seq_ids[b], dk = p.dk, dv = p.dv, g = h / (p.H / p.G), dtype = p.dtype;
    const bool fresh = p.tok_pos[t0] == 0;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane & 7, cg = lane >> 3;
    const int cta_col = blockIdx.z * COLS, col_l = warp * 4 * CPT + cg * CPT;      // this lane's first column, in the CTA
    const bool sliced = gridDim.z > 1;
    float* st = p.state + ((int64_t)seq * p.H + h) * dk * dv;
    float S[R][CPT];
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int d = 32 * (r >> 2) + 4 * rg + (r & 3);
#pragma unroll
        for (int c = 0; c < CPT; c++) {
            const int col = cta_col + col_l + c;
            S[r][c] = (!fresh && d < dk && col < dv) ? st[(int64_t)d * dv + col] : 0.f;
        }
    }
    float m_run = 0.f;
    if constexpr (!DELTA) {
        const float* ns = p.nstate + ((int64_t)seq * p.H + h) * dk;
        for (int d = tid; d < DKP; d += HD_WARPS * 32) us[d] = (!fresh && d < dk) ? ns[d] : 0.f;
        if (!fresh) m_run = p.mstate[(int64_t)seq * p.H + h];
    }
    uint32_t rq[NQ], rk[NQ], rv[CPT];
    float fa = 0.f, fb = 0.f;
    auto fetch = [&](int i0) {                                           // warp w: token w of the batch
        const int64_t t = t0 + i0 + warp;
        const bool live = i0 + warp < n;
#pragma unroll
        for (int e = 0; e < NQ; e++) {
            const int d = lane + 32 * e;
            const bool ok = live && d < dk;
            rq[e] = ok ? hd_raw(p.q, t * p.q_stride + (int64_t)g * dk + d, dtype) : 0u;
            rk[e] = ok ? hd_raw(p.k, t * p.k_stride + (int64_t)g * dk + d, dtype) : 0u;
        }
#pragma unroll
        for (int c = 0; c < CPT; c++) {
            const int col = cta_col + lane + 32 * c;
            rv[c] = live && col < dv ? hd_raw(p.v, t * p.v_stride + (int64_t)h * dv + col, dtype) : 0u;
        }
        if (live) hd_gates<DELTA>(p, t, h, fa, fb);
        else { fa = 0.f; fb = DELTA ? 0.f : -INFINITY; }                  // past the end: no decay, nothing written
    };
    // norm, gate and store of batch `i0`'s token `warp` (its read-outs are in `os`)
    auto finish = [&](int i0) {
        if (i0 + warp >= n) return;
        const int64_t t = t0 + i0 + warp;
        float o[CPT], ss = 0.f;
#pragma unroll
        for (int c = 0; c < CPT; c++) {
            o[c] = cta_col + lane + 32 * c < dv ? os[warp * COLS + lane + 32 * c] : 0.f;
            ss += o[c] * o[c];
        }
        const float f = sliced ? 1.f : 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
#pragma unroll
        for (int c = 0; c < CPT; c++) {
            const int col = cta_col + lane + 32 * c;
            if (col >= dv) continue;
            if (sliced) p.o_raw[(t * p.H + h) * dv + col] = o[c];
            else
                hd_store(p.out, t * p.out_stride + (int64_t)h * dv + col,
                         o[c] * f * p.norm_w[h * p.norm_step + col] * hd_out_gate<DELTA>(p, t, (int64_t)h * dv + col), dtype);
        }
    };
    fetch(0);
    for (int i0 = 0; i0 < n; i0 += HD_TOKENS) {
        const int buf = (i0 / HD_TOKENS) & 1;
        float* qb = qs + buf * HD_TOKENS * P;
        float* kb = ks + buf * HD_TOKENS * P;
        float* vb = vs + buf * HD_TOKENS * COLS;
        {
            float x[NQ], y[NQ], fq = p.q_scale, fk = 1.f;
#pragma unroll
            for (int e = 0; e < NQ; e++) { x[e] = hd_val(rq[e], dtype); y[e] = hd_val(rk[e], dtype); }
            if constexpr (DELTA) {
                float sq = 0.f, sk = 0.f;
#pragma unroll
                for (int e = 0; e < NQ; e++) { sq += x[e] * x[e]; sk += y[e] * y[e]; }
                fq *= 1.f / sqrtf(warp_sum(sq) + HD_UNIT_EPS);
                fk = 1.f / sqrtf(warp_sum(sk) + HD_UNIT_EPS);
            }
#pragma unroll
            for (int e = 0; e < NQ; e++) {
                qb[warp * P + lane + 32 * e] = x[e] * fq;
                kb[warp * P + lane + 32 * e] = y[e] * fk;
            }
#pragma unroll
            for (int c = 0; c < CPT; c++) vb[warp * COLS + lane + 32 * c] = hd_val(rv[c], dtype);
            if (lane == 0) { ga[buf * HD_TOKENS + warp] = fa; gb[buf * HD_TOKENS + warp] = fb; }
        }
        __syncthreads();                                                 // the batch is staged; the last one's read-outs are in `os`
        if (i0 + HD_TOKENS < n) fetch(i0 + HD_TOKENS);                   // in flight while this batch is worked on
        if (i0 > 0) finish(i0 - HD_TOKENS);
        // ---- row `warp` of the small matrices: lane = (l, quarter of the head)
        {
            float lg[HD_TOKENS], wl[HD_TOKENS], floor_j = 0.f;
#pragma unroll
            for (int i = 0; i < HD_TOKENS; i++) {
                const float a = ga[buf * HD_TOKENS + i], bb = gb[buf * HD_TOKENS + i];
                if constexpr (DELTA) {
                    lg[i] = a;
                    wl[i] = bb;                                          // beta
                } else {
                    const float m_new = fmaxf(a + m_run, bb);
                    lg[i] = a + m_run - m_new;
                    wl[i] = expf(bb - m_new);
                    m_run = m_new;
                    if (i == warp) floor_j = expf(-m_new);
                }
            }
            const int l = lane & 7, quarter = lane >> 3;
            float sum = 0.f, upto = 0.f, w_l = 0.f;
#pragma unroll
            for (int i = 0; i < HD_TOKENS; i++) {
                if (i > l && i <= warp) sum += lg[i];
                if (i <= warp) upto += lg[i];
                if (i == l) w_l = wl[i];
            }
            float kk = 0.f, kq = 0.f, nq = 0.f;
            const float* kl = kb + l * P + quarter * (DKP / 4);
            const float* kj = kb + warp * P + quarter * (DKP / 4);
            const float* qj = qb + warp * P + quarter * (DKP / 4);
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
            const float D = expf(sum), d_upto = expf(upto);
            const float m2 = l <= warp ? D * kq * (DELTA ? 1.f : w_l) : 0.f;
            if constexpr (!DELTA) {
                for (int d = lane; d < DKP; d += 32) nq += us[d] * qb[warp * P + d];
                nq = warp_sum(nq) * d_upto;
                float in = m2;                                           // every quarter holds the same eight entries
                in += __shfl_xor_sync(0xffffffffu, in, 1);
                in += __shfl_xor_sync(0xffffffffu, in, 2);
                in += __shfl_xor_sync(0xffffffffu, in, 4);
                nq += in;
            }
            if (quarter == 0) {
                if constexpr (DELTA) M1[warp * HD_TOKENS + l] = l < warp ? D * kk : 0.f;
                M2[warp * HD_TOKENS + l] = m2;
                if (warp == HD_TOKENS - 1) tail[l] = D * (DELTA ? 1.f : w_l);
                if (l == 0) dj[warp] = d_upto;
                if (l == warp) bj[warp] = DELTA ? w_l : 1.f / (fmaxf(fabsf(nq), floor_j) + HD_DEN_EPS);
            }
        }
        // ---- the state against the batch's vectors
        float r[HD_TOKENS];
        int mine = 0;                                                    // which of the lane's columns r belongs to
        {
            float accB[HD_TOKENS][CPT];
            float accA[DELTA ? HD_TOKENS : 1][CPT];
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++)
#pragma unroll
                for (int c = 0; c < CPT; c++) {
                    accB[j][c] = 0.f;
                    if constexpr (DELTA) accA[j][c] = 0.f;
                }
#pragma unroll
            for (int i = 0; i < R / 4; i++) {
#pragma unroll
                for (int j = 0; j < HD_TOKENS; j++) {
                    const float4 q4 = *reinterpret_cast<const float4*>(qb + j * P + 32 * i + 4 * rg);
                    const float qe[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                    for (int e = 0; e < 4; e++)
#pragma unroll
                        for (int c = 0; c < CPT; c++) accB[j][c] = fmaf(S[4 * i + e][c], qe[e], accB[j][c]);
                    if constexpr (DELTA) {
                        const float4 k4 = *reinterpret_cast<const float4*>(kb + j * P + 32 * i + 4 * rg);
                        const float ke[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                        for (int e = 0; e < 4; e++)
#pragma unroll
                            for (int c = 0; c < CPT; c++) accA[j][c] = fmaf(S[4 * i + e][c], ke[e], accA[j][c]);
                    }
                }
            }
            if constexpr (DELTA) {                                       // even lanes take S^T k, odd lanes S^T q
                const bool odd = lane & 1;
                float z[HD_TOKENS][CPT];
#pragma unroll
                for (int j = 0; j < HD_TOKENS; j++)
#pragma unroll
                    for (int c = 0; c < CPT; c++) {
                        const float give = odd ? accA[j][c] : accB[j][c], keep = odd ? accB[j][c] : accA[j][c];
                        z[j][c] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
                    }
                hd_reduce<1, CPT>(z, lane, mine, r);
            } else {
                hd_reduce<0, CPT>(accB, lane, mine, r);
            }
        }
        __syncthreads();                                                 // the small matrices are written, `os` is read
        // ---- one column per lane (several lanes hold the same one): the triangular system and the read-outs
        const int col = col_l + mine;
        if constexpr (DELTA) {
            float u[HD_TOKENS];
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++) {
                float pre = dj[j] * r[j];
#pragma unroll
                for (int l = 0; l < j; l++) pre = fmaf(M1[j * HD_TOKENS + l], u[l], pre);
                u[j] = bj[j] * (vb[j * COLS + col] - pre);
            }
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++) u[j] = __shfl_sync(0xffffffffu, u[j], lane & ~1);
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++) {
                float o = dj[j] * r[j];
#pragma unroll
                for (int l = 0; l <= j; l++) o = fmaf(M2[j * HD_TOKENS + l], u[l], o);
                if (lane & 1) os[j * COLS + col] = o;
                else us[j * COLS + col] = u[j] * tail[j];
            }
            __syncwarp();
        } else {
#pragma unroll
            for (int j = 0; j < HD_TOKENS; j++) {
                float o = dj[j] * r[j];
#pragma unroll
                for (int l = 0; l <= j; l++) o = fmaf(M2[j * HD_TOKENS + l], vb[l * COLS + col], o);
                os[j * COLS + col] = o * bj[j];
            }
            for (int d = tid; d < DKP; d += HD_WARPS * 32) {             // read again only behind the next barrier
                float x = us[d] * dj[HD_TOKENS - 1];
#pragma unroll
                for (int l = 0; l < HD_TOKENS; l++) x = fmaf(tail[l], kb[l * P + d], x);
                us[d] = x;
            }
        }
        // ---- the state moves on
        const float keep = dj[HD_TOKENS - 1];
#pragma unroll
        for (int r_ = 0; r_ < R; r_++)
#pragma unroll
            for (int c = 0; c < CPT; c++) S[r_][c] *= keep;
#pragma unroll
        for (int l = 0; l < HD_TOKENS; l++) {
            float w[CPT];
#pragma unroll
            for (int c = 0; c < CPT; c++)
                w[c] = DELTA ? us[l * COLS + col_l + c] : vb[l * COLS + col_l + c] * tail[l];
#pragma unroll
            for (int i = 0; i < R / 4; i++) {
                const float4 k4 = *reinterpret_cast<const float4*>(kb + l * P + 32 * i + 4 * rg);
                const float ke[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int e = 0; e < 4; e++)
#pragma unroll
                    for (int c = 0; c < CPT; c++) S[4 * i + e][c] = fmaf(ke[e], w[c], S[4 * i + e][c]);
            }
        }
    }
    __syncthreads();
    finish((n - 1) / HD_TOKENS * HD_TOKENS);
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int d = 32 * (r >> 2) + 4 * rg + (r & 3);
#pragma unroll
        for (int c = 0; c < CPT; c++) {
            const int col = cta_col + col_l + c;
            if (d < dk && col < dv) st[(int64_t)d * dv + col] = S[r][c];
        }
    }
    if constexpr (!DELTA) {
        if (blockIdx.z != 0) return;
        // another CTA of this head may not have read the old n and m yet: they wait in `carry` for the head norm's launch
        float* ns = sliced ? p.carry + ((int64_t)b * p.H + h) * (dk + 1) : p.nstate + ((int64_t)seq * p.H + h) * dk;
        for (int d = tid; d < dk; d += HD_WARPS * 32) ns[d] = us[d];
        if (tid == 0) *(sliced ? ns + dk : p.mstate + (int64_t)seq * p.H + h) = m_run;
    }
}

// One warp per (row, head): the norm and the gate of a head whose columns several CTAs computed (prompt portions' rows are the first).
template <bool DELTA>
__global__ void __launch_bounds__(256) hd_norm_kernel(const HeadDecayArgs p, int64_t units) {
    const int lane = threadIdx.x & 31;
    const int64_t unit = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= units) return;
    const int64_t t = unit / p.H;
    const int h = (int)(unit % p.H);
    const float* o = p.o_raw + unit * p.dv;
    float ss = 0.f;
    for (int d = lane; d < p.dv; d += 32) ss += o[d] * o[d];
    const float f = 1.f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
    for (int d = lane; d < p.dv; d += 32)
        hd_store(p.out, t * p.out_stride + (int64_t)h * p.dv + d,
                 o[d] * f * p.norm_w[h * p.norm_step + d] * hd_out_gate<DELTA>(p, t, (int64_t)h * p.dv + d), p.dtype);
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

// One single decoded token: grid (segments, heads), 8 warps.  Warp w takes state rows w, w + 8, .. (RB of them, in registers between the
// read and the write), a lane V neighbouring columns of each 32 V.  Dynamic shared memory: (16 + 2) * 32 V + 2 dk + 2 dv floats.
template <bool DELTA, int V, int RB>
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
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dk = p.dk, dv = p.dv, g = h / (p.H / p.G), dtype = p.dtype;
    const bool fresh = p.tok_pos[t] == 0;
    const int64_t row = (int64_t)p.seq_ids[b] * p.H + h;
    float* st = p.state + row * dk * dv;
    float S[RB][V];
    auto load_rows = [&](int c0) {
#pragma unroll
        for (int r = 0; r < RB; r++) {
            const int d = warp + r * HD_WARPS;
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
    load_rows(lane * V);                                                // in flight while the vectors are staged
    float ga, gb;
    hd_gates<DELTA>(p, t, h, ga, gb);
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
    float s0 = 0.f, s1 = 0.f, s2 = 0.f;                                 // DELTA: q.q, k.k, k.q;  memory: n.q, -, k.q
    for (int d = tid; d < dk; d += HD_WARPS * 32) {
        const float x = hd_load(p.q, t * p.q_stride + (int64_t)g * dk + d, dtype), y = hd_load(p.k, t * p.k_stride + (int64_t)g * dk + d, dtype);
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
    for (int d = tid; d < dv; d += HD_WARPS * 32) vv[d] = hd_load(p.v, t * p.v_stride + (int64_t)h * dv + d, dtype);
    s0 = warp_sum(s0); s1 = warp_sum(s1); s2 = warp_sum(s2);
    if (lane == 0) { sums[0][warp] = s0; sums[1][warp] = s1; sums[2][warp] = s2; }
    __syncthreads();                                                    // (memory: every thread has read m)
    s0 = s1 = s2 = 0.f;
#pragma unroll
    for (int w = 0; w < HD_WARPS; w++) { s0 += sums[0][w]; s1 += sums[1][w]; s2 += sums[2][w]; }
    float fq = p.q_scale, fk = 1.f, inv_den = 1.f;
    if constexpr (DELTA) {
        fq *= 1.f / sqrtf(s0 + HD_UNIT_EPS);
        fk = 1.f / sqrtf(s1 + HD_UNIT_EPS);
    } else {
        inv_den = 1.f / (fmaxf(fabsf(s0 * fq), expf(-m_new)) + HD_DEN_EPS);
        if (tid == 0) p.mstate[row] = m_new;
    }
    const float kq = s2 * fq * fk;
    for (int cb = 0; cb < dv; cb += CB) {
        const int c0 = cb + lane * V;
        if (cb > 0) load_rows(c0);
        float A[V], B[V];
#pragma unroll
        for (int c = 0; c < V; c++) A[c] = B[c] = 0.f;
#pragma unroll
        for (int r = 0; r < RB; r++) {
            const int d = warp + r * HD_WARPS;
            const float y = d < dk ? kv[d] : 0.f, x = d < dk ? qv[d] : 0.f;
#pragma unroll
            for (int c = 0; c < V; c++) {
                if constexpr (DELTA) A[c] = fmaf(S[r][c], y, A[c]);
                B[c] = fmaf(S[r][c], x, B[c]);
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
        float u[V];
#pragma unroll
        for (int c = 0; c < V; c++) {
            const float val = c0 + c < dv ? vv[c0 + c] : 0.f;
            if constexpr (DELTA) u[c] = take * (val - decay * fk * tot[lane * V + c]);
            else u[c] = take * val;
            if (warp == 0 && c0 + c < dv) ov[c0 + c] = (decay * fq * tot[CB + lane * V + c] + kq * u[c]) * inv_den;
            u[c] *= fk;
        }
        if (c0 < dv) {
#pragma unroll
            for (int r = 0; r < RB; r++) {
                const int d = warp + r * HD_WARPS;
                if (d >= dk) break;
                const float y = kv[d];
                float* s = st + (int64_t)d * dv + c0;
#pragma unroll
                for (int c = 0; c < V; c++) S[r][c] = fmaf(decay, S[r][c], y * u[c]);
                if constexpr (V == 4) *reinterpret_cast<float4*>(s) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
                else *s = S[r][0];
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int d = tid; d < dv; d += HD_WARPS * 32) ss += ov[d] * ov[d];
    const float f = 1.f / sqrtf(block_sum(ss, bsum) / (float)dv + p.eps);
    for (int d = tid; d < dv; d += HD_WARPS * 32)
        hd_store(p.out, t * p.out_stride + (int64_t)h * dv + d,
                 ov[d] * f * p.norm_w[h * p.norm_step + d] * hd_out_gate<DELTA>(p, t, (int64_t)h * dv + d), dtype);
}

// ---------------------------------------------------------------- launchers
template <bool DELTA, int R, int CPT> static int hd_launch_prompt(const HeadDecayArgs& a, cudaStream_t stream) {
    static unsigned long long attr_mask = 0;
    auto kern = hd_prompt_kernel<DELTA, R, CPT>;
    const size_t smem = sizeof(float) * hd_prompt_smem_floats<DELTA, R, CPT>();
    if (first_use_on_this_device(attr_mask)) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    kern<<<dim3((unsigned)a.num_segs, (unsigned)a.H, (unsigned)cdiv(a.dv, 32 * CPT)), HD_WARPS * 32, smem, stream>>>(a);
    return cdiv(a.dv, 32 * CPT);
}

template <bool DELTA> static int hd_run(HeadDecayArgs a, int64_t num_tokens, int64_t num_prefill_tokens, int num_prefill_segs,
                                        int64_t workspace_floats, cudaStream_t s) {
    const int total_segs = a.num_segs;
    SLLM_REQUIRE(num_tokens >= 0 && total_segs >= 0 && a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.dk > 0 && a.dv > 0 &&
                 a.dk <= 512 && a.dv <= 4096, "head decay: bad shape (heads %d / %d, dk %d <= 512, dv %d <= 4096)", a.H, a.G, a.dk, a.dv);
    SLLM_REQUIRE(a.dtype == SLLM_F16 || a.dtype == SLLM_BF16 || a.dtype == SLLM_F32, "head decay: unknown dtype tag %d", a.dtype);
    SLLM_REQUIRE(num_prefill_segs >= 0 && num_prefill_segs <= total_segs && num_prefill_tokens >= 0 && num_prefill_tokens <= num_tokens &&
                 num_tokens - num_prefill_tokens == total_segs - num_prefill_segs,
                 "head decay: %d prompt segments of %d with %lld of %lld tokens: every other segment is one token", num_prefill_segs,
                 total_segs, (long long)num_prefill_tokens, (long long)num_tokens);
    if (num_tokens == 0 || total_segs == 0) return 0;
    SLLM_REQUIRE(a.q && a.k && a.v && a.gate && a.ga && a.gb && a.pa && a.pb && a.norm_w && a.state && a.seg_starts && a.seq_ids &&
                 a.tok_pos && a.out && (DELTA || (a.nstate && a.mstate)), "head decay: null pointer");
    if (num_prefill_segs > 0 && num_prefill_tokens > 0) {
        const int64_t raw = num_prefill_tokens * a.H * a.dv, carry = DELTA ? 0 : (int64_t)num_prefill_segs * a.H * (a.dk + 1);
        SLLM_REQUIRE(a.o_raw && workspace_floats >= raw + carry, "head decay: workspace of %lld floats, need %lld",
                     (long long)workspace_floats, (long long)(raw + carry));
        a.carry = a.o_raw + raw;
        a.num_segs = num_prefill_segs;
        int num_sms = 0;
        cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, current_device());
        // columns per lane: a whole head per CTA where segments x heads fill the GPU, else the widest slice that still does
        const int64_t units = (int64_t)num_prefill_segs * a.H;
        const int rows = cdiv(a.dk, 8);
        int want = 1;
        if (a.dv > 64 && units * cdiv(a.dv, 128) >= num_sms) want = 4;
        else if (a.dv > 32 && units * cdiv(a.dv, 64) >= num_sms) want = 2;
        int slices;
        if (rows <= 8) slices = want >= 4 ? hd_launch_prompt<DELTA, 8, 4>(a, s) : want >= 2 ? hd_launch_prompt<DELTA, 8, 2>(a, s) : hd_launch_prompt<DELTA, 8, 1>(a, s);
        else if (rows <= 16) slices = want >= 4 ? hd_launch_prompt<DELTA, 16, 4>(a, s) : want >= 2 ? hd_launch_prompt<DELTA, 16, 2>(a, s) : hd_launch_prompt<DELTA, 16, 1>(a, s);
        else if (rows <= 32) slices = want >= 2 ? hd_launch_prompt<DELTA, 32, 2>(a, s) : hd_launch_prompt<DELTA, 32, 1>(a, s);
        else slices = hd_launch_prompt<DELTA, 64, 1>(a, s);
        if (check_launch("head decay (prompt portions)")) return 1;
        if (slices > 1) {
            const int64_t n = num_prefill_tokens * a.H;
            hd_norm_kernel<DELTA><<<(unsigned)cdiv(n, 8), 256, 0, s>>>(a, n);
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
        const dim3 grid((unsigned)a.num_segs, (unsigned)a.H);
        const bool wide = a.dv % 4 == 0 && ((uintptr_t)a.state & 15) == 0 && a.dk <= 256;
        const size_t smem = sizeof(float) * (18 * 32 * (wide ? 4 : 1) + 2 * (size_t)a.dk + 2 * (size_t)a.dv);
        static unsigned long long attr_mask = 0;
        if (first_use_on_this_device(attr_mask)) {
            cudaFuncSetAttribute(hd_decode_kernel<DELTA, 4, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
            cudaFuncSetAttribute(hd_decode_kernel<DELTA, 4, 16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
            cudaFuncSetAttribute(hd_decode_kernel<DELTA, 4, 32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
            cudaFuncSetAttribute(hd_decode_kernel<DELTA, 1, 64>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
        }
        if (!wide) hd_decode_kernel<DELTA, 1, 64><<<grid, HD_WARPS * 32, smem, s>>>(a);
        else if (a.dk <= 64) hd_decode_kernel<DELTA, 4, 8><<<grid, HD_WARPS * 32, smem, s>>>(a);
        else if (a.dk <= 128) hd_decode_kernel<DELTA, 4, 16><<<grid, HD_WARPS * 32, smem, s>>>(a);
        else hd_decode_kernel<DELTA, 4, 32><<<grid, HD_WARPS * 32, smem, s>>>(a);
        return check_launch("head decay (decode)");
    }
    return 0;
}

}  // namespace sllm
