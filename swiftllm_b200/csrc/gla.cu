// Gated linear attention: linear attention whose state decays per KEY CHANNEL by a factor that depends on the token,
//     alpha[t, h, d] = sigmoid(z[t, h, d] + bias[h, d])^(1 / tau),
//     S[h] <- diag(alpha[t, h]) S[h] + k[t, h] v[t, h]^T   (dk x dv per head),      o[t, h] = S[h]^T (q[t, h] * q_scale),
//     out[t, h] = o / sqrt(mean(o^2) + eps) * norm_w * silu(gate[t, h]).
// The state lives per SEQUENCE (row `seq` of a state tensor, the sequence's block-table row), in fp32, and is carried from step to
// step.  A step brings SEGMENTS: rows seg_starts[b] .. seg_starts[b+1] - 1 of the packed batch are consecutive positions of sequence
// seq_ids[b].  A segment that starts at position 0 starts from the zero state whatever its row holds (rows are used again without
// being cleared).  Decays (from fp32 logits z), their logarithms and products, the state, the read-out and the norm are fp32 for
// every storage type T of q, k, v and the gate.
#include <type_traits>

#include "mma_helpers.cuh"
#include "typed_io.cuh"

namespace sllm {

constexpr int GL_TOKENS = 8;               // tokens per staged batch
constexpr int GL_WARPS = 8;
// largest decay exponent (natural log, over a batch) that is folded into the staged vectors
constexpr float GL_MAX_FOLD = 40.f;

// log sigmoid(z), without overflow on either side
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

template <typename T> __device__ __forceinline__ float silu_gate(const T* p) {
    const float z = ldf(p);
    return z / (1.f + expf(-z));
}

// The columns of a head's state never mix, so a CTA owns 32 CPT columns of one (segment, head): grid (segments, heads,
// ceil(dv / (32 CPT))), 8 warps.  Lane j: columns j, j + 32, .. (CPT of them); warp w: rows (key channels) w R .. w R + R - 1, in
// registers for the whole segment.  Tokens are staged GL_TOKENS at a time; inside a batch the decays are folded into the staged
// vectors: with c_i[d] = sum_{j <= i} log alpha_j[d] the state after token i is e^(c_i) (S_start + sum_{j <= i} e^(-c_j) k_j v_j^T),
// so k_j is staged times e^(-c_j), q_i times e^(c_i), and the update is ONE fused multiply-add per state entry (plus one for the dot
// product); the rows are scaled by e^(c_last) once per batch.  A batch whose c falls below -GL_MAX_FOLD takes the direct form.
// When the CTA owns all columns of the head (norm_w given) the head's norm and gate are applied before `out` (type T) is written;
// otherwise o goes to `o_raw` (fp32 [T, H * dv]) for gla_head_norm_kernel.
template <typename T, int R, int CPT>
__global__ void __launch_bounds__(GL_WARPS * 32) gla_kernel(
    const T* __restrict__ q, int64_t q_stride, const T* __restrict__ k, int64_t k_stride, const T* __restrict__ v, int64_t v_stride,
    const float* __restrict__ z, int64_t z_stride, const float* __restrict__ bias, float inv_tau, float q_scale,
    float* __restrict__ state, const int* __restrict__ seg_starts, const int* __restrict__ seq_ids, const int* __restrict__ tok_pos,
    float* __restrict__ o_raw, const float* __restrict__ norm_w, float eps, const T* __restrict__ gate, int64_t gate_stride,
    T* __restrict__ out, int64_t out_stride, int H, int dk, int dv) {
    constexpr int DKP = GL_WARPS * R;                                   // padded rows
    constexpr int COLS = 32 * CPT;
    extern __shared__ __align__(16) unsigned char gl_smem[];
    float (*qs)[DKP] = reinterpret_cast<float (*)[DKP]>(gl_smem);                                    // [GL_TOKENS][DKP]
    float (*ks)[DKP] = qs + GL_TOKENS;
    float (*as)[DKP] = ks + GL_TOKENS;                                                                // log alpha, or alpha (direct form)
    float* es = reinterpret_cast<float*>(as + GL_TOKENS);                                             // [DKP] e^(c_last)
    float (*vs)[COLS] = reinterpret_cast<float (*)[COLS]>(es + DKP);                                  // [GL_TOKENS][COLS]
    float (*red)[GL_TOKENS][COLS] = reinterpret_cast<float (*)[GL_TOKENS][COLS]>(vs + GL_TOKENS);     // [GL_WARPS][GL_TOKENS][COLS]
    const int b = blockIdx.x, h = blockIdx.y;
    const int t0 = seg_starts[b], n = seg_starts[b + 1] - t0;
    if (n <= 0) return;
    const int seq = seq_ids[b], p0 = tok_pos[t0];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int col0 = blockIdx.z * COLS + lane;                          // this thread's columns: col0 + 32 c
    float* st = state + ((int64_t)seq * H + h) * dk * dv;
    float S[R][CPT];
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int d = warp * R + r;
#pragma unroll
        for (int c = 0; c < CPT; c++)
            S[r][c] = (col0 + 32 * c < dv && d < dk && p0 > 0) ? st[(int64_t)d * dv + col0 + 32 * c] : 0.f;
    }
    // raw inputs of one batch: NQ entries of q, k and z (entry idx = tid + e * 256 of the padded [GL_TOKENS][DKP] tile), CPT of v
    // (warp i stages token i's columns)
    constexpr int NQ = GL_TOKENS * DKP / (GL_WARPS * 32);
    T rq[NQ], rk[NQ], rv[CPT];
    float rz[NQ];
    auto fetch = [&](int i0) {
        const int nt = min(GL_TOKENS, n - i0);
#pragma unroll
        for (int e = 0; e < NQ; e++) {
            const int idx = tid + e * (GL_WARPS * 32);
            const int i = idx / DKP, d = idx - i * DKP;
            if (i < nt && d < dk) {
                const int64_t t = t0 + i0 + i;
                rq[e] = q[t * q_stride + (int64_t)h * dk + d];
                rk[e] = k[t * k_stride + (int64_t)h * dk + d];
                rz[e] = z[t * z_stride + (int64_t)h * dk + d];
            }
        }
#pragma unroll
        for (int c = 0; c < CPT; c++)
            if (warp < nt && col0 + 32 * c < dv) rv[c] = v[(int64_t)(t0 + i0 + warp) * v_stride + (int64_t)h * dv + col0 + 32 * c];
    };
    fetch(0);
    for (int i0 = 0; i0 < n; i0 += GL_TOKENS) {
        const int nt = min(GL_TOKENS, n - i0);
        float la[NQ];
#pragma unroll
        for (int e = 0; e < NQ; e++) {
            const int idx = tid + e * (GL_WARPS * 32);
            const int i = idx / DKP, d = idx - i * DKP;
            la[e] = (i < nt && d < dk) ? log_sigmoid(rz[e] + bias[h * dk + d]) * inv_tau : 0.f;
            as[i][d] = la[e];
        }
        __syncthreads();
        int steep = 0;
#pragma unroll
        for (int e = 0; e < NQ; e++) {
            const int idx = tid + e * (GL_WARPS * 32);
            const int i = idx / DKP, d = idx - i * DKP;
            float c = 0.f;
            for (int j = 0; j <= i; j++) c += as[j][d];
            steep |= c < -GL_MAX_FOLD;
            const bool live = i < nt && d < dk;
            const float up = expf(c);
            qs[i][d] = live ? ldf(&rq[e]) * q_scale * up : 0.f;
            ks[i][d] = live ? ldf(&rk[e]) * expf(-c) : 0.f;
            if (i == GL_TOKENS - 1) es[d] = up;                         // tokens past the segment's end have log alpha = 0
        }
#pragma unroll
        for (int c = 0; c < CPT; c++) vs[warp][lane + 32 * c] = (warp < nt && col0 + 32 * c < dv) ? ldf(&rv[c]) : 0.f;
        steep = __syncthreads_or(steep);                                // staged (and `as` read) by every thread
        if (steep) {                                                    // direct form: plain vectors beside the decays
#pragma unroll
            for (int e = 0; e < NQ; e++) {
                const int idx = tid + e * (GL_WARPS * 32);
                const int i = idx / DKP, d = idx - i * DKP;
                const bool live = i < nt && d < dk;
                qs[i][d] = live ? ldf(&rq[e]) * q_scale : 0.f;
                ks[i][d] = live ? ldf(&rk[e]) : 0.f;
                as[i][d] = expf(la[e]);
            }
            __syncthreads();
        }
        if (i0 + GL_TOKENS < n) fetch(i0 + GL_TOKENS);                  // in flight while this batch is multiplied
        auto multiply = [&](auto fold) {
            constexpr bool FOLD = decltype(fold)::value;
#pragma unroll
            for (int i = 0; i < GL_TOKENS; i++) {
                float part[CPT];
#pragma unroll
                for (int c = 0; c < CPT; c++) part[c] = 0.f;
                if (i < nt) {                                           // uniform over the CTA
                    float vj[CPT];
#pragma unroll
                    for (int c = 0; c < CPT; c++) vj[c] = vs[i][lane + 32 * c];
#pragma unroll
                    for (int r = 0; r < R; r += 4) {
                        const float4 k4 = *reinterpret_cast<const float4*>(&ks[i][warp * R + r]);
                        const float4 q4 = *reinterpret_cast<const float4*>(&qs[i][warp * R + r]);
                        float4 a4 = make_float4(1.f, 1.f, 1.f, 1.f);
                        if constexpr (!FOLD) a4 = *reinterpret_cast<const float4*>(&as[i][warp * R + r]);
                        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w}, aa[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
                        for (int e = 0; e < 4; e++) {
#pragma unroll
                            for (int c = 0; c < CPT; c++) {
                                if constexpr (FOLD) S[r + e][c] = fmaf(kk[e], vj[c], S[r + e][c]);
                                else S[r + e][c] = fmaf(aa[e], S[r + e][c], kk[e] * vj[c]);
                                part[c] = fmaf(S[r + e][c], qq[e], part[c]);
                            }
                        }
                    }
                }
#pragma unroll
                for (int c = 0; c < CPT; c++) red[warp][i][lane + 32 * c] = part[c];
            }
            if constexpr (FOLD) {
#pragma unroll
                for (int r = 0; r < R; r++) {
                    const float back = es[warp * R + r];
#pragma unroll
                    for (int c = 0; c < CPT; c++) S[r][c] *= back;
                }
            }
        };
        if (steep) multiply(std::false_type{});
        else multiply(std::true_type{});
        __syncthreads();                    // partial sums visible; the staged vectors are done with
        if (warp < nt) {                    // warp i adds up token i
            const int64_t t = t0 + i0 + warp;
            float o[CPT], ss = 0.f;
#pragma unroll
            for (int c = 0; c < CPT; c++) {
                o[c] = 0.f;
                if (col0 + 32 * c < dv) {
#pragma unroll
                    for (int w = 0; w < GL_WARPS; w++) o[c] += red[w][warp][lane + 32 * c];
                    ss += o[c] * o[c];
                }
            }
            if (norm_w != nullptr) {
                const float f = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
#pragma unroll
                for (int c = 0; c < CPT; c++) {
                    const int d = col0 + 32 * c;
                    if (d < dv)
                        stf(out + t * out_stride + (int64_t)h * dv + d,
                            o[c] * f * norm_w[d] * silu_gate(gate + t * gate_stride + (int64_t)h * dv + d));
                }
            } else {
#pragma unroll
                for (int c = 0; c < CPT; c++)
                    if (col0 + 32 * c < dv) o_raw[(t * H + h) * dv + col0 + 32 * c] = o[c];
            }
        }
        // the next batch writes `red` only after its own barriers, which every warp reaches after this read
    }
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int d = warp * R + r;
#pragma unroll
        for (int c = 0; c < CPT; c++)
            if (col0 + 32 * c < dv && d < dk) st[(int64_t)d * dv + col0 + 32 * c] = S[r][c];
    }
}

// One warp per (row, head): the norm and the gate of a head whose columns several CTAs computed.
template <typename T>
__global__ void __launch_bounds__(256) gla_head_norm_kernel(const float* __restrict__ o_raw, const float* __restrict__ norm_w, float eps,
                                                            const T* __restrict__ gate, int64_t gate_stride, T* __restrict__ out,
                                                            int64_t out_stride, int64_t row0, int64_t units, int H, int dv) {
    const int lane = threadIdx.x & 31;
    const int64_t unit = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= units) return;
    const int64_t t = row0 + unit / H;
    const int h = (int)(unit % H);
    const float* o = o_raw + (t * H + h) * dv;
    float ss = 0.f;
    for (int d = lane; d < dv; d += 32) ss += o[d] * o[d];
    const float f = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
    const T* g = gate + t * gate_stride + (int64_t)h * dv;
    for (int d = lane; d < dv; d += 32) stf(out + t * out_stride + (int64_t)h * dv + d, o[d] * f * norm_w[d] * silu_gate(g + d));
}

struct GlaArgs {
    const void *q, *k, *v, *z, *bias, *norm_w, *gate;
    int64_t q_stride, k_stride, v_stride, z_stride, gate_stride, out_stride;
    float inv_tau, q_scale, eps;
    void *state, *o_raw, *out;
    const int *seg_starts, *seq_ids, *tok_pos;
    int num_segs, H, dk, dv;
};

template <typename T, int R, int CPT>
static bool launch_gla_as(const GlaArgs& a, cudaStream_t stream) {
    static unsigned long long attr_mask = 0;
    auto kern = gla_kernel<T, R, CPT>;
    if (first_use_on_this_device(attr_mask)) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
    constexpr int DKP = GL_WARPS * R, COLS = 32 * CPT;
    const size_t smem = sizeof(float) * (3 * GL_TOKENS * DKP + DKP + GL_TOKENS * COLS + GL_WARPS * GL_TOKENS * COLS);
    const bool whole = a.dv <= COLS;
    kern<<<dim3((unsigned)a.num_segs, (unsigned)a.H, (unsigned)cdiv(a.dv, COLS)), GL_WARPS * 32, smem, stream>>>(
        (const T*)a.q, a.q_stride, (const T*)a.k, a.k_stride, (const T*)a.v, a.v_stride, (const float*)a.z, a.z_stride,
        (const float*)a.bias, a.inv_tau, a.q_scale, (float*)a.state, a.seg_starts, a.seq_ids, a.tok_pos, (float*)a.o_raw,
        whole ? (const float*)a.norm_w : nullptr, a.eps, (const T*)a.gate, a.gate_stride, (T*)a.out, a.out_stride, a.H, a.dk, a.dv);
    return whole;
}

// -> whether the head norm was applied.  want: columns per thread the caller would like (1, 2 or 4); R * CPT <= 64 registers of state.
template <typename T>
static bool launch_gla(const GlaArgs& a, int want, cudaStream_t stream) {
    const int rows = cdiv(a.dk, GL_WARPS);                              // state rows per warp, rounded up to 4, 8, 16, 32 or 64
#define GLA_BY_CPT(R, MAXC)                                                                                                    \
    do {                                                                                                                       \
        if (want >= 4 && MAXC >= 4) return launch_gla_as<T, R, (MAXC >= 4 ? 4 : MAXC)>(a, stream);                             \
        if (want >= 2 && MAXC >= 2) return launch_gla_as<T, R, (MAXC >= 2 ? 2 : 1)>(a, stream);                                \
        return launch_gla_as<T, R, 1>(a, stream);                                                                              \
    } while (0)
    if (rows <= 4) GLA_BY_CPT(4, 4);
    if (rows <= 8) GLA_BY_CPT(8, 4);
    if (rows <= 16) GLA_BY_CPT(16, 4);
    if (rows <= 32) GLA_BY_CPT(32, 2);
    GLA_BY_CPT(64, 1);
#undef GLA_BY_CPT
}

}  // namespace sllm

using namespace sllm;

extern "C" {

int sllm_gla(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride, const void* z,
             int64_t z_stride, const void* bias, float inv_tau, float q_scale, const void* norm_w, float eps, const void* gate,
             int64_t gate_stride, void* state, const void* seg_starts, const void* seq_ids, const void* tok_pos, void* o_workspace,
             void* out, int64_t out_stride, int64_t num_tokens, int64_t num_prefill_tokens, int num_segs, int num_prefill_segs,
             int num_heads, int dk, int dv, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && num_segs >= 0 && num_heads > 0 && dk > 0 && dv > 0 && dk <= 64 * GL_WARPS && cdiv(dv, 32) <= 65535,
                 "gla: bad shape (dk %d <= %d, dv %d)", dk, 64 * GL_WARPS, dv);
    SLLM_REQUIRE(num_prefill_segs >= 0 && num_prefill_segs <= num_segs && num_prefill_tokens >= 0 && num_prefill_tokens <= num_tokens,
                 "gla: bad number of prompt segments (%d of %d)", num_prefill_segs, num_segs);
    if (num_tokens == 0 || num_segs == 0) return 0;
    SLLM_REQUIRE(q && k && v && z && bias && norm_w && gate && state && seg_starts && seq_ids && tok_pos && o_workspace && out,
                 "gla: null pointer");
    int num_sms = 0;
    cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, current_device());
    const int64_t parts[2][2] = {{0, num_prefill_segs}, {num_prefill_segs, num_segs - num_prefill_segs}};
    for (int p = 0; p < 2; p++) {
        const int64_t first = parts[p][0], count = parts[p][1];
        if (count <= 0) continue;
        GlaArgs a{q, k, v, z, bias, norm_w, gate, q_stride, k_stride, v_stride, z_stride, gate_stride, out_stride, inv_tau, q_scale, eps,
                  state, o_workspace, out, (const int*)seg_starts + first, (const int*)seq_ids + first, (const int*)tok_pos,
                  (int)count, num_heads, dk, dv};
        // columns per thread: single decoded tokens take a whole head per CTA (the norm is fused); prompt portions the widest
        // slice that still gives every SM a CTA
        const int64_t units = count * num_heads;
        int want = 1;
        if (p == 1) want = dv > 64 ? 4 : dv > 32 ? 2 : 1;
        else if (dv > 64 && units * cdiv(dv, 128) >= num_sms) want = 4;
        else if (dv > 32 && units * cdiv(dv, 64) >= num_sms) want = 2;
        const int64_t row0 = p == 0 ? 0 : num_prefill_tokens, rows = p == 0 ? num_prefill_tokens : num_tokens - num_prefill_tokens;
        bool normed = false;
        SLLM_DISPATCH_DTYPE_F32(dtype, normed = launch_gla<T>(a, want, (cudaStream_t)stream));
        if (check_launch("gla")) return 1;
        if (!normed && rows > 0) {
            SLLM_DISPATCH_DTYPE_F32(dtype, (gla_head_norm_kernel<T><<<(unsigned)cdiv(rows * num_heads, 8), 256, 0, (cudaStream_t)stream>>>(
                (const float*)o_workspace, (const float*)norm_w, eps, (const T*)gate, gate_stride, (T*)out, out_stride, row0,
                rows * num_heads, num_heads, dv)));
            if (check_launch("gla (head norm)")) return 1;
        }
    }
    return 0;
}

}  // extern "C"
