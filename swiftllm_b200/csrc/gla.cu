// Gated linear attention: linear attention whose state decays per KEY CHANNEL by a factor that depends on the token,
//     alpha[t, h, d] = sigmoid(z[t, h, d] + bias[h, d])^(1 / tau),
//     S[h] <- diag(alpha[t, h]) S[h] + k[t, h] v[t, h]^T   (dk x dv per head),      o[t, h] = S[h]^T (q[t, h] * q_scale),
//     out[t, h] = o / sqrt(mean(o^2) + eps) * norm_w * silu(gate[t, h]).
// The state lives per SEQUENCE (row `seq` of a state tensor, the sequence's block-table row), in fp32, and is carried from step to
// step.  A step brings SEGMENTS: rows seg_starts[b] .. seg_starts[b+1] - 1 of the packed batch are consecutive positions of sequence
// seq_ids[b].  A segment that starts at position 0 starts from the zero state whatever its row holds (rows are used again without
// being cleared).  Decays (from fp32 logits z), their logarithms and products, the state, the read-out and the norm are fp32 for
// every storage type T of q, k, v and the gate.
//
// Single decoded tokens: gla_decode_kernel streams the state once (read, update, write) and applies the head's norm and gate.
// Prompt portions: gla_kernel walks a segment's tokens with the state in registers.  When segments x heads are too few CTAs to fill
// the GPU a segment is cut into CHUNKS: one pass gives every chunk's own contribution to the state and its total decay (from the
// zero state, all chunks in parallel), gla_chunk_scan_kernel turns them into the state at every chunk's start, and a second pass
// computes the outputs of all chunks in parallel.  The recurrence is linear in the state, so this is exact algebra; in floating point
// the result differs from the token-by-token walk by rounding only.
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

// The columns of a head's state never mix, so a CTA owns 32 CPT columns of one (segment chunk, head): grid (segments x chunks, heads,
// ceil(dv / (32 CPT))), 8 warps.  Lane j: columns j, j + 32, .. (CPT of them); warp w: rows (key channels) w R .. w R + R - 1, in
// registers for the whole chunk.  Tokens are staged GL_TOKENS at a time; inside a batch the decays are folded into the staged
// vectors: with c_i[d] = sum_{j <= i} log alpha_j[d] the state after token i is e^(c_i) (S_start + sum_{j <= i} e^(-c_j) k_j v_j^T),
// so k_j is staged times e^(-c_j), q_i times e^(c_i), and the update is ONE fused multiply-add per state entry (plus one for the dot
// product); the rows are scaled by e^(c_last) once per batch.  A batch whose c falls below -GL_MAX_FOLD takes the direct form.
// When the CTA owns all columns of the head (norm_w given) the head's norm and gate are applied before `out` (type T) is written;
// otherwise o goes to `o_raw` (fp32 [T, H * dv]) for gla_head_norm_kernel.
// STATE_ONLY: no outputs; the chunk's final state from zero goes to chunk_states and its decays' product to chunk_decays.
// chunk_states [segments, chunks, H, dk, dv] (null: one chunk per segment, which starts from and ends in `state`): the state at each
// chunk's start; the segment's last chunk leaves its final state in `state`.
template <typename T, int R, int CPT, bool STATE_ONLY>
__global__ void __launch_bounds__(GL_WARPS * 32) gla_kernel(
    const T* __restrict__ q, int64_t q_stride, const T* __restrict__ k, int64_t k_stride, const T* __restrict__ v, int64_t v_stride,
    const float* __restrict__ z, int64_t z_stride, const float* __restrict__ bias, float inv_tau, float q_scale,
    float* __restrict__ state, const int* __restrict__ seg_starts, const int* __restrict__ seq_ids, const int* __restrict__ tok_pos,
    float* __restrict__ o_raw, const float* __restrict__ norm_w, float eps, const T* __restrict__ gate, int64_t gate_stride,
    T* __restrict__ out, int64_t out_stride, int H, int dk, int dv, int chunks, int chunk_len, float* __restrict__ chunk_states,
    float* __restrict__ chunk_decays) {
    constexpr int DKP = GL_WARPS * R;                                   // padded rows
    constexpr int COLS = 32 * CPT;
    extern __shared__ __align__(16) unsigned char gl_smem[];
    float (*qs)[DKP] = reinterpret_cast<float (*)[DKP]>(gl_smem);                                    // [GL_TOKENS][DKP]
    float (*ks)[DKP] = qs + GL_TOKENS;
    float (*as)[DKP] = ks + GL_TOKENS;                                                                // log alpha, or alpha (direct form)
    float* es = reinterpret_cast<float*>(as + GL_TOKENS);                                             // [DKP] e^(c_last)
    float (*vs)[COLS] = reinterpret_cast<float (*)[COLS]>(es + DKP);                                  // [GL_TOKENS][COLS]
    float (*red)[GL_TOKENS][COLS] = reinterpret_cast<float (*)[GL_TOKENS][COLS]>(vs + GL_TOKENS);     // [GL_WARPS][GL_TOKENS][COLS]
    const int b = blockIdx.x / chunks, chunk = blockIdx.x - b * chunks, h = blockIdx.y;
    const int seg0 = seg_starts[b], seg_n = seg_starts[b + 1] - seg0;
    const int t0 = seg0 + chunk * chunk_len, n = min(chunk_len, seg_n - chunk * chunk_len);
    const bool last = chunk * chunk_len + n >= seg_n;                   // the segment's last chunk
    if (n <= 0 || (STATE_ONLY && last)) return;                         // nothing follows the last chunk inside the segment
    const int seq = seq_ids[b];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int col0 = blockIdx.z * COLS + lane;                          // this thread's columns: col0 + 32 c
    float* st = state + ((int64_t)seq * H + h) * dk * dv;
    float* cst = chunk_states != nullptr ? chunk_states + ((int64_t)blockIdx.x * H + h) * dk * dv : nullptr;
    const float* from = STATE_ONLY ? nullptr : cst != nullptr ? cst : tok_pos[seg0] > 0 ? st : nullptr;      // null: the zero state
    float S[R][CPT];
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int d = warp * R + r;
#pragma unroll
        for (int c = 0; c < CPT; c++)
            S[r][c] = (from != nullptr && col0 + 32 * c < dv && d < dk) ? from[(int64_t)d * dv + col0 + 32 * c] : 0.f;
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
                if constexpr (!STATE_ONLY) rq[e] = q[t * q_stride + (int64_t)h * dk + d];
                rk[e] = k[t * k_stride + (int64_t)h * dk + d];
                rz[e] = z[t * z_stride + (int64_t)h * dk + d];
            }
        }
#pragma unroll
        for (int c = 0; c < CPT; c++)
            if (warp < nt && col0 + 32 * c < dv) rv[c] = v[(int64_t)(t0 + i0 + warp) * v_stride + (int64_t)h * dv + col0 + 32 * c];
    };
    fetch(0);
    float total[NQ];                                                    // STATE_ONLY: log decays summed over the chunk, per staged entry
#pragma unroll
    for (int e = 0; e < NQ; e++) total[e] = 0.f;
    for (int i0 = 0; i0 < n; i0 += GL_TOKENS) {
        const int nt = min(GL_TOKENS, n - i0);
        float la[NQ];
#pragma unroll
        for (int e = 0; e < NQ; e++) {
            const int idx = tid + e * (GL_WARPS * 32);
            const int i = idx / DKP, d = idx - i * DKP;
            la[e] = (i < nt && d < dk) ? log_sigmoid(rz[e] + bias[h * dk + d]) * inv_tau : 0.f;
            as[i][d] = la[e];
            if constexpr (STATE_ONLY) total[e] += la[e];
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
            if constexpr (!STATE_ONLY) qs[i][d] = live ? ldf(&rq[e]) * q_scale * up : 0.f;
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
                if constexpr (!STATE_ONLY) qs[i][d] = live ? ldf(&rq[e]) * q_scale : 0.f;
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
                        float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f);
                        if constexpr (!STATE_ONLY) q4 = *reinterpret_cast<const float4*>(&qs[i][warp * R + r]);
                        float4 a4 = make_float4(1.f, 1.f, 1.f, 1.f);
                        if constexpr (!FOLD) a4 = *reinterpret_cast<const float4*>(&as[i][warp * R + r]);
                        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w}, aa[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
                        for (int e = 0; e < 4; e++) {
#pragma unroll
                            for (int c = 0; c < CPT; c++) {
                                if constexpr (FOLD) S[r + e][c] = fmaf(kk[e], vj[c], S[r + e][c]);
                                else S[r + e][c] = fmaf(aa[e], S[r + e][c], kk[e] * vj[c]);
                                if constexpr (!STATE_ONLY) part[c] = fmaf(S[r + e][c], qq[e], part[c]);
                            }
                        }
                    }
                }
                if constexpr (!STATE_ONLY) {
#pragma unroll
                    for (int c = 0; c < CPT; c++) red[warp][i][lane + 32 * c] = part[c];
                }
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
        if (!STATE_ONLY && warp < nt) {     // warp i adds up token i
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
    if (STATE_ONLY || last) {
        float* to = STATE_ONLY ? cst : st;
#pragma unroll
        for (int r = 0; r < R; r++) {
            const int d = warp * R + r;
#pragma unroll
            for (int c = 0; c < CPT; c++)
                if (col0 + 32 * c < dv && d < dk) to[(int64_t)d * dv + col0 + 32 * c] = S[r][c];
        }
    }
    if constexpr (STATE_ONLY) {
        if (blockIdx.z != 0) return;                                    // uniform over the CTA
        __syncthreads();                                                // `as` is done with
#pragma unroll
        for (int e = 0; e < NQ; e++) {
            const int idx = tid + e * (GL_WARPS * 32);
            as[idx / DKP][idx % DKP] = total[e];
        }
        __syncthreads();
        for (int d = tid; d < dk; d += GL_WARPS * 32) {
            float c = 0.f;
#pragma unroll
            for (int i = 0; i < GL_TOKENS; i++) c += as[i][d];
            chunk_decays[((int64_t)blockIdx.x * H + h) * dk + d] = expf(c);
        }
    }
}

// chunk_states[segment, c]: in: chunk c's own contribution to the state (chunks 0 .. of the segment but the last); out: the state at
// chunk c's start.  One thread per state entry; grid (segments, heads, ceil(dk * dv / 256)).
__global__ void __launch_bounds__(256) gla_chunk_scan_kernel(const float* __restrict__ state, const int* __restrict__ seg_starts,
                                                             const int* __restrict__ seq_ids, const int* __restrict__ tok_pos,
                                                             float* __restrict__ chunk_states, const float* __restrict__ chunk_decays,
                                                             int H, int dk, int dv, int chunks, int chunk_len) {
    const int b = blockIdx.x, h = blockIdx.y;
    const int64_t size = (int64_t)dk * dv, i = (int64_t)blockIdx.z * blockDim.x + threadIdx.x;
    const int seg0 = seg_starts[b], seg_n = seg_starts[b + 1] - seg0;
    if (i >= size || seg_n <= 0) return;
    const int live = min(chunks, (seg_n + chunk_len - 1) / chunk_len), d = (int)(i / dv);
    float S = tok_pos[seg0] > 0 ? state[((int64_t)seq_ids[b] * H + h) * size + i] : 0.f;
    float* p = chunk_states + (((int64_t)b * chunks) * H + h) * size + i;
    const float* a = chunk_decays + (((int64_t)b * chunks) * H + h) * dk + d;
    const int64_t step = H * size;
    constexpr int AHEAD = 8;                                            // contributions in flight
    for (int c0 = 0; c0 < live; c0 += AHEAD) {
        float add[AHEAD], f[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; j++) {
            const bool more = c0 + j + 1 < live;                        // the last chunk left no contribution
            add[j] = more ? p[j * step] : 0.f;
            f[j] = more ? a[(int64_t)j * H * dk] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < AHEAD; j++) {
            if (c0 + j < live) p[j * step] = S;
            S = f[j] * S + add[j];
        }
        p += AHEAD * step;
        a += (int64_t)AHEAD * H * dk;
    }
}

// One single decoded token: grid (segments, heads), 8 warps.  The head's state is streamed once: warp w takes rows w, w + 8, .., a lane
// V neighbouring columns of each 32 V (V = 4: 16-byte accesses, dv % 4 == 0), RB rows in flight; the partial read-outs of the warps
// meet in shared memory, then the norm and the gate.  Dynamic shared memory: 3 dk + 9 dv floats.
template <typename T, int V, int RB>
__global__ void __launch_bounds__(GL_WARPS * 32) gla_decode_kernel(
    const T* __restrict__ q, int64_t q_stride, const T* __restrict__ k, int64_t k_stride, const T* __restrict__ v, int64_t v_stride,
    const float* __restrict__ z, int64_t z_stride, const float* __restrict__ bias, float inv_tau, float q_scale,
    float* __restrict__ state, const int* __restrict__ seg_starts, const int* __restrict__ seq_ids, const int* __restrict__ tok_pos,
    const float* __restrict__ norm_w, float eps, const T* __restrict__ gate, int64_t gate_stride, T* __restrict__ out,
    int64_t out_stride, int H, int dk, int dv) {
    extern __shared__ __align__(16) unsigned char gl_smem[];
    float* red = reinterpret_cast<float*>(gl_smem);                     // [GL_WARPS][dv]
    float* vv = red + GL_WARPS * dv;                                    // [dv]
    float* qv = vv + dv;                                                // [dk] query, key, decay
    float* kv = qv + dk;
    float* av = kv + dk;
    __shared__ float sums[32];
    const int b = blockIdx.x, h = blockIdx.y;
    const int64_t t = seg_starts[b];
    if (seg_starts[b + 1] <= t) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bool fresh = tok_pos[t] == 0;
    float* st = state + ((int64_t)seq_ids[b] * H + h) * dk * dv;
    float S[RB][V];
    auto load_rows = [&](int d0, int c0) {
#pragma unroll
        for (int r = 0; r < RB; r++) {
            const int d = d0 + r * GL_WARPS;
#pragma unroll
            for (int c = 0; c < V; c++) S[r][c] = 0.f;
            if (!fresh && d < dk && c0 < dv) {
                const float* p = st + (int64_t)d * dv + c0;
                if constexpr (V == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(p);
                    S[r][0] = x.x; S[r][1] = x.y; S[r][2] = x.z; S[r][3] = x.w;
                } else {
                    S[r][0] = *p;
                }
            }
        }
    };
    load_rows(warp, lane * V);                                          // in flight while the vectors are staged
    for (int d = tid; d < dk; d += GL_WARPS * 32) {
        qv[d] = ldf(q + t * q_stride + (int64_t)h * dk + d) * q_scale;
        kv[d] = ldf(k + t * k_stride + (int64_t)h * dk + d);
        av[d] = expf(log_sigmoid(z[t * z_stride + (int64_t)h * dk + d] + bias[h * dk + d]) * inv_tau);
    }
    for (int d = tid; d < dv; d += GL_WARPS * 32) vv[d] = ldf(v + t * v_stride + (int64_t)h * dv + d);
    __syncthreads();
    for (int cb = 0; cb < dv; cb += 32 * V) {
        const int c0 = cb + lane * V;
        float x[V], acc[V];
#pragma unroll
        for (int c = 0; c < V; c++) { x[c] = c0 < dv ? vv[c0 + c] : 0.f; acc[c] = 0.f; }
        for (int d0 = warp; d0 < dk; d0 += RB * GL_WARPS) {
            if (cb > 0 || d0 > warp) load_rows(d0, c0);
#pragma unroll
            for (int r = 0; r < RB; r++) {
                const int d = d0 + r * GL_WARPS;
                if (d >= dk) break;
                const float a = av[d], kk = kv[d], qq = qv[d];
#pragma unroll
                for (int c = 0; c < V; c++) {
                    S[r][c] = fmaf(a, S[r][c], kk * x[c]);
                    acc[c] = fmaf(S[r][c], qq, acc[c]);
                }
                if (c0 < dv) {
                    float* p = st + (int64_t)d * dv + c0;
                    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
                    else *p = S[r][0];
                }
            }
        }
        if (c0 < dv) {
#pragma unroll
            for (int c = 0; c < V; c++) red[warp * dv + c0 + c] = acc[c];
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int d = tid; d < dv; d += GL_WARPS * 32) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < GL_WARPS; w++) o += red[w * dv + d];
        red[d] = o;                                                     // read back by this thread only
        ss += o * o;
    }
    const float f = 1.f / sqrtf(block_sum(ss, sums) / (float)dv + eps);
    for (int d = tid; d < dv; d += GL_WARPS * 32)
        stf(out + t * out_stride + (int64_t)h * dv + d, red[d] * f * norm_w[d] * silu_gate(gate + t * gate_stride + (int64_t)h * dv + d));
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
    int chunks, chunk_len;
    float *chunk_states, *chunk_decays;
};

template <typename T, int R, int CPT, bool STATE_ONLY>
static bool launch_gla_as(const GlaArgs& a, cudaStream_t stream) {
    static unsigned long long attr_mask = 0;
    auto kern = gla_kernel<T, R, CPT, STATE_ONLY>;
    if (first_use_on_this_device(attr_mask)) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
    constexpr int DKP = GL_WARPS * R, COLS = 32 * CPT;
    const size_t smem = sizeof(float) * (3 * GL_TOKENS * DKP + DKP + GL_TOKENS * COLS + (STATE_ONLY ? 0 : GL_WARPS * GL_TOKENS * COLS));
    const bool whole = a.dv <= COLS;
    kern<<<dim3((unsigned)(a.num_segs * a.chunks), (unsigned)a.H, (unsigned)cdiv(a.dv, COLS)), GL_WARPS * 32, smem, stream>>>(
        (const T*)a.q, a.q_stride, (const T*)a.k, a.k_stride, (const T*)a.v, a.v_stride, (const float*)a.z, a.z_stride,
        (const float*)a.bias, a.inv_tau, a.q_scale, (float*)a.state, a.seg_starts, a.seq_ids, a.tok_pos, (float*)a.o_raw,
        whole ? (const float*)a.norm_w : nullptr, a.eps, (const T*)a.gate, a.gate_stride, (T*)a.out, a.out_stride, a.H, a.dk, a.dv,
        a.chunks, a.chunk_len, a.chunk_states, a.chunk_decays);
    return whole;
}

// -> whether the head norm was applied.  want: columns per thread the caller would like (1, 2 or 4); R * CPT <= 64 registers of state.
template <typename T, bool STATE_ONLY>
static bool launch_gla(const GlaArgs& a, int want, cudaStream_t stream) {
    const int rows = cdiv(a.dk, GL_WARPS);                              // state rows per warp, rounded up to 4, 8, 16, 32 or 64
#define GLA_BY_CPT(R, MAXC)                                                                                                    \
    do {                                                                                                                       \
        if (want >= 4 && MAXC >= 4) return launch_gla_as<T, R, (MAXC >= 4 ? 4 : MAXC), STATE_ONLY>(a, stream);                 \
        if (want >= 2 && MAXC >= 2) return launch_gla_as<T, R, (MAXC >= 2 ? 2 : 1), STATE_ONLY>(a, stream);                    \
        return launch_gla_as<T, R, 1, STATE_ONLY>(a, stream);                                                                  \
    } while (0)
    if (rows <= 4) GLA_BY_CPT(4, 4);
    if (rows <= 8) GLA_BY_CPT(8, 4);
    if (rows <= 16) GLA_BY_CPT(16, 4);
    if (rows <= 32) GLA_BY_CPT(32, 2);
    GLA_BY_CPT(64, 1);
#undef GLA_BY_CPT
}

template <typename T>
static int launch_gla_decode(const GlaArgs& a, cudaStream_t stream) {
    const size_t smem = sizeof(float) * (3 * (size_t)a.dk + 9 * (size_t)a.dv);
    static unsigned long long attr_mask = 0;
    auto wide = gla_decode_kernel<T, 4, 8>;
    auto narrow = gla_decode_kernel<T, 1, 8>;
    if (smem > 48 * 1024 && first_use_on_this_device(attr_mask)) {
        cudaFuncSetAttribute(wide, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
        cudaFuncSetAttribute(narrow, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
    }
    (a.dv % 4 == 0 && ((uintptr_t)a.state & 15) == 0 ? wide : narrow)<<<dim3((unsigned)a.num_segs, (unsigned)a.H), GL_WARPS * 32, smem, stream>>>(
        (const T*)a.q, a.q_stride, (const T*)a.k, a.k_stride, (const T*)a.v, a.v_stride, (const float*)a.z, a.z_stride,
        (const float*)a.bias, a.inv_tau, a.q_scale, (float*)a.state, a.seg_starts, a.seq_ids, a.tok_pos, (const float*)a.norm_w, a.eps,
        (const T*)a.gate, a.gate_stride, (T*)a.out, a.out_stride, a.H, a.dk, a.dv);
    return check_launch("gla (decode)");
}

// Chunks per segment for a prompt step whose longest segment has max_len tokens: enough CTAs for about four waves of one CTA per SM,
// chunks of at least 64 tokens, one chunk when the segments alone fill half of that.
static int gla_chunk_count(int64_t num_segs, int64_t max_len, int H, int num_sms) {
    const int64_t units = num_segs * H;
    if (units <= 0 || units >= 2 * (int64_t)num_sms) return 1;
    int64_t n = cdiv((int64_t)4 * num_sms, units);
    if (n > max_len / 64) n = max_len / 64;
    return n < 1 ? 1 : (int)n;
}

}  // namespace sllm

using namespace sllm;

extern "C" {

int64_t sllm_gla_workspace_floats(int64_t num_tokens, int num_prefill_segs, int64_t max_prefill_len, int num_heads, int dk, int dv) {
    int num_sms = 0;
    cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, current_device());
    const int64_t chunks = gla_chunk_count(num_prefill_segs, max_prefill_len, num_heads, num_sms);
    const int64_t per = (int64_t)num_prefill_segs * chunks * num_heads;
    return num_tokens * num_heads * dv + (chunks > 1 ? per * dk * dv + per * dk : 0);
}

int sllm_gla(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride, const void* z,
             int64_t z_stride, const void* bias, float inv_tau, float q_scale, const void* norm_w, float eps, const void* gate,
             int64_t gate_stride, void* state, const void* seg_starts, const void* seq_ids, const void* tok_pos, void* workspace,
             int64_t workspace_floats, void* out, int64_t out_stride, int64_t num_tokens, int64_t num_prefill_tokens, int num_segs,
             int num_prefill_segs, int64_t max_prefill_len, int num_heads, int dk, int dv, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && num_segs >= 0 && num_heads > 0 && dk > 0 && dv > 0 && dk <= 64 * GL_WARPS && dv <= 4096,
                 "gla: bad shape (dk %d <= %d, dv %d <= 4096)", dk, 64 * GL_WARPS, dv);
    SLLM_REQUIRE(num_prefill_segs >= 0 && num_prefill_segs <= num_segs && num_prefill_tokens >= 0 && num_prefill_tokens <= num_tokens &&
                 max_prefill_len >= 0 && max_prefill_len <= num_prefill_tokens &&
                 num_tokens - num_prefill_tokens == num_segs - num_prefill_segs,
                 "gla: %d prompt segments of %d with %lld of %lld tokens: every other segment is one token", num_prefill_segs, num_segs,
                 (long long)num_prefill_tokens, (long long)num_tokens);
    if (num_tokens == 0 || num_segs == 0) return 0;
    SLLM_REQUIRE(q && k && v && z && bias && norm_w && gate && state && seg_starts && seq_ids && tok_pos && workspace && out,
                 "gla: null pointer");
    SLLM_REQUIRE(workspace_floats >= sllm_gla_workspace_floats(num_tokens, num_prefill_segs, max_prefill_len, num_heads, dk, dv),
                 "gla: workspace of %lld floats is too small", (long long)workspace_floats);
    const cudaStream_t s = (cudaStream_t)stream;
    GlaArgs a{q, k, v, z, bias, norm_w, gate, q_stride, k_stride, v_stride, z_stride, gate_stride, out_stride, inv_tau, q_scale, eps,
              state, workspace, out, (const int*)seg_starts, (const int*)seq_ids, (const int*)tok_pos, num_prefill_segs, num_heads, dk, dv,
              1, 0, nullptr, nullptr};
    if (num_prefill_segs > 0 && max_prefill_len > 0) {
        int num_sms = 0;
        cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, current_device());
        a.chunks = gla_chunk_count(num_prefill_segs, max_prefill_len, num_heads, num_sms);
        a.chunk_len = (int)(cdiv(cdiv(max_prefill_len, (int64_t)a.chunks), (int64_t)GL_TOKENS) * GL_TOKENS);
        // columns per thread: a whole head per CTA where the chunks fill the GPU, else the widest slice that still does
        const int64_t units = (int64_t)num_prefill_segs * a.chunks * num_heads;
        int want = 1;
        if (dv > 64 && units * cdiv(dv, 128) >= num_sms) want = 4;
        else if (dv > 32 && units * cdiv(dv, 64) >= num_sms) want = 2;
        if (a.chunks > 1) {
            const int64_t per = (int64_t)num_prefill_segs * a.chunks * num_heads;
            a.chunk_states = (float*)workspace + num_tokens * num_heads * dv;
            a.chunk_decays = a.chunk_states + per * dk * dv;
            SLLM_DISPATCH_DTYPE_F32(dtype, (launch_gla<T, true>(a, want, s)));
            if (check_launch("gla (chunk states)")) return 1;
            gla_chunk_scan_kernel<<<dim3((unsigned)num_prefill_segs, (unsigned)num_heads, (unsigned)cdiv((int64_t)dk * dv, 256)), 256, 0, s>>>(
                (const float*)state, a.seg_starts, a.seq_ids, a.tok_pos, a.chunk_states, a.chunk_decays, num_heads, dk, dv, a.chunks,
                a.chunk_len);
            if (check_launch("gla (chunk scan)")) return 1;
        }
        bool normed = false;
        SLLM_DISPATCH_DTYPE_F32(dtype, (normed = launch_gla<T, false>(a, want, s)));
        if (check_launch("gla")) return 1;
        if (!normed) {
            SLLM_DISPATCH_DTYPE_F32(dtype, (gla_head_norm_kernel<T><<<(unsigned)cdiv(num_prefill_tokens * num_heads, 8), 256, 0, s>>>(
                (const float*)workspace, (const float*)norm_w, eps, (const T*)gate, gate_stride, (T*)out, out_stride, 0,
                num_prefill_tokens * num_heads, num_heads, dv)));
            if (check_launch("gla (head norm)")) return 1;
        }
    }
    if (num_segs > num_prefill_segs) {
        a.seg_starts += num_prefill_segs;
        a.seq_ids += num_prefill_segs;
        a.num_segs = num_segs - num_prefill_segs;
        SLLM_DISPATCH_DTYPE_F32(dtype, return launch_gla_decode<T>(a, s));
    }
    return 0;
}

}  // extern "C"
