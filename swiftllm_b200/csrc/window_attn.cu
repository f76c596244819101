// Gated sliding-window attention with grouped key/value heads and an optional softmax sink, over a paged cache that holds per
// token and layer ONE row [ k (G heads x dk, rotary applied) | v (G heads x dv) ].
//   score(i, j) = rope(q[i,h]) . k[j, g(h)] * scale          g(h) = h / (H / G)
//   p(i, j)     = exp(score) / (sink + sum_j' exp(score))     sink = 1 when the softmax has a value-less sink of score 0, else 0
//   out[i, h]   = sigmoid(gate[i, h, :]) * sum_j p(i, j) v[j, g(h)]          (element-wise gate; no gate when null)
// Every token of the step is a query with its own (block-table row, position): prompt portions and single decoded tokens go
// through the same kernel, so the result at a position does not depend on how its sequence was cut into steps.  A query at
// position p sees the positions max(0, p - window + 1) .. p (window <= 0: all of 0 .. p).  Rotary pairs are interleaved
// ((2i, 2i+1)) or halves ((i, i + rot_dims/2)) of the first rot_dims entries of a head; the rest pass through; the caller's
// cos / sin tables carry the frequencies (and any common factor on both).  Softmax, rotation and the weighted sum of values
// run in fp32 for every storage type.
// Options that other designs use (all off for the plain gated window attention):
//   qk_norm_eps >= 0   rotated queries and keys are divided by sqrt(mean over the head + eps)
//   softcap > 0        score <- softcap * tanh(score / softcap) after the scale
//   vcos / vsin        the value at position j is stored turned by j (pairs (m, m + dv/2) when `halves`, else (2m, 2m+1), angle
//                      tables [T, dv/2]) and the head's output at position i is turned back by -i
//   out_scale          factor on the output (a mixer that is summed with another one folds its weight here)
//   pre-norm weights   queries / keys are RMS-normed over the head (x / sqrt(mean + prenorm_eps) * weight[dk]) BEFORE they turn
//   chunk > 0          a query at position p sees only keys of its own chunk: positions >= floor(p / chunk) * chunk
//   vshare > 1         `vshare` neighbouring key heads share ONE value head (value head = key head / vshare; the cache row holds
//                      G keys and G / vshare values): several score maps over the same values, each its own query head
//   out_f32            the output is written as fp32 whatever the storage type (a combine step follows)
//   slopes             a bias on the distance: score <- score - slopes[h] * (i - j) after the scale (and cap)
//   keep_first > 0     with a window: the sequence's first keep_first positions stay visible (at their true positions)
//   gate_per_head      ONE gate logit per query head ([T, H]) instead of one per output entry
//   shared_kv          the values are the un-normed keys: the cache row is [ inv (G fp32 values in 2 G elements, rounded up to 8) |
//                      k (G x dk as projected, rounded up to 8) ], inv = 1 / sqrt(mean(k^2) + eps) of the head; the norm's weight
//                      belongs to the query weights (q . (inv k w) = inv (q w) . k), so ONE staged tile serves as K and V
//   krot > 0           shared_kv with rotation: a key head's part of the row is [ k as projected (dk) | its first krot entries times
//                      the norm's weight, turned (not divided by the rms) ], and queries arrive as [ entries krot .. dk - 1 times the
//                      key norm's weight | the turned entries ] (whole_norm_rope_store), so the score is inv q . (columns krot ..
//                      krot + dk - 1 of the key part) and the value its first dk columns
//   sinks              a learned number per head: the softmax's denominator also contains exp(sinks[h])
// diff_combine: per token and head, o = a1 - lambda * a2 of two maps' outputs, o / sqrt(mean(o^2) + eps) * factor * sigmoid(gate).
#include "mma_helpers.cuh"
#include "typed_io.cuh"

namespace sllm {

// entry j of a head row x turned by the token's angles (cs / sn: the token's table rows); entries from rot_dims on pass through
// nw: weight of a norm over the head that comes BEFORE the turn (entry j is x[j] * inv * nw[j]), or null
template <typename T>
__device__ __forceinline__ float pre_entry(const T* __restrict__ x, int j, float inv, const float* __restrict__ nw) {
    const float v = ldf(x + j);
    return nw != nullptr ? v * inv * nw[j] : v;
}
template <typename T>
__device__ __forceinline__ float rot_entry(const T* __restrict__ x, int j, int rot_dims, int halves, const float* __restrict__ cs,
                                           const float* __restrict__ sn, float inv = 1.f, const float* __restrict__ nw = nullptr) {
    if (j >= rot_dims) return pre_entry(x, j, inv, nw);
    if (halves) {
        const int half = rot_dims >> 1;
        if (j < half) return pre_entry(x, j, inv, nw) * cs[j] - pre_entry(x, j + half, inv, nw) * sn[j];
        return pre_entry(x, j, inv, nw) * cs[j - half] + pre_entry(x, j - half, inv, nw) * sn[j - half];
    }
    const int i = j >> 1;
    const float a = pre_entry(x, 2 * i, inv, nw), b = pre_entry(x, 2 * i + 1, inv, nw);
    return (j & 1) ? b * cs[i] + a * sn[i] : a * cs[i] - b * sn[i];
}

// the shared_kv cache row: first element of the keys, elements per row
__host__ __device__ __forceinline__ int shared_kv_key_offset(int G) { return (2 * G + 7) / 8 * 8; }
__host__ __device__ __forceinline__ int shared_kv_row(int G, int dk) { return shared_kv_key_offset(G) + (G * dk + 7) / 8 * 8; }

// bytes between the rows of a shared-memory tile of `cols` 16-bit entries (cols % 8 == 0): an odd number of 16-byte pieces, so that the
// eight rows an ldmatrix reads fall into different bank groups
__host__ __device__ __forceinline__ int tile_pitch(int cols) { const int c = cols >> 3; return (c + 1 + (c & 1)) * 16; }

// What a query at position p sees, walked as ONE list of keys: entries 0 .. nk - 1 are the kept first positions that lie before the
// window's start `lo`, the rest are lo, lo + 1, ..
__device__ __forceinline__ int key_position(int v, int nk, int lo) { return v < nk ? v : v - nk + lo; }

// ------------------------------------------------------------------ cache store
// One CTA per token, one warp per key/value head at a time: rotate k (and divide it by its root mean square), rotate or copy v,
// write the token's row of cache slot `slot`.
template <typename T>
__global__ void __launch_bounds__(128) window_kv_store_kernel(
    const T* __restrict__ k, int64_t k_stride, const T* __restrict__ v, int64_t v_stride, const float* __restrict__ cosb,
    const float* __restrict__ sinb, const int* __restrict__ tok_seq, const int* __restrict__ tok_pos,
    const int* __restrict__ block_table, int max_blocks_per_seq, T* __restrict__ cache, int n_slots, int slot, int block_size,
    int G, int dk, int dv, int rot_dims, int halves, float qk_norm_eps, const float* __restrict__ vcos,
    const float* __restrict__ vsin, const float* __restrict__ knorm_w, float prenorm_eps, int vshare) {
    const int64_t t = blockIdx.x;
    const int pos = tok_pos[t];
    const int blk = block_table[(int64_t)tok_seq[t] * max_blocks_per_seq + pos / block_size];
    const int GV = G / vshare;
    const int kw = G * dk, vw = GV * dv;
    T* dst = cache + (((int64_t)blk * n_slots + slot) * block_size + pos % block_size) * (kw + vw);
    const T* kr = k + t * k_stride;
    const T* vr = v + t * v_stride;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    const float* cs = cosb != nullptr ? cosb + t * (rot_dims >> 1) : nullptr;
    const float* sn = sinb != nullptr ? sinb + t * (rot_dims >> 1) : nullptr;
    for (int g = warp; g < G; g += nwarps) {
        const T* x = kr + g * dk;
        float pinv = 1.f;
        if (knorm_w != nullptr) {
            float ss = 0.f;
            for (int j = lane; j < dk; j += 32) { const float o = ldf(x + j); ss += o * o; }
            pinv = 1.f / sqrtf(warp_sum(ss) / (float)dk + prenorm_eps);
        }
        float inv = 1.f;
        if (qk_norm_eps >= 0.f) {
            float ss = 0.f;
            for (int j = lane; j < dk; j += 32) { const float o = rot_entry(x, j, rot_dims, halves, cs, sn, pinv, knorm_w); ss += o * o; }
            inv = 1.f / sqrtf(warp_sum(ss) / (float)dk + qk_norm_eps);
        }
        for (int j = lane; j < dk; j += 32) stf(dst + g * dk + j, rot_entry(x, j, rot_dims, halves, cs, sn, pinv, knorm_w) * inv);
        if (g >= GV) continue;                          // value heads: the first G / vshare turns of this loop
        const T* y = vr + g * dv;
        if (vcos != nullptr) {
            const float* vc = vcos + t * (dv >> 1);
            const float* vs = vsin + t * (dv >> 1);
            for (int j = lane; j < dv; j += 32) stf(dst + kw + g * dv + j, rot_entry(y, j, dv, halves, vc, vs));
        } else {
            for (int j = lane; j < dv; j += 32) dst[kw + g * dv + j] = y[j];
        }
    }
}

// One CTA per token, one warp per key head at a time: the row of the shared_kv layout (see the top of the file).
template <typename T>
__global__ void __launch_bounds__(128) shared_kv_store_kernel(
    const T* __restrict__ k, int64_t k_stride, const int* __restrict__ tok_seq, const int* __restrict__ tok_pos,
    const int* __restrict__ block_table, int max_blocks_per_seq, T* __restrict__ cache, int n_slots, int slot, int block_size,
    int G, int dk, float eps) {
    const int64_t t = blockIdx.x;
    const int pos = tok_pos[t];
    const int blk = block_table[(int64_t)tok_seq[t] * max_blocks_per_seq + pos / block_size];
    const int koff = shared_kv_key_offset(G);
    T* dst = cache + (((int64_t)blk * n_slots + slot) * block_size + pos % block_size) * shared_kv_row(G, dk);
    float* inv = reinterpret_cast<float*>(dst);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    for (int g = warp; g < G; g += nwarps) {
        const T* x = k + t * k_stride + g * dk;
        float ss = 0.f;
        for (int j = lane; j < dk; j += 32) {
            const T v = x[j];
            const float f = ldf(&v);
            ss += f * f;
            dst[koff + g * dk + j] = v;
        }
        ss = warp_sum(ss);
        if (lane == 0) inv[g] = 1.f / sqrtf(ss / (float)dk + eps);
    }
}

// Queries and keys that are RMS-normed over their WHOLE projection (all heads together, weights qw [H * dk], kw [G * dk]) and then turned
// on their first rot entries, with the un-normed keys as values: one CTA per token writes the cache row (shared_kv with krot = rot, see
// the top of the file) and the queries in the order the attention kernels read them.  Both rows wait in shared memory as fp32
// ((H + G) dk floats, with the token's angles behind them) between the sums and the writes; then a warp takes a head at a time.  VEC: 16 bytes a load (rows aligned)
// and four entries a store (dk and rot multiples of 4).
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) whole_norm_rope_store_kernel(
    const T* __restrict__ q, int64_t q_stride, const T* __restrict__ k, int64_t k_stride, const float* __restrict__ qw,
    const float* __restrict__ kw, float eps, const float* __restrict__ cosb, const float* __restrict__ sinb,
    const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, const int* __restrict__ block_table, int max_blocks_per_seq,
    T* __restrict__ cache, int n_slots, int slot, int block_size, T* __restrict__ q_out, int H, int G, int dk, int rot, int halves) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float red[32];
    constexpr int N = VEC ? 4 : 1;
    const int64_t t = blockIdx.x;
    float* qs = smem;                          // [H * dk]
    float* ks = qs + H * dk;                   // [G * dk]
    const int pos = tok_pos[t];
    const int blk = block_table[(int64_t)tok_seq[t] * max_blocks_per_seq + pos / block_size];
    const int koff = shared_kv_key_offset(G), kw_cols = dk + rot, hq = H / G, pass = dk - rot;
    T* dst = cache + (((int64_t)blk * n_slots + slot) * block_size + pos % block_size) * shared_kv_row(G, kw_cols);
    const int half = rot >> 1;
    float* cs = ks + G * dk;                   // [half] each
    float* sn = cs + half;
    for (int i = threadIdx.x; i < half; i += blockDim.x) { cs[i] = cosb[t * half + i]; sn[i] = sinb[t * half + i]; }
    auto stage = [&](const T* src, float* to, int n) {
        float ss = 0.f;
        if constexpr (VEC) {
            constexpr int E = 16 / sizeof(T);
            for (int i = threadIdx.x * E; i < n; i += blockDim.x * E) {
                const uint4 u = *reinterpret_cast<const uint4*>(src + i);
                const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
                for (int j = 0; j < E; j += 4) {
                    const float4 v = make_float4(ldf(e + j), ldf(e + j + 1), ldf(e + j + 2), ldf(e + j + 3));
                    *reinterpret_cast<float4*>(to + i + j) = v;
                    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                }
            }
        } else {
            for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = ldf(src + i); to[i] = v; ss += v * v; }
        }
        return ss;
    };
    const float sq = stage(q + t * q_stride, qs, H * dk), sk = stage(k + t * k_stride, ks, G * dk);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    const float wq = warp_sum(sq), wk_ = warp_sum(sk);
    if (lane == 0) { red[warp] = wq; red[16 + warp] = wk_; }
    __syncthreads();                                                     // both rows, the angles and the warps' sums are staged
    float q2 = 0.f, k2 = 0.f;
    for (int w = 0; w < nwarps; w++) { q2 += red[w]; k2 += red[16 + w]; }
    const float qinv = 1.f / sqrtf(q2 / (float)(H * dk) + eps), kinv = 1.f / sqrtf(k2 / (float)(G * dk) + eps);
    for (int g = threadIdx.x; g < G; g += blockDim.x) reinterpret_cast<float*>(dst)[g] = kinv;
    auto put = [&](T* to, const float* v) {                              // N neighbouring entries
        if constexpr (VEC) {
            struct alignas(4 * sizeof(T)) Pack { T e[4]; } x;
#pragma unroll
            for (int e = 0; e < 4; e++) stf(x.e + e, v[e]);
            *reinterpret_cast<Pack*>(to) = x;
        } else {
            stf(to, v[0]);
        }
    };
    // the turned entries of a head x (weights w): pair i of `half`
    auto turn = [&](T* to, const float* x, const float* w, float inv) {
        for (int i = lane; i < half; i += 32) {
            const int ia = halves ? i : 2 * i, ib = halves ? i + half : 2 * i + 1;
            const float a = x[ia] * inv * w[ia], b = x[ib] * inv * w[ib];
            stf(to + ia, a * cs[i] - b * sn[i]);
            stf(to + ib, b * cs[i] + a * sn[i]);
        }
    };
    for (int unit = warp; unit < H + G; unit += nwarps) {
        if (unit < G) {
            const int g = unit;
            T* to = dst + koff + g * kw_cols;
            for (int j = lane * N; j < dk; j += 32 * N) put(to + j, ks + g * dk + j);
            turn(to + dk, ks + g * dk, kw + g * dk, 1.f);
        } else {
            const int h = unit - G, g = h / hq;
            T* to = q_out + (t * H + h) * dk;
            const float* x = qs + h * dk + rot;
            const float* w = qw + h * dk + rot;
            const float* wk = kw + g * dk + rot;
            for (int j = lane * N; j < pass; j += 32 * N) {
                float v[N];
#pragma unroll
                for (int e = 0; e < N; e++) v[e] = x[j + e] * qinv * w[j + e] * wk[j + e];
                put(to + j, v);
            }
            turn(to + pass, qs + h * dk, qw + h * dk, qinv);
        }
    }
}

// ------------------------------------------------------------------ attention (fp32 CUDA cores)
constexpr int WA_TILE = 32;        // keys per tile: one per lane in the score phase
constexpr int WA_MAX_HPB = 8;      // query heads (warps) per CTA: heads of ONE key/value group, they share the staged tile

// grid (tokens, H / hpb), hpb warps; hpb divides H / G.  KR: per-lane accumulator registers, dv <= 32 * KR.
template <typename T, int KR>
__global__ void __launch_bounds__(WA_MAX_HPB * 32) window_attn_kernel(
    const T* __restrict__ q, int64_t q_stride_t,                                 // [T, H, dk] (un-rotated; rotated here)
    const float* __restrict__ cosb, const float* __restrict__ sinb,            // [T, rot_dims / 2]
    const T* __restrict__ gate, int64_t gate_stride_t,                          // [T, H, dv] gate logits, or null
    const T* __restrict__ cache, int n_slots, int slot, int block_size,
    const int* __restrict__ block_table, int max_blocks_per_seq, const int* __restrict__ tok_seq,
    const int* __restrict__ tok_pos, T* __restrict__ out, int64_t out_stride_t,  // [T, H, dv]
    int H, int G, int dk, int dv, int rot_dims, int window, float scale, float sink, int halves, float qk_norm_eps,
    float softcap, const float* __restrict__ vcos, const float* __restrict__ vsin, float out_scale,
    const float* __restrict__ qnorm_w, float prenorm_eps, int chunk, int vshare, int out_f32, const float* __restrict__ slopes,
    int keep_first, int gate_per_head, int shared_kv, int krot, const float* __restrict__ sinks) {
    extern __shared__ float smem[];
    const int KW = dk + krot, KP = KW + 1;      // entries of a key head in the cache row; row pitch of the tile
    const int hpb = blockDim.x >> 5;
    float* qs = smem;                          // [hpb][dk]
    float* kt = qs + hpb * dk;                 // [WA_TILE][KP]
    float* vt = kt + WA_TILE * KP;             // [WA_TILE][dv] (not with shared_kv)
    float* os = shared_kv ? vt : vt + WA_TILE * dv;      // [hpb][dv]: the head's output before it is turned back (vcos only)
    float* kinv = os + hpb * dv;               // [WA_TILE]: the keys' 1 / rms (shared_kv only)
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t t = blockIdx.x;
    const int h = blockIdx.y * hpb + warp;
    const int g = (blockIdx.y * hpb) / (H / G);
    const int pos = tok_pos[t];
    const int* bt = block_table + (int64_t)tok_seq[t] * max_blocks_per_seq;
    const int row = shared_kv ? shared_kv_row(G, KW) : G * dk + (G / vshare) * dv;
    const int koff = shared_kv ? shared_kv_key_offset(G) : 0;
    const float slope = slopes != nullptr ? slopes[h] : 0.f;

    {
        float* qw = qs + warp * dk;
        const T* qr = q + t * q_stride_t + (int64_t)h * dk;
        const float* cs = cosb != nullptr ? cosb + t * (rot_dims >> 1) : nullptr;
        const float* sn = sinb != nullptr ? sinb + t * (rot_dims >> 1) : nullptr;
        float pinv = 1.f;
        if (qnorm_w != nullptr) {
            float s0 = 0.f;
            for (int j = lane; j < dk; j += 32) { const float o = ldf(qr + j); s0 += o * o; }
            pinv = 1.f / sqrtf(warp_sum(s0) / (float)dk + prenorm_eps);
        }
        float ss = 0.f;
        for (int j = lane; j < dk; j += 32) {
            const float o = rot_entry(qr, j, rot_dims, halves, cs, sn, pinv, qnorm_w);
            qw[j] = o;
            ss += o * o;
        }
        const float f = qk_norm_eps >= 0.f ? scale / sqrtf(warp_sum(ss) / (float)dk + qk_norm_eps) : scale;
        for (int j = lane; j < dk; j += 32) qw[j] *= f;            // every lane rescales what it wrote itself
    }

    // a sink takes part in the normalisation only: it enters the running (maximum, sum) as a key of score 0 without a value
    float m = sinks != nullptr ? sinks[h] : sink > 0.f ? 0.f : -INFINITY, l = sinks != nullptr ? 1.f : sink;
    float acc[KR];
#pragma unroll
    for (int k = 0; k < KR; k++) acc[k] = 0.f;

    int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    const int nk = window > 0 ? min(keep_first, lo) : 0;
    const int total = nk + pos - lo + 1;
    const float* vbase = shared_kv ? kt : vt;
    const int VP = shared_kv ? KP : dv;
    for (int base = 0; base < total; base += WA_TILE) {
        __syncthreads();                       // the previous tile is no longer read (and qs is written, first time round)
        const int nkeys = min(WA_TILE, total - base);
        for (int jj = warp; jj < nkeys; jj += hpb) {
            const int kp = key_position(base + jj, nk, lo);
            const T* src = cache + (((int64_t)bt[kp / block_size] * n_slots + slot) * block_size + kp % block_size) * row;
            const T* ks = src + koff + g * KW;
            for (int d = lane; d < KW; d += 32) kt[jj * KP + d] = ldf(ks + d);
            if (shared_kv) {
                if (lane == 0) kinv[jj] = reinterpret_cast<const float*>(src)[g];
                continue;
            }
            const T* vs = src + G * dk + (g / vshare) * dv;
            for (int d = lane; d < dv; d += 32) vt[jj * dv + d] = ldf(vs + d);
        }
        __syncthreads();
        const float* qw = qs + warp * dk;
        float s = -INFINITY;
        if (lane < nkeys) {
            const float* kr = kt + lane * KP + krot;
            float a = 0.f;
            for (int d = 0; d < dk; d++) a += qw[d] * kr[d];
            if (shared_kv) a *= kinv[lane];
            s = softcap > 0.f ? softcap * tanhf(a / softcap) : a;
            s -= slope * (float)(pos - key_position(base + lane, nk, lo));
        }
        const float m_new = fmaxf(m, warp_max(s));          // finite: every tile has a visible key
        const float alpha = expf(m - m_new);                // 0 on the first tile without a sink (m = -inf)
        const float p = lane < nkeys ? expf(s - m_new) : 0.f;
        l = l * alpha + warp_sum(p);
#pragma unroll
        for (int k = 0; k < KR; k++) acc[k] *= alpha;
        for (int jj = 0; jj < nkeys; jj++) {
            const float pj = __shfl_sync(0xffffffffu, p, jj);
            const float* vr = vbase + jj * VP;
#pragma unroll
            for (int k = 0; k < KR; k++) {
                const int d = lane + 32 * k;
                if (d < dv) acc[k] += pj * vr[d];
            }
        }
        m = m_new;
    }
    float denom = l;
    T* o = out + t * out_stride_t + (int64_t)h * dv;
    const T* gr = gate != nullptr && !gate_per_head ? gate + t * gate_stride_t + (int64_t)h * dv : nullptr;
    if (gate != nullptr && gate_per_head) out_scale *= 1.f / (1.f + expf(-ldf(gate + t * gate_stride_t + h)));
    if (vcos != nullptr) {
        // the sum of turned values is turned back by the query's own position: pair (a, b) -> (a c + b s, b c - a s)
        float* ow = os + warp * dv;
#pragma unroll
        for (int k = 0; k < KR; k++) {
            const int d = lane + 32 * k;
            if (d < dv) ow[d] = acc[k] / denom;
        }
        __syncwarp();
        const int hv = dv >> 1;
        const float* vc = vcos + t * hv;
        const float* vs = vsin + t * hv;
#pragma unroll
        for (int k = 0; k < KR; k++) {
            const int d = lane + 32 * k;
            if (d < dv) {
                int m, second;
                if (halves) { second = d >= hv; m = second ? d - hv : d; } else { second = d & 1; m = d >> 1; }
                const float a = halves ? ow[m] : ow[2 * m], b = halves ? ow[m + hv] : ow[2 * m + 1];
                acc[k] = second ? b * vc[m] - a * vs[m] : a * vc[m] + b * vs[m];
            }
        }
        denom = 1.f;
    }
#pragma unroll
    for (int k = 0; k < KR; k++) {
        const int d = lane + 32 * k;
        if (d < dv) {
            float y = acc[k] / denom * out_scale;
            if (gr != nullptr) y *= 1.f / (1.f + expf(-ldf(gr + d)));
            if (out_f32) reinterpret_cast<float*>(out)[t * out_stride_t + (int64_t)h * dv + d] = y;
            else stf(o + d, y);
        }
    }
}


// ------------------------------------------------------------------ attention (tensor cores, 16-bit storage)
// One CTA = up to 64 query ROWS of one key/value group: row r is (token r / hqp of the CTA's token range, head r % hqp of the
// group), hqp = heads per group rounded up to a power of two.  The CTA walks its tokens in SEGMENTS (runs of one sequence at
// consecutive positions - a prompt portion; a decoded token is a segment of one), and a segment's rows share every staged key
// tile: WT_KEYS keys x (dk + dv), gathered through the block table with cp.async into a two-stage ring while the previous tile is
// multiplied (32-key tiles for prompt portions and large decode batches, see the launcher).  Warp w owns rows 16 w .. 16 w + 15: S = Q K^T (mma.sync m16n8k16, fp32 accumulate), per-row window mask, online
// softmax in fp32 (base 2, the sink enters as a key of score 0), P rounded to the storage type and fed from registers into
// O += P V.  dk, dv multiples of 16, at most DMAX.  Rows of 16-bit tiles are padded by 16 bytes: the eight rows an ldmatrix
// reads then fall into eight different bank groups for every dk / dv.
constexpr int WT_ROWS = 64;

// EXT: the kernel knows slopes, kept first positions, gates per head and shared_kv rows (compiled out otherwise).
// WT_KEYS: keys per tile (32 or 64).  Smaller tiles leave room for more CTAs per SM (prompt portions: many CTAs, latency-bound);
// larger ones keep more bytes in flight per CTA (decoded tokens: few CTAs that walk their window alone).
template <typename T, int DMAX, int WT_KEYS, bool EXT>
__global__ void __launch_bounds__(128, WT_KEYS == 32 ? 3 : 2) window_attn_mma_kernel(
    const T* __restrict__ q, int64_t q_stride_t, const float* __restrict__ cosb, const float* __restrict__ sinb,
    const T* __restrict__ gate, int64_t gate_stride_t, const T* __restrict__ cache, int n_slots, int slot, int block_size,
    const int* __restrict__ block_table, int max_blocks_per_seq, const int* __restrict__ tok_seq,
    const int* __restrict__ tok_pos, T* __restrict__ out, int64_t out_stride_t, int row0, int nrows, int qt, int hq, int hqp_log2,
    int H, int G, int dk, int dv, int rot_dims, int window, float scale_log2, float sink, int halves, float qk_norm_eps,
    float softcap, const float* __restrict__ vcos, const float* __restrict__ vsin, float out_scale,
    const float* __restrict__ qnorm_w, float prenorm_eps, int chunk, int vshare, int out_f32, const float* __restrict__ slopes_,
    int keep_first_, int gate_per_head_, int shared_kv_, int krot_, const float* __restrict__ sinks_) {
    const float* slopes = EXT ? slopes_ : nullptr;
    const float* sinks = EXT ? sinks_ : nullptr;
    const int keep_first = EXT ? keep_first_ : 0, krot = EXT ? krot_ : 0;
    const bool gate_per_head = EXT && gate_per_head_, shared_kv = EXT && shared_kv_;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int KW = dk + krot;                                                  // entries of a key head in the cache row
    const int PQ = dk * 2 + 16, PK = tile_pitch(KW), PV = shared_kv ? PK : dv * 2 + 16;      // row pitches in bytes
    unsigned char* Qs = smem_raw;                                              // [64][PQ]
    unsigned char* Ks = Qs + WT_ROWS * PQ;                                     // [2][64][PK]
    unsigned char* Vs = shared_kv ? Ks : Ks + 2 * WT_KEYS * PK;                // [2][64][PV] (shared_kv: the key tile itself)
    float* kinv = reinterpret_cast<float*>(Ks + 2 * WT_KEYS * PK);             // [2][64]: the keys' 1 / rms (shared_kv only)
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = blockIdx.y;
    const int hqp = 1 << hqp_log2;
    const int t_first = row0 + blockIdx.x * qt;
    const int ntok = min(qt, row0 + nrows - t_first);
    const int row_elems = shared_kv ? shared_kv_row(G, KW) : G * dk + (G / vshare) * dv;
    const int koff = shared_kv ? shared_kv_key_offset(G) : 0;
    const int ck = KW >> 3, cv = dv >> 3;                                      // 16-byte chunks per key / value row
    const int half = rot_dims >> 1;
    // with a score cap: cap * tanh(s * scale / cap), then to base 2
    const float cap_in = softcap > 0.f ? scale_log2 * 0.6931471805599453f / softcap : 0.f;
    const float cap_out = softcap * 1.4426950408889634f;

    for (int i0 = 0; i0 < ntok;) {
        // ---- the segment: tokens t_first + i0 .. + n - 1 of one sequence at consecutive positions
        const int ts = t_first + i0;
        const int seq = tok_seq[ts], pos0 = tok_pos[ts];
        int n = 1;
        while (i0 + n < ntok && tok_seq[ts + n] == seq && tok_pos[ts + n] == pos0 + n) n++;
        const int* bt = block_table + (int64_t)seq * max_blocks_per_seq;
        int lo = (window > 0 && pos0 - window + 1 > 0) ? pos0 - window + 1 : 0;
        if (chunk > 0) lo = max(lo, pos0 / chunk * chunk);
        const int hi = pos0 + n - 1;
        const int nk = EXT && window > 0 ? min(keep_first, lo) : 0;
        const int total = nk + hi - lo + 1;                                    // keys the segment's rows see together
        const int ntiles = (total - 1) / WT_KEYS + 1;
        __syncthreads();                                                       // the previous segment's tiles and queries are done with

        // two threads per key row, alternating 16-byte chunks: ONE block-table lookup and address per thread and tile
        auto load_tile = [&](int it) {
            constexpr int TPR = 128 / WT_KEYS;                                 // threads per key row
            const int st = it & 1, jj = tid / TPR, part = tid % TPR;
            const int kp = key_position(it * WT_KEYS + jj, nk, lo);
            const bool ok = kp <= hi;
            const T* krow = cache;
            const T* vrow = cache;
            if (ok) {
                const int b = kp / block_size;
                const int64_t rowi = ((int64_t)bt[b] * n_slots + slot) * block_size + (kp - b * block_size);
                krow = cache + rowi * row_elems + koff + g * KW;
                vrow = cache + rowi * row_elems + G * dk + (g / vshare) * dv;
                if (shared_kv && part == 0) cp_async4(smem_u32(kinv + st * WT_KEYS + jj), cache + rowi * row_elems + 2 * g);
            } else if (shared_kv && part == 0) {
                kinv[st * WT_KEYS + jj] = 0.f;
            }
            const int nb = ok ? 16 : 0;
            const uint32_t kd = smem_u32(Ks + (st * WT_KEYS + jj) * PK), vd = smem_u32(Vs + (st * WT_KEYS + jj) * PV);
            for (int ch = part; ch < ck; ch += TPR) cp_async16(kd + ch * 16, ok ? krow + ch * 8 : krow, nb);
            if (!shared_kv)
                for (int ch = part; ch < cv; ch += TPR) cp_async16(vd + ch * 16, ok ? vrow + ch * 8 : vrow, nb);
            cp_async_commit();
        };
        load_tile(0);

        // ---- queries of the segment: rotated (and divided by their root mean square) in fp32, rounded to the storage type;
        // dead rows are zeros.  Two threads per row (neighbouring lanes), each takes every other pair of entries.
        {
            const int r = tid >> 1;                                            // 128 threads, 64 rows: one row per thread pair
            const int j = r >> hqp_log2, hh = r & (hqp - 1);
            const bool live = j < n && hh < hq;
            const int64_t t = ts + j;
            const T* qr = q + t * q_stride_t + (int64_t)(g * hq + hh) * dk;
            const float* cs = cosb != nullptr ? cosb + t * half : nullptr;
            const float* sn = sinb != nullptr ? sinb + t * half : nullptr;
            float pinv = 1.f;
            if (qnorm_w != nullptr) {
                float s0 = 0.f;
                if (live)
                    for (int i = tid & 1; i < (dk >> 1); i += 2) {
                        const float a = ldf(qr + 2 * i), b = ldf(qr + 2 * i + 1);
                        s0 += a * a + b * b;
                    }
                s0 += __shfl_xor_sync(0xffffffffu, s0, 1);
                pinv = 1.f / sqrtf(s0 / (float)dk + prenorm_eps);
            }
            float inv = 1.f;
            if (qk_norm_eps >= 0.f) {
                float ss = 0.f;
                if (live)
                    for (int i = tid & 1; i < (dk >> 1); i += 2) {
                        const float a = rot_entry(qr, 2 * i, rot_dims, halves, cs, sn, pinv, qnorm_w),
                                    b = rot_entry(qr, 2 * i + 1, rot_dims, halves, cs, sn, pinv, qnorm_w);
                        ss += a * a + b * b;
                    }
                ss += __shfl_xor_sync(0xffffffffu, ss, 1);
                inv = 1.f / sqrtf(ss / (float)dk + qk_norm_eps);
            }
            for (int i = tid & 1; i < (dk >> 1); i += 2) {
                float a = 0.f, b = 0.f;
                if (live) {
                    a = rot_entry(qr, 2 * i, rot_dims, halves, cs, sn, pinv, qnorm_w) * inv;
                    b = rot_entry(qr, 2 * i + 1, rot_dims, halves, cs, sn, pinv, qnorm_w) * inv;
                }
                *reinterpret_cast<uint32_t*>(Qs + r * PQ + i * 4) = pack2<T>(a, b);
            }
        }

        // ---- per-thread state: rows (lane / 4) and (lane / 4) + 8 of the warp's 16
        const int r_a = warp * 16 + (lane >> 2), r_b = r_a + 8;
        const int j_a = r_a >> hqp_log2, j_b = r_b >> hqp_log2;
        const bool live_a = j_a < n && (r_a & (hqp - 1)) < hq, live_b = j_b < n && (r_b & (hqp - 1)) < hq;
        const int pos_a = pos0 + j_a, pos_b = pos0 + j_b;
        int lo_a = window > 0 ? pos_a - window + 1 : 0, lo_b = window > 0 ? pos_b - window + 1 : 0;
        if (chunk > 0) { lo_a = max(lo_a, pos_a / chunk * chunk); lo_b = max(lo_b, pos_b / chunk * chunk); }
        // keys any row of this warp can see (warp-uniform): tiles outside are skipped
        const int wj_min = (warp * 16) >> hqp_log2, wj_max = min((warp * 16 + 15) >> hqp_log2, n - 1);
        const bool warp_live = wj_min < n;
        int w_lo = window > 0 ? max(0, pos0 + wj_min - window + 1) : 0;
        if (chunk > 0) w_lo = max(w_lo, (pos0 + wj_min) / chunk * chunk);
        const int w_hi = pos0 + wj_max;
        const float sl_a = slopes != nullptr && live_a ? slopes[g * hq + (r_a & (hqp - 1))] * 1.4426950408889634f : 0.f;
        const float sl_b = slopes != nullptr && live_b ? slopes[g * hq + (r_b & (hqp - 1))] * 1.4426950408889634f : 0.f;
        float m_a = sink > 0.f ? 0.f : -INFINITY, m_b = m_a;
        float l_a = (lane & 3) == 0 ? sink : 0.f, l_b = l_a;
        if (sinks != nullptr) {
            if (live_a) m_a = sinks[g * hq + (r_a & (hqp - 1))] * 1.4426950408889634f;
            if (live_b) m_b = sinks[g * hq + (r_b & (hqp - 1))] * 1.4426950408889634f;
            l_a = l_b = (lane & 3) == 0 ? 1.f : 0.f;
        }
        float o[DMAX / 8][4];
#pragma unroll
        for (int nt = 0; nt < DMAX / 8; nt++) { o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f; }

        for (int it = 0; it < ntiles; it++) {
            if (it + 1 < ntiles) { load_tile(it + 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
            __syncthreads();                                                   // tile `it` (and, first time, the queries) visible
            const int base = it * WT_KEYS;                                     // the tile's first entry in the list of visible keys
            const int kp_first = key_position(base, nk, lo), kp_last = key_position(base + WT_KEYS - 1, nk, lo);
            if (warp_live && kp_first <= w_hi && (kp_last >= w_lo || (EXT && kp_first < keep_first))) {
                const unsigned char* Kt = Ks + (it & 1) * WT_KEYS * PK;
                const unsigned char* Vt = Vs + (it & 1) * WT_KEYS * PV;
                float sc[WT_KEYS / 8][4];
#pragma unroll
                for (int nt = 0; nt < WT_KEYS / 8; nt++) { sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f; }
#pragma unroll
                for (int kk = 0; kk < DMAX / 16; kk++) {
                    if (kk * 16 < dk) {
                        uint32_t a[4];
                        ldmatrix_x4(smem_u32(Qs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PQ + (kk * 16 + (lane >> 4) * 8) * 2),
                                    a[0], a[1], a[2], a[3]);
#pragma unroll
                        for (int np = 0; np < WT_KEYS / 16; np++) {
                            uint32_t b0, b1, b2, b3;
                            ldmatrix_x4(smem_u32(Kt + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * PK + (krot + kk * 16 + ((lane >> 3) & 1) * 8) * 2),
                                        b0, b1, b2, b3);
                            mma_16816<T>(sc[2 * np], a, b0, b1);
                            mma_16816<T>(sc[2 * np + 1], a, b2, b3);
                        }
                    }
                }
                if (shared_kv) {
                    const float* ki = kinv + (it & 1) * WT_KEYS + (lane & 3) * 2;
#pragma unroll
                    for (int nt = 0; nt < WT_KEYS / 8; nt++) {
                        const float2 f = *reinterpret_cast<const float2*>(ki + nt * 8);
                        sc[nt][0] *= f.x; sc[nt][1] *= f.y; sc[nt][2] *= f.x; sc[nt][3] *= f.y;
                    }
                }
                // mask, running maximum
                float mx_a = -INFINITY, mx_b = -INFINITY;
#pragma unroll
                for (int nt = 0; nt < WT_KEYS / 8; nt++) {
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        const int kp = key_position(base + nt * 8 + (lane & 3) * 2 + e, nk, lo);
                        const bool kept = EXT && kp < keep_first;
                        const bool va = live_a && kp <= pos_a && (kp >= lo_a || kept), vb = live_b && kp <= pos_b && (kp >= lo_b || kept);
                        float sa = softcap > 0.f ? cap_out * tanhf(sc[nt][e] * cap_in) : sc[nt][e] * scale_log2;
                        float sb = softcap > 0.f ? cap_out * tanhf(sc[nt][2 + e] * cap_in) : sc[nt][2 + e] * scale_log2;
                        if (EXT) {
                            sa -= sl_a * (float)(pos_a - kp);
                            sb -= sl_b * (float)(pos_b - kp);
                        }
                        sc[nt][e] = va ? sa : -INFINITY;
                        sc[nt][2 + e] = vb ? sb : -INFINITY;
                        mx_a = fmaxf(mx_a, sc[nt][e]);
                        mx_b = fmaxf(mx_b, sc[nt][2 + e]);
                    }
                }
                mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1)); mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
                mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1)); mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
                const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
                const float ref_a = mn_a == -INFINITY ? 0.f : mn_a, ref_b = mn_b == -INFINITY ? 0.f : mn_b;   // nothing seen yet
                const float al_a = exp2f(m_a - ref_a), al_b = exp2f(m_b - ref_b);                             // exp2(-inf) = 0
                m_a = mn_a; m_b = mn_b;
                l_a *= al_a; l_b *= al_b;
#pragma unroll
                for (int nt = 0; nt < DMAX / 8; nt++) { o[nt][0] *= al_a; o[nt][1] *= al_a; o[nt][2] *= al_b; o[nt][3] *= al_b; }
                uint32_t pa[WT_KEYS / 16][4];
#pragma unroll
                for (int nt = 0; nt < WT_KEYS / 8; nt++) {
                    const float p0 = exp2f(sc[nt][0] - ref_a), p1 = exp2f(sc[nt][1] - ref_a);
                    const float p2 = exp2f(sc[nt][2] - ref_b), p3 = exp2f(sc[nt][3] - ref_b);
                    l_a += p0 + p1; l_b += p2 + p3;
                    pa[nt >> 1][(nt & 1) * 2] = pack2<T>(p0, p1);
                    pa[nt >> 1][(nt & 1) * 2 + 1] = pack2<T>(p2, p3);
                }
#pragma unroll
                for (int kk = 0; kk < WT_KEYS / 16; kk++) {                    // 16 keys per step
#pragma unroll
                    for (int np = 0; np < DMAX / 16; np++) {
                        if (np * 16 < dv) {
                            uint32_t b0, b1, b2, b3;
                            ldmatrix_x4_trans(smem_u32(Vt + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PV + (np * 16 + (lane >> 4) * 8) * 2),
                                              b0, b1, b2, b3);
                            mma_16816<T>(o[2 * np], pa[kk], b0, b1);
                            mma_16816<T>(o[2 * np + 1], pa[kk], b2, b3);
                        }
                    }
                }
            }
            __syncthreads();                                                   // stage it & 1 may be overwritten by tile it + 2
        }

        // ---- normalise, (turn back,) gate, store
        l_a += __shfl_xor_sync(0xffffffffu, l_a, 1); l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
        l_b += __shfl_xor_sync(0xffffffffu, l_b, 1); l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
        if (vcos != nullptr) {
            // values were stored turned by their own position: the normalised sums go through shared memory (the tiles are done
            // with: the loop ended on a barrier), where every pair is turned back by the query's position
            float* Os = reinterpret_cast<float*>(smem_raw);                    // [64][dv]
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int r = e ? r_b : r_a;
                const float inv = 1.f / (e ? l_b : l_a);
#pragma unroll
                for (int nt = 0; nt < DMAX / 8; nt++) {
                    const int d = nt * 8 + (lane & 3) * 2;
                    if (d < dv) { Os[r * dv + d] = o[nt][2 * e] * inv; Os[r * dv + d + 1] = o[nt][2 * e + 1] * inv; }
                }
            }
            __syncthreads();
            const int hv = dv >> 1;
            for (int idx = tid; idx < WT_ROWS * hv; idx += 128) {
                const int r = idx / hv, m = idx - r * hv;
                const int j = r >> hqp_log2, hh = r & (hqp - 1);
                if (j >= n || hh >= hq) continue;
                const int64_t t = ts + j;
                const int da = halves ? m : 2 * m, db = halves ? m + hv : 2 * m + 1;
                const float a = Os[r * dv + da], b = Os[r * dv + db];
                const float c = vcos[t * hv + m], sn = vsin[t * hv + m];
                float ya = (a * c + b * sn) * out_scale, yb = (b * c - a * sn) * out_scale;
                T* orow = out + t * out_stride_t + (int64_t)(g * hq + hh) * dv;
                if (gate != nullptr) {
                    const T* grow = gate + t * gate_stride_t + (gate_per_head ? g * hq + hh : (int64_t)(g * hq + hh) * dv);
                    ya *= 1.f / (1.f + __expf(-ldf(grow + (gate_per_head ? 0 : da))));
                    yb *= 1.f / (1.f + __expf(-ldf(grow + (gate_per_head ? 0 : db))));
                }
                stf(orow + da, ya);
                stf(orow + db, yb);
            }
            i0 += n;
            continue;                                                          // the next segment starts with a barrier
        }
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const bool live = e ? live_b : live_a;
            if (!live) continue;
            const int r = e ? r_b : r_a;
            const int64_t t = ts + (r >> hqp_log2);
            const int h = g * hq + (r & (hqp - 1));
            float inv = out_scale / (e ? l_b : l_a);
            if (gate != nullptr && gate_per_head) inv *= 1.f / (1.f + __expf(-ldf(gate + t * gate_stride_t + h)));
            T* orow = out + t * out_stride_t + (int64_t)h * dv;
            const T* grow = gate != nullptr && !gate_per_head ? gate + t * gate_stride_t + (int64_t)h * dv : nullptr;
#pragma unroll
            for (int nt = 0; nt < DMAX / 8; nt++) {
                const int d = nt * 8 + (lane & 3) * 2;
                if (d < dv) {
                    float y0 = o[nt][2 * e] * inv, y1 = o[nt][2 * e + 1] * inv;
                    if (grow != nullptr) {
                        y0 *= 1.f / (1.f + __expf(-ldf(grow + d)));
                        y1 *= 1.f / (1.f + __expf(-ldf(grow + d + 1)));
                    }
                    if (out_f32) {
                        float* o32 = reinterpret_cast<float*>(out) + t * out_stride_t + (int64_t)h * dv + d;
                        o32[0] = y0; o32[1] = y1;
                    } else {
                        *reinterpret_cast<uint32_t*>(orow + d) = pack2<T>(y0, y1);
                    }
                }
            }
        }
        i0 += n;
    }
}

// ------------------------------------------------------------------ attention of single decoded tokens (tensor cores, 16-bit storage)
// One CTA = one token and key/value group of at most 8 NH query heads.  The token's visible keys are split over the CTA's
// WARPS (4 or 8): warp w walks the tiles w, w + WD_WARPS, .. of KT keys through a cp.async ring of its own (no CTA barrier inside the loop) with its own
// running (maximum, sum, output); the results are merged through shared memory at the end.  The products are taken transposed, so
// that the few heads are the narrow side of the MMA tiles: S^T [keys, heads] = K Q^T with Q^T in registers for the whole walk, then
// O^T [dv, heads] += V^T P^T, where P^T is S^T's fragment turned by movmatrix.  Same options as the kernel above.
constexpr int WD_STAGES = 3;

// the 8 x 8 matrix of 16-bit entries held by the warp, transposed
__device__ __forceinline__ uint32_t movmatrix_trans(uint32_t x) {
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}

template <typename T, int DMAX, int KT, int NH, int WD_WARPS, bool EXT>
__global__ void __launch_bounds__(WD_WARPS * 32) window_attn_decode_kernel(
    const T* __restrict__ q, int64_t q_stride_t, const float* __restrict__ cosb, const float* __restrict__ sinb,
    const T* __restrict__ gate, int64_t gate_stride_t, const T* __restrict__ cache, int n_slots, int slot, int block_size,
    const int* __restrict__ block_table, int max_blocks_per_seq, const int* __restrict__ tok_seq,
    const int* __restrict__ tok_pos, T* __restrict__ out, int64_t out_stride_t, int row0, int hq,
    int G, int dk, int dv, int rot_dims, int window, float scale_log2, float sink, int halves, float qk_norm_eps,
    float softcap, const float* __restrict__ vcos, const float* __restrict__ vsin, float out_scale,
    const float* __restrict__ qnorm_w, float prenorm_eps, int chunk, int vshare, int out_f32, const float* __restrict__ slopes_,
    int keep_first_, int gate_per_head_, int shared_kv_, int krot_, const float* __restrict__ sinks_) {
    const float* slopes = EXT ? slopes_ : nullptr;
    const float* sinks = EXT ? sinks_ : nullptr;
    const int keep_first = EXT ? keep_first_ : 0, krot = EXT ? krot_ : 0;
    const bool gate_per_head = EXT && gate_per_head_, shared_kv = EXT && shared_kv_;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int KW = dk + krot;                                                  // entries of a key head in the cache row
    const int PQ = dk * 2 + 16, PK = tile_pitch(KW), PV = dv * 2 + 16;         // row pitches in bytes
    const int stage_bytes = KT * (PK + (shared_kv ? (int)sizeof(float) : PV));
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    unsigned char* Qs = smem_raw;                                              // [16][PQ]
    unsigned char* Ws = Qs + 16 * PQ + warp * WD_STAGES * stage_bytes;         // this warp's stages: K [KT][PK], V [KT][PV] | 1 / rms [KT]
    const uint32_t ws_a = smem_u32(Ws);
    const int g = blockIdx.y;
    const int64_t t = row0 + blockIdx.x;
    const int pos = tok_pos[t];
    const int* bt = block_table + (int64_t)tok_seq[t] * max_blocks_per_seq;
    const int row_elems = shared_kv ? shared_kv_row(G, KW) : G * dk + (G / vshare) * dv;
    int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    const int nk = EXT && window > 0 ? min(keep_first, lo) : 0;
    const int total = nk + pos - lo + 1;
    const int ntiles = (total - 1) / KT + 1;

    // lane l < KT looks up where row l of tile `it` lies in the cache (-1: past the visible keys); the copies then take whole rows with
    // LPR neighbouring lanes, one 16-byte piece of the key and of the value each
    constexpr int LPR = DMAX / 8, RPI = 32 / LPR;
    const int piece = lane % LPR;
    const bool has_k = piece * 8 < KW, has_v = !shared_kv && piece * 8 < dv;
    const bool has_k2 = EXT && (piece + LPR) * 8 < KW;                         // key parts wider than LPR pieces (krot <= dk)
    const int k_elem = (shared_kv ? shared_kv_key_offset(G) : 0) + g * KW + piece * 8, v_elem = G * dk + (g / vshare) * dv + piece * 8;
    auto find_row = [&](int it) -> int {
        const int e = it * KT + lane;
        if (lane >= KT || e >= total) return -1;
        const int kp = key_position(e, nk, lo), b = kp / block_size;
        return (bt[b] * n_slots + slot) * block_size + (kp - b * block_size);  // cache rows are numbered below 2^31
    };
    auto load_tile = [&](int row, int st) {
        const uint32_t K = ws_a + st * stage_bytes, V = K + KT * PK;
        if (shared_kv && lane < KT) {
            if (row >= 0) cp_async4(V + lane * 4, cache + (int64_t)row * row_elems + 2 * g);
            else *reinterpret_cast<float*>(Ws + st * stage_bytes + KT * PK + lane * 4) = 0.f;
        }
#pragma unroll
        for (int i = 0; i < KT / RPI; i++) {
            const int r = i * RPI + lane / LPR;
            const int src = __shfl_sync(0xffffffffu, row, r);
            const T* base = cache + (int64_t)max(src, 0) * row_elems;
            const int nb = src >= 0 ? 16 : 0;
            if (has_k) cp_async16(K + r * PK + piece * 16, base + k_elem, nb);
            if (EXT && has_k2) cp_async16(K + r * PK + (piece + LPR) * 16, base + k_elem + LPR * 8, nb);
            if (has_v) cp_async16(V + r * PV + piece * 16, base + v_elem, nb);
        }
        cp_async_commit();
    };
    int row_next = warp < ntiles ? find_row(warp) : -1;
#pragma unroll
    for (int i = 0; i < WD_STAGES - 1; i++) {
        const int it = warp + i * WD_WARPS;
        if (it < ntiles) { load_tile(row_next, i); row_next = it + WD_WARPS < ntiles ? find_row(it + WD_WARPS) : -1; }
        else cp_async_commit();                                                // an empty group keeps the count
    }

    // ---- queries: rows past the group's heads are zeros
    {
        constexpr int TPR = WD_WARPS * 2;                                      // threads per row (16 rows)
        const int r = tid / TPR, part = tid % TPR;
        const bool live = r < hq;
        const int half = rot_dims >> 1;
        const T* qr = q + t * q_stride_t + (int64_t)(g * hq + (live ? r : 0)) * dk;
        const float* cs = cosb != nullptr ? cosb + t * half : nullptr;
        const float* sn = sinb != nullptr ? sinb + t * half : nullptr;
        float pinv = 1.f;
        if (qnorm_w != nullptr) {
            float s0 = 0.f;
            for (int i = part; i < dk; i += TPR) { const float a = ldf(qr + i); s0 += a * a; }
            s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2); s0 += __shfl_xor_sync(0xffffffffu, s0, 4);
            if constexpr (TPR == 16) s0 += __shfl_xor_sync(0xffffffffu, s0, 8);
            pinv = 1.f / sqrtf(s0 / (float)dk + prenorm_eps);
        }
        float inv = 1.f;
        if (qk_norm_eps >= 0.f) {
            float ss = 0.f;
            for (int i = part; i < dk; i += TPR) { const float a = rot_entry(qr, i, rot_dims, halves, cs, sn, pinv, qnorm_w); ss += a * a; }
            ss += __shfl_xor_sync(0xffffffffu, ss, 1); ss += __shfl_xor_sync(0xffffffffu, ss, 2); ss += __shfl_xor_sync(0xffffffffu, ss, 4);
            if constexpr (TPR == 16) ss += __shfl_xor_sync(0xffffffffu, ss, 8);
            inv = 1.f / sqrtf(ss / (float)dk + qk_norm_eps);
        }
        for (int i = part; i < (dk >> 1); i += TPR) {
            float a = 0.f, b = 0.f;
            if (live) {
                a = rot_entry(qr, 2 * i, rot_dims, halves, cs, sn, pinv, qnorm_w) * inv;
                b = rot_entry(qr, 2 * i + 1, rot_dims, halves, cs, sn, pinv, qnorm_w) * inv;
            }
            *reinterpret_cast<uint32_t*>(Qs + r * PQ + i * 4) = pack2<T>(a, b);
        }
    }
    __syncthreads();
    uint32_t qf[DMAX / 16][NH][2];                                             // Q^T as B fragments: heads 8 n .. 8 n + 7
#pragma unroll
    for (int kk = 0; kk < DMAX / 16; kk++)
        if (kk * 16 < dk) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(smem_u32(Qs + ((lane & 7) + (lane >> 4) * 8) * PQ + (kk * 16 + ((lane >> 3) & 1) * 8) * 2), b0, b1, b2, b3);
            qf[kk][0][0] = b0; qf[kk][0][1] = b1;
            if constexpr (NH == 2) { qf[kk][1][0] = b2; qf[kk][1][1] = b3; }
        }

    // this lane's heads: 8 n + 2 (lane % 4) + e; its keys within a 16-key block: lane / 4 and lane / 4 + 8
    const float cap_in = softcap > 0.f ? scale_log2 * 0.6931471805599453f / softcap : 0.f;
    const float cap_out = softcap * 1.4426950408889634f;
    float m[NH][2], l[NH][2], sl[NH][2];
#pragma unroll
    for (int n = 0; n < NH; n++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int hh = n * 8 + 2 * (lane & 3) + e;
            m[n][e] = sink > 0.f && warp == 0 ? 0.f : -INFINITY;
            l[n][e] = lane < 4 && warp == 0 ? sink : 0.f;
            if (sinks != nullptr && warp == 0 && hh < hq) {
                m[n][e] = sinks[g * hq + hh] * 1.4426950408889634f;
                l[n][e] = lane < 4 ? 1.f : 0.f;
            }
            sl[n][e] = slopes != nullptr && hh < hq ? slopes[g * hq + hh] * 1.4426950408889634f : 0.f;
        }
    float o[DMAX / 16][NH][4];
#pragma unroll
    for (int mt = 0; mt < DMAX / 16; mt++)
#pragma unroll
        for (int n = 0; n < NH; n++) { o[mt][n][0] = o[mt][n][1] = o[mt][n][2] = o[mt][n][3] = 0.f; }

    int st = 0;
    for (int it = warp; it < ntiles; it += WD_WARPS) {
        {
            const int ahead = it + (WD_STAGES - 1) * WD_WARPS;
            const int st_ahead = st + WD_STAGES - 1 >= WD_STAGES ? st - 1 : st + WD_STAGES - 1;
            if (ahead < ntiles) {
                load_tile(row_next, st_ahead);
                row_next = ahead + WD_WARPS < ntiles ? find_row(ahead + WD_WARPS) : -1;
            } else {
                cp_async_commit();
            }
        }
        cp_async_wait<WD_STAGES - 1>();
        __syncwarp();                                                          // the tile is visible to the whole warp
        const uint32_t Kt = ws_a + st * stage_bytes, Vt = shared_kv ? Kt : Kt + KT * PK;
        const int PVt = shared_kv ? PK : PV;
        float sc[KT / 16][NH][4];
#pragma unroll
        for (int b = 0; b < KT / 16; b++)
#pragma unroll
            for (int n = 0; n < NH; n++) { sc[b][n][0] = sc[b][n][1] = sc[b][n][2] = sc[b][n][3] = 0.f; }
        const uint32_t k_addr = Kt + ((lane & 7) + ((lane >> 3) & 1) * 8) * PK + krot * 2 + (lane >> 4) * 16;
#pragma unroll
        for (int kk = 0; kk < DMAX / 16; kk++) {
            if (kk * 16 < dk) {
#pragma unroll
                for (int b = 0; b < KT / 16; b++) {
                    uint32_t a[4];
                    ldmatrix_x4(k_addr + b * 16 * PK + kk * 32, a[0], a[1], a[2], a[3]);
#pragma unroll
                    for (int n = 0; n < NH; n++) mma_16816<T>(sc[b][n], a, qf[kk][n][0], qf[kk][n][1]);
                }
            }
        }
        float mx[NH][2];
#pragma unroll
        for (int n = 0; n < NH; n++) { mx[n][0] = mx[n][1] = -INFINITY; }
        const float* ki = reinterpret_cast<const float*>(Ws + st * stage_bytes + KT * PK) + (lane >> 2);
#pragma unroll
        for (int b = 0; b < KT / 16; b++) {
#pragma unroll
            for (int half = 0; half < 2; half++) {
                const int v = it * KT + b * 16 + half * 8 + (lane >> 2);       // every entry of the list below `total` is visible
                const float kinv = shared_kv ? ki[b * 16 + half * 8] : 1.f;
                const float dist = EXT ? (float)(pos - key_position(v, nk, lo)) : 0.f;
#pragma unroll
                for (int n = 0; n < NH; n++)
#pragma unroll
                    for (int e = 0; e < 2; e++) {
                        float x = sc[b][n][2 * half + e];
                        if (shared_kv) x *= kinv;
                        x = softcap > 0.f ? cap_out * tanhf(x * cap_in) : x * scale_log2;
                        if (EXT) x -= sl[n][e] * dist;
                        x = v < total ? x : -INFINITY;
                        sc[b][n][2 * half + e] = x;
                        mx[n][e] = fmaxf(mx[n][e], x);
                    }
            }
        }
        float al[NH][2];
#pragma unroll
        for (int n = 0; n < NH; n++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                float x = mx[n][e];
                x = fmaxf(x, __shfl_xor_sync(0xffffffffu, x, 4));
                x = fmaxf(x, __shfl_xor_sync(0xffffffffu, x, 8));
                x = fmaxf(x, __shfl_xor_sync(0xffffffffu, x, 16));
                x = fmaxf(x, m[n][e]);                                         // finite: a tile has at least one visible key
                al[n][e] = exp2f(m[n][e] - x);
                m[n][e] = x;
                l[n][e] *= al[n][e];
            }
#pragma unroll
        for (int mt = 0; mt < DMAX / 16; mt++)
#pragma unroll
            for (int n = 0; n < NH; n++) {
                o[mt][n][0] *= al[n][0]; o[mt][n][1] *= al[n][1]; o[mt][n][2] *= al[n][0]; o[mt][n][3] *= al[n][1];
            }
        const uint32_t v_addr = Vt + ((lane & 7) + (lane >> 4) * 8) * PVt + ((lane >> 3) & 1) * 16;
#pragma unroll
        for (int b = 0; b < KT / 16; b++) {                                    // 16 keys per step
            uint32_t pb[NH][2];
#pragma unroll
            for (int n = 0; n < NH; n++)
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    const float p0 = exp2f(sc[b][n][2 * half] - m[n][0]), p1 = exp2f(sc[b][n][2 * half + 1] - m[n][1]);
                    l[n][0] += p0; l[n][1] += p1;
                    pb[n][half] = movmatrix_trans(pack2<T>(p0, p1));
                }
#pragma unroll
            for (int mt = 0; mt < DMAX / 16; mt++) {
                if (mt * 16 < dv) {
                    uint32_t a[4];
                    ldmatrix_x4_trans(v_addr + b * 16 * PVt + mt * 32, a[0], a[1], a[2], a[3]);
#pragma unroll
                    for (int n = 0; n < NH; n++) mma_16816<T>(o[mt][n], a, pb[n][0], pb[n][1]);
                }
            }
        }
        __syncwarp();                                                          // the stage may be overwritten
        st = st + 1 == WD_STAGES ? 0 : st + 1;
    }

    // ---- merge the warps, (turn back,) gate, store
    cp_async_wait<0>();
    __syncthreads();                                                           // every warp is done with its tiles
    float* Om = reinterpret_cast<float*>(smem_raw);                            // [WD_WARPS][hq][dv]
    float* Ms = Om + WD_WARPS * hq * dv;                                       // [WD_WARPS][16] maximum, then [WD_WARPS][16] sum
#pragma unroll
    for (int n = 0; n < NH; n++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float x = l[n][e];
            x += __shfl_xor_sync(0xffffffffu, x, 4);
            x += __shfl_xor_sync(0xffffffffu, x, 8);
            x += __shfl_xor_sync(0xffffffffu, x, 16);
            const int hh = n * 8 + 2 * (lane & 3) + e;
            if (hh >= hq) continue;
            if (lane < 4) { Ms[warp * 16 + hh] = m[n][e]; Ms[(WD_WARPS + warp) * 16 + hh] = x; }
#pragma unroll
            for (int mt = 0; mt < DMAX / 16; mt++) {
                const int d = mt * 16 + (lane >> 2);
                if (mt * 16 < dv) {
                    Om[(warp * hq + hh) * dv + d] = o[mt][n][e];
                    Om[(warp * hq + hh) * dv + d + 8] = o[mt][n][2 + e];
                }
            }
        }
    __syncthreads();
    const int n_out = hq * dv;
    for (int i = tid; i < n_out; i += WD_WARPS * 32) {                         // slot 0 <- the normalised output
        const int r = i / dv;
        float M = Ms[r];
#pragma unroll
        for (int w = 1; w < WD_WARPS; w++) M = fmaxf(M, Ms[w * 16 + r]);
        float L = 0.f, y = 0.f;
#pragma unroll
        for (int w = 0; w < WD_WARPS; w++) {
            const float f = exp2f(Ms[w * 16 + r] - M);                         // 0 for a warp that saw no key
            L += f * Ms[(WD_WARPS + w) * 16 + r];
            y += f * Om[w * n_out + i];
        }
        Om[i] = y / L;
    }
    if (vcos != nullptr) __syncthreads();                                      // the turn back reads a neighbour's entry
    const int hv = dv >> 1;
    for (int i = tid; i < n_out; i += WD_WARPS * 32) {
        const int r = i / dv, d = i - r * dv;
        float y = Om[i];
        if (vcos != nullptr) {
            int m, second;
            if (halves) { second = d >= hv; m = second ? d - hv : d; } else { second = d & 1; m = d >> 1; }
            const float a = Om[r * dv + (halves ? m : 2 * m)], b = Om[r * dv + (halves ? m + hv : 2 * m + 1)];
            const float c = vcos[t * hv + m], sn = vsin[t * hv + m];
            y = second ? b * c - a * sn : a * c + b * sn;
        }
        y *= out_scale;
        const int64_t h = g * hq + r;
        if (gate != nullptr) y *= 1.f / (1.f + __expf(-ldf(gate + t * gate_stride_t + (gate_per_head ? h : h * dv + d))));
        if (out_f32) reinterpret_cast<float*>(out)[t * out_stride_t + h * dv + d] = y;
        else stf(out + t * out_stride_t + h * dv + d, y);
    }
}

// ------------------------------------------------------------------ two maps -> one head
// a: fp32 [T, G, 2, hq, dv] (the attention above with vshare = 2 and queries ordered [key/value head][map][head of the group]).
// One warp per (token, head h = g hq + hh): o = a[g, 0, hh] - lambda a[g, 1, hh]; out = o / sqrt(mean(o^2) + eps) * factor *
// sigmoid(gate[t, h]) in the storage type, heads in their natural order.  KR: registers per lane, dv <= 32 KR.
template <typename T, int KR>
__global__ void __launch_bounds__(256) diff_combine_kernel(const float* __restrict__ a, const T* __restrict__ gate,
                                                           int64_t gate_stride_t, T* __restrict__ out, int64_t out_stride_t,
                                                           int64_t units, int H, int hq, int dv, float lambda, float eps,
                                                           float factor) {
    const int lane = threadIdx.x & 31;
    const int64_t unit = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (unit >= units) return;
    const int64_t t = unit / H;
    const int h = (int)(unit - t * H), g = h / hq, hh = h - g * hq;
    const float* a1 = a + (t * 2 * H + (int64_t)(g * 2 * hq + hh)) * dv;
    const float* a2 = a1 + (int64_t)hq * dv;
    float o[KR], ss = 0.f;
#pragma unroll
    for (int k = 0; k < KR; k++) {
        const int d = lane + 32 * k;
        o[k] = d < dv ? a1[d] - lambda * a2[d] : 0.f;
        ss += o[k] * o[k];
    }
    const float f = factor / sqrtf(warp_sum(ss) / (float)dv + eps);
    const T* gr = gate != nullptr ? gate + t * gate_stride_t + (int64_t)h * dv : nullptr;
    T* orow = out + t * out_stride_t + (int64_t)h * dv;
#pragma unroll
    for (int k = 0; k < KR; k++) {
        const int d = lane + 32 * k;
        if (d < dv) {
            float y = o[k] * f;
            if (gr != nullptr) y *= 1.f / (1.f + expf(-ldf(gr + d)));
            stf(orow + d, y);
        }
    }
}

static bool g_window_simt = false;

// rows [0, num_prefill) are prompt portions (many consecutive tokens of a sequence share a CTA), the rest single decoded tokens
template <typename T, int DMAX, bool EXT>
static int launch_window_attn_mma(const void* q, int64_t q_stride_t, const void* cosb, const void* sinb, const void* gate,
                                  int64_t gate_stride_t, const void* cache, int n_slots, int slot, int block_size,
                                  const void* block_table, int max_blocks_per_seq, const void* tok_seq, const void* tok_pos,
                                  void* out, int64_t out_stride_t, int64_t num_tokens, int64_t num_prefill, int H, int G, int dk,
                                  int dv, int rot_dims, int window, float scale, float sink, int halves, float qk_norm_eps,
                                  float softcap, const void* vcos, const void* vsin, float out_scale, const void* qnorm_w,
                                  float prenorm_eps, int chunk, int vshare, int out_f32, const void* slopes, int keep_first,
                                  int gate_per_head, int shared_kv, int krot, const void* sinks, cudaStream_t stream) {
    static unsigned long long attr_mask = 0;
    const int hq = H / G;
    int hqp_log2 = 0;
    while ((1 << hqp_log2) < hq) hqp_log2++;
    auto kern_prompt = window_attn_mma_kernel<T, DMAX, 32, EXT>;
    auto kern_decode = window_attn_mma_kernel<T, DMAX, 64, EXT>;
    // single decoded tokens of up to 16 heads per group: keys split over the warps of a CTA; small tiles where a row is long
    // (eight warps where a key row is also the value row and a stage is half as large)
    constexpr int KT = DMAX == 64 ? 32 : 16, WD_WARPS = EXT ? 8 : 4;
    auto kern_split = hq <= 8 ? window_attn_decode_kernel<T, DMAX, KT, 1, WD_WARPS, EXT> : window_attn_decode_kernel<T, DMAX, KT, 2, WD_WARPS, EXT>;
    if (first_use_on_this_device(attr_mask)) {
        cudaFuncSetAttribute(window_attn_decode_kernel<T, DMAX, KT, 1, WD_WARPS, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
        cudaFuncSetAttribute(window_attn_decode_kernel<T, DMAX, KT, 2, WD_WARPS, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
        cudaFuncSetAttribute(kern_prompt, cudaFuncAttributeMaxDynamicSharedMemorySize, 120 * 1024);
        cudaFuncSetAttribute(kern_decode, cudaFuncAttributeMaxDynamicSharedMemorySize, 120 * 1024);
    }
    int num_sms = 0;
    cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, current_device());
    const float scale_log2 = scale * 1.4426950408889634f;
    const int64_t parts[2][2] = {{0, num_prefill}, {num_prefill, num_tokens - num_prefill}};
    for (int k = 0; k < 2; k++) {
        const int64_t first = parts[k][0], count = parts[k][1];
        if (count <= 0) continue;
        if (k == 1 && hq <= 16) {
            size_t smem = 16 * (size_t)(dk * 2 + 16) + WD_WARPS * WD_STAGES * (size_t)KT * (tile_pitch(dk + krot) + (shared_kv ? sizeof(float) : dv * 2 + 16));
            const size_t merge = ((size_t)WD_WARPS * hq * dv + 2 * WD_WARPS * 16) * sizeof(float);
            if (smem < merge) smem = merge;
            kern_split<<<dim3((unsigned)count, (unsigned)G), WD_WARPS * 32, smem, stream>>>(
                (const T*)q, q_stride_t, (const float*)cosb, (const float*)sinb, (const T*)gate, gate_stride_t, (const T*)cache,
                n_slots, slot, block_size, (const int*)block_table, max_blocks_per_seq, (const int*)tok_seq, (const int*)tok_pos,
                (T*)out, out_stride_t, (int)first, hq, G, dk, dv, rot_dims, window, scale_log2, sink, halves, qk_norm_eps, softcap,
                (const float*)vcos, (const float*)vsin, out_scale, (const float*)qnorm_w, prenorm_eps, chunk, vshare, out_f32,
                (const float*)slopes, keep_first, gate_per_head, shared_kv, krot, (const float*)sinks);
            continue;
        }
        const int qt = k == 0 ? WT_ROWS >> hqp_log2 : 1;
        // measured on B200 (128 + 128 per head): prompt portions 24 - 26 % faster with 32-key tiles (three CTAs per SM instead of
        // two); decoded tokens faster with 64-key tiles at 512 CTAs (357 vs 385 us), with 32-key tiles at 2048 CTAs (950 vs 1220 us)
        const int keys = (k == 0 || count * G >= 7 * (int64_t)num_sms) ? 32 : 64;
        size_t smem = (size_t)WT_ROWS * (dk * 2 + 16) + 2 * (size_t)keys * (tile_pitch(dk + krot) + (shared_kv ? sizeof(float) : dv * 2 + 16));
        if (vcos != nullptr && smem < (size_t)WT_ROWS * dv * sizeof(float)) smem = (size_t)WT_ROWS * dv * sizeof(float);
        (keys == 32 ? kern_prompt : kern_decode)<<<dim3((unsigned)cdiv(count, qt), (unsigned)G), 128, smem, stream>>>(
            (const T*)q, q_stride_t, (const float*)cosb, (const float*)sinb, (const T*)gate, gate_stride_t, (const T*)cache,
            n_slots, slot, block_size, (const int*)block_table, max_blocks_per_seq, (const int*)tok_seq, (const int*)tok_pos,
            (T*)out, out_stride_t, (int)first, (int)count, qt, hq, hqp_log2, H, G, dk, dv, rot_dims, window, scale_log2, sink,
            halves, qk_norm_eps, softcap, (const float*)vcos, (const float*)vsin, out_scale, (const float*)qnorm_w, prenorm_eps,
            chunk, vshare, out_f32, (const float*)slopes, keep_first, gate_per_head, shared_kv, krot, (const float*)sinks);
    }
    return check_launch("window_attention (tensor cores)");
}

static int heads_per_cta(int hq) {
    for (int n = WA_MAX_HPB; n > 1; n--)
        if (hq % n == 0) return n;
    return 1;
}

template <typename T, int KR>
static int launch_window_attn(const void* q, int64_t q_stride_t, const void* cosb, const void* sinb, const void* gate,
                              int64_t gate_stride_t, const void* cache, int n_slots, int slot, int block_size,
                              const void* block_table, int max_blocks_per_seq, const void* tok_seq, const void* tok_pos, void* out,
                              int64_t out_stride_t, int64_t num_tokens, int H, int G, int dk, int dv, int rot_dims, int window,
                              float scale, float sink, int halves, float qk_norm_eps, float softcap, const void* vcos,
                              const void* vsin, float out_scale, const void* qnorm_w, float prenorm_eps, int chunk, int vshare,
                              int out_f32, const void* slopes, int keep_first, int gate_per_head, int shared_kv, int krot,
                              const void* sinks, cudaStream_t stream) {
    static unsigned long long attr_mask = 0;
    const int hpb = heads_per_cta(H / G);
    const size_t smem = ((size_t)hpb * dk + (size_t)WA_TILE * (dk + krot + 1) + (shared_kv ? 0 : (size_t)WA_TILE * dv) + (size_t)hpb * dv + WA_TILE) * sizeof(float);
    SLLM_REQUIRE(smem <= 200 * 1024, "window_attention: head sizes %d / %d need %zu bytes of shared memory", dk, dv, smem);
    auto kern = window_attn_kernel<T, KR>;
    if (first_use_on_this_device(attr_mask))
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    kern<<<dim3((unsigned)num_tokens, (unsigned)(H / hpb)), hpb * 32, smem, stream>>>(
        (const T*)q, q_stride_t, (const float*)cosb, (const float*)sinb, (const T*)gate, gate_stride_t, (const T*)cache, n_slots,
        slot, block_size, (const int*)block_table, max_blocks_per_seq, (const int*)tok_seq, (const int*)tok_pos, (T*)out,
        out_stride_t, H, G, dk, dv, rot_dims, window, scale, sink, halves, qk_norm_eps, softcap, (const float*)vcos,
        (const float*)vsin, out_scale, (const float*)qnorm_w, prenorm_eps, chunk, vshare, out_f32, (const float*)slopes, keep_first,
        gate_per_head, shared_kv, krot, (const float*)sinks);
    return check_launch("window_attention");
}

}  // namespace sllm

using namespace sllm;

extern "C" {

int sllm_window_kv_store(const void* k, int64_t k_row_stride, const void* v, int64_t v_row_stride, const void* cosb,
                         const void* sinb, const void* tok_seq, const void* tok_pos, const void* block_table,
                         int max_blocks_per_seq, void* cache, int n_slots, int slot, int block_size, int64_t num_tokens,
                         int num_kv_heads, int dk, int dv, int rot_dims, int pair_halves, float qk_norm_eps, const void* vcos,
                         const void* vsin, const void* knorm_w, float prenorm_eps, int vshare, sllm_dtype_t dtype,
                         sllm_stream_t stream) {
    SLLM_REQUIRE(vshare >= 1 && num_kv_heads % vshare == 0, "window_kv_store: %d key heads cannot share values in runs of %d",
                 num_kv_heads, vshare);
    SLLM_REQUIRE(num_tokens >= 0 && num_kv_heads > 0 && dk > 0 && dv > 0 && rot_dims >= 0 && rot_dims <= dk && rot_dims % 2 == 0,
                 "window_kv_store: bad shape (kv heads %d, dk %d, dv %d, rot_dims %d)", num_kv_heads, dk, dv, rot_dims);
    SLLM_REQUIRE((vcos == nullptr) == (vsin == nullptr) && (vcos == nullptr || dv % 2 == 0),
                 "window_kv_store: turned values need both angle tables and an even value size (dv %d)", dv);
    SLLM_REQUIRE(slot >= 0 && slot < n_slots && block_size > 0, "window_kv_store: bad cache slot %d of %d", slot, n_slots);
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(k && v && tok_seq && tok_pos && block_table && cache && (rot_dims == 0 || (cosb && sinb)),
                 "window_kv_store: null pointer");
    SLLM_DISPATCH_DTYPE_F32(dtype, (window_kv_store_kernel<T><<<(unsigned)num_tokens, 128, 0, (cudaStream_t)stream>>>(
        (const T*)k, k_row_stride, (const T*)v, v_row_stride, (const float*)cosb, (const float*)sinb, (const int*)tok_seq,
        (const int*)tok_pos, (const int*)block_table, max_blocks_per_seq, (T*)cache, n_slots, slot, block_size, num_kv_heads,
        dk, dv, rot_dims, pair_halves, qk_norm_eps, (const float*)vcos, (const float*)vsin, (const float*)knorm_w, prenorm_eps,
        vshare)));
    return check_launch("window_kv_store");
}

int sllm_shared_kv_store(const void* k, int64_t k_row_stride, const void* tok_seq, const void* tok_pos, const void* block_table,
                         int max_blocks_per_seq, void* cache, int n_slots, int slot, int block_size, int64_t num_tokens,
                         int num_kv_heads, int dk, float eps, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && num_kv_heads > 0 && dk > 0, "shared_kv_store: bad shape (kv heads %d, dk %d)", num_kv_heads, dk);
    SLLM_REQUIRE(slot >= 0 && slot < n_slots && block_size > 0, "shared_kv_store: bad cache slot %d of %d", slot, n_slots);
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(k && tok_seq && tok_pos && block_table && cache, "shared_kv_store: null pointer");
    SLLM_DISPATCH_DTYPE_F32(dtype, (shared_kv_store_kernel<T><<<(unsigned)num_tokens, 128, 0, (cudaStream_t)stream>>>(
        (const T*)k, k_row_stride, (const int*)tok_seq, (const int*)tok_pos, (const int*)block_table, max_blocks_per_seq,
        (T*)cache, n_slots, slot, block_size, num_kv_heads, dk, eps)));
    return check_launch("shared_kv_store");
}

int sllm_whole_norm_rope_store(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* q_norm_w,
                               const void* k_norm_w, float eps, const void* cosb, const void* sinb, const void* tok_seq,
                               const void* tok_pos, const void* block_table, int max_blocks_per_seq, void* cache, int n_slots, int slot,
                               int block_size, void* q_out, int64_t num_tokens, int num_heads, int num_kv_heads, int dk, int rot_dims,
                               int pair_halves, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && num_heads > 0 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dk > 0 && rot_dims >= 0 &&
                 rot_dims <= dk && rot_dims % 2 == 0, "whole_norm_rope_store: bad shape (heads %d / %d, dk %d, rot_dims %d)", num_heads,
                 num_kv_heads, dk, rot_dims);
    SLLM_REQUIRE(slot >= 0 && slot < n_slots && block_size > 0, "whole_norm_rope_store: bad cache slot %d of %d", slot, n_slots);
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(q && k && q_norm_w && k_norm_w && tok_seq && tok_pos && block_table && cache && q_out && (rot_dims == 0 || (cosb && sinb)),
                 "whole_norm_rope_store: null pointer");
    const size_t smem = ((size_t)(num_heads + num_kv_heads) * dk + rot_dims) * sizeof(float);
    SLLM_REQUIRE(smem <= 200 * 1024, "whole_norm_rope_store: %d + %d heads of %d entries do not fit in shared memory", num_heads,
                 num_kv_heads, dk);
    const int per = dtype == SLLM_F32 ? 4 : 8;
    const bool vec = dk % 4 == 0 && rot_dims % 4 == 0 && (num_heads * dk) % per == 0 && (num_kv_heads * dk) % per == 0 && q_row_stride % per == 0 &&
                     k_row_stride % per == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)q_out | (uintptr_t)cache) & 15) == 0;
    SLLM_DISPATCH_DTYPE_F32(dtype, {
        static unsigned long long attr_mask = 0;
        if (first_use_on_this_device(attr_mask)) {
            cudaFuncSetAttribute(whole_norm_rope_store_kernel<T, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
            cudaFuncSetAttribute(whole_norm_rope_store_kernel<T, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        }
        (vec ? whole_norm_rope_store_kernel<T, true> : whole_norm_rope_store_kernel<T, false>)<<<(unsigned)num_tokens, 256, smem,
                                                                                             (cudaStream_t)stream>>>(
            (const T*)q, q_row_stride, (const T*)k, k_row_stride, (const float*)q_norm_w, (const float*)k_norm_w, eps, (const float*)cosb,
            (const float*)sinb, (const int*)tok_seq, (const int*)tok_pos, (const int*)block_table, max_blocks_per_seq, (T*)cache, n_slots,
            slot, block_size, (T*)q_out, num_heads, num_kv_heads, dk, rot_dims, pair_halves);
    });
    return check_launch("whole_norm_rope_store");
}

int sllm_window_attention_set_simt(int on) {
    const int old = g_window_simt ? 1 : 0;
    g_window_simt = on != 0;
    return old;
}

int sllm_window_attention(const void* q, int64_t q_stride_t, const void* cosb, const void* sinb, const void* gate,
                          int64_t gate_stride_t, const void* cache, int n_slots, int slot, int block_size,
                          const void* block_table, int max_blocks_per_seq, const void* tok_seq, const void* tok_pos, void* out,
                          int64_t out_stride_t, int64_t num_tokens, int64_t num_prefill_tokens, int num_heads, int num_kv_heads,
                          int dk, int dv, int rot_dims, int window, float scale, int sink, int pair_halves, float qk_norm_eps,
                          float softcap, const void* vcos, const void* vsin, float out_scale, const void* qnorm_w,
                          float prenorm_eps, int chunk, int vshare, int out_f32, const void* slopes, int keep_first,
                          int gate_per_head, int shared_kv, int krot, const void* sinks, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(krot >= 0 && krot <= dk && (krot == 0 || shared_kv), "window_attention: %d turned entries beside shared keys of %d", krot, dk);
    SLLM_REQUIRE(!(sink && sinks), "window_attention: a sink of score 0 or learned sinks, not both");
    SLLM_REQUIRE(keep_first >= 0 && (keep_first == 0 || chunk == 0), "window_attention: kept first positions (%d) exclude chunks",
                 keep_first);
    SLLM_REQUIRE(!shared_kv || (dk == dv && vshare == 1 && rot_dims == 0 && qk_norm_eps < 0.f && vcos == nullptr),
                 "window_attention: values that are the un-normed keys need dk = dv and no rotation (dk %d, dv %d)", dk, dv);
    SLLM_REQUIRE(vshare >= 1 && num_kv_heads % vshare == 0 && chunk >= 0 && (!out_f32 || vcos == nullptr),
                 "window_attention: %d key heads in runs of %d; chunk %d >= 0; fp32 output excludes turned values", num_kv_heads,
                 vshare, chunk);
    SLLM_REQUIRE((vcos == nullptr) == (vsin == nullptr) && (vcos == nullptr || dv % 2 == 0) && softcap >= 0.f,
                 "window_attention: turned values need both angle tables and an even value size (dv %d); softcap >= 0", dv);
    SLLM_REQUIRE(num_tokens >= 0 && num_heads > 0 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dk > 0 && dv > 0 &&
                 dv <= 256 && rot_dims >= 0 && rot_dims <= dk && rot_dims % 2 == 0,
                 "window_attention: bad shape (heads %d / %d, dk %d, dv %d <= 256, rot_dims %d)", num_heads, num_kv_heads, dk,
                 dv, rot_dims);
    SLLM_REQUIRE(slot >= 0 && slot < n_slots && block_size > 0, "window_attention: bad cache slot %d of %d", slot, n_slots);
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(q && tok_seq && tok_pos && block_table && cache && out && (rot_dims == 0 || (cosb && sinb)),
                 "window_attention: null pointer");
    SLLM_REQUIRE(num_prefill_tokens >= 0 && num_prefill_tokens <= num_tokens, "window_attention: bad number of prompt rows");
    const float sinkw = sink ? 1.f : 0.f;
    const int hq = num_heads / num_kv_heads;
    if (!g_window_simt && dtype != SLLM_F32 && dk % 16 == 0 && dv % 16 == 0 && krot % 8 == 0 && dk <= 128 && dv <= 128 && hq <= WT_ROWS &&
        num_tokens < (1ll << 31)) {
#define WA_MMA(DMAX, EXT)                                                                                                        \
    SLLM_DISPATCH_DTYPE(dtype, return (launch_window_attn_mma<T, DMAX, EXT>(q, q_stride_t, cosb, sinb, gate, gate_stride_t, cache,  \
        n_slots, slot, block_size, block_table, max_blocks_per_seq, tok_seq, tok_pos, out, out_stride_t, num_tokens,         \
        num_prefill_tokens, num_heads, num_kv_heads, dk, dv, rot_dims, window, scale, sinkw, pair_halves, qk_norm_eps, softcap, \
        vcos, vsin, out_scale, qnorm_w, prenorm_eps, chunk, vshare, out_f32, slopes, keep_first, gate_per_head, shared_kv, krot, sinks, \
        (cudaStream_t)stream)))
        const bool ext = slopes != nullptr || keep_first > 0 || gate_per_head || shared_kv || sinks != nullptr;
        const bool small = dk <= 64 && dv <= 64;
        if (ext) { if (small) { WA_MMA(64, true); } else { WA_MMA(128, true); } }
        else if (small) { WA_MMA(64, false); }
        else { WA_MMA(128, false); }
#undef WA_MMA
    }
#define WA_LAUNCH(KR)                                                                                                      \
    SLLM_DISPATCH_DTYPE_F32(dtype, return (launch_window_attn<T, KR>(q, q_stride_t, cosb, sinb, gate, gate_stride_t, cache,   \
        n_slots, slot, block_size, block_table, max_blocks_per_seq, tok_seq, tok_pos, out, out_stride_t, num_tokens,        \
        num_heads, num_kv_heads, dk, dv, rot_dims, window, scale, sinkw, pair_halves, qk_norm_eps, softcap, vcos, vsin,      \
        out_scale, qnorm_w, prenorm_eps, chunk, vshare, out_f32, slopes, keep_first, gate_per_head, shared_kv, krot, sinks, \
        (cudaStream_t)stream)))
    if (dv <= 32) { WA_LAUNCH(1); }
    else if (dv <= 64) { WA_LAUNCH(2); }
    else if (dv <= 128) { WA_LAUNCH(4); }
    else { WA_LAUNCH(8); }
#undef WA_LAUNCH
    return 0;
}

int sllm_diff_combine(const void* a, const void* gate, int64_t gate_stride_t, void* out, int64_t out_stride_t, int64_t num_tokens,
                      int num_heads, int num_kv_heads, int dv, float lambda, float eps, float factor, sllm_dtype_t dtype,
                      sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && num_heads > 0 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dv > 0 && dv <= 256,
                 "diff_combine: bad shape (heads %d / %d, dv %d <= 256)", num_heads, num_kv_heads, dv);
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(a && out, "diff_combine: null pointer");
    const int64_t units = num_tokens * num_heads;
    const int hq = num_heads / num_kv_heads;
#define DC_LAUNCH(KR)                                                                                                       \
    SLLM_DISPATCH_DTYPE_F32(dtype, (diff_combine_kernel<T, KR><<<(unsigned)cdiv(units, 8), 256, 0, (cudaStream_t)stream>>>(   \
        (const float*)a, (const T*)gate, gate_stride_t, (T*)out, out_stride_t, units, num_heads, hq, dv, lambda, eps, factor)))
    if (dv <= 32) { DC_LAUNCH(1); }
    else if (dv <= 64) { DC_LAUNCH(2); }
    else if (dv <= 128) { DC_LAUNCH(4); }
    else { DC_LAUNCH(8); }
#undef DC_LAUNCH
    return check_launch("diff_combine");
}

}  // extern "C"
