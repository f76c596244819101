// Row-wise kernels of SEQUENTIAL decoder blocks whose sublayers read the fp32 residual stream itself and whose OUTPUT is
// normalised before it is added (x <- x + gain * y / rms(y), a scalar gain or one per channel), with an optional learned weighted sum
// over the results of all earlier layers ("depth mix"), plus the embedding with a hashed table of token pairs, the tanh cap
// of logits, and the router / activation of a mixture of SiLU-gated experts with sigmoid scores.
// The stream, sums, norms and the router are fp32 whatever the storage type T (half, bf16 or float) of the projections is; every
// kernel that updates the stream also writes its rounding to T, which is what the next projections read.
// Algorithmic bytes (s = sizeof(T)): postnorm_add_mix  T*W*(8 + 2s) + 4*T*W*(1 + mixed layers).
// Also here: the SiLU gated linear unit and the element-wise sigmoid gate of a mixer's output.
#include "typed_io.cuh"

namespace sllm {

// x[t] = embed[token] * scale + pairs[row]; row = (previous * mul_prev + token * mul_cur) mod buckets, where `previous` is the token
// before it: the row above when that is the same sequence's previous position, else the sequence's stored last token; a
// sequence's first token (position 0) takes row `buckets`.  One CTA per token.
template <typename T>
__global__ void __launch_bounds__(256) embed_pair_hash_kernel(
    const int* __restrict__ tokens, const int* __restrict__ tok_seq, const int* __restrict__ tok_pos,
    const int* __restrict__ last_token, const T* __restrict__ embed, const T* __restrict__ pairs, int buckets, int64_t mul_prev,
    int64_t mul_cur, float scale, float* __restrict__ x, float* __restrict__ x_copy, T* __restrict__ h, int width) {
    const int64_t t = blockIdx.x;
    const int tok = tokens[t], pos = tok_pos[t], seq = tok_seq[t];
    const T* er = embed + (int64_t)tok * width;
    const T* pr = nullptr;
    if (pairs != nullptr) {
        int64_t row = buckets;
        if (pos > 0) {
            const bool above = t > 0 && tok_seq[t - 1] == seq && tok_pos[t - 1] == pos - 1;
            const int64_t prev = above ? tokens[t - 1] : last_token[seq];
            row = (prev * mul_prev + (int64_t)tok * mul_cur) % buckets;
            if (row < 0) row += buckets;
        }
        pr = pairs + row * width;
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        float v = ldf(er + i) * scale;
        if (pr != nullptr) v += ldf(pr + i);
        x[t * width + i] = v;
        if (x_copy != nullptr) x_copy[t * width + i] = v;
        if (h != nullptr) stf(h + t * width + i, v);
    }
}

// last_token[seq of segment b] = the segment's last token.  Runs after the embedding has read the old values.
__global__ void store_last_tokens_kernel(const int* __restrict__ tokens, const int* __restrict__ seg_starts,
                                         const int* __restrict__ seq_ids, int* __restrict__ last_token, int num_segs) {
    const int b = blockIdx.x * blockDim.x + threadIdx.x;
    if (b < num_segs && seg_starts[b + 1] > seg_starts[b]) last_token[seq_ids[b]] = tokens[seg_starts[b + 1] - 1];
}

// X = x[t] + gain * y[t] / sqrt(mean(y[t]^2) + eps)     (X = x[t] when y is null; gain: one number, or [width] with gain_step = 1)
// history[slot][t] = X (when history is given); x[t] <- sum_{j <= slot} mix[j] * history[j][t] (when mix is given), else X;
// h[t] = T(x[t]).  One CTA per token.
template <typename T>
__global__ void __launch_bounds__(256) postnorm_add_mix_kernel(
    float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ gain, int gain_step, float eps, float* __restrict__ history,
    int slot, int64_t hist_stride, const float* __restrict__ mix, T* __restrict__ h, int width) {
    __shared__ float red[32];
    const int64_t t = blockIdx.x;
    float f = 0.f;
    if (y != nullptr) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < width; i += blockDim.x) { const float v = ldf(y + t * width + i); ss += v * v; }
        f = 1.f / sqrtf(block_sum(ss, red) / (float)width + eps);
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        float v = x[t * width + i];
        if (y != nullptr) v += ldf(y + t * width + i) * (f * gain[i * gain_step]);
        if (history != nullptr) history[slot * hist_stride + t * width + i] = v;
        if (mix != nullptr) {
            float acc = mix[slot] * v;
            for (int j = 0; j < slot; j++) acc += mix[j] * history[j * hist_stride + t * width + i];
            v = acc;
        }
        x[t * width + i] = v;
        stf(h + t * width + i, v);
    }
}

// The same add without history: one row per CTA of `NT` threads, four entries a thread and turn (width % 4 == 0, rows 16-byte
// aligned), y kept in registers between the two passes (width <= 4 * NT * RY).
template <typename T> struct Quad;
template <> struct Quad<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
    static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <typename T> struct Quad {
    static __device__ __forceinline__ float4 load(const T* p) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const T* e = reinterpret_cast<const T*>(&u);
        return make_float4(ldf(e), ldf(e + 1), ldf(e + 2), ldf(e + 3));
    }
    static __device__ __forceinline__ void store(T* p, float4 v) {
        uint2 u;
        T* e = reinterpret_cast<T*>(&u);
        stf(e, v.x); stf(e + 1, v.y); stf(e + 2, v.z); stf(e + 3, v.w);
        *reinterpret_cast<uint2*>(p) = u;
    }
};

template <typename T, int RY>
__global__ void __launch_bounds__(256) postnorm_add_quad_kernel(float* __restrict__ x, const T* __restrict__ y,
                                                                const float* __restrict__ gain, int gain_step, float eps,
                                                                T* __restrict__ h, int width) {
    __shared__ float red[32];
    const int64_t base = (int64_t)blockIdx.x * width;
    float4 v[RY], xv[RY];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < RY; k++) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        v[k] = xv[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < width) {
            v[k] = Quad<T>::load(y + base + i);
            xv[k] = *reinterpret_cast<const float4*>(x + base + i);
        }
        ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    }
    const float f = 1.f / sqrtf(block_sum(ss, red) / (float)width + eps);
#pragma unroll
    for (int k = 0; k < RY; k++) {
        const int i = 4 * (threadIdx.x + k * blockDim.x);
        if (i >= width) break;
        float4 g;
        if (gain_step) g = *reinterpret_cast<const float4*>(gain + i);
        else g.x = g.y = g.z = g.w = gain[0];
        const float4 o = make_float4(xv[k].x + v[k].x * (f * g.x), xv[k].y + v[k].y * (f * g.y), xv[k].z + v[k].z * (f * g.z),
                                     xv[k].w + v[k].w * (f * g.w));
        *reinterpret_cast<float4*>(x + base + i) = o;
        Quad<T>::store(h + base + i, o);
    }
}

// u [T, 2 F] = [gate | up] -> y [T, F] = silu(gate) * up; V entries a thread (F % V == 0)
template <typename T, int V>
__global__ void silu_glu_kernel(const T* __restrict__ u, T* __restrict__ y, int64_t n, int ff) {
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= n) return;
    const int64_t t = i / ff;
    const int f = (int)(i - t * ff);
    const T* ur = u + t * 2 * ff;
    if constexpr (V == 4) {
        const float4 g = Quad<T>::load(ur + f), v = Quad<T>::load(ur + ff + f);
        Quad<T>::store(y + i, make_float4(g.x / (1.f + expf(-g.x)) * v.x, g.y / (1.f + expf(-g.y)) * v.y,
                                          g.z / (1.f + expf(-g.z)) * v.z, g.w / (1.f + expf(-g.w)) * v.w));
    } else {
        const float g = ldf(ur + f);
        stf(y + i, g / (1.f + expf(-g)) * ldf(ur + ff + f));
    }
}

// x [T, n] (contiguous) *= sigmoid(gate [T, n]) (row-strided); V entries a thread
template <typename T, int V>
__global__ void sigmoid_gate_kernel(T* __restrict__ x, const T* __restrict__ gate, int64_t gate_stride, int64_t total, int n) {
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= total) return;
    const int64_t t = i / n;
    const T* g = gate + t * gate_stride + (i - t * n);
    if constexpr (V == 4) {
        const float4 a = Quad<T>::load(x + i), b = Quad<T>::load(g);
        Quad<T>::store(x + i, make_float4(a.x / (1.f + expf(-b.x)), a.y / (1.f + expf(-b.y)), a.z / (1.f + expf(-b.z)),
                                          a.w / (1.f + expf(-b.w))));
    } else {
        stf(x + i, ldf(x + i) / (1.f + expf(-ldf(g))));
    }
}

template <typename T>
__global__ void tanh_cap_kernel(T* __restrict__ x, int64_t n, float cap) {
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) stf(x + i, cap * tanhf(ldf(x + i) / cap));
}

// One warp per token.  s = sigmoid(logits); the `top` experts with the largest s + bias are chosen (equal values: the lower
// expert index wins); weights[t, e] = s_e at the chosen experts (not renormalised), 0 elsewhere.  groups > 1: only experts of the
// `keep` best of `groups` equal groups of neighbours can be chosen (a group's score: the sum of its two largest s + bias).
// Dynamic shared memory: warps * (2 * experts + groups) floats.
__global__ void __launch_bounds__(128) moe_route_sigmoid_kernel(const float* __restrict__ logits, const float* __restrict__ bias,
                                                                float* __restrict__ weights, int64_t num_tokens, int experts,
                                                                int top, int groups, int keep) {
    extern __shared__ float vals[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t t = (int64_t)blockIdx.x * (blockDim.x >> 5) + warp;
    if (t >= num_tokens) return;
    float* s = vals + warp * (2 * experts + groups);     // scores
    float* c = s + experts;                   // choice scores
    float* gs = c + experts;                  // group scores
    for (int e = lane; e < experts; e += 32) {
        s[e] = 1.f / (1.f + expf(-logits[t * experts + e]));
        c[e] = s[e] + (bias != nullptr ? bias[e] : 0.f);
        weights[t * experts + e] = 0.f;
    }
    __syncwarp();
    if (keep < groups) {
        const int size = experts / groups;
        for (int g = lane; g < groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;           // the two largest
            for (int e = g * size; e < (g + 1) * size; e++) {
                const float v = c[e];
                if (v > a) { b = a; a = v; } else if (v > b) b = v;
            }
            gs[g] = size > 1 ? a + b : a;
        }
        __syncwarp();
        for (int g = lane; g < groups; g += 32) {         // a group stays when fewer than `keep` groups are before it
            int before = 0;
            for (int o = 0; o < groups; o++) before += gs[o] > gs[g] || (gs[o] == gs[g] && o < g);
            if (before >= keep)
                for (int e = g * size; e < (g + 1) * size; e++) c[e] = -INFINITY;
        }
        __syncwarp();
    }
    for (int k = 0; k < top; k++) {
        float best = -INFINITY;
        int bi = 0x7fffffff;
        for (int e = lane; e < experts; e += 32) {
            const float v = c[e];
            if (v > best) { best = v; bi = e; }
        }
        if (best == -INFINITY) bi = 0x7fffffff;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
        }
        if (lane == 0 && bi != 0x7fffffff) { weights[t * experts + bi] = s[bi]; c[bi] = -INFINITY; }
        __syncwarp();
    }
}

// u [T, experts * 2 * ff] holds per expert e the rows [gate_e (ff) | up_e (ff)]; y[t, e * ff + f] = silu(gate) * up * w[t, e]:
// exact zeros for the experts a token does not use, so ONE down projection over the concatenated experts sums the chosen ones.
// V entries a thread (ff % V == 0: one expert's).
template <typename T, int V>
__global__ void moe_silu_glu_scale_kernel(const T* __restrict__ u, const float* __restrict__ w, T* __restrict__ y, int64_t n,
                                          int experts, int ff) {
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= n) return;
    const int64_t cols = (int64_t)experts * ff;
    const int64_t t = i / cols;
    const int64_t c = i - t * cols;
    const int e = (int)(c / ff), f = (int)(c - (int64_t)e * ff);
    const float wt = w[t * experts + e];
    const T* ur = u + t * 2 * cols + (int64_t)e * 2 * ff;
    if constexpr (V == 4) {
        if (wt == 0.f) { Quad<T>::store(y + i, make_float4(0.f, 0.f, 0.f, 0.f)); return; }
        const float4 g = Quad<T>::load(ur + f), v = Quad<T>::load(ur + ff + f);
        Quad<T>::store(y + i, make_float4(g.x / (1.f + expf(-g.x)) * v.x * wt, g.y / (1.f + expf(-g.y)) * v.y * wt,
                                          g.z / (1.f + expf(-g.z)) * v.z * wt, g.w / (1.f + expf(-g.w)) * v.w * wt));
    } else {
        if (wt == 0.f) { stf(y + i, 0.f); return; }
        const float g = ldf(ur + f), v = ldf(ur + ff + f);
        stf(y + i, g / (1.f + expf(-g)) * v * wt);
    }
}

}  // namespace sllm

using namespace sllm;

extern "C" {

int sllm_embed_pair_hash(const void* tokens, const void* tok_seq, const void* tok_pos, const void* last_token, const void* embed,
                         const void* pairs, int buckets, int64_t mul_prev, int64_t mul_cur, float scale, void* x, void* x_copy, void* h,
                         int64_t num_tokens, int width, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && width > 0 && (pairs == nullptr || buckets > 0), "embed_pair_hash: bad shape");
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(tokens && tok_seq && tok_pos && embed && x && (pairs == nullptr || last_token), "embed_pair_hash: null pointer");
    SLLM_DISPATCH_DTYPE_F32(dtype, (embed_pair_hash_kernel<T><<<(unsigned)num_tokens, 256, 0, (cudaStream_t)stream>>>(
        (const int*)tokens, (const int*)tok_seq, (const int*)tok_pos, (const int*)last_token, (const T*)embed, (const T*)pairs,
        buckets, mul_prev, mul_cur, scale, (float*)x, (float*)x_copy, (T*)h, width)));
    return check_launch("embed_pair_hash");
}

int sllm_store_last_tokens(const void* tokens, const void* seg_starts, const void* seq_ids, void* last_token, int num_segs,
                           sllm_stream_t stream) {
    if (num_segs <= 0) return 0;
    SLLM_REQUIRE(tokens && seg_starts && seq_ids && last_token, "store_last_tokens: null pointer");
    store_last_tokens_kernel<<<(unsigned)cdiv(num_segs, 128), 128, 0, (cudaStream_t)stream>>>(
        (const int*)tokens, (const int*)seg_starts, (const int*)seq_ids, (int*)last_token, num_segs);
    return check_launch("store_last_tokens");
}

int sllm_postnorm_add_mix(void* x, const void* y, const void* gain, int gain_per_channel, float eps, void* history, int slot,
                          const void* mix, void* h, int64_t num_tokens, int width, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && width > 0 && slot >= 0, "postnorm_add_mix: bad shape");
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(x && h && (y == nullptr || gain) && (mix == nullptr || history), "postnorm_add_mix: null pointer");
    const int step = gain_per_channel ? 1 : 0;
    const bool aligned = (((uintptr_t)x | (uintptr_t)y | (uintptr_t)h | (step ? (uintptr_t)gain : 0)) & 15) == 0;
    if (y != nullptr && history == nullptr && width % 4 == 0 && width <= 8192 && aligned) {
        int threads = 32;
        while (threads < 256 && threads * 4 < width) threads *= 2;
#define PNA(RY)                                                                                                            \
    SLLM_DISPATCH_DTYPE_F32(dtype, (postnorm_add_quad_kernel<T, RY><<<(unsigned)num_tokens, threads, 0, (cudaStream_t)stream>>>( \
        (float*)x, (const T*)y, (const float*)gain, step, eps, (T*)h, width)))
        if (width <= 4 * threads) { PNA(1); }
        else if (width <= 8 * threads) { PNA(2); }
        else if (width <= 16 * threads) { PNA(4); }
        else { PNA(8); }
#undef PNA
        return check_launch("postnorm_add_mix");
    }
    SLLM_DISPATCH_DTYPE_F32(dtype, (postnorm_add_mix_kernel<T><<<(unsigned)num_tokens, 256, 0, (cudaStream_t)stream>>>(
        (float*)x, (const T*)y, (const float*)gain, step, eps, (float*)history, slot, num_tokens * (int64_t)width, (const float*)mix,
        (T*)h, width)));
    return check_launch("postnorm_add_mix");
}

int sllm_silu_glu(const void* u, void* y, int64_t num_tokens, int ff, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && ff > 0, "silu_glu: bad shape");
    const int64_t n = num_tokens * ff;
    if (n == 0) return 0;
    SLLM_REQUIRE(u && y, "silu_glu: null pointer");
    const bool quad = ff % 4 == 0 && (((uintptr_t)u | (uintptr_t)y) & 15) == 0;
    SLLM_DISPATCH_DTYPE_F32(dtype, {
        if (quad) silu_glu_kernel<T, 4><<<(unsigned)cdiv(n / 4, 256), 256, 0, (cudaStream_t)stream>>>((const T*)u, (T*)y, n, ff);
        else silu_glu_kernel<T, 1><<<(unsigned)cdiv(n, 256), 256, 0, (cudaStream_t)stream>>>((const T*)u, (T*)y, n, ff);
    });
    return check_launch("silu_glu");
}

int sllm_sigmoid_gate_inplace(void* x, const void* gate, int64_t gate_stride, int64_t num_tokens, int n, sllm_dtype_t dtype,
                              sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && n > 0, "sigmoid_gate_inplace: bad shape");
    const int64_t total = num_tokens * n;
    if (total == 0) return 0;
    SLLM_REQUIRE(x && gate, "sigmoid_gate_inplace: null pointer");
    const bool quad = n % 4 == 0 && gate_stride % 4 == 0 && (((uintptr_t)x | (uintptr_t)gate) & 15) == 0;
    SLLM_DISPATCH_DTYPE_F32(dtype, {
        if (quad) sigmoid_gate_kernel<T, 4><<<(unsigned)cdiv(total / 4, 256), 256, 0, (cudaStream_t)stream>>>((T*)x, (const T*)gate, gate_stride, total, n);
        else sigmoid_gate_kernel<T, 1><<<(unsigned)cdiv(total, 256), 256, 0, (cudaStream_t)stream>>>((T*)x, (const T*)gate, gate_stride, total, n);
    });
    return check_launch("sigmoid_gate_inplace");
}

int sllm_tanh_cap_inplace(void* x, int64_t n, float cap, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(n >= 0 && cap > 0.f, "tanh_cap_inplace: need a positive cap");
    if (n == 0) return 0;
    SLLM_REQUIRE(x, "tanh_cap_inplace: null pointer");
    SLLM_DISPATCH_DTYPE_F32(dtype, (tanh_cap_kernel<T><<<(unsigned)cdiv(n, 256), 256, 0, (cudaStream_t)stream>>>((T*)x, n, cap)));
    return check_launch("tanh_cap_inplace");
}

int sllm_moe_route_sigmoid(const void* logits, const void* bias, void* weights, int64_t num_tokens, int experts, int top, int groups,
                           int keep, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && experts > 0 && top > 0 && top <= experts && experts <= 2048,
                 "moe_route_sigmoid: need 0 < top <= experts <= 2048 (got top %d, experts %d)", top, experts);
    SLLM_REQUIRE(groups >= 1 && experts % groups == 0 && keep >= 1 && keep <= groups && top <= keep * (experts / groups),
                 "moe_route_sigmoid: %d experts from %d of %d groups of %d", top, keep, groups, experts / (groups > 0 ? groups : 1));
    if (num_tokens == 0) return 0;
    SLLM_REQUIRE(logits && weights, "moe_route_sigmoid: null pointer");
    moe_route_sigmoid_kernel<<<(unsigned)cdiv(num_tokens, 4), 128, 4 * (2 * experts + groups) * sizeof(float), (cudaStream_t)stream>>>(
        (const float*)logits, (const float*)bias, (float*)weights, num_tokens, experts, top, groups, keep);
    return check_launch("moe_route_sigmoid");
}

int sllm_moe_silu_glu_scale(const void* u, const void* weights, void* y, int64_t num_tokens, int experts, int ff,
                            sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_tokens >= 0 && experts > 0 && ff > 0, "moe_silu_glu_scale: bad shape");
    const int64_t n = num_tokens * (int64_t)experts * ff;
    if (n == 0) return 0;
    SLLM_REQUIRE(u && y && weights, "moe_silu_glu_scale: null pointer");
    const bool quad = ff % 4 == 0 && (((uintptr_t)u | (uintptr_t)y) & 15) == 0;
    SLLM_DISPATCH_DTYPE_F32(dtype, {
        if (quad) moe_silu_glu_scale_kernel<T, 4><<<(unsigned)cdiv(n / 4, 256), 256, 0, (cudaStream_t)stream>>>((const T*)u, (const float*)weights, (T*)y, n, experts, ff);
        else moe_silu_glu_scale_kernel<T, 1><<<(unsigned)cdiv(n, 256), 256, 0, (cudaStream_t)stream>>>((const T*)u, (const float*)weights, (T*)y, n, experts, ff);
    });
    return check_launch("moe_silu_glu_scale");
}

}  // extern "C"
