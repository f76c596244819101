// Several residual streams per token (hyper-connections): a sublayer reads a weighted sum of the streams through an RMS norm,
//     h = rms(sum_s in[s] x_s) * norm_w,
// and its output y goes back into all of them at once,
//     x_t <- sum_s mix[s, t] x_s + share[t] y.
// ONE kernel does a sublayer's write and the next sublayer's read: the streams are read once and written once.  The streams, both sums
// and the norm are fp32 for every storage type T of y and h.  Algorithmic bytes: width * (8 streams + 2 s) per token (s = sizeof(T)).
#include "typed_io.cuh"

namespace sllm {

template <typename T, int V> struct HsVec;
template <typename T> struct HsVec<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = ldf(p); }
    static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { stf(p, v[0]); }
};
template <> struct HsVec<float, 4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
};
template <typename T> struct HsVec<T, 4> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[4]) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
        for (int i = 0; i < 4; i++) v[i] = ldf(e + i);
    }
    static __device__ __forceinline__ void store(T* p, const float (&v)[4]) {
        uint2 u;
        T* e = reinterpret_cast<T*>(&u);
#pragma unroll
        for (int i = 0; i < 4; i++) stf(e + i, v[i]);
        *reinterpret_cast<uint2*>(p) = u;
    }
};

// One CTA per row; row i of `h` is token rows[i] (or i).  x_in: [T, S, width], or [T, width] when all streams are still equal
// (one_stream).  y null: the streams stay as they are.  x_out (may be x_in, unless one_stream) null: not written.  h null: no read.
// SMAX: streams held in registers (S <= SMAX); V entries a thread and turn.  Dynamic shared memory: width floats.
template <typename T, int SMAX, int V>
__global__ void __launch_bounds__(256, SMAX <= 4 ? 4 : 1) stream_mix_norm_kernel(const float* x_in, int one_stream, int S, const T* __restrict__ y,
                                                              const float* __restrict__ mix, const float* __restrict__ share,
                                                              const float* __restrict__ in, const float* __restrict__ norm_w,
                                                              float eps, float* x_out, T* __restrict__ h,
                                                              const int* __restrict__ rows, int width) {
    extern __shared__ __align__(16) float u_row[];                     // [width]
    __shared__ float ms[SMAX * SMAX], sh[SMAX], ins[SMAX], red[32];
    const int64_t i = blockIdx.x, t = rows != nullptr ? rows[i] : i;
    for (int k = threadIdx.x; k < SMAX * SMAX; k += blockDim.x) {
        const int s = k / SMAX, to = k % SMAX;
        ms[k] = y != nullptr && s < S && to < S ? mix[s * S + to] : 0.f;
    }
    if (threadIdx.x < SMAX) {
        sh[threadIdx.x] = y != nullptr && threadIdx.x < S ? share[threadIdx.x] : 0.f;
        ins[threadIdx.x] = h != nullptr && threadIdx.x < S ? in[threadIdx.x] : 0.f;
    }
    __syncthreads();
    const float* xr = x_in + t * (one_stream ? 1 : S) * (int64_t)width;
    float* xo = x_out != nullptr ? x_out + t * S * (int64_t)width : nullptr;
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        float x[SMAX][V], u[V];
#pragma unroll
        for (int s = 0; s < SMAX; s++) {
            if (s < S && (s == 0 || !one_stream)) HsVec<float, V>::load(xr + (int64_t)s * width + c, x[s]);
            else {
#pragma unroll
                for (int e = 0; e < V; e++) x[s][e] = s < S ? x[0][e] : 0.f;
            }
        }
#pragma unroll
        for (int e = 0; e < V; e++) u[e] = 0.f;
        if (y != nullptr) {
            float yv[V];
            HsVec<T, V>::load(y + t * width + c, yv);
#pragma unroll
            for (int to = 0; to < SMAX; to++) {
                if (to >= S) break;
                float o[V];
#pragma unroll
                for (int e = 0; e < V; e++) o[e] = sh[to] * yv[e];
#pragma unroll
                for (int s = 0; s < SMAX; s++)
#pragma unroll
                    for (int e = 0; e < V; e++) o[e] = fmaf(ms[s * SMAX + to], x[s][e], o[e]);
                if (xo != nullptr) HsVec<float, V>::store(xo + (int64_t)to * width + c, o);
#pragma unroll
                for (int e = 0; e < V; e++) u[e] = fmaf(ins[to], o[e], u[e]);
            }
        } else {
#pragma unroll
            for (int s = 0; s < SMAX; s++) {
                if (xo != nullptr && s < S) HsVec<float, V>::store(xo + (int64_t)s * width + c, x[s]);
#pragma unroll
                for (int e = 0; e < V; e++) u[e] = fmaf(ins[s], x[s][e], u[e]);
            }
        }
        if (h != nullptr) {
            HsVec<float, V>::store(u_row + c, u);                      // read back by this thread only
#pragma unroll
            for (int e = 0; e < V; e++) ss += u[e] * u[e];
        }
    }
    if (h == nullptr) return;
    const float f = 1.f / sqrtf(block_sum(ss, red) / (float)width + eps);
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        float u[V], w[V];
        HsVec<float, V>::load(u_row + c, u);
        HsVec<float, V>::load(norm_w + c, w);
#pragma unroll
        for (int e = 0; e < V; e++) u[e] *= f * w[e];
        HsVec<T, V>::store(h + i * width + c, u);
    }
}

template <typename T, int SMAX>
static int launch_stream_mix_norm(const void* x_in, int one_stream, int S, const void* y, const void* mix, const void* share,
                                  const void* in, const void* norm_w, float eps, void* x_out, void* h, const void* rows,
                                  int64_t num_rows, int width, cudaStream_t stream) {
    const bool quad = width % 4 == 0 && (((uintptr_t)x_in | (uintptr_t)y | (uintptr_t)x_out | (uintptr_t)h | (uintptr_t)norm_w) & 15) == 0;
    int threads = 32;
    while (threads < 256 && threads * (quad ? 4 : 1) < width) threads *= 2;
    const size_t smem = (size_t)width * sizeof(float);
    auto kern = quad ? stream_mix_norm_kernel<T, SMAX, 4> : stream_mix_norm_kernel<T, SMAX, 1>;
    if (smem > 40 * 1024) {
        SLLM_REQUIRE(smem <= 200 * 1024, "stream_mix_norm: rows of %d entries do not fit in shared memory", width);
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    }
    kern<<<(unsigned)num_rows, threads, smem, stream>>>((const float*)x_in, one_stream, S, (const T*)y, (const float*)mix,
                                                        (const float*)share, (const float*)in, (const float*)norm_w, eps, (float*)x_out,
                                                        (T*)h, (const int*)rows, width);
    return check_launch("stream_mix_norm");
}

}  // namespace sllm

using namespace sllm;

extern "C" int sllm_stream_mix_norm(const void* x_in, int one_stream, int streams, const void* y, const void* mix, const void* share,
                                    const void* in, const void* norm_w, float eps, void* x_out, void* h, const void* rows,
                                    int64_t num_rows, int width, sllm_dtype_t dtype, sllm_stream_t stream) {
    SLLM_REQUIRE(num_rows >= 0 && width > 0 && streams >= 1 && streams <= 16, "stream_mix_norm: 1 <= streams <= 16 (got %d), width %d",
                 streams, width);
    if (num_rows == 0) return 0;
    SLLM_REQUIRE(x_in && (y == nullptr || (mix && share)) && (h == nullptr || (in && norm_w)) && (x_out || h), "stream_mix_norm: null pointer");
    SLLM_REQUIRE(!(one_stream && streams > 1 && x_in == x_out), "stream_mix_norm: one stream cannot become several in place");
#define SMN(SMAX)                                                                                                          \
    SLLM_DISPATCH_DTYPE_F32(dtype, return (launch_stream_mix_norm<T, SMAX>(x_in, one_stream, streams, y, mix, share, in, norm_w, eps,  \
        x_out, h, rows, num_rows, width, (cudaStream_t)stream)))
    if (streams == 1) { SMN(1); }
    else if (streams == 2) { SMN(2); }
    else if (streams <= 4) { SMN(4); }
    else if (streams <= 8) { SMN(8); }
    else { SMN(16); }
#undef SMN
    return 0;
}
