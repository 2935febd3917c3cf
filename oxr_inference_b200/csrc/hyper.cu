// Several residual streams beside each other (hyper-connections), kept in fp32 as x [tokens, S, hidden]. A sublayer reads the norm of a weighted
// sum of the streams; its result y goes to every stream with a weight of that stream's, while the streams are mixed by a small matrix. What
// stands between two sublayers is one kernel, one pass over the rows:
//
//   x'_t = sum_s mix[s, t] x_s + out[t] * (scale * y)         t, s = 0 .. S - 1; `scale` (a number per entry) is optional; without a y: x' = x
//   h    = u / rms(u) * w      with  u = sum_t in[t] x'_t     the next sublayer's input, when it has one
//   sum  = sum_t x'_t                                         what leaves the streams, behind the last sublayer
//
// x may have a stream stride of zero (all streams equal, as they are in front of the first sublayer: nobody writes the copies out). x' may
// be x itself. All arithmetic fp32, h rounded once to T. One block per token; a thread keeps u of its entries in registers between the pass
// over the streams and the norm.
#include "common.cuh"

constexpr int HYPER_MAX_STREAMS = 16;

struct HyperArgs {
    const float* x;
    long long x_row, x_stream;
    float* x_out;            // [tokens, S, hidden], or null
    float* sum_out;          // [tokens, hidden], or null
    const float* mix;        // [S from, S to]
    const float* out_w;      // [S]
    const float* scale;      // [hidden], or null
    const float* in_w;       // [S], with h
    const float* w;          // [hidden], with h
    float eps;
    int hidden;
};

__device__ __forceinline__ void hy_load(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void hy_load(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x; v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void hy_store(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void hy_store(__nv_bfloat16* p, const float (&v)[8]) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
}

// Rows of whole 8-entry words, VPT words per thread.
template <typename T, int S, int VPT>
__global__ void __launch_bounds__(VPT <= 2 ? 512 : 1024) hyper_words_kernel(T* __restrict__ h, const T* __restrict__ y, const HyperArgs a) {
    __shared__ float red[32];
    const size_t row = blockIdx.x;
    const int hidden = a.hidden, nvec = hidden / 8;
    float u[VPT][8];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 8;
#pragma unroll
        for (int i = 0; i < 8; ++i) u[k][i] = 0.f;
        if (c >= nvec * 8) continue;
        float x[S][8], yv[8];
#pragma unroll
        for (int s = 0; s < S; ++s) hy_load(a.x + row * a.x_row + s * a.x_stream + c, x[s]);
        if (y != nullptr) {
            hy_load(y + row * hidden + c, yv);
            if (a.scale != nullptr) {
                float sc[8];
                hy_load(a.scale + c, sc);
#pragma unroll
                for (int i = 0; i < 8; ++i) yv[i] *= sc[i];
            }
        }
#pragma unroll
        for (int t = 0; t < S; ++t) {
            float v[8];
            if (y != nullptr) {
                const float ow = a.out_w[t];
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] = a.mix[t] * x[0][i];
#pragma unroll
                for (int s = 1; s < S; ++s) {
                    const float m = a.mix[s * S + t];
#pragma unroll
                    for (int i = 0; i < 8; ++i) v[i] = fmaf(m, x[s][i], v[i]);
                }
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] = fmaf(ow, yv[i], v[i]);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] = x[t][i];
            }
            if (a.x_out != nullptr) hy_store(a.x_out + (row * S + t) * hidden + c, v);
            const float iw = h != nullptr ? a.in_w[t] : 1.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) u[k][i] = fmaf(iw, v[i], u[k][i]);
        }
        if (a.sum_out != nullptr) hy_store(a.sum_out + row * hidden + c, u[k]);
#pragma unroll
        for (int i = 0; i < 8; ++i) ss = fmaf(u[k][i], u[k][i], ss);
    }
    if (h == nullptr) return;
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)hidden + a.eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 8;
        if (c >= nvec * 8) continue;
        float w[8];
        hy_load(a.w + c, w);
#pragma unroll
        for (int i = 0; i < 8; ++i) w[i] = u[k][i] * inv * w[i];
        hy_store(h + row * hidden + c, w);
    }
}

// Any width and number of streams, entry by entry; u of the row stands in shared memory between the two passes.
template <typename T>
__global__ void __launch_bounds__(256) hyper_kernel(T* __restrict__ h, const T* __restrict__ y, const HyperArgs a, int S) {
    extern __shared__ float hy_u[];
    __shared__ float red[32];
    const size_t row = blockIdx.x;
    float ss = 0.f;
    for (int c = threadIdx.x; c < a.hidden; c += blockDim.x) {
        float x[HYPER_MAX_STREAMS];
#pragma unroll
        for (int s = 0; s < HYPER_MAX_STREAMS; ++s) x[s] = s < S ? a.x[row * a.x_row + s * a.x_stream + c] : 0.f;
        float yv = 0.f;
        if (y != nullptr) yv = Num<T>::to_f32(y[row * a.hidden + c]) * (a.scale != nullptr ? a.scale[c] : 1.f);
        float u = 0.f;
        for (int t = 0; t < S; ++t) {
            float v = 0.f;
            if (y != nullptr) {
#pragma unroll
                for (int s = 0; s < HYPER_MAX_STREAMS; ++s)
                    if (s < S) v = fmaf(a.mix[s * S + t], x[s], v);
                v = fmaf(a.out_w[t], yv, v);
            } else {
                v = a.x[row * a.x_row + t * a.x_stream + c];
            }
            if (a.x_out != nullptr) a.x_out[(row * S + t) * a.hidden + c] = v;
            u = fmaf(h != nullptr ? a.in_w[t] : 1.f, v, u);
        }
        if (a.sum_out != nullptr) a.sum_out[row * a.hidden + c] = u;
        if (h != nullptr) hy_u[c] = u;      // read again by this same thread
        ss = fmaf(u, u, ss);
    }
    if (h == nullptr) return;
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.hidden + a.eps);
    for (int c = threadIdx.x; c < a.hidden; c += blockDim.x) h[row * a.hidden + c] = Num<T>::from_f32(hy_u[c] * inv * a.w[c]);
}

template <typename T>
static int hyper_launch(T* h, const T* y, const HyperArgs& a, int S, int n, cudaStream_t stream) {
    const bool words = S <= 4 && a.hidden % 8 == 0 && a.hidden <= 32768 && a.x_row % 4 == 0 && a.x_stream % 4 == 0 && (uintptr_t)a.x % 16 == 0 &&
                       (uintptr_t)a.x_out % 16 == 0 && (uintptr_t)a.sum_out % 16 == 0 && (uintptr_t)a.scale % 16 == 0 && (uintptr_t)a.w % 16 == 0 &&
                       (uintptr_t)h % 16 == 0 && (uintptr_t)y % 16 == 0;
    if (words) {
        const int nvec = a.hidden / 8;
        const int vpt = nvec <= 512 ? 1 : (nvec <= 1024 ? 2 : 4);
        const int threads = ((nvec + vpt - 1) / vpt + 31) / 32 * 32;
#define OXR_HY(NS) \
    do { \
        if (vpt == 1) hyper_words_kernel<T, NS, 1><<<n, threads, 0, stream>>>(h, y, a); \
        else if (vpt == 2) hyper_words_kernel<T, NS, 2><<<n, threads, 0, stream>>>(h, y, a); \
        else hyper_words_kernel<T, NS, 4><<<n, threads, 0, stream>>>(h, y, a); \
    } while (0)
        if (S == 1) OXR_HY(1);
        else if (S == 2) OXR_HY(2);
        else if (S == 3) OXR_HY(3);
        else OXR_HY(4);
#undef OXR_HY
        return oxr_launch_status();
    }
    const size_t smem = h != nullptr ? (size_t)a.hidden * sizeof(float) : 0;
    if (smem > 200 * 1024) return OXR_BAD_ARGUMENT;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(hyper_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return 1000 + (int)e;
    }
    hyper_kernel<T><<<n, a.hidden >= 1024 ? 256 : 128, smem, stream>>>(h, y, a, S);
    return oxr_launch_status();
}

// h, y: [n, hidden] of `dtype`; h null: no norm (in_w, w unused); y null: the streams pass unchanged (mix, out_w unused).
OXR_API int oxr_hyper_mix(void* h, const void* y, const float* x, long long x_row, long long x_stream, float* x_out, float* sum_out, const float* mix,
                          const float* out_w, const float* scale, const float* in_w, const float* w, float eps, int n, int S, int hidden, int dtype,
                          cudaStream_t stream) {
    if (n <= 0) return 0;
    if (hidden <= 0 || S <= 0 || S > HYPER_MAX_STREAMS || x == nullptr || x_row < hidden || (x_stream != 0 && x_stream < hidden) ||
        (y != nullptr && (mix == nullptr || out_w == nullptr)) || (h != nullptr && (in_w == nullptr || w == nullptr)) ||
        (h != nullptr && sum_out != nullptr) || (x_out == x && (x_stream != hidden || x_row != (long long)S * hidden)))
        return OXR_BAD_ARGUMENT;
    HyperArgs a;
    a.x = x; a.x_row = x_row; a.x_stream = x_stream; a.x_out = x_out; a.sum_out = sum_out; a.mix = mix; a.out_w = out_w; a.scale = scale;
    a.in_w = in_w; a.w = w; a.eps = eps; a.hidden = hidden;
    if (dtype == 0) return hyper_launch<float>((float*)h, (const float*)y, a, S, n, stream);
    return hyper_launch<__nv_bfloat16>((__nv_bfloat16*)h, (const __nv_bfloat16*)y, a, S, n, stream);
}
