// The norm in front of a mixer whose input is blended with the previous token's (a token shift), on a residual stream that is kept whole in
// fp32, together with the add that the block before left to do:
//
//   s_t   = stream_t + y_t / rms(y_t) * w_post          (only with a pending y; s goes to a new buffer, see below)
//   h_t   = s_t / rms(s_t) * w
//   out_t = h_t + (h_(t-1) - h_t) * mu                   h_(t-1): the previous token of the same request, zeros before the first one
//
// The previous token of a request's first token in the step is in the request's state row (fp32 [hidden], zero for a new request), which
// the kernel moves on to the request's last token. All arithmetic fp32, one rounding to T.
//
// A block takes R neighbouring tokens of the packed step and keeps h of the last one in registers for the next; the token before its first
// one it computes again from `stream` and `y` (which is why s is written to a buffer of its own: the rows that other blocks read again stay
// as they were). The block that holds a request's FIRST token also owns its state row: it reads the row before it writes h of the request's
// last token there, computed again as well, so no other block touches it.
//
// VEC neighbouring entries per word (8 for bf16 rows of whole 16-byte words, else 1), VPT words per thread.
#include "common.cuh"

struct ShiftNormArgs {
    const float* stream;
    float* stream_out;       // with a pending y
    const float* w_post;
    float eps_post;
    const float* w;
    float eps;
    const float* mu;
    float* state;            // row of slot s: state + s * state_stride
    long long state_stride;
    const int* req_of_token;
    const int* cu_q;
    const int* state_slots;
    int n_tokens;
    int hidden;
};

template <int VEC> __device__ __forceinline__ void sn_load_f32(const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 8) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = p[i];
    }
}
template <int VEC> __device__ __forceinline__ void sn_store_f32(float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 8) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) p[i] = v[i];
    }
}
template <typename T, int VEC> __device__ __forceinline__ void sn_load(const T* p, float (&v)[VEC]) {
    if constexpr (VEC == 8 && sizeof(T) == 2) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = Num<T>::to_f32(p[i]);
    }
}
template <typename T, int VEC> __device__ __forceinline__ void sn_store(T* p, const float (&v)[VEC]) {
    if constexpr (VEC == 8 && sizeof(T) == 2) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) p[i] = Num<T>::from_f32(v[i]);
    }
}

template <typename T, int VEC, int VPT>
__global__ void __launch_bounds__(VEC == 8 && VPT <= 2 ? 512 : 1024) shift_norm_kernel(T* __restrict__ out, const T* __restrict__ y, const ShiftNormArgs a, int rows_per_block) {
    __shared__ float red[32];
    const int hidden = a.hidden, nvec = hidden / VEC;
    float prev[VPT][VEC], h[VPT][VEC];

    // h of token t; the block's own tokens (`write`) also leave the new stream row
    auto normed = [&](int t, float (&v)[VPT][VEC], bool write) {
        const size_t at = (size_t)t * hidden;
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int idx = threadIdx.x + k * blockDim.x;
            if (idx < nvec) sn_load_f32<VEC>(a.stream + at + VEC * idx, v[k]);
            else {
#pragma unroll
                for (int i = 0; i < VEC; ++i) v[k][i] = 0.f;
            }
        }
        if (y != nullptr) {
            float yv[VPT][VEC];
            float ss = 0.f;
#pragma unroll
            for (int k = 0; k < VPT; ++k) {
                const int idx = threadIdx.x + k * blockDim.x;
                if (idx < nvec) {
                    sn_load<T, VEC>(y + at + VEC * idx, yv[k]);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) ss = fmaf(yv[k][i], yv[k][i], ss);
                }
            }
            ss = block_sum(ss, red);
            const float inv = 1.f / sqrtf(ss / (float)hidden + a.eps_post);
#pragma unroll
            for (int k = 0; k < VPT; ++k) {
                const int idx = threadIdx.x + k * blockDim.x;
                if (idx < nvec) {
                    float w[VEC];
                    sn_load_f32<VEC>(a.w_post + VEC * idx, w);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) v[k][i] += yv[k][i] * inv * w[i];
                    if (write) sn_store_f32<VEC>(a.stream_out + at + VEC * idx, v[k]);
                }
            }
        }
        float s2 = 0.f;
#pragma unroll
        for (int k = 0; k < VPT; ++k)
#pragma unroll
            for (int i = 0; i < VEC; ++i) s2 = fmaf(v[k][i], v[k][i], s2);
        s2 = block_sum(s2, red);
        const float inv = 1.f / sqrtf(s2 / (float)hidden + a.eps);
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int idx = threadIdx.x + k * blockDim.x;
            if (idx < nvec) {
                float w[VEC];
                sn_load_f32<VEC>(a.w + VEC * idx, w);
#pragma unroll
                for (int i = 0; i < VEC; ++i) v[k][i] = v[k][i] * inv * w[i];
            }
        }
    };

    const int t0 = blockIdx.x * rows_per_block, t_end = min(t0 + rows_per_block, a.n_tokens);
    if (t0 > a.cu_q[a.req_of_token[t0]]) normed(t0 - 1, prev, false);
    for (int t = t0; t < t_end; ++t) {
        const int r = a.req_of_token[t], first = a.cu_q[r], end = a.cu_q[r + 1];
        float* state = a.state + (long long)a.state_slots[r] * a.state_stride;
        if (t == first) {
#pragma unroll
            for (int k = 0; k < VPT; ++k) {
                const int idx = threadIdx.x + k * blockDim.x;
                if (idx < nvec) sn_load_f32<VEC>(state + VEC * idx, prev[k]);
            }
        }
        normed(t, h, true);
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
            const int idx = threadIdx.x + k * blockDim.x;
            if (idx < nvec) {
                float mu[VEC], o[VEC];
                sn_load_f32<VEC>(a.mu + VEC * idx, mu);
#pragma unroll
                for (int i = 0; i < VEC; ++i) o[i] = h[k][i] + (prev[k][i] - h[k][i]) * mu[i];
                sn_store<T, VEC>(out + (size_t)t * hidden + VEC * idx, o);
            }
        }
        if (t == first) {
            if (end - first > 1) normed(end - 1, prev, false);
            else {
#pragma unroll
                for (int k = 0; k < VPT; ++k)
#pragma unroll
                    for (int i = 0; i < VEC; ++i) prev[k][i] = h[k][i];
            }
#pragma unroll
            for (int k = 0; k < VPT; ++k) {
                const int idx = threadIdx.x + k * blockDim.x;
                if (idx < nvec) sn_store_f32<VEC>(state + VEC * idx, prev[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < VPT; ++k)
#pragma unroll
            for (int i = 0; i < VEC; ++i) prev[k][i] = h[k][i];
    }
}

OXR_API int oxr_shift_norm(void* out, const float* stream, const void* y, float* stream_out, const float* w_post, float eps_post, const float* w,
                           float eps, const float* mu, float* state, long long state_stride, const int* req_of_token, const int* cu_q,
                           const int* state_slots, int n_tokens, int hidden, int rows_per_block, int dtype, cudaStream_t stream_) {
    if (n_tokens <= 0) return 0;
    if (hidden <= 0 || rows_per_block <= 0 || state == nullptr || (y != nullptr && (stream_out == nullptr || stream_out == stream || w_post == nullptr)))
        return OXR_BAD_ARGUMENT;
    ShiftNormArgs a;
    a.stream = stream; a.stream_out = stream_out; a.w_post = w_post; a.eps_post = eps_post; a.w = w; a.eps = eps; a.mu = mu; a.state = state;
    a.state_stride = state_stride; a.req_of_token = req_of_token; a.cu_q = cu_q; a.state_slots = state_slots; a.n_tokens = n_tokens; a.hidden = hidden;
    const int blocks = (n_tokens + rows_per_block - 1) / rows_per_block;
    const bool words = dtype == 1 && hidden % 8 == 0 && hidden <= 32768 && (uintptr_t)stream % 16 == 0 && (uintptr_t)stream_out % 16 == 0 &&
                       (uintptr_t)y % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)w_post % 16 == 0 && (uintptr_t)w % 16 == 0 &&
                       (uintptr_t)mu % 16 == 0 && (uintptr_t)state % 16 == 0 && state_stride % 4 == 0;
#define OXR_SN(T, VEC, VPT) \
    shift_norm_kernel<T, VEC, VPT><<<blocks, ((hidden / VEC + VPT - 1) / VPT + 31) / 32 * 32, 0, stream_>>>((T*)out, (const T*)y, a, rows_per_block)
    if (words) {
        const int nvec = hidden / 8;
        if (nvec <= 512) OXR_SN(__nv_bfloat16, 8, 1);
        else if (nvec <= 1024) OXR_SN(__nv_bfloat16, 8, 2);
        else OXR_SN(__nv_bfloat16, 8, 4);
        return oxr_launch_status();
    }
#define OXR_SN_T(T) \
    do { \
        if (hidden <= 1024) OXR_SN(T, 1, 1); \
        else if (hidden <= 4096) OXR_SN(T, 1, 4); \
        else if (hidden <= 16384) OXR_SN(T, 1, 16); \
        else return OXR_BAD_ARGUMENT; \
    } while (0)
    if (dtype == 0) OXR_SN_T(float);
    else OXR_SN_T(__nv_bfloat16);
#undef OXR_SN_T
#undef OXR_SN
    return oxr_launch_status();
}
