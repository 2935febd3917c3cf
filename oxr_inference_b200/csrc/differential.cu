// Differential attention between its projections, the softmax attention kernels and its output projection.
//
// A head has two score maps over the same values: query row [q1 | q2] and key row [k1 | k2] of 2 D entries, map m scoring q_m . k_m. Both maps
// run as ordinary attention heads over the SAME cached key row: the query heads 2h and 2h + 1 are [q1 | 0] and [0 | q2], so a key row is kept
// and read once, head 2h + m reads the key/value head of head h, and any attention kernel that takes rows of W >= 2 D entries serves.
//
//   diff_prep:    q[t, 2h + m] = the m-th half of (projection + bias), zeros elsewhere; key row = projection + bias; value row likewise; the
//                 rows of the pools are WK and WV entries wide (entries behind 2 D and DV stay as the pool was made: zero).
//   diff_combine: o = o1 - lambda o2 per head (o1, o2 the two heads' outputs, rows of W entries of which DV count), then
//                 o / sqrt(mean(o^2) + eps) * factor.
#include "common.cuh"

struct DiffArgs {
    int stride, q_col0, k_col0, v_col0;
    int H, G, D, DV, W, WV;      // W: width of a query head and of a key row; WV: width of a value row
    const float* bias;           // [2 H D | 2 G D | G DV] or null
    const int* slots;
    long long pool_slots;
    int* status;
};

template <typename T, int VEC> struct DiffWord;
template <typename T> struct DiffWord<T, 1> {
    float v[1];
    __device__ __forceinline__ void load(const T* p) { v[0] = Num<T>::to_f32(*p); }
    __device__ __forceinline__ void store(T* p) const { *p = Num<T>::from_f32(v[0]); }
};
template <> struct DiffWord<__nv_bfloat16, 8> {
    float v[8];
    __device__ __forceinline__ void load(const __nv_bfloat16* p) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x; v[2 * i + 1] = f.y;
        }
    }
    __device__ __forceinline__ void store(__nv_bfloat16* p) const {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
};

// grid (words of a token's output / 128, tokens)
template <typename T, int VEC>
__global__ void __launch_bounds__(128) diff_prep_kernel(T* __restrict__ q_out, T* __restrict__ k_pool, T* __restrict__ v_pool, const T* __restrict__ proj,
                                                        const DiffArgs a) {
    const int t = blockIdx.y;
    int i = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    const int q_cols = 2 * a.H * a.W, k_cols = 2 * a.G * a.D, v_cols = a.G * a.DV;
    if (i >= q_cols + k_cols + v_cols) return;
    const T* row = proj + (size_t)t * a.stride;
    DiffWord<T, VEC> w;
    const float* bias = nullptr;
    T* dst;
    if (i < q_cols) {
        const int head = i / a.W, d = i - head * a.W, m = head & 1;
        dst = q_out + (size_t)t * q_cols + i;
        if (d < m * a.D || d >= (m + 1) * a.D) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) w.v[k] = 0.f;
            w.store(dst);
            return;
        }
        const int c = (head >> 1) * 2 * a.D + d;
        w.load(row + a.q_col0 + c);
        if (a.bias != nullptr) bias = a.bias + c;
    } else {
        const int slot = a.slots[t];
        if (slot < 0) return;
        if (slot >= a.pool_slots) { oxr_report(a.status, OXR_BAD_SLOT, t); return; }
        i -= q_cols;
        if (i < k_cols) {
            const int g = i / (2 * a.D), d = i - g * 2 * a.D;
            dst = k_pool + ((long long)slot * a.G + g) * a.W + d;
            w.load(row + a.k_col0 + i);
            if (a.bias != nullptr) bias = a.bias + 2 * a.H * a.D + i;
        } else {
            i -= k_cols;
            const int g = i / a.DV, d = i - g * a.DV;
            dst = v_pool + ((long long)slot * a.G + g) * a.WV + d;
            w.load(row + a.v_col0 + i);
            if (a.bias != nullptr) bias = a.bias + 2 * (a.H + a.G) * a.D + i;
        }
    }
    if (bias != nullptr) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) w.v[k] += bias[k];
    }
    w.store(dst);
}

OXR_API int oxr_diff_prep(void* q_out, void* k_pool, void* v_pool, const void* proj, int n_tokens, int stride, int q_col0, int k_col0, int v_col0, int H,
                          int G, int D, int DV, int W, int WV, const float* bias, const int* slots, long long pool_slots, int dtype, int* status,
                          cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0 || DV <= 0 || W < 2 * D || WV < DV || n_tokens > 65535) return OXR_BAD_ARGUMENT;
    DiffArgs a;
    a.stride = stride; a.q_col0 = q_col0; a.k_col0 = k_col0; a.v_col0 = v_col0; a.H = H; a.G = G; a.D = D; a.DV = DV; a.W = W; a.WV = WV; a.bias = bias;
    a.slots = slots; a.pool_slots = pool_slots; a.status = status;
    const int cols = 2 * H * W + 2 * G * D + G * DV;
    const bool words = dtype == 1 && D % 8 == 0 && DV % 8 == 0 && W % 8 == 0 && WV % 8 == 0 && stride % 8 == 0 && q_col0 % 8 == 0 && k_col0 % 8 == 0 &&
                       v_col0 % 8 == 0 && (uintptr_t)proj % 16 == 0 && (uintptr_t)q_out % 16 == 0 && (uintptr_t)k_pool % 16 == 0 && (uintptr_t)v_pool % 16 == 0;
    if (words)
        diff_prep_kernel<__nv_bfloat16, 8><<<dim3((cols / 8 + 127) / 128, n_tokens), 128, 0, stream>>>((__nv_bfloat16*)q_out, (__nv_bfloat16*)k_pool,
                                                                                                      (__nv_bfloat16*)v_pool, (const __nv_bfloat16*)proj, a);
    else if (dtype == 0)
        diff_prep_kernel<float, 1><<<dim3((cols + 127) / 128, n_tokens), 128, 0, stream>>>((float*)q_out, (float*)k_pool, (float*)v_pool, (const float*)proj, a);
    else
        diff_prep_kernel<__nv_bfloat16, 1><<<dim3((cols + 127) / 128, n_tokens), 128, 0, stream>>>((__nv_bfloat16*)q_out, (__nv_bfloat16*)k_pool,
                                                                                                  (__nv_bfloat16*)v_pool, (const __nv_bfloat16*)proj, a);
    return oxr_launch_status();
}

// G lanes per (token, head), G a power of two: the head's entries stay in registers when they fit (KEEP words a lane), else they are read twice
template <typename T, int VEC, int G>
__global__ void __launch_bounds__(128) diff_combine_kernel(T* __restrict__ out, const T* __restrict__ o, int o_head, int H, int DV, const float* __restrict__ lambda,
                                                           float eps, float factor, int n_tokens) {
    const int l = threadIdx.x % G;
    const long long at = (long long)blockIdx.x * (128 / G) + threadIdx.x / G;
    const bool live = at < (long long)n_tokens * H;      // the others walk along: the sums are for whole warps
    const float lam = *lambda;
    const T* o1 = o + (live ? at : 0) * 2 * o_head;
    const T* o2 = o1 + o_head;
    constexpr int KEEP = 4;
    DiffWord<T, VEC> kept[KEEP];
    const int nw = DV / VEC;
    float sq = 0.f;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int w = l + G * k;
        if (w < nw) {
            DiffWord<T, VEC> b;
            kept[k].load(o1 + w * VEC);
            b.load(o2 + w * VEC);
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                kept[k].v[i] -= lam * b.v[i];
                sq = fmaf(kept[k].v[i], kept[k].v[i], sq);
            }
        }
    }
    for (int w = l + G * KEEP; w < nw; w += G) {
        DiffWord<T, VEC> a, b;
        a.load(o1 + w * VEC);
        b.load(o2 + w * VEC);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float v = a.v[i] - lam * b.v[i];
            sq = fmaf(v, v, sq);
        }
    }
#pragma unroll
    for (int s = G >> 1; s > 0; s >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, s);
    if (!live) return;
    const float inv = factor / sqrtf(sq / (float)DV + eps);
    T* dst = out + at * DV;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int w = l + G * k;
        if (w < nw) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) kept[k].v[i] *= inv;
            kept[k].store(dst + w * VEC);
        }
    }
    for (int w = l + G * KEEP; w < nw; w += G) {
        DiffWord<T, VEC> a, b;
        a.load(o1 + w * VEC);
        b.load(o2 + w * VEC);
#pragma unroll
        for (int i = 0; i < VEC; ++i) a.v[i] = (a.v[i] - lam * b.v[i]) * inv;
        a.store(dst + w * VEC);
    }
}

OXR_API int oxr_diff_combine(void* out, const void* o, int n_tokens, int o_head, int H, int DV, const float* lambda, float eps, float factor, int dtype,
                             cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (H <= 0 || DV <= 0 || o_head < DV) return OXR_BAD_ARGUMENT;
    const long long total = (long long)n_tokens * H;
#define OXR_COMBINE(T, VEC, G) \
    diff_combine_kernel<T, VEC, G><<<(unsigned)((total + 128 / G - 1) / (128 / G)), 128, 0, stream>>>((T*)out, (const T*)o, o_head, H, DV, lambda, eps, factor, n_tokens)
    if (dtype == 1 && DV % 8 == 0 && o_head % 8 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)o % 16 == 0) {
        // two words a lane where a head has that many
        if (DV <= 128) OXR_COMBINE(__nv_bfloat16, 8, 8);
        else if (DV <= 256) OXR_COMBINE(__nv_bfloat16, 8, 16);
        else OXR_COMBINE(__nv_bfloat16, 8, 32);
    } else if (dtype == 0) {
        OXR_COMBINE(float, 1, 32);
    } else {
        OXR_COMBINE(__nv_bfloat16, 1, 32);
    }
#undef OXR_COMBINE
    return oxr_launch_status();
}
