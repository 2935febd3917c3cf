// A delta-rule recurrence with a decay per key channel, between its in- and out-projections.
//
// Per request and head the state is a matrix S [DK, DV] (zero for a new request). Per token, with u the key over its length and decay w
// and removal rate a per key channel,
//
//   u_t = k_t / sqrt(sum k_t^2 + len_eps)      w_t = exp(-rate * sigmoid(zw_t + w0))      a_t = sigmoid(za_t + ab)
//   S_t = diag(w_t) S_(t-1) - (a_t * u_t) (u_t^T S_(t-1)) + k_t v_t^T          o_t = S_t^T r_t
//
// k, v, r are columns of the projections (type T); zw and za are fp32; everything behind them is fp32. Written over the old state alone,
//
//   d1 = S^T u        d2 = S^T (w * r)        o = d2 - ((a * u) . r) d1 + (k . r) v        S <- w S - (a * u) d1 + k v
//
// so a token has ONE sum over the key channels to wait for (both dot products of a column together), and o does not wait for the update.
//
// Columns of S (one value entry each) are independent: a block takes COLS of them of one head of one request. A warp takes 32 / J columns
// times CPT; J neighbouring lanes share a column: lane j holds the key entries 4 (j + J i) .. + 3 for i < 4 (16 entries of CPT columns in
// registers), so that the J lanes' shared-memory words are neighbours and their sum is a butterfly of log2 J steps. In memory the state lies
// column by column ([DV, DK] per head): those words are neighbours there, too. J = ceil(DK / 16) rounded up to a power of two; entries from
// DK on are zero. Tokens go through shared memory a tile of TT at a time, one warp preparing one token (unit key, decay, rate, and the two
// scalar products), with the next tile's loads in flight in registers while this one is computed.
//
// Token by token in the order of the sequence whatever the cut, so a position's result does not depend on how a prompt was cut into steps.
#include "common.cuh"

struct DeltaArgs {
    int stride, r_col0, k_col0, v_col0;       // projections
    const float* zw; int zw_stride;           // [tokens, heads DK]
    const float* w0;
    const float* za; int za_stride;
    const float* ab;
    float rate, len_eps;
    int heads, DK, DV;
    float* state;
    long long slot_stride;
    const int* cu_q;
    const int* state_slots;
};

constexpr int DELTA_NW = 8, DELTA_TT = 8;     // warps per block; tokens per tile (one per warp)

__device__ __forceinline__ float delta_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

template <typename T, int J, int CPT>
__global__ void __launch_bounds__(32 * DELTA_NW) delta_scan_kernel(float* __restrict__ y, const T* __restrict__ proj, const DeltaArgs a) {
    constexpr int DKP = 16 * J, CPW = 32 / J, COLS = DELTA_NW * CPW * CPT;   // key entries with padding; column groups per warp; columns per block
    constexpr int KL = (DKP + 31) / 32;                                       // key entries per lane when a warp prepares a token
    constexpr int VL = (COLS + 31) / 32;                                      // value entries per lane likewise
    extern __shared__ __align__(16) float dsm[];
    float* us = dsm;                              // [TT][DKP]: unit key, w * r, w, k, a * u
    float* wrs = us + DELTA_TT * DKP;
    float* ws = wrs + DELTA_TT * DKP;
    float* ks = ws + DELTA_TT * DKP;
    float* aus = ks + DELTA_TT * DKP;
    float* vs = aus + DELTA_TT * DKP;             // [TT][COLS]
    float* os = vs + DELTA_TT * COLS;             // [TT][COLS]
    float* sc = os + DELTA_TT * COLS;             // [TT][2]: (a u) . r and k . r
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, j = lane % J, grp = lane / J;
    const int p0 = blockIdx.x * COLS, h = blockIdx.y, r = blockIdx.z;
    const int t0 = a.cu_q[r], t1 = a.cu_q[r + 1];
    if (t1 <= t0) return;
    const int DK = a.DK, DV = a.DV;
    float* S = a.state + (long long)a.state_slots[r] * a.slot_stride + (long long)h * DK * DV;
    const bool words = DK % 4 == 0 && (((uintptr_t)S) & 15) == 0;

    float s[CPT][16];
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int p = p0 + (warp * CPT + c) * CPW + grp;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = 4 * (j + J * i);
            if (words) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (p < DV && e < DK) v = *reinterpret_cast<const float4*>(S + (size_t)p * DK + e);
                s[c][4 * i] = v.x; s[c][4 * i + 1] = v.y; s[c][4 * i + 2] = v.z; s[c][4 * i + 3] = v.w;
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q) s[c][4 * i + q] = (p < DV && e + q < DK) ? S[(size_t)p * DK + e + q] : 0.f;
            }
        }
    }

    // the loads of one token (this warp's of the tile): raw values in registers
    float kr[KL], rr[KL], zwr[KL], zar[KL], vr[VL];
    auto fetch = [&](int tile) {
        const int t = tile + warp;
        const bool live = t < t1;
        const T* row = proj + (size_t)(live ? t : t0) * a.stride;
#pragma unroll
        for (int i = 0; i < KL; ++i) {
            const int e = lane + 32 * i;
            const bool ok = live && e < DK;
            kr[i] = ok ? Num<T>::to_f32(row[a.k_col0 + h * DK + e]) : 0.f;
            rr[i] = ok ? Num<T>::to_f32(row[a.r_col0 + h * DK + e]) : 0.f;
            zwr[i] = ok ? a.zw[(size_t)t * a.zw_stride + h * DK + e] + a.w0[h * DK + e] : 0.f;
            zar[i] = ok ? a.za[(size_t)t * a.za_stride + h * DK + e] + a.ab[h * DK + e] : 0.f;
        }
#pragma unroll
        for (int i = 0; i < VL; ++i) {
            const int c = lane + 32 * i;
            vr[i] = (live && c < COLS && p0 + c < DV) ? Num<T>::to_f32(row[a.v_col0 + h * DV + p0 + c]) : 0.f;
        }
    };
    auto prepare = [&]() {
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < KL; ++i) sq = fmaf(kr[i], kr[i], sq);
        const float inv = 1.f / sqrtf(warp_sum(sq) + a.len_eps);
        float aur = 0.f, kdr = 0.f;
#pragma unroll
        for (int i = 0; i < KL; ++i) {
            const int e = lane + 32 * i;
            const float u = kr[i] * inv, w = expf(-a.rate * delta_sigmoid(zwr[i])), au = delta_sigmoid(zar[i]) * u;
            aur = fmaf(au, rr[i], aur);
            kdr = fmaf(kr[i], rr[i], kdr);
            if (e < DKP) {
                us[warp * DKP + e] = u;
                wrs[warp * DKP + e] = w * rr[i];
                ws[warp * DKP + e] = w;
                ks[warp * DKP + e] = kr[i];
                aus[warp * DKP + e] = au;
            }
        }
        aur = warp_sum(aur);
        kdr = warp_sum(kdr);
        if (lane == 0) { sc[2 * warp] = aur; sc[2 * warp + 1] = kdr; }
#pragma unroll
        for (int i = 0; i < VL; ++i) {
            const int c = lane + 32 * i;
            if (c < COLS) vs[warp * COLS + c] = vr[i];
        }
    };

    fetch(t0);
    prepare();
    __syncthreads();
    for (int tile = t0; tile < t1; tile += DELTA_TT) {
        const int nt = min(DELTA_TT, t1 - tile);
        const bool more = tile + DELTA_TT < t1;
        if (more) fetch(tile + DELTA_TT);
        for (int t = 0; t < nt; ++t) {
            const float4* u4 = reinterpret_cast<const float4*>(us + t * DKP) + j;
            const float4* wr4 = reinterpret_cast<const float4*>(wrs + t * DKP) + j;
            float d1[CPT][2], d2[CPT][2];      // two chains each, added in a fixed order
#pragma unroll
            for (int c = 0; c < CPT; ++c) d1[c][0] = d1[c][1] = d2[c][0] = d2[c][1] = 0.f;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float4 uu = u4[J * i], wr = wr4[J * i];
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    d1[c][0] = fmaf(s[c][4 * i], uu.x, d1[c][0]);
                    d1[c][1] = fmaf(s[c][4 * i + 1], uu.y, d1[c][1]);
                    d2[c][0] = fmaf(s[c][4 * i], wr.x, d2[c][0]);
                    d2[c][1] = fmaf(s[c][4 * i + 1], wr.y, d2[c][1]);
                    d1[c][0] = fmaf(s[c][4 * i + 2], uu.z, d1[c][0]);
                    d1[c][1] = fmaf(s[c][4 * i + 3], uu.w, d1[c][1]);
                    d2[c][0] = fmaf(s[c][4 * i + 2], wr.z, d2[c][0]);
                    d2[c][1] = fmaf(s[c][4 * i + 3], wr.w, d2[c][1]);
                }
            }
            float a1[CPT], a2[CPT], v[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                a1[c] = d1[c][0] + d1[c][1];
                a2[c] = d2[c][0] + d2[c][1];
                v[c] = vs[t * COLS + (warp * CPT + c) * CPW + grp];
            }
#pragma unroll
            for (int o = J >> 1; o > 0; o >>= 1)
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    a1[c] += __shfl_xor_sync(0xffffffffu, a1[c], o);
                    a2[c] += __shfl_xor_sync(0xffffffffu, a2[c], o);
                }
            const float4* w4 = reinterpret_cast<const float4*>(ws + t * DKP) + j;
            const float4* k4 = reinterpret_cast<const float4*>(ks + t * DKP) + j;
            const float4* au4 = reinterpret_cast<const float4*>(aus + t * DKP) + j;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float4 w = w4[J * i], k = k4[J * i], au = au4[J * i];
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    s[c][4 * i] = fmaf(w.x, s[c][4 * i], fmaf(k.x, v[c], -au.x * a1[c]));
                    s[c][4 * i + 1] = fmaf(w.y, s[c][4 * i + 1], fmaf(k.y, v[c], -au.y * a1[c]));
                    s[c][4 * i + 2] = fmaf(w.z, s[c][4 * i + 2], fmaf(k.z, v[c], -au.z * a1[c]));
                    s[c][4 * i + 3] = fmaf(w.w, s[c][4 * i + 3], fmaf(k.w, v[c], -au.w * a1[c]));
                }
            }
            if (j == 0) {
                const float aur = sc[2 * t], kdr = sc[2 * t + 1];
#pragma unroll
                for (int c = 0; c < CPT; ++c) os[t * COLS + (warp * CPT + c) * CPW + grp] = a2[c] - aur * a1[c] + kdr * v[c];
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nt * COLS; i += 32 * DELTA_NW) {
            const int t = i / COLS, c = i - t * COLS;
            if (p0 + c < DV) y[(size_t)(tile + t) * a.heads * DV + h * DV + p0 + c] = os[i];
        }
        if (more) {
            prepare();        // the tile's vectors have been read by every warp (the barrier above)
            __syncthreads();
        }
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const int p = p0 + (warp * CPT + c) * CPW + grp;
        if (p >= DV) continue;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = 4 * (j + J * i);
            if (words) {
                if (e < DK) *reinterpret_cast<float4*>(S + (size_t)p * DK + e) = make_float4(s[c][4 * i], s[c][4 * i + 1], s[c][4 * i + 2], s[c][4 * i + 3]);
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (e + q < DK) S[(size_t)p * DK + e + q] = s[c][4 * i + q];
            }
        }
    }
}

template <typename T, int J, int CPT>
static int delta_launch(float* y, const T* proj, const DeltaArgs& a, int n_requests, cudaStream_t stream) {
    constexpr int DKP = 16 * J, COLS = DELTA_NW * (32 / J) * CPT;
    constexpr size_t smem = (size_t)DELTA_TT * (5 * DKP + 2 * COLS + 2) * sizeof(float);
    if constexpr (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<T, J, CPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return 1000 + (int)e;
    }
    dim3 grid((a.DV + COLS - 1) / COLS, a.heads, n_requests);
    delta_scan_kernel<T, J, CPT><<<grid, 32 * DELTA_NW, smem, stream>>>(y, proj, a);
    return oxr_launch_status();
}

template <typename T>
static int delta_launch_j(float* y, const T* proj, const DeltaArgs& a, int n_requests, int cpt, cudaStream_t stream) {
    const int j = (a.DK + 15) / 16;
#define OXR_DELTA(J) return cpt == 2 ? delta_launch<T, J, 2>(y, proj, a, n_requests, stream) : delta_launch<T, J, 1>(y, proj, a, n_requests, stream)
    if (j <= 1) OXR_DELTA(1);
    if (j <= 2) OXR_DELTA(2);
    if (j <= 4) OXR_DELTA(4);
    if (j <= 8) OXR_DELTA(8);
    OXR_DELTA(16);
#undef OXR_DELTA
}

OXR_API int oxr_delta_scan(float* y, const void* proj, int n_requests, int stride, int r_col0, int k_col0, int v_col0, const float* zw, int zw_stride,
                           const float* w0, const float* za, int za_stride, const float* ab, float rate, float len_eps, int heads, int DK, int DV,
                           float* state, long long slot_stride, const int* cu_q, const int* state_slots, int dtype, int columns_per_thread,
                           cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (heads <= 0 || DK <= 0 || DK > 256 || DV <= 0 || heads > 65535 || n_requests > 65535 || !(rate > 0.f) || !(len_eps > 0.f)) return OXR_BAD_ARGUMENT;
    DeltaArgs a;
    a.stride = stride; a.r_col0 = r_col0; a.k_col0 = k_col0; a.v_col0 = v_col0; a.zw = zw; a.zw_stride = zw_stride; a.w0 = w0; a.za = za;
    a.za_stride = za_stride; a.ab = ab; a.rate = rate; a.len_eps = len_eps; a.heads = heads; a.DK = DK; a.DV = DV; a.state = state;
    a.slot_stride = slot_stride; a.cu_q = cu_q; a.state_slots = state_slots;
    if (dtype == 0) return delta_launch_j<float>(y, (const float*)proj, a, n_requests, columns_per_thread, stream);
    return delta_launch_j<__nv_bfloat16>(y, (const __nv_bfloat16*)proj, a, n_requests, columns_per_thread, stream);
}

// out[t, c] = tanh(z[t, col0 + c]), evaluated in fp32 and rounded once: the activation inside a low-rank map whose first half left fp32.
template <typename T>
__global__ void tanh_cols_kernel(T* __restrict__ out, const float* __restrict__ z, int stride, int col0, int width, size_t total) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t t = i / width;
    out[i] = Num<T>::from_f32(tanhf(z[t * stride + col0 + (int)(i - t * width)]));
}

OXR_API int oxr_tanh_cols(void* out, const float* z, int n, int stride, int col0, int width, int dtype, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (width <= 0 || col0 < 0 || col0 + width > stride) return OXR_BAD_ARGUMENT;
    const size_t total = (size_t)n * width;
    const unsigned blocks = (unsigned)((total + 127) / 128);
    if (dtype == 0) tanh_cols_kernel<float><<<blocks, 128, 0, stream>>>((float*)out, z, stride, col0, width, total);
    else tanh_cols_kernel<__nv_bfloat16><<<blocks, 128, 0, stream>>>((__nv_bfloat16*)out, z, stride, col0, width, total);
    return oxr_launch_status();
}
