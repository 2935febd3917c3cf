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
// Columns of S (one value entry each) are independent: a block takes 32 of them of one head of one request, 8 per computing warp. J lanes share
// a group of CPT = J / 4 columns: lane j holds the key entries 4 (j + J i) .. + 3, i < KW, of each (J = DK / 4 rounded up to a power of two, 4 to
// 32; KW = 2 for keys of more than 128 entries), as pairs for the packed fp32 multiply-add; entries from DK on are zero. So every vector read
// from shared memory is read once per group, and the 2 CPT dot products of a token meet in a butterfly that halves their number with every
// step: lane j ends with number j / 2 of them, and a column's d1 goes back to the group by one shuffle. In memory the state lies column by
// column ([DV, DK] per head), which makes a column's lanes neighbours there, too.
// A warp per token of a tile prepares it (unit key, decay, rate, the two scalar products), a tile of TT tokens ahead of the computing warps in a
// second buffer, from raw values that cp.async brings in two more tiles ahead, and writes the finished tile's results out. A step of single tokens runs a
// kernel of its own (below).
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
    int async;                                // every row piece is whole 16-byte words: copied ahead by cp.async
};

constexpr int DELTA_TT = 8, DELTA_COLS = 32, DELTA_WARPS = 4, DELTA_PREP_WARPS = DELTA_TT,      // tokens per tile; columns per block; computing warps; preparing warps, one per token
              DELTA_STAGES = 4;                                                           // tiles of raw values on their way or waiting

__device__ __forceinline__ float delta_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

typedef unsigned long long f32x2;      // two floats, the lower half first
__device__ __forceinline__ f32x2 pack2(float lo, float hi) { f32x2 d; asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi)); return d; }
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) { f32x2 d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) { f32x2 d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }

template <int J, int KW> struct DeltaShape {
    static constexpr int DKP = 4 * J * KW, CPT = J / 4, NV = 2 * CPT;
    static constexpr int VEC = DELTA_TT * DKP;                                            // one vector of every token of a tile
    static constexpr int TILE = 5 * VEC + DELTA_TT * DELTA_COLS + 2 * DELTA_TT;           // floats of a tile's buffer
    template <typename T> static constexpr int TOKEN = (2 * DKP + DELTA_COLS) * (int)sizeof(T) + 8 * DKP;      // bytes of a token's raw values
    template <typename T> static constexpr size_t SMEM =
        (size_t)(2 * TILE + 2 * DELTA_TT * DELTA_COLS) * sizeof(float) + (size_t)DELTA_STAGES * DELTA_TT * TOKEN<T>;
    static_assert(DELTA_WARPS * (32 / J) * CPT == DELTA_COLS, "the warps hold the block's columns");
};

// The sums of v[0 .. N - 1] over a group of 2 N neighbouring lanes, number j / 2 of them for lane j of the group: every step sends half of the
// numbers that are left to the lane N, N / 2, ... away and keeps the other half; the last step adds the two lanes of a pair.
template <int N> __device__ __forceinline__ float delta_reduce(float (&v)[N], int lane) {
    if constexpr (N == 1) return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
    else {
        float half[N / 2];
        const bool up = (lane & N) != 0;       // this lane keeps the upper half of the numbers
#pragma unroll
        for (int i = 0; i < N / 2; ++i) {
            const float send = up ? v[i] : v[N / 2 + i], keep = up ? v[N / 2 + i] : v[i];
            half[i] = keep + __shfl_xor_sync(0xffffffffu, send, N);
        }
        return delta_reduce<N / 2>(half, lane);
    }
}

// N neighbouring floats from an address that is a multiple of N
template <int N> __device__ __forceinline__ void delta_columns(const float* p, float (&v)[N]) {
    if constexpr (N >= 4) {
#pragma unroll
        for (int i = 0; i < N / 4; ++i) {
            const float4 x = reinterpret_cast<const float4*>(p)[i];
            v[4 * i] = x.x; v[4 * i + 1] = x.y; v[4 * i + 2] = x.z; v[4 * i + 3] = x.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = p[i];
    }
}

template <typename T, int J, int KW>
__global__ void __launch_bounds__(32 * (DELTA_WARPS + DELTA_PREP_WARPS), 1) delta_scan_kernel(float* __restrict__ y, const T* __restrict__ proj, const DeltaArgs a) {
    using Sh = DeltaShape<J, KW>;
    constexpr int DKP = Sh::DKP, CPT = Sh::CPT, KL = (DKP + 31) / 32;      // KL: key entries per lane when a warp prepares a token
    extern __shared__ __align__(16) float dsm[];      // [2][TILE], then the results [2][TT][COLS]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int p0 = blockIdx.x * DELTA_COLS, h = blockIdx.y, r = blockIdx.z;
    const int t0 = a.cu_q[r], t1 = a.cu_q[r + 1];
    if (t1 <= t0) return;
    const int DK = a.DK, DV = a.DV, n_tiles = (t1 - t0 + DELTA_TT - 1) / DELTA_TT;
    float* results = dsm + 2 * Sh::TILE;

    if (warp >= DELTA_WARPS) {
        // ---- preparing warps: token `slot` of every tile
        const int slot = warp - DELTA_WARPS;
        float w0[KL], ab[KL];
#pragma unroll
        for (int i = 0; i < KL; ++i) {
            const int e = lane + 32 * i;
            w0[i] = e < DK ? a.w0[h * DK + e] : 0.f;
            ab[i] = e < DK ? a.ab[h * DK + e] : 0.f;
        }
        // a token's raw values in a stage: k | r | v (32 columns) | decay logits | rate logits; every warp copies and reads its own tokens only.
        // Copy m of this lane: 16 bytes from `from[m]` + t * `pace[m]` bytes to `to[m]` within the token's stage.
        constexpr int KB = DKP * (int)sizeof(T), VB = DELTA_COLS * (int)sizeof(T), ZB = DKP * 4, NM = (Sh::template TOKEN<T> / 16 + 31) / 32;
        char* stages = reinterpret_cast<char*>(results + 2 * DELTA_TT * DELTA_COLS) + slot * Sh::template TOKEN<T>;
        const char* from[NM];
        int pace[NM], to[NM];
        if (a.async) {
            const int nk = DK * (int)sizeof(T) / 16, nv = min(VB, (DV - p0) * (int)sizeof(T)) / 16, nz = DK / 4;
            const char* row = reinterpret_cast<const char*>(proj);
#pragma unroll
            for (int m = 0; m < NM; ++m) {
                int i = lane + 32 * m;
                pace[m] = a.stride * (int)sizeof(T);
                if (i < nk) { from[m] = row + (a.k_col0 + h * DK) * (int)sizeof(T) + 16 * i; to[m] = 16 * i; }
                else if ((i -= nk) < nk) { from[m] = row + (a.r_col0 + h * DK) * (int)sizeof(T) + 16 * i; to[m] = KB + 16 * i; }
                else if ((i -= nk) < nv) { from[m] = row + (a.v_col0 + h * DV + p0) * (int)sizeof(T) + 16 * i; to[m] = 2 * KB + 16 * i; }
                else if ((i -= nv) < nz) { from[m] = reinterpret_cast<const char*>(a.zw + h * DK) + 16 * i; to[m] = 2 * KB + VB + 16 * i; pace[m] = a.zw_stride * 4; }
                else if ((i -= nz) < nz) { from[m] = reinterpret_cast<const char*>(a.za + h * DK) + 16 * i; to[m] = 2 * KB + VB + ZB + 16 * i; pace[m] = a.za_stride * 4; }
                else to[m] = -1;
            }
        }
        auto fetch = [&](int tile) {
            __syncwarp();      // the stage's last values have been read by every lane
            const int t = t0 + tile * DELTA_TT + slot;
            if (a.async && t < t1) {
                const uint32_t dst = (uint32_t)__cvta_generic_to_shared(stages + (size_t)(tile % DELTA_STAGES) * DELTA_TT * Sh::template TOKEN<T>);
#pragma unroll
                for (int m = 0; m < NM; ++m)
                    if (to[m] >= 0)
                        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + to[m]), "l"(from[m] + (size_t)t * pace[m]) : "memory");
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        auto prepare = [&](int tile) {
            asm volatile("cp.async.wait_group %0;" ::"n"(DELTA_STAGES - 2) : "memory");      // this tile's copies have arrived
            __syncwarp();
            const int t = t0 + tile * DELTA_TT + slot;
            if (t >= t1) return;
            float* buf = dsm + (tile & 1) * Sh::TILE;
            float k[KL], rd[KL], w[KL], au[KL], v;
            float sq = 0.f, kdr = 0.f, akr = 0.f;
            if (a.async) {
                const char* src = stages + (size_t)(tile % DELTA_STAGES) * DELTA_TT * Sh::template TOKEN<T>;
#pragma unroll
                for (int i = 0; i < KL; ++i) {
                    const int e = lane + 32 * i;
                    const bool ok = e < DK;
                    k[i] = ok ? Num<T>::to_f32(reinterpret_cast<const T*>(src)[e]) : 0.f;
                    rd[i] = ok ? Num<T>::to_f32(reinterpret_cast<const T*>(src + KB)[e]) : 0.f;
                    w[i] = ok ? reinterpret_cast<const float*>(src + 2 * KB + VB)[e] : 0.f;
                    au[i] = ok ? reinterpret_cast<const float*>(src + 2 * KB + VB + ZB)[e] : 0.f;
                }
                v = p0 + lane < DV ? Num<T>::to_f32(reinterpret_cast<const T*>(src + 2 * KB)[lane]) : 0.f;
            } else {       // sizes whose rows are not whole 16-byte words
                const T* row = proj + (size_t)t * a.stride;
#pragma unroll
                for (int i = 0; i < KL; ++i) {
                    const int e = lane + 32 * i;
                    const bool ok = e < DK;
                    k[i] = ok ? Num<T>::to_f32(row[a.k_col0 + h * DK + e]) : 0.f;
                    rd[i] = ok ? Num<T>::to_f32(row[a.r_col0 + h * DK + e]) : 0.f;
                    w[i] = ok ? a.zw[(size_t)t * a.zw_stride + h * DK + e] : 0.f;
                    au[i] = ok ? a.za[(size_t)t * a.za_stride + h * DK + e] : 0.f;
                }
                v = p0 + lane < DV ? Num<T>::to_f32(row[a.v_col0 + h * DV + p0 + lane]) : 0.f;
            }
#pragma unroll
            for (int i = 0; i < KL; ++i) {
                w[i] = expf(-a.rate * delta_sigmoid(w[i] + w0[i]));
                au[i] = delta_sigmoid(au[i] + ab[i]) * k[i];
                sq = fmaf(k[i], k[i], sq);
                kdr = fmaf(k[i], rd[i], kdr);
                akr = fmaf(au[i], rd[i], akr);
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {      // the three sums side by side
                sq += __shfl_xor_sync(0xffffffffu, sq, o);
                kdr += __shfl_xor_sync(0xffffffffu, kdr, o);
                akr += __shfl_xor_sync(0xffffffffu, akr, o);
            }
            const float inv = 1.f / sqrtf(sq + a.len_eps);
#pragma unroll
            for (int i = 0; i < KL; ++i) {
                const int e = lane + 32 * i;
                if (e < DKP) {
                    float* at = buf + slot * DKP + e;
                    at[0] = k[i] * inv;
                    at[Sh::VEC] = w[i] * rd[i];
                    at[2 * Sh::VEC] = w[i];
                    at[3 * Sh::VEC] = k[i];
                    at[4 * Sh::VEC] = -au[i] * inv;
                }
            }
            float* tail = buf + 5 * Sh::VEC;
            tail[slot * DELTA_COLS + lane] = v;
            if (lane == 0) {
                tail[DELTA_TT * DELTA_COLS + 2 * slot] = akr * inv;
                tail[DELTA_TT * DELTA_COLS + 2 * slot + 1] = kdr;
            }
        };
        auto write_out = [&](int tile) {
            const int t = t0 + tile * DELTA_TT + slot;
            if (t < t1 && p0 + lane < DV) y[(size_t)t * a.heads * DV + h * DV + p0 + lane] = results[((tile & 1) * DELTA_TT + slot) * DELTA_COLS + lane];
        };
#pragma unroll
        for (int tile = 0; tile < DELTA_STAGES - 1; ++tile) fetch(tile);
        prepare(0);
        __syncthreads();
        for (int tile = 0; tile < n_tiles; ++tile) {
            fetch(tile + DELTA_STAGES - 1);
            if (tile + 1 < n_tiles) prepare(tile + 1);
            if (tile > 0) write_out(tile - 1);
            __syncthreads();
        }
        write_out(n_tiles - 1);
        return;
    }

    // ---- computing warps
    const int j = lane % J, c0 = (warp * (32 / J) + lane / J) * CPT;     // this thread's first column of the block
    float* S = a.state + (long long)a.state_slots[r] * a.slot_stride + (long long)h * DK * DV;
    const bool words = DK % 4 == 0 && (((uintptr_t)S) & 15) == 0;
    f32x2 s[CPT][2 * KW];
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < KW; ++i) {
            const int e = 4 * (j + J * i), p = p0 + c0 + c;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (p < DV && e < DK) {
                const float* src = S + (size_t)p * DK + e;
                if (words) v = *reinterpret_cast<const float4*>(src);
                else {
                    v.x = src[0];
                    if (e + 1 < DK) v.y = src[1];
                    if (e + 2 < DK) v.z = src[2];
                    if (e + 3 < DK) v.w = src[3];
                }
            }
            s[c][2 * i] = pack2(v.x, v.y);
            s[c][2 * i + 1] = pack2(v.z, v.w);
        }
    const int mine = j >> 1;                                   // which of the 2 CPT sums this lane ends with: d1 of column mine, or d2 of column mine - CPT
    const bool writes = mine >= CPT && (j & 1) == 0;
    const int out_col = c0 + mine - CPT;
    __syncthreads();
    for (int tile = 0; tile < n_tiles; ++tile) {
        const float* buf = dsm + (tile & 1) * Sh::TILE;
        const float* tail = buf + 5 * Sh::VEC;
        float* os = results + (tile & 1) * DELTA_TT * DELTA_COLS;
        const int nt = min(DELTA_TT, t1 - t0 - tile * DELTA_TT);
        ulonglong2 uu[KW], wr[KW];
#pragma unroll
        for (int i = 0; i < KW; ++i) {
            uu[i] = reinterpret_cast<const ulonglong2*>(buf)[j + J * i];
            wr[i] = reinterpret_cast<const ulonglong2*>(buf + Sh::VEC)[j + J * i];
        }
        for (int t = 0; t < nt; ++t) {
            const ulonglong2* vec = reinterpret_cast<const ulonglong2*>(buf + t * DKP) + j;     // 4 floats a word; vectors VEC / 4 words apart
            ulonglong2 w[KW], k[KW], au[KW];
#pragma unroll
            for (int i = 0; i < KW; ++i) {
                w[i] = vec[2 * (Sh::VEC / 4) + J * i];
                k[i] = vec[3 * (Sh::VEC / 4) + J * i];
                au[i] = vec[4 * (Sh::VEC / 4) + J * i];      // negated
            }
            float d[2 * CPT], v[CPT];
            delta_columns<CPT>(tail + t * DELTA_COLS + c0, v);
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                f32x2 d1 = mul2(s[c][0], uu[0].x), d2 = mul2(s[c][0], wr[0].x);
                d1 = fma2(s[c][1], uu[0].y, d1);
                d2 = fma2(s[c][1], wr[0].y, d2);
#pragma unroll
                for (int i = 1; i < KW; ++i) {
                    d1 = fma2(s[c][2 * i], uu[i].x, d1);
                    d2 = fma2(s[c][2 * i], wr[i].x, d2);
                    d1 = fma2(s[c][2 * i + 1], uu[i].y, d1);
                    d2 = fma2(s[c][2 * i + 1], wr[i].y, d2);
                }
                float lo, hi;
                unpack2(d1, lo, hi);
                d[c] = lo + hi;
                unpack2(d2, lo, hi);
                d[CPT + c] = lo + hi;
            }
#pragma unroll
            for (int i = 0; i < KW; ++i) {      // the next token's (behind the tile's last one: not used), on their way while this one's sums meet
                uu[i] = vec[DKP / 4 + J * i];
                wr[i] = vec[Sh::VEC / 4 + DKP / 4 + J * i];
            }
            const float sum = delta_reduce<2 * CPT>(d, lane);
            // the part of the update that does not wait for the sums
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const f32x2 v2 = pack2(v[c], v[c]);
#pragma unroll
                for (int i = 0; i < KW; ++i) {
                    s[c][2 * i] = fma2(w[i].x, s[c][2 * i], mul2(k[i].x, v2));
                    s[c][2 * i + 1] = fma2(w[i].y, s[c][2 * i + 1], mul2(k[i].y, v2));
                }
            }
            const float held = __shfl_xor_sync(0xffffffffu, sum, J / 2);      // d1 of the column whose d2 this lane has
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                const float a1 = __shfl_sync(0xffffffffu, sum, 2 * c, J);
                const f32x2 h2 = pack2(a1, a1);
#pragma unroll
                for (int i = 0; i < KW; ++i) {
                    s[c][2 * i] = fma2(au[i].x, h2, s[c][2 * i]);
                    s[c][2 * i + 1] = fma2(au[i].y, h2, s[c][2 * i + 1]);
                }
            }
            if (writes) {
                const float aur = tail[DELTA_TT * DELTA_COLS + 2 * t], kdr = tail[DELTA_TT * DELTA_COLS + 2 * t + 1];
                os[t * DELTA_COLS + out_col] = sum - aur * held + kdr * tail[t * DELTA_COLS + out_col];
            }
        }
        __syncthreads();      // the tile's results are there; its buffer may be filled again
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < KW; ++i) {
            const int e = 4 * (j + J * i), p = p0 + c0 + c;
            if (p >= DV || e >= DK) continue;
            float4 v;
            unpack2(s[c][2 * i], v.x, v.y);
            unpack2(s[c][2 * i + 1], v.z, v.w);
            float* dst = S + (size_t)p * DK + e;
            if (words) *reinterpret_cast<float4*>(dst) = v;
            else {
                dst[0] = v.x;
                if (e + 1 < DK) dst[1] = v.y;
                if (e + 2 < DK) dst[2] = v.z;
                if (e + 3 < DK) dst[3] = v.w;
            }
        }
}

// One token per request (a decode step), where a step is its state's way through the registers: the same layout of columns over lanes without
// shared memory; every group of lanes prepares the token's vectors for its own key entries. grid (columns / 32, heads, requests).
template <typename T, int J, int KW>
__global__ void __launch_bounds__(32 * DELTA_WARPS) delta_step_kernel(float* __restrict__ y, const T* __restrict__ proj, const DeltaArgs a) {
    constexpr int CPT = DeltaShape<J, KW>::CPT;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, j = lane % J, c0 = (warp * (32 / J) + lane / J) * CPT;
    const int p0 = blockIdx.x * DELTA_COLS + c0, h = blockIdx.y, r = blockIdx.z, DK = a.DK, DV = a.DV;
    const int t = a.cu_q[r];
    if (a.cu_q[r + 1] <= t) return;
    float* S = a.state + (long long)a.state_slots[r] * a.slot_stride + (long long)h * DK * DV;
    const bool words = DK % 4 == 0 && (((uintptr_t)S) & 15) == 0;
    float s[CPT][4 * KW];
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < KW; ++i) {
            const int e = 4 * (j + J * i);
            const float* src = S + (size_t)(p0 + c) * DK + e;
            if (words) {
                const float4 v = p0 + c < DV && e < DK ? *reinterpret_cast<const float4*>(src) : make_float4(0.f, 0.f, 0.f, 0.f);
                s[c][4 * i] = v.x; s[c][4 * i + 1] = v.y; s[c][4 * i + 2] = v.z; s[c][4 * i + 3] = v.w;
            } else {
#pragma unroll
                for (int q = 0; q < 4; ++q) s[c][4 * i + q] = p0 + c < DV && e + q < DK ? src[q] : 0.f;
            }
        }
    const T* row = proj + (size_t)t * a.stride;
    float k[4 * KW], rd[4 * KW], w[4 * KW], u[4 * KW], au[4 * KW], v[CPT];
    float sq = 0.f, aur = 0.f, kdr = 0.f;
#pragma unroll
    for (int i = 0; i < 4 * KW; ++i) {
        const int e = 4 * (j + J * (i / 4)) + i % 4, at = min(e, DK - 1);
        const float zw = a.zw[(size_t)t * a.zw_stride + h * DK + at] + a.w0[h * DK + at], za = a.za[(size_t)t * a.za_stride + h * DK + at] + a.ab[h * DK + at];
        k[i] = e < DK ? Num<T>::to_f32(row[a.k_col0 + h * DK + at]) : 0.f;
        rd[i] = e < DK ? Num<T>::to_f32(row[a.r_col0 + h * DK + at]) : 0.f;
        w[i] = expf(-a.rate * delta_sigmoid(zw));
        au[i] = delta_sigmoid(za);
        sq = fmaf(k[i], k[i], sq);
        kdr = fmaf(k[i], rd[i], kdr);
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c) v[c] = Num<T>::to_f32(row[a.v_col0 + h * DV + min(p0 + c, DV - 1)]);
#pragma unroll
    for (int o = J / 2; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        kdr += __shfl_xor_sync(0xffffffffu, kdr, o);
    }
    const float inv = 1.f / sqrtf(sq + a.len_eps);
#pragma unroll
    for (int i = 0; i < 4 * KW; ++i) {
        u[i] = k[i] * inv;
        au[i] *= u[i];
        aur = fmaf(au[i], rd[i], aur);
        rd[i] *= w[i];
    }
#pragma unroll
    for (int o = J / 2; o > 0; o >>= 1) aur += __shfl_xor_sync(0xffffffffu, aur, o);
    float d[2 * CPT];
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        d[c] = d[CPT + c] = 0.f;
#pragma unroll
        for (int i = 0; i < 4 * KW; ++i) {
            d[c] = fmaf(s[c][i], u[i], d[c]);
            d[CPT + c] = fmaf(s[c][i], rd[i], d[CPT + c]);
        }
    }
    const float sum = delta_reduce<2 * CPT>(d, lane), held = __shfl_xor_sync(0xffffffffu, sum, J / 2);
    const int mine = (j >> 1) - CPT;
#pragma unroll
    for (int c = 0; c < CPT; ++c) {
        const float a1 = __shfl_sync(0xffffffffu, sum, 2 * c, J);
#pragma unroll
        for (int i = 0; i < 4 * KW; ++i) s[c][i] = fmaf(-au[i], a1, fmaf(w[i], s[c][i], k[i] * v[c]));
        if (mine == c && (j & 1) == 0 && p0 + c < DV) y[(size_t)t * a.heads * DV + h * DV + p0 + c] = sum - aur * held + kdr * v[c];
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < KW; ++i) {
            const int e = 4 * (j + J * i);
            if (p0 + c >= DV || e >= DK) continue;
            float* dst = S + (size_t)(p0 + c) * DK + e;
            if (words) *reinterpret_cast<float4*>(dst) = make_float4(s[c][4 * i], s[c][4 * i + 1], s[c][4 * i + 2], s[c][4 * i + 3]);
            else {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (e + q < DK) dst[q] = s[c][4 * i + q];
            }
        }
}

template <typename T, int J, int KW>
static int delta_launch(float* y, const T* proj, const DeltaArgs& a, int n_requests, bool single, cudaStream_t stream) {
    using Sh = DeltaShape<J, KW>;
    const dim3 grid((a.DV + DELTA_COLS - 1) / DELTA_COLS, a.heads, n_requests);
    if (single) {
        delta_step_kernel<T, J, KW><<<grid, 32 * DELTA_WARPS, 0, stream>>>(y, proj, a);
        return oxr_launch_status();
    }
    constexpr size_t SMEM = Sh::template SMEM<T>;
    static_assert(SMEM <= 227 * 1024, "fits a block");
    if constexpr (SMEM > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<T, J, KW>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
        if (e != cudaSuccess) return 1000 + (int)e;
    }
    delta_scan_kernel<T, J, KW><<<grid, 32 * (DELTA_WARPS + DELTA_PREP_WARPS), SMEM, stream>>>(y, proj, a);
    return oxr_launch_status();
}

template <typename T>
static int delta_launch_j(float* y, const T* proj, const DeltaArgs& a, int n_requests, bool single, cudaStream_t stream) {
    if (a.DK <= 16) return delta_launch<T, 4, 1>(y, proj, a, n_requests, single, stream);
    if (a.DK <= 32) return delta_launch<T, 8, 1>(y, proj, a, n_requests, single, stream);
    if (a.DK <= 64) return delta_launch<T, 16, 1>(y, proj, a, n_requests, single, stream);
    if (a.DK <= 128) return delta_launch<T, 32, 1>(y, proj, a, n_requests, single, stream);
    return delta_launch<T, 32, 2>(y, proj, a, n_requests, single, stream);
}

OXR_API int oxr_delta_scan(float* y, const void* proj, int n_requests, int stride, int r_col0, int k_col0, int v_col0, const float* zw, int zw_stride,
                           const float* w0, const float* za, int za_stride, const float* ab, float rate, float len_eps, int heads, int DK, int DV,
                           float* state, long long slot_stride, const int* cu_q, const int* state_slots, int single, int dtype,
                           cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (heads <= 0 || DK <= 0 || DK > 256 || DV <= 0 || heads > 65535 || n_requests > 65535 || !(rate > 0.f) || !(len_eps > 0.f)) return OXR_BAD_ARGUMENT;
    DeltaArgs a;
    a.stride = stride; a.r_col0 = r_col0; a.k_col0 = k_col0; a.v_col0 = v_col0; a.zw = zw; a.zw_stride = zw_stride; a.w0 = w0; a.za = za;
    a.za_stride = za_stride; a.ab = ab; a.rate = rate; a.len_eps = len_eps; a.heads = heads; a.DK = DK; a.DV = DV; a.state = state;
    a.slot_stride = slot_stride; a.cu_q = cu_q; a.state_slots = state_slots;
    const int word = dtype == 0 ? 4 : 8;      // elements of the projections per 16 bytes
    a.async = DK % word == 0 && DK % 4 == 0 && DV % word == 0 && stride % word == 0 && r_col0 % word == 0 && k_col0 % word == 0 && v_col0 % word == 0 &&
              zw_stride % 4 == 0 && za_stride % 4 == 0 && (uintptr_t)proj % 16 == 0 && (uintptr_t)zw % 16 == 0 && (uintptr_t)za % 16 == 0;
    if (dtype == 0) return delta_launch_j<float>(y, (const float*)proj, a, n_requests, single != 0, stream);
    return delta_launch_j<__nv_bfloat16>(y, (const __nv_bfloat16*)proj, a, n_requests, single != 0, stream);
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
