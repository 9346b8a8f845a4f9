// The residual sum with several waiting addends, the norm behind it and the token shift, one kernel, all float arithmetic.
//
//   v[t]  = x[t] (+ base[t]) (+ row) + sum_i scale_i * a_i[t]      a_i of the activation type, scale_i a vector over the width
//                                                                  (a layer scale; null: ones), base float [T, W], row [W]
//   n[t]  = v[t] / sqrt(mean(v[t]^2) + eps) * w
//   h[t]  = n[t] + (n[t-1] - n[t]) * shift                         shift [W]; null: h = n
// n[t-1] is the row of the request's token in front of t: the row in front in the step, or, for the first row of a request's
// portion, what the request's slot of `prev` (float [slots, W]) holds, or zeros at position 0.  The block that owns a
// portion's first row leaves n of the portion's LAST row in the slot after it has read the slot, so a launch both reads and
// renews the state and no two blocks touch the same slot.
// A row's neighbour is normalised again by the block that needs it (NR rows a block, NR + 1 norms), from the same inputs in
// the same order of additions, so the result does not depend on how a step was cut.  With a shift x is therefore left as it
// is (the addends stay with the caller until a norm without a shift writes them); without one x takes v (`write_x`).
// `rows` picks rows (no shift; x is left alone); `h` null: only the sum.
#include "common.cuh"

constexpr int SUM_ADDENDS = 3;

struct SumNormArgs {
    float* x; int W;
    const void* add[SUM_ADDENDS]; const float* scale[SUM_ADDENDS]; int n_add;
    const float* base; const float* row;
    const void* w; float eps;
    void* h;
    const int* rows; int T; int write_x;
    const float* shift; float* prev; long long prev_stride;
    const int* pos; const int* req_slot; const int* q_start; int B; int single;
};

template <int VEC> struct Pack;
template <> struct Pack<4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
        const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[4]) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&t.x), b = *reinterpret_cast<const __nv_bfloat162*>(&t.y);
        v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[4]) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 t; t.x = *reinterpret_cast<uint32_t*>(&a); t.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = t;
    }
};
template <> struct Pack<1> {
    template <typename T> static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f<T>(*p); }
    template <typename T> static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_f<T>(v[0]); }
};

// v of L rows in this thread's columns, and the thread's shares of the sums of their squares.  `at`: the rows' first elements, or
// -1 for a row that is not there (its v is zero).  Source after source, so that the loads of all rows are in flight together.
template <typename TA, int VEC, int NV, int L>
__device__ __forceinline__ void sum_rows(const SumNormArgs& A, const long long (&at)[L], int nvec, float (&v)[L][NV][VEC], float (&ss)[L]) {
    using P = Pack<VEC>;
    auto place = [&](int k) { return (size_t)(threadIdx.x + k * blockDim.x) * VEC; };
    auto here = [&](int k) { return threadIdx.x + k * blockDim.x < nvec; };
#pragma unroll
    for (int j = 0; j < L; ++j)
#pragma unroll
        for (int k = 0; k < NV; ++k) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[j][k][e] = 0.f;
            if (at[j] >= 0 && here(k)) P::load(A.x + at[j] + place(k), v[j][k]);
        }
    if (A.base) {
        float b[L][NV][VEC];
#pragma unroll
        for (int j = 0; j < L; ++j)
#pragma unroll
            for (int k = 0; k < NV; ++k) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) b[j][k][e] = 0.f;
                if (at[j] >= 0 && here(k)) P::load(A.base + at[j] + place(k), b[j][k]);
            }
#pragma unroll
        for (int j = 0; j < L; ++j)
#pragma unroll
            for (int k = 0; k < NV; ++k)
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[j][k][e] += b[j][k][e];
    }
    if (A.row) {
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            if (!here(k)) continue;
            float b[VEC]; P::load(A.row + place(k), b);
#pragma unroll
            for (int j = 0; j < L; ++j)
#pragma unroll
                for (int e = 0; e < VEC; ++e) if (at[j] >= 0) v[j][k][e] += b[e];
        }
    }
#pragma unroll
    for (int i = 0; i < SUM_ADDENDS; ++i) {
        if (i < A.n_add) {
            const TA* a = (const TA*)A.add[i];
            float av[L][NV][VEC];
#pragma unroll
            for (int j = 0; j < L; ++j)
#pragma unroll
                for (int k = 0; k < NV; ++k) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) av[j][k][e] = 0.f;
                    if (at[j] >= 0 && here(k)) P::load(a + at[j] + place(k), av[j][k]);
                }
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                float sv[VEC];
#pragma unroll
                for (int e = 0; e < VEC; ++e) sv[e] = 1.0f;
                if (A.scale[i] && here(k)) P::load(A.scale[i] + place(k), sv);
#pragma unroll
                for (int j = 0; j < L; ++j)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) v[j][k][e] = fmaf(sv[e], av[j][k][e], v[j][k][e]);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < L; ++j) {
        ss[j] = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k)
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss[j] = fmaf(v[j][k][e], v[j][k][e], ss[j]);
    }
}

// L sums over the block at once; the order of additions is that of one sum alone.  red: [L][33] floats.
template <int L>
__device__ __forceinline__ void block_sums(float (&s)[L], float (*red)[33]) {
    const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
#pragma unroll
    for (int j = 0; j < L; ++j) s[j] = warp_sum(s[j]);
    __syncthreads();
    if (lane == 0) {
#pragma unroll
        for (int j = 0; j < L; ++j) red[j][wid] = s[j];
    }
    __syncthreads();
    for (int j = wid; j < L; j += nw) {
        float t = lane < nw ? red[j][lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) red[j][32] = t;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < L; ++j) s[j] = red[j][32];
}

template <typename TA, typename TW, int VEC, int NV, int NR, bool SHIFT>
__global__ void __launch_bounds__(1024) sum_norm_kernel(const SumNormArgs A) {
    using P = Pack<VEC>;
    constexpr int L = NR + (SHIFT ? 1 : 0);
    __shared__ float red[L][33];
    const int nvec = A.W / VEC;
    const int t0 = blockIdx.x * NR;
    float wv[NV][VEC], mu[NV][VEC];
    const bool early = gridDim.x <= 128;                     // few rows: the weights, nobody's output, come before the wait
    auto load_w = [&]() {
        if (A.h == nullptr) return;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * blockDim.x;
            if (c < nvec) {
                P::load((const TW*)A.w + (size_t)c * VEC, wv[k]);
                if (SHIFT) P::load(A.shift + (size_t)c * VEC, mu[k]);
            }
        }
    };
    if (early) load_w();
    grid_dependency_wait();
    grid_dependency_trigger();
    if (!early) load_w();
    int slot_of[NR];                                         // which rows are the first of their request's portion, and where its state lies
    unsigned firsts = 0, starts = 0;
    if (SHIFT) {
#pragma unroll
        for (int j = 0; j < NR; ++j) {
            const int t = t0 + j;
            slot_of[j] = 0;
            if (t >= A.T) continue;
            slot_of[j] = A.req_slot[t];
            const int before = t > 0 ? A.req_slot[t - 1] : -1, p = A.pos[t];
            if (A.single || before != slot_of[j]) { firsts |= 1u << j; if (p == 0) starts |= 1u << j; }
        }
    }
    float v[L][NV][VEC], ss[L];
    float pv_early[NV][VEC];                                 // one row a block: the state's row comes with the others
    if (SHIFT && NR == 1 && firsts && !starts) {
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * blockDim.x;
            if (c < nvec) P::load(A.prev + (size_t)slot_of[0] * A.prev_stride + (size_t)c * VEC, pv_early[k]);
        }
    }
    long long at[L];
#pragma unroll
    for (int j = 0; j < L; ++j) {
        const int t = t0 + j - (SHIFT ? 1 : 0);
        at[j] = t >= 0 && t < A.T && !(SHIFT && j == 0 && A.single) ? (long long)(A.rows ? A.rows[t] : t) * A.W : -1;
    }
    sum_rows<TA, VEC, NV, L>(A, at, nvec, v, ss);
    if (!SHIFT && A.write_x) {
#pragma unroll
        for (int j = 0; j < L; ++j)
            if (t0 + j < A.T)
#pragma unroll
                for (int k = 0; k < NV; ++k) {
                    const int c = threadIdx.x + k * blockDim.x;
                    if (c < nvec) P::store(A.x + (size_t)(t0 + j) * A.W + (size_t)c * VEC, v[j][k]);
                }
    }
    if (A.h == nullptr) return;
    block_sums<L>(ss, red);
#pragma unroll
    for (int j = 0; j < L; ++j) {
        const float rstd = 1.0f / sqrtf(ss[j] / (float)A.W + A.eps);
#pragma unroll
        for (int k = 0; k < NV; ++k)
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[j][k][e] = v[j][k][e] * rstd * wv[k][e];
    }
    TA* h = (TA*)A.h;
    if (!SHIFT) {
#pragma unroll
        for (int j = 0; j < L; ++j)
            if (t0 + j < A.T)
#pragma unroll
                for (int k = 0; k < NV; ++k) {
                    const int c = threadIdx.x + k * blockDim.x;
                    if (c < nvec) P::store(h + (size_t)(t0 + j) * A.W + (size_t)c * VEC, v[j][k]);
                }
        return;
    }
#pragma unroll
    for (int j = 0; j < NR; ++j) {
        const int t = t0 + j;
        if (t >= A.T) continue;
        const bool first = (firsts >> j) & 1u, start = (starts >> j) & 1u;
        const float* st = A.prev + (size_t)slot_of[j] * A.prev_stride;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * blockDim.x;
            if (c < nvec) {
                float pv[VEC], o[VEC];
                if (start) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) pv[e] = 0.f;
                } else if (first && NR == 1) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) pv[e] = pv_early[k][e];
                } else if (first) P::load(st + (size_t)c * VEC, pv);
                else {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) pv[e] = v[j][k][e];
                }
#pragma unroll
                for (int e = 0; e < VEC; ++e) o[e] = fmaf(pv[e] - v[j + 1][k][e], mu[k][e], v[j + 1][k][e]);
                P::store(h + (size_t)t * A.W + (size_t)c * VEC, o);
            }
        }
    }
    // the state: n of the portion's last row, by the block (and the threads) that have just read the slot
#pragma unroll 1
    for (int j = 0; j < NR; ++j) {
        if (!((firsts >> j) & 1u)) continue;
        const int t = t0 + j;
        float* st = A.prev + (size_t)A.req_slot[t] * A.prev_stride;
        int last = t;
        if (!A.single) {                                     // the request whose rows start at t
            int lo = 0, hi = A.B - 1;
            while (lo < hi) { const int mid = (lo + hi) >> 1; if (A.q_start[mid] < t) lo = mid + 1; else hi = mid; }
            last = A.q_start[lo + 1] - 1;
        }
        if (NR == 1 && last == t) {                          // a single token: its own row
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                const int c = threadIdx.x + k * blockDim.x;
                if (c < nvec) P::store(st + (size_t)c * VEC, v[L - 1][k]);
            }
            continue;
        }
        float n[1][NV][VEC], s1[1];
        const long long where[1] = {(long long)last * A.W};
        sum_rows<TA, VEC, NV, 1>(A, where, nvec, n, s1);
        block_sums<1>(s1, red);
        const float rstd = 1.0f / sqrtf(s1[0] / (float)A.W + A.eps);
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            const int c = threadIdx.x + k * blockDim.x;
            if (c < nvec) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) n[0][k][e] = n[0][k][e] * rstd * wv[k][e];
                P::store(st + (size_t)c * VEC, n[0][k]);
            }
        }
    }
}

template <typename TA, typename TW, int VEC>
static int launch_sum_norm(const SumNormArgs& A, cudaStream_t stream) {
    const int nvec = A.W / VEC;
    const bool shift = A.shift != nullptr;
    // one thread count for a width whatever the step (the order of additions), rows a block by how many there are
#define SN(NV, NR, S) launch_after_wait(sum_norm_kernel<TA, TW, VEC, NV, NR, S>, dim3((A.T + NR - 1) / NR), dim3(((nvec + NV - 1) / NV + 31) / 32 * 32), 0, stream, A)
    if (nvec <= 1024) {
        if (shift) return A.single || A.T < 256 ? SN(1, 1, true) : A.T < 1024 ? SN(1, 3, true) : SN(1, 7, true);
        return SN(1, 1, false);
    }
    if (nvec <= 2048) return shift ? SN(2, 1, true) : SN(2, 1, false);
    if (nvec <= 8192) return shift ? SN(8, 1, true) : SN(8, 1, false);
#undef SN
    return 1;
}

TL_EXPORT int tl_sum_norm(float* x, int W, int T, const void* a0, const float* s0, const void* a1, const float* s1, const void* a2,
                          const float* s2, int n_add, int act_dtype, const float* base, const float* row, const void* w, int w_dtype,
                          float eps, void* h, const int* rows, int write_x, const float* shift, float* prev, long long prev_stride,
                          const int* pos, const int* req_slot, const int* q_start, int B, int single, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (n_add < 0 || n_add > SUM_ADDENDS || (shift && (rows || write_x || !h || !prev || !pos || !req_slot || !q_start)) || (rows && write_x)) return 1;
    const SumNormArgs A{x, W, {a0, a1, a2}, {s0, s1, s2}, n_add, base, row, w, eps, h, rows, T, write_x, shift, prev, prev_stride,
                        pos, req_slot, q_start, B, single};
    const uintptr_t all = (uintptr_t)x | (uintptr_t)a0 | (uintptr_t)s0 | (uintptr_t)a1 | (uintptr_t)s1 | (uintptr_t)a2 | (uintptr_t)s2 |
                          (uintptr_t)base | (uintptr_t)row | (uintptr_t)w | (uintptr_t)h | (uintptr_t)shift | (uintptr_t)prev;
    const bool vec = (W & 3) == 0 && (prev_stride & 3) == 0 && (all & 15) == 0;
#define SNT(TA, TW) (vec ? launch_sum_norm<TA, TW, 4>(A, stream) : launch_sum_norm<TA, TW, 1>(A, stream))
    if (act_dtype == TL_F32) return w_dtype == TL_F32 ? SNT(float, float) : SNT(float, bf16);
    return w_dtype == TL_F32 ? SNT(bf16, float) : SNT(bf16, bf16);
#undef SNT
}
