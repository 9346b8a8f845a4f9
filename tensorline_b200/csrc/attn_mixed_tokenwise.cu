// Paged causal attention whose heads' softmax weights are mixed before they meet the values (Shazeer et al.,
// "Talking-Heads Attention"), in exact order: one block a token, all heads.
//
//   P_g(j)  = exp(s_g(j) - m_g) / l_g,  s_g(j) = (q_g . k_g'(j)) * scale over the keys j <= p of the request (g' = g's KV head)
//   P'_h(j) = sum_g mix[h, g] P_g(j)
//   o_h     = sum_j P'_h(j) v_h'(j)
// A weight needs its head's whole denominator before it is mixed, so the keys are walked twice: first every head's m and l
// (a warp a head), then, tile by tile of 32 keys, every head's weights into shared memory, the mix and the values (a warp an
// output head).  Tiles are aligned to position 0 and every sum's order depends on the position alone, so a position's result
// is bit-identical under every schedule.  The true 32-bit engine uses this kernel for everything; the bfloat16 engine for
// sizes its own kernels do not take, and the tests as an on-device reference.
#include "common.cuh"

#define MIX_MAX_D 512

template <typename TA>
__global__ void __launch_bounds__(1024, 1) attn_mixed_tokenwise_kernel(const TA* __restrict__ q, int q_stride, TA* __restrict__ out,
                                                                       const TA* __restrict__ k_pages, const TA* __restrict__ v_pages,
                                                                       const int* __restrict__ table, int max_pages, int page_size,
                                                                       const int* __restrict__ pos, const int* __restrict__ req_slot,
                                                                       int nq, int nkv, int d, float scale, const float* __restrict__ mix,
                                                                       const TlLimits L) {
    extern __shared__ float sm[];
    float* qs = sm;                          // [nq][d]
    float* ms = qs + (size_t)nq * d;         // [nq]
    float* ls = ms + nq;                     // [nq]
    float* ps = ls + nq;                     // [nq][33]
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    const int p = pos[t], grp = nq / nkv;
    const int* tab = table + (size_t)tl_checked(req_slot[t], L.table_rows, L, TL_K_TOKENWISE) * max_pages;
    for (int e = threadIdx.x; e < nq * d; e += blockDim.x) qs[e] = to_f<TA>(q[(size_t)t * q_stride + e]);
    __syncthreads();

    auto row_of = [&](int j, int kh) {
        const int page = tl_checked(tab[tl_checked(j / page_size, max_pages, L, TL_K_TOKENWISE)], L.total_pages, L, TL_K_TOKENWISE);
        return (((size_t)page * nkv + kh) * page_size + (j % page_size)) * d;
    };
    auto score = [&](int g, int j) {
        const TA* kr = k_pages + row_of(j, g / grp);
        const float* qg = qs + (size_t)g * d;
        float dot = 0.f;
        for (int e = 0; e < d; ++e) dot = fmaf(qg[e], to_f<TA>(kr[e]), dot);
        return dot * scale;
    };
    for (int g = warp; g < nq; g += nw) {
        float m = -INFINITY, l = 0.f;
        for (int j0 = 0; j0 <= p; j0 += 32) {
            const int j = j0 + lane;
            const float s = j <= p ? score(g, j) : -INFINITY;
            const float m_new = fmaxf(m, warp_max(s));
            l = l * expf(m - m_new) + warp_sum(j <= p ? expf(s - m_new) : 0.f);
            m = m_new;
        }
        if (lane == 0) { ms[g] = m; ls[g] = 1.0f / l; }
    }
    __syncthreads();

    constexpr int MAXC = MIX_MAX_D / 32;
    for (int h0 = 0; h0 < nq; h0 += nw) {                    // as many output heads at a time as there are warps
        const int h = h0 + warp;
        float acc[MAXC];
#pragma unroll
        for (int c = 0; c < MAXC; ++c) acc[c] = 0.f;
        for (int j0 = 0; j0 <= p; j0 += 32) {
            const int j = j0 + lane;
            for (int g = warp; g < nq; g += nw) ps[g * 33 + lane] = j <= p ? expf(score(g, j) - ms[g]) * ls[g] : 0.f;
            __syncthreads();
            if (h < nq) {
                float pm = 0.f;
                for (int g = 0; g < nq; ++g) pm = fmaf(mix[h * nq + g], ps[g * 33 + lane], pm);
                const size_t row = j <= p ? row_of(j, h / grp) : 0;
                const int n_here = min(32, p - j0 + 1);
                for (int jj = 0; jj < n_here; ++jj) {
                    const float pb = __shfl_sync(0xffffffffu, pm, jj);
                    const TA* vr = v_pages + __shfl_sync(0xffffffffu, (unsigned long long)row, jj);
#pragma unroll
                    for (int c = 0; c < MAXC; ++c) {
                        const int e = lane + 32 * c;
                        if (e < d) acc[c] = fmaf(pb, to_f<TA>(vr[e]), acc[c]);
                    }
                }
            }
            __syncthreads();
        }
        if (h < nq) {
            TA* orow = out + ((size_t)t * nq + h) * d;
#pragma unroll
            for (int c = 0; c < MAXC; ++c) {
                const int e = lane + 32 * c;
                if (e < d) orow[e] = from_f<TA>(acc[c]);
            }
        }
    }
}

template <typename TA>
static int launch_mixed_tokenwise(const void* q, int q_stride, void* out, const void* k_pages, const void* v_pages, const int* table,
                                  int max_pages, int page_size, const int* pos, const int* req_slot, int T, int nq, int nkv, int d,
                                  float scale, const float* mix, const TlLimits& L, cudaStream_t stream) {
    const size_t smem = ((size_t)nq * d + 2 * nq + 33 * (size_t)nq) * sizeof(float);
    if (smem > 227 * 1024) return 1;
    if (smem > 48 * 1024) {
        static int raised[TL_MAX_DEVICES] = {};
        const int dev = tl_device_index();
        if (dev < 0) return 1;
        if (raised[dev] < (int)smem) {
            const cudaError_t e = cudaFuncSetAttribute(attn_mixed_tokenwise_kernel<TA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (e != cudaSuccess) return (int)e;
            raised[dev] = (int)smem;
        }
    }
    attn_mixed_tokenwise_kernel<TA><<<T, 32 * (nq < 32 ? nq : 32), smem, stream>>>((const TA*)q, q_stride, (TA*)out, (const TA*)k_pages,
        (const TA*)v_pages, table, max_pages, page_size, pos, req_slot, nq, nkv, d, scale, mix, L);
    return tl_launch_status();
}

TL_EXPORT int tl_attn_mixed_tokenwise(const void* q, int q_stride, void* out, int act_dtype, const void* k_pages, const void* v_pages,
                                      const int* table, int max_pages, int page_size, const int* pos, const int* req_slot, int T, int nq,
                                      int nkv, int d, float scale, const float* mix, int table_rows, int total_pages, int* fault,
                                      cudaStream_t stream) {
    const TlLimits L{table_rows, total_pages, fault};
    if (T <= 0) return 0;
    if (d > MIX_MAX_D || nq % nkv) return 1;
    if (act_dtype == TL_F32)
        return launch_mixed_tokenwise<float>(q, q_stride, out, k_pages, v_pages, table, max_pages, page_size, pos, req_slot, T, nq, nkv, d, scale, mix, L, stream);
    return launch_mixed_tokenwise<bf16>(q, q_stride, out, k_pages, v_pages, table, max_pages, page_size, pos, req_slot, T, nq, nkv, d, scale, mix, L, stream);
}
