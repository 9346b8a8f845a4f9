// The steps around attention whose heads are made of maps (differential attention: Ye et al., "Differential Transformer") and
// whose queries, keys and values pass a short causal convolution over time.
//
//   conv_heads      y[t, c] = sum_j w[c, j] u[t - (taps - 1) + j, c] for every channel c of the step's q|k|v projection u (zeros
//                   before a request's start; the taps - 1 rows before the step come from the request's slot, which is then
//                   brought up to date), the RMS norm of every map of a q or k head over its `dim` channels with a weight, and
//                   the rows of the attention kernels: map m of a head of `maps` maps keeps to columns [m dim, (m + 1) dim) of a
//                   row of d, q's other columns are zeros, a key's maps lie side by side in its page row, values in theirs.
//                   A query of map m then meets map m of the key and nothing else, so ONE run of a paged attention kernel over
//                   maps * heads query heads reads every key and value once for all maps.
//   map_difference  o = a_1 - lambda a_2 per head, divided by its root mean square over the head's dv values, times a constant
//
// Sums, statistics and the difference are float; projections, rows and outputs are of the activation type.
#include "common.cuh"

struct ConvHeads {
    const void* proj; int stride;          // [T, stride]: q [nq, maps, dim], k [nkv, maps, dim], v [nkv, dv]
    const void* taps_w; int taps;          // [C, taps]
    void* state; long long slot_stride;    // [slots][taps - 1][C] of the activation type, oldest row first; null with one tap
    const int* q_start; const int* slots; const int* start_pos;
    const int* table; int max_pages, page_size;
    const float* q_norm; const float* k_norm; float eps;     // [dim] each or both null
    void* q_out; void* k_pages; void* v_pages;
    int nq, nkv, maps, dim, dv, d, C;
    TlLimits lim;
};

// Where the values of one map of q or k, or of one v head, go for the token at position p of the request in `slot`.
template <typename TA>
__device__ __forceinline__ TA* conv_heads_row(const ConvHeads& A, int unit, int t, int p, int slot) {
    const int nqm = A.nq * A.maps, nkm = A.nkv * A.maps;
    if (unit < nqm) return (TA*)A.q_out + ((size_t)t * nqm + unit) * A.d;
    const int* tab = A.table + (size_t)tl_checked(slot, A.lim.table_rows, A.lim, TL_K_ROPE) * A.max_pages;
    const int page = tl_checked(tab[tl_checked(p / A.page_size, A.max_pages, A.lim, TL_K_ROPE)], A.lim.total_pages, A.lim, TL_K_ROPE);
    const int head = unit < nqm + nkm ? (unit - nqm) / A.maps : unit - nqm - nkm;
    return (TA*)(unit < nqm + nkm ? A.k_pages : A.v_pages) + (((size_t)page * A.nkv + head) * A.page_size + p % A.page_size) * A.d;
}

// Any type and size.  grid (requests, chunks of `chunk` >= taps - 1 tokens, units / 4): a warp a unit (a map of a q or k head,
// a v head), its tokens one after the other; the warp of a request's first chunk also keeps the unit's part of the state.
template <typename TA, typename TW>
__global__ void __launch_bounds__(128) conv_heads_kernel(const ConvHeads A, int chunk) {
    const int b = blockIdx.x, lane = threadIdx.x & 31, unit = blockIdx.z * 4 + (threadIdx.x >> 5);
    grid_dependency_wait();
    grid_dependency_trigger();
    const int nqm = A.nq * A.maps, nkm = A.nkv * A.maps;
    if (unit >= nqm + nkm + A.nkv) return;
    const int t0 = A.q_start[b], t1 = A.q_start[b + 1], n = t1 - t0, slot = A.slots[b], p0 = A.start_pos[b];
    const int c0 = t0 + blockIdx.y * chunk, c1 = min(t1, c0 + chunk);
    if (c0 >= t1) return;
    const bool is_q = unit < nqm, is_k = !is_q && unit < nqm + nkm;
    const int width = is_q || is_k ? A.dim : A.dv, base = is_q || is_k ? unit * A.dim : (nqm + nkm) * A.dim + (unit - nqm - nkm) * A.dv;
    const int map = is_q ? unit % A.maps : is_k ? (unit - nqm) % A.maps : 0;
    const float* nw = is_q ? A.q_norm : is_k ? A.k_norm : nullptr;
    const TA* proj = (const TA*)A.proj;
    const TW* tw = (const TW*)A.taps_w;
    TA* st = (TA*)A.state + (size_t)slot * A.slot_stride;
    for (int t = c0; t < c1; ++t) {
        auto conv_at = [&](int c) {
            float acc = 0.f;
            for (int j = 0; j < A.taps; ++j) {
                const int src = t - t0 - (A.taps - 1) + j;   // the row's place in the step; negative: the slot's
                const float u = src >= 0 ? to_f<TA>(proj[(size_t)(t0 + src) * A.stride + c]) : to_f<TA>(st[(size_t)(A.taps - 1 + src) * A.C + c]);
                acc = fmaf(to_f<TW>(tw[(size_t)c * A.taps + j]), u, acc);
            }
            return acc;
        };
        float rstd = 1.0f;
        if (nw) {
            float ss = 0.f;
            for (int e = lane; e < width; e += 32) { const float y = conv_at(base + e); ss = fmaf(y, y, ss); }
            rstd = 1.0f / sqrtf(warp_sum(ss) / (float)width + A.eps);
        }
        TA* row = conv_heads_row<TA>(A, unit, t, p0 + (t - t0), slot);
        const int off = map * A.dim;
        for (int e = lane; e < width; e += 32) {
            const float y = conv_at(base + e);
            row[off + e] = from_f<TA>(nw ? y * rstd * nw[e] : y);
        }
        // zeros: a query's other columns, what lies behind the last map of a key and behind a value
        if (is_q) { for (int e = lane; e < off; e += 32) row[e] = from_f<TA>(0.f); }
        if (is_q || !is_k || map == A.maps - 1) { for (int e = off + width + lane; e < A.d; e += 32) row[e] = from_f<TA>(0.f); }
    }
    if (A.taps > 1 && blockIdx.y == 0) {                     // oldest place first: each reads a place behind it or the step's rows
        for (int e = lane; e < width; e += 32) {
            for (int j = 0; j < A.taps - 1; ++j) {
                const int src = n - (A.taps - 1) + j;
                st[(size_t)j * A.C + base + e] = src >= 0 ? proj[(size_t)(t0 + src) * A.stride + base + e] : st[(size_t)(j + n) * A.C + base + e];
            }
        }
    }
}

// bfloat16, dim 8 .. 256 a power of two, dv and d multiples of 8, weights in bfloat16.  A thread owns eight channels and walks
// `tiles` tiles of TT tokens of a request: the TAPS - 1 rows in front of a tile are carried along, the next tile's rows (16 bytes
// each) are on their way while a tile is worked through, a map's sum of squares is finished by shuffles over the dim / 8 lanes
// that share it.  The thread of a request's first tile holds the slot's rows in registers before it overwrites them.  The sums
// are those of the kernel above, in its order but for the squares.
__device__ __forceinline__ void conv_unpack(const uint4 x, float (&v)[8]) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&x);
#pragma unroll
    for (int k = 0; k < 4; ++k) { v[2 * k] = __low2float(h[k]); v[2 * k + 1] = __high2float(h[k]); }
}

template <int TAPS, int TT>
__global__ void __launch_bounds__(128) conv_heads_vec_kernel(const ConvHeads A, int tiles) {
    __shared__ size_t place[TT == 1 ? 1 : 128];              // the block's tokens: row of head 0 in the pages
    const int b = blockIdx.x, nqm = A.nq * A.maps, nkm = A.nkv * A.maps;
    const int n8 = A.C >> 3, mine = blockIdx.z * blockDim.x + threadIdx.x, c8 = min(mine, n8 - 1), c = c8 * 8;      // whole warps: the lanes exchange
    const int qk8 = (nqm + nkm) * A.dim >> 3;
    const bool qk = c8 < qk8;
    const int unit = qk ? c / A.dim : nqm + nkm + (c - (nqm + nkm) * A.dim) / A.dv;
    const int width = qk ? A.dim : A.dv, e0 = qk ? c % A.dim : (c - (nqm + nkm) * A.dim) % A.dv;
    const bool is_q = unit < nqm;
    const int map = is_q ? unit % A.maps : qk ? (unit - nqm) % A.maps : 0;
    const float* nw = is_q ? A.q_norm : qk ? A.k_norm : nullptr;
    float w[8][TAPS], g[8];
    {
        uint4 raw[TAPS];                                     // eight channels x TAPS weights lie side by side: 16 * TAPS bytes
#pragma unroll
        for (int j = 0; j < TAPS; ++j) raw[j] = *reinterpret_cast<const uint4*>((const bf16*)A.taps_w + (size_t)c * TAPS + j * 8);
        float flat[8 * TAPS];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) conv_unpack(raw[j], reinterpret_cast<float(&)[8]>(flat[j * 8]));
#pragma unroll
        for (int k = 0; k < 8; ++k)
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[k][j] = flat[k * TAPS + j];
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) g[k] = nw ? nw[e0 + k] : 1.0f;
    grid_dependency_wait();
    grid_dependency_trigger();
    const int t0 = A.q_start[b], t1 = A.q_start[b + 1], n = t1 - t0, slot = A.slots[b], p0 = A.start_pos[b];
    const int first = blockIdx.y * TT * tiles, count = min(TT * tiles, n - first);             // the block's place in the step
    if (count <= 0) return;
    for (int i = threadIdx.x; i < count; i += blockDim.x) {
        const int p = p0 + first + i;
        const int* tab = A.table + (size_t)tl_checked(slot, A.lim.table_rows, A.lim, TL_K_ROPE) * A.max_pages;
        const int page = tl_checked(tab[tl_checked(p / A.page_size, A.max_pages, A.lim, TL_K_ROPE)], A.lim.total_pages, A.lim, TL_K_ROPE);
        place[i] = (size_t)page * A.nkv * A.page_size + p % A.page_size;
    }
    const bf16* proj = (const bf16*)A.proj + (size_t)t0 * A.stride + c;
    bf16* st = (bf16*)A.state + (size_t)slot * A.slot_stride + c;
    auto row_at = [&](int src) {                             // a row of the step, or what the request left in front of it
        if (src < 0) return *reinterpret_cast<const uint4*>(st + (size_t)(TAPS - 1 + src) * A.C);
        if (src < n) return *reinterpret_cast<const uint4*>(proj + (size_t)src * A.stride);
        return make_uint4(0, 0, 0, 0);
    };
    uint4 next[TT], last[TAPS > 1 ? TAPS - 1 : 1];
    float back[TAPS > 1 ? TAPS - 1 : 1][8];                  // the TAPS - 1 rows in front of the tile
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) conv_unpack(row_at(first + j - (TAPS - 1)), back[j]);
#pragma unroll
    for (int i = 0; i < TT; ++i) next[i] = row_at(first + i);
    if (first == 0 && TAPS > 1) {                            // the slot's rows after the step: loaded before any is written
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int src = n - (TAPS - 1) + j;
            last[j] = row_at(src);
        }
    }
    const int lanes = A.dim >> 3;
    const int head = is_q ? unit : qk ? (unit - nqm) / A.maps : unit - nqm - nkm;
    bf16* const pages = (bf16*)(qk ? A.k_pages : A.v_pages) + (size_t)head * A.page_size * A.d;
    bf16* const queries = (bf16*)A.q_out + ((size_t)(t0 + first) * nqm + unit) * A.d;
    __syncthreads();
    for (int at = 0; at < count; at += TT) {
        float u[TAPS - 1 + TT][8];
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
            for (int k = 0; k < 8; ++k) u[j][k] = back[j][k];
#pragma unroll
        for (int i = 0; i < TT; ++i) conv_unpack(next[i], u[TAPS - 1 + i]);
        if (TT > 1) {
#pragma unroll
            for (int i = 0; i < TT; ++i) if (at + TT < count) next[i] = row_at(first + at + TT + i);
        }
#pragma unroll
        for (int i = 0; i < TT; ++i) {
            if (at + i >= count) break;                      // the same for the whole block
            float y[8];
#pragma unroll
            for (int k = 0; k < 8; ++k) y[k] = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j)
#pragma unroll
                for (int k = 0; k < 8; ++k) y[k] = fmaf(w[k][j], u[i + j][k], y[k]);
            float ss = 0.f;
#pragma unroll
            for (int k = 0; k < 8; ++k) ss = fmaf(y[k], y[k], ss);
            for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);      // values join in and ignore the sum
            if (nw) {
                const float rstd = 1.0f / sqrtf(ss / (float)A.dim + A.eps);
#pragma unroll
                for (int k = 0; k < 8; ++k) y[k] = y[k] * rstd * g[k];
            }
            if (mine >= n8) continue;
            uint4 out;
            __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
            for (int k = 0; k < 4; ++k) o2[k] = __floats2bfloat162_rn(y[2 * k], y[2 * k + 1]);
            bf16* row = is_q ? queries + (size_t)(at + i) * nqm * A.d : pages + place[at + i] * A.d;
            *reinterpret_cast<uint4*>(row + map * A.dim + e0) = out;
            const uint4 zero = make_uint4(0, 0, 0, 0);
            if (is_q) {                                      // a query's other maps
                for (int m = 0; m < A.maps; ++m) if (m != map) *reinterpret_cast<uint4*>(row + m * A.dim + e0) = zero;
            }
            if (is_q || !qk || map == A.maps - 1) {          // behind the last map, behind a value
                for (int e = (qk ? A.maps * A.dim : A.dv) + e0; e < A.d; e += width) *reinterpret_cast<uint4*>(row + e) = zero;
            }
        }
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
            for (int k = 0; k < 8; ++k) back[j][k] = u[TT + j][k];
    }
    if (first == 0 && TAPS > 1 && mine < n8) {
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) *reinterpret_cast<uint4*>(st + (size_t)j * A.C) = last[j];
    }
}

constexpr int CONV_HEADS_TT = 4, CONV_HEADS_TILES = 4;       // tokens a tile, tiles a block in long steps (128 tokens at most)

TL_EXPORT int tl_conv_heads(const void* proj, int act_dtype, int stride, const void* taps_w, int w_dtype, int taps, void* state,
                            long long slot_stride, const int* q_start, const int* slots, const int* start_pos, const int* table,
                            int max_pages, int page_size, const float* q_norm, const float* k_norm, float eps, void* q_out,
                            void* k_pages, void* v_pages, int nq, int nkv, int maps, int dim, int dv, int d, int B, int max_q_len,
                            int table_rows, int total_pages, int* fault, cudaStream_t stream) {
    if (B <= 0 || max_q_len <= 0) return 0;
    if (taps < 1 || (taps > 1 && !state) || maps < 1 || maps * dim > d || dv > d || (q_norm == nullptr) != (k_norm == nullptr)) return 1;
    const ConvHeads A{proj, stride, taps_w, taps, state, slot_stride, q_start, slots, start_pos, table, max_pages, page_size, q_norm, k_norm, eps,
                      q_out, k_pages, v_pages, nq, nkv, maps, dim, dv, d, (nq + nkv) * maps * dim + nkv * dv,
                      TlLimits{table_rows, total_pages, fault}};
    const uintptr_t bases = (uintptr_t)proj | (uintptr_t)taps_w | (uintptr_t)state | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages;
    if (act_dtype == TL_BF16 && w_dtype == TL_BF16 && taps <= 4 && dim >= 8 && dim <= 256 && (dim & (dim - 1)) == 0 && (dv & 7) == 0 &&
        (d & 7) == 0 && (stride & 7) == 0 && (slot_stride & 7) == 0 && (bases & 15) == 0) {
        const int n8 = A.C >> 3;
        const bool one = max_q_len == 1;
        // a few tiles a block once the blocks of single tiles would fill the GPU more than twice
        const long long single_tiles = (long long)B * ((max_q_len + CONV_HEADS_TT - 1) / CONV_HEADS_TT) * ((n8 + 127) / 128);
        const int tiles = one || single_tiles < 8LL * tl_num_sms() ? 1 : CONV_HEADS_TILES;
        const dim3 grid(B, one ? 1 : (max_q_len + CONV_HEADS_TT * tiles - 1) / (CONV_HEADS_TT * tiles), (n8 + 127) / 128);
        if (grid.y > 65535 || grid.z > 65535) return 1;
#define CH(TAPS) (one ? launch_after_wait(conv_heads_vec_kernel<TAPS, 1>, grid, dim3(128), 0, stream, A, tiles) \
                      : launch_after_wait(conv_heads_vec_kernel<TAPS, CONV_HEADS_TT>, grid, dim3(128), 0, stream, A, tiles))
        const int e = taps == 1 ? CH(1) : taps == 2 ? CH(2) : taps == 3 ? CH(3) : CH(4);
#undef CH
        return e ? e : tl_launch_status();
    }
    const int chunk = taps - 1 > 4 ? taps - 1 : 4;           // only a request's first chunk may read the slot's rows
    const dim3 grid(B, (max_q_len + chunk - 1) / chunk, ((nq + nkv) * maps + nkv + 3) / 4);
    if (grid.y > 65535 || grid.z > 65535) return 1;
#define CG(TA, TW) launch_after_wait(conv_heads_kernel<TA, TW>, grid, dim3(128), 0, stream, A, chunk)
    int e;
    if (act_dtype == TL_F32) e = w_dtype == TL_F32 ? CG(float, float) : CG(float, bf16);
    else e = w_dtype == TL_F32 ? CG(bf16, float) : CG(bf16, bf16);
#undef CG
    return e ? e : tl_launch_status();
}

// ------------------------------------------------------------------ the two maps' outputs, combined
// a: [T, H, 2, d] (a head's maps one behind the other, values in the first dv of d columns); y: [T, H * dv].  A warp a (token, head).
template <typename TA>
__global__ void __launch_bounds__(128) map_difference_kernel(const TA* __restrict__ a, TA* __restrict__ y, long long heads, int d, int dv,
                                                             float lambda, float eps, float out_scale) {
    const long long i = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    grid_dependency_wait();
    grid_dependency_trigger();
    if (i >= heads) return;
    const TA* a1 = a + i * 2 * d;
    const TA* a2 = a1 + d;
    float ss = 0.f;
    for (int e = lane; e < dv; e += 32) { const float o = to_f<TA>(a1[e]) - lambda * to_f<TA>(a2[e]); ss = fmaf(o, o, ss); }
    const float r = out_scale / sqrtf(warp_sum(ss) / (float)dv + eps);
    for (int e = lane; e < dv; e += 32) y[i * dv + e] = from_f<TA>((to_f<TA>(a1[e]) - lambda * to_f<TA>(a2[e])) * r);
}

// bfloat16, dv / 8 a power of two of at most 32 lanes, d a multiple of 8: eight values a lane, dv / 8 lanes a (token, head).
__global__ void __launch_bounds__(128) map_difference_vec_kernel(const bf16* __restrict__ a, bf16* __restrict__ y, long long heads, int d, int dv,
                                                                 float lambda, float eps, float out_scale) {
    const int lanes = dv >> 3;
    const long long item = (long long)blockIdx.x * 128 + threadIdx.x, last = heads * lanes - 1;
    grid_dependency_wait();
    grid_dependency_trigger();
    const long long at = item < last ? item : last;          // whole warps: the lanes exchange
    const long long i = at / lanes;
    const int e0 = (int)(at - i * lanes) * 8;
    float x[8], z[8];
    conv_unpack(*reinterpret_cast<const uint4*>(a + i * 2 * d + e0), x);
    conv_unpack(*reinterpret_cast<const uint4*>(a + i * 2 * d + d + e0), z);
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) { x[k] -= lambda * z[k]; ss = fmaf(x[k], x[k], ss); }
    for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float r = out_scale / sqrtf(ss / (float)dv + eps);
    if (item > last) return;
    uint4 out;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int k = 0; k < 4; ++k) o2[k] = __floats2bfloat162_rn(x[2 * k] * r, x[2 * k + 1] * r);
    *reinterpret_cast<uint4*>(y + i * dv + e0) = out;
}

TL_EXPORT int tl_map_difference(const void* a, void* y, int act_dtype, int T, int H, int d, int dv, float lambda, float eps,
                                float out_scale, cudaStream_t stream) {
    if (T <= 0 || H <= 0) return 0;
    if (dv < 1 || dv > d) return 1;
    const long long heads = (long long)T * H;
    const int lanes = dv >> 3;
    int e;
    if (act_dtype == TL_BF16 && (dv & 7) == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0 && (d & 7) == 0 && ((((uintptr_t)a | (uintptr_t)y) & 15) == 0))
        e = launch_after_wait(map_difference_vec_kernel, dim3((unsigned)((heads * lanes + 127) / 128)), dim3(128), 0, stream, (const bf16*)a,
                              (bf16*)y, heads, d, dv, lambda, eps, out_scale);
    else if (act_dtype == TL_F32)
        e = launch_after_wait(map_difference_kernel<float>, dim3((unsigned)((heads + 3) / 4)), dim3(128), 0, stream, (const float*)a, (float*)y,
                              heads, d, dv, lambda, eps, out_scale);
    else
        e = launch_after_wait(map_difference_kernel<bf16>, dim3((unsigned)((heads + 3) / 4)), dim3(128), 0, stream, (const bf16*)a, (bf16*)y,
                              heads, d, dv, lambda, eps, out_scale);
    return e ? e : tl_launch_status();
}
