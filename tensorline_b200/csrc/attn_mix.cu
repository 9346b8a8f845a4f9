// Paged causal attention whose heads' softmax weights are mixed before they meet the values (Shazeer et al., "Talking-Heads
// Attention"), bfloat16 engine, compiled for one head size (-DHEAD_DIM=d, a multiple of 64 up to 256).
//
//   P_g(i, j)  = softmax over j <= i of scale q_g(i) . k_g'(j)          g' = g's KV head
//   P'_h(i, j) = sum_g mix[h, g] P_g(i, j);   o_h(i) = sum_j P'_h(i, j) v_h'(j)
//
// A weight needs its head's whole denominator and every other head's weight at the same place before it is of use, so the
// usual one-pass form (rescale O while the maximum grows) is not open: an output head would need one accumulator per head it
// listens to.  The work is cut where the heads meet instead; every piece is a product or a stream of its own:
//   prompts    scores   S_h = Q_h K_h^T per 128 rows x 64 keys on tcgen05, float scores to scratch, log2 of the denominators
//              mix      P = exp2(S - L) in float, P' = mix P on mma.sync: `mix` is exact in bfloat16, P is the sum of three
//                       bfloat16 parts, so products and sums carry a float's 24 bits; P' rounded to bfloat16 for the values
//              values   O_h = P'_h V_h on tcgen05, accumulated in tensor memory over the row's whole range of keys
//   decoding   scores   a block a (request, KV head, range of keys): scores and the range's (m, l)
//              mix and values   a block a (request, range of keys, group of KV heads): P' of the range, then its share of O
//              sum      the ranges' shares added up (they need no rescaling: the weights are normalised already)
//              or, where a request's keys fit the shared memory of a cluster of blocks, all of it in one launch
// Scratch is laid out in the order its reader wants it: scores in 128 x 64 tiles, a row's 16-byte pieces exclusive-ored with the
// row number (the writer's shared-memory image, stored by one bulk copy); P' as the swizzled A-operand tile, loaded by one.
// Every wait is bounded; a block whose wait runs out records a code in `status` and leaves.
#include "common.cuh"
#include "umma.cuh"

#ifndef HEAD_DIM
#error "compile with -DHEAD_DIM=<head size>"
#endif
#if HEAD_DIM % 64 != 0 || HEAD_DIM < 64 || HEAD_DIM > 256
#error "the mixed-head attention kernels take head sizes 64, 128, 192, 256"
#endif

namespace {

constexpr int D = HEAD_DIM;
constexpr int BM = 128;                  // query rows a tile
constexpr int BN = 64;                   // keys a tile
constexpr int CH = D / 8;                // 16-byte pieces of a head's row
constexpr int Q_BYTES = BM * D * 2, K_BYTES = BN * D * 2, P_BYTES = BM * BN * 2, S_BYTES = BM * BN * 4;
constexpr uint32_t O_COLS = D <= 64 ? 64 : D <= 128 ? 128 : 256;

struct MixArgs {
    const bf16* q; int q_stride;         // rows of the step's q|k|v
    bf16* out;                           // [T, nq * D]
    const bf16* k_pages; const bf16* v_pages;
    const int* table; int max_pages; int page_size;
    const int* q_start; const int* start_pos; const int* slots;
    int nq, nkv;
    float scale_log2;
    const int4* tiles; int n_tiles;      // row tiles: (request, tile of 128 rows, first unit in the scratch, key tiles)
    const int2* parts; int n_parts;      // runs of a row tile's key tiles, a block of the scores each: (row tile, number of the run)
    const int* unit_tile; int n_units;   // unit (row tile x key tile) -> its row tile
    float* scores;                       // [units][nq][128][64]
    float2* part_ml;                     // [T][nq][MAX_PARTS]  maximum and sum of each run, in the scores' scaled base-2 units
    float* lse;                          // [T][nq]  log2 of the denominator
    bf16* mixed;                         // [units][nq][128][64]
    const bf16* mix; int hp;             // [hp][hp], nq padded with zeros to a multiple of 16
    int* status;
    TlLimits lim;
};

// A row tile's key tiles are dealt out to several blocks of the scores kernel, in runs of eight or of a sixteenth of them.
constexpr int MAX_PARTS = 16;
__host__ __device__ __forceinline__ int part_tiles(int n_kt) { return n_kt > 8 * MAX_PARTS ? (n_kt + MAX_PARTS - 1) / MAX_PARTS : 8; }

// Keys [key0, key0 + 64) of one KV head as TMA boxes (a page, 64 elements wide), by one thread: pages of 8 tokens or more.
__device__ __forceinline__ void pages_of(int (&page)[8], const int* tab, int max_pages, int ps_shift, int key0, const TlLimits& L) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
        if (i < (BN >> ps_shift)) page[i] = tl_checked(tab[min((key0 >> ps_shift) + i, max_pages - 1)], L.total_pages, L, TL_K_TC_PREFILL);
}
__device__ __forceinline__ void fetch_keys(uint32_t dst, const CUtensorMap* map, uint64_t* bar, const int (&page)[8], int ps_shift, int nkv, int kh) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        if (i >= (BN >> ps_shift)) break;
#pragma unroll
        for (int db = 0; db < D / 64; ++db)
            tma_box(dst + db * (BN * 128) + ((i << ps_shift) * 128), map, bar, db * 64, (page[i] * nkv + kh) << ps_shift);
    }
}

// Copy of keys [key0, key0 + 64) of one KV head into a swizzled [64][D] tile; the calling thread is number `part` of PARTS;
// keys past last_key are zeros.
template <int PARTS>
__device__ __forceinline__ void copy_keys(uint32_t dst, const bf16* pages, const int* tab, int ps_shift, size_t page_stride, int key0,
                                          int last_key, int part, const TlLimits& L) {
    const int ps_mask = (1 << ps_shift) - 1;
#pragma unroll 8
    for (int i = 0; i < BN * CH / PARTS; ++i) {
        const int idx = part + i * PARTS, key = idx / CH, c = idx - key * CH;
        const bool valid = key0 + key <= last_key;
        const int page = valid ? tl_checked(tab[(key0 + key) >> ps_shift], L.total_pages, L, TL_K_TC_PREFILL) : 0;
        const bf16* src = pages + (size_t)page * page_stride + (size_t)((key & ps_mask) * D + c * 8);
        cp_async16(dst + swz(BN, key, c), src, valid);
    }
}
__device__ __forceinline__ int shift_of(int page_size) { int s = 0; while ((1 << s) < page_size) ++s; return s; }
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(dst), "l"(src), "r"(bytes), "r"(smem_addr(bar)) : "memory");
}
__device__ __forceinline__ void bulk_store(void* dst, uint32_t src, uint32_t bytes) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(src), "r"(bytes) : "memory");
    asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}

// ------------------------------------------------------------------------------------------------ prompts: scores
// Warps 0..3: one row a thread (scores out of tensor memory, mask, running maximum and sum, the tile to scratch through
// shared memory); warp 4: MMA issue; warps 5, 6: K, by TMA (warp 5) or by asynchronous copies, every other tile each.
constexpr int S_THREADS = 224;
constexpr int SS_TILES = Q_BYTES + 2 * K_BYTES + S_BYTES;          // two blocks an SM up to head size 128
constexpr int SS_SMEM = SS_TILES + 1024 + 128;
constexpr uint32_t SS_COLS = 128;        // two score slots of 64 columns

template <bool TMA>
__global__ void __launch_bounds__(S_THREADS, D <= 128 ? 2 : 1)
mix_scores_kernel(const __grid_constant__ CUtensorMap map_k, const MixArgs A) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const uint32_t sQ = smem_addr(base), sK = sQ + Q_BYTES, sS = sK + 2 * K_BYTES;
    uint64_t* bars = reinterpret_cast<uint64_t*>(base + SS_TILES);
    uint64_t* bar_q = bars;              // the Q tile is in shared memory
    uint64_t* bar_k = bars + 1;          // [2] K has landed
    uint64_t* bar_s = bars + 3;          // [2] S is complete (commit); the K slot is free
    uint64_t* bar_f = bars + 5;          // [2] the 128 rows have read the S slot
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 7);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x % A.nq, kh = h / (A.nq / A.nkv);
    const int2 pt = A.parts[blockIdx.x / A.nq];
    const int4 tl = A.tiles[pt.x];
    const int b = tl.x, row0 = tl.y * BM, kt0 = pt.y * part_tiles(tl.w), n_kt = min(part_tiles(tl.w), tl.w - kt0);
    const int qs = A.q_start[b], qlen = A.q_start[b + 1] - qs, sp = A.start_pos[b];
    const int row_end = min(row0 + BM, qlen), pos_hi = sp + row_end - 1;
    const int* tab = A.table + (size_t)tl_checked(A.slots[b], A.lim.table_rows, A.lim, TL_K_TC_PREFILL) * A.max_pages;
    tl_checked(pos_hi / A.page_size, A.max_pages, A.lim, TL_K_TC_PREFILL);

    if (tid == 0) {
        mbar_init(bar_q, BM);
        for (int i = 0; i < 2; ++i) { mbar_init(bar_k + i, TMA ? 1 : 32); mbar_init(bar_s + i, 1); mbar_init(bar_f + i, BM); }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 4) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(tmem_slot)), "r"(SS_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;

    if (warp < 4) {
        for (int idx = tid; idx < BM * CH; idx += BM) {
            const int r = idx / CH, c = idx - r * CH;
            const bool valid = row0 + r < qlen;
            cp_async16(sQ + swz(BM, r, c), valid ? A.q + (size_t)(qs + row0 + r) * A.q_stride + (size_t)h * D + c * 8 : A.q, valid);
        }
        cp_async_wait_all();
        fence_async_proxy();
        mbar_arrive(bar_q);
        const int R = row0 + tid, pos_r = R < qlen ? sp + R : -1;
        const uint32_t lane_addr = tmem + ((uint32_t)(warp * 32) << 16);
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        for (int i = 0; i < n_kt; ++i) {
            const int sl = i & 1;
            if (ok) ok = mbar_wait(bar_s + sl, (i >> 1) & 1, abort_flag, A.status, 41);
            float s[BN];
            if (__all_sync(0xffffffffu, ok)) {
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                tmem_ld32(lane_addr + sl * BN, reinterpret_cast<float(&)[32]>(s[0]));
                tmem_ld32(lane_addr + sl * BN + 32, reinterpret_cast<float(&)[32]>(s[32]));
                tmem_ld_wait();
                asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                mbar_arrive(bar_f + sl);
            } else {
                ok = false;
#pragma unroll
                for (int c = 0; c < BN; ++c) s[c] = 0.f;
            }
#pragma unroll
            for (int c = 0; c < BN; ++c) s[c] *= A.scale_log2;
            const int key0 = (kt0 + i) * BN;
            if (key0 + BN - 1 > pos_r) {
#pragma unroll
                for (int c = 0; c < BN; ++c) if (key0 + c > pos_r) s[c] = -INFINITY;
            }
            const float mx = row_max(s);
            const float m_new = fmaxf(m, mx), m_use = m_new == -INFINITY ? 0.f : m_new;
            float l4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int c = 0; c < BN; ++c) l4[c & 3] += fast_exp2(s[c] - m_use);
            l = l * fast_exp2(m - m_use) + ((l4[0] + l4[1]) + (l4[2] + l4[3]));
            m = m_new;
            // a warp's 32 rows are 8 KB in a row of the tile's image: it stages and stores them by itself
            if (lane == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");     // its last store has read the place
            __syncwarp();
#pragma unroll
            for (int c = 0; c < BN / 4; ++c)
                asm volatile("st.shared.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(sS + tid * 256 + ((c ^ (tid & 7)) << 4)),
                             "f"(s[4 * c]), "f"(s[4 * c + 1]), "f"(s[4 * c + 2]), "f"(s[4 * c + 3]) : "memory");
            fence_async_proxy();
            __syncwarp();
            if (lane == 0) bulk_store(A.scores + ((size_t)(tl.z + kt0 + i) * A.nq + h) * (BM * BN) + warp * (32 * BN), sS + warp * (32 * BN * 4), 32 * BN * 4);
        }
        if (R < qlen) A.part_ml[((size_t)(qs + R) * A.nq + h) * MAX_PARTS + pt.y] = make_float2(m, l);
        if (lane == 0) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    } else if (warp == 4) {
        if (lane == 0) {
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(BM >> 4) << 24);
            bool ok = mbar_wait(bar_q, 0, abort_flag, A.status, 42, true);
            for (int j = 0; j < n_kt && ok; ++j) {
                const int sl = j & 1;
                ok = mbar_wait(bar_k + sl, (j >> 1) & 1, abort_flag, A.status, 43, true);
                if (ok && j >= 2) ok = mbar_wait(bar_f + sl, ((j - 2) >> 1) & 1, abort_flag, A.status, 44, true);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t k_addr = sK + sl * K_BYTES;
#pragma unroll
                for (int k = 0; k < D / 16; ++k)
                    umma(tmem + sl * BN, desc_kmajor(sQ + (k >> 2) * BM * 128 + (k & 3) * 32),
                         desc_kmajor(k_addr + (k >> 2) * BN * 128 + (k & 3) * 32), idesc, k > 0 ? 1u : 0u);
                umma_commit(bar_s + sl);
            }
        }
    } else {
        const int ps_shift = shift_of(A.page_size);
        const size_t page_stride = (size_t)A.nkv * A.page_size * D;
        const bf16* pages = A.k_pages + (size_t)kh * A.page_size * D;
        bool ok = true;
        if (TMA) {
            if (warp == 5 && lane == 0) {
                asm volatile("prefetch.tensormap [%0];" ::"l"(&map_k) : "memory");
                int j = 0;
                for (; j < n_kt && ok; ++j) {
                    const int sl = j & 1;
                    int page[8];
                    pages_of(page, tab, A.max_pages, ps_shift, (kt0 + j) * BN, A.lim);       // asked for before the wait
                    if (j >= 2) ok = mbar_wait(bar_s + sl, ((j - 2) >> 1) & 1, abort_flag, A.status, 45, true);
                    if (!ok) break;
                    mbar_expect_tx(bar_k + sl, K_BYTES);
                    fetch_keys(sK + sl * K_BYTES, &map_k, bar_k + sl, page, ps_shift, A.nkv, kh);
                }
                for (int i = max(0, j - 2); !ok && i < j; ++i) {         // a block that gives up waits (bounded) for its own copies
                    const long long t0 = clock64();
                    while (!mbar_try_wait(bar_k + (i & 1), (i >> 1) & 1) && clock64() - t0 < 2000000LL) { }
                }
            }
        } else for (int j = warp - 5; j < n_kt && ok; j += 2) {
            const int sl = j & 1;
            if (j >= 2) ok = mbar_wait(bar_s + sl, ((j - 2) >> 1) & 1, abort_flag, A.status, 45, true);
            if (!ok) break;
            copy_keys<32>(sK + sl * K_BYTES, pages, tab, ps_shift, page_stride, (kt0 + j) * BN, pos_hi, lane, A.lim);
            cp_async_wait_all();
            fence_async_proxy();
            mbar_arrive(bar_k + sl);
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (*abort_flag) {
        const long long t0 = clock64();
        while (clock64() - t0 < 2000000LL) { }
    }
    if (warp == 4) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(SS_COLS) : "memory");
    }
}

// ------------------------------------------------------------------------------------------------ the mix
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// a pair of floats as three packed pairs of bfloat16 whose sums are the floats (24 bits in three times 8)
__device__ __forceinline__ void split3(float x, float y, uint32_t (&o)[3]) {
#pragma unroll
    for (int k = 0; k < 3; ++k) {
        const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
        o[k] = *reinterpret_cast<const uint32_t*>(&v);
        x -= __low2float(v); y -= __high2float(v);
    }
}

// One row's P' over 32 keys by one warp.  Lane (n = lane / 4, c = lane % 4) reads, for the heads 2c, 2c + 1, 2c + 8, 2c + 9 of
// every 16, the scores of keys 4n .. 4n + 3 (`load(g)` -> float4) and makes their weights exp2(s - L_g), L[t][..] of group t;
// product e of four takes key 4n + e as its column n, so the lane's results are keys 8c .. 8c + 7 of the heads lane / 4 and
// lane / 4 + 8 of every 16: acc[m][e][0..1] (keys 8c + e, 8c + 4 + e) and acc[m][e][2..3].  `live` = number of the 32 keys that
// are visible.
__device__ __forceinline__ int mix_head(int t, int k, int c) { return t * 16 + 2 * c + (k & 1) + (k >> 1) * 8; }

template <int MT, typename Load>
__device__ __forceinline__ void mix_row(float (&acc)[MT][4][4], const bf16* mix, int hp, int nq, int lane, int live, const float (&L)[MT][4], Load load) {
    const int n = lane >> 2, c = lane & 3;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[m][e][k] = 0.f;
#pragma unroll
    for (int t = 0; t < MT; ++t) {
        float p[4][4];                                       // [head of the lane][key e]
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const int g = mix_head(t, k, c);
            float4 s = make_float4(-INFINITY, -INFINITY, -INFINITY, -INFINITY);
            if (g < nq) s = load(g);
            p[k][0] = fast_exp2(s.x - L[t][k]); p[k][1] = fast_exp2(s.y - L[t][k]);
            p[k][2] = fast_exp2(s.z - L[t][k]); p[k][3] = fast_exp2(s.w - L[t][k]);
        }
        if (live < 32) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
#pragma unroll
                for (int e = 0; e < 4; ++e) if (4 * n + e >= live) p[k][e] = 0.f;
        }
        uint32_t b0[4][3], b1[4][3];
#pragma unroll
        for (int e = 0; e < 4; ++e) { split3(p[0][e], p[1][e], b0[e]); split3(p[2][e], p[3][e], b1[e]); }
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            uint32_t a[4];
            const bf16* w = mix + (size_t)(m * 16 + n) * hp + t * 16 + 2 * c;
            a[0] = *reinterpret_cast<const uint32_t*>(w);     a[1] = *reinterpret_cast<const uint32_t*>(w + 8 * hp);
            a[2] = *reinterpret_cast<const uint32_t*>(w + 8); a[3] = *reinterpret_cast<const uint32_t*>(w + 8 * hp + 8);
#pragma unroll
            for (int e = 0; e < 4; ++e)
#pragma unroll
                for (int k = 2; k >= 0; --k) mma16816(acc[m][e], a, b0[e][k], b1[e][k]);       // the small parts first
        }
    }
}

// L of every (row, head) of the row tiles from its runs, in their order.
__global__ void __launch_bounds__(256) mix_lse_kernel(const MixArgs A) {
    const int4 tl = A.tiles[blockIdx.x];
    const int qs = A.q_start[tl.x], qlen = A.q_start[tl.x + 1] - qs, np = (tl.w + part_tiles(tl.w) - 1) / part_tiles(tl.w);
    for (int i = blockIdx.y * 256 + threadIdx.x; i < BM * A.nq; i += gridDim.y * 256) {
        const int R = tl.y * BM + i / A.nq;
        if (R >= qlen) return;
        const size_t at = (size_t)(qs + R) * A.nq + i % A.nq;
        float m = -INFINITY, l = 0.f;
        for (int p = 0; p < np; ++p) {                       // a run behind the row's position holds (-inf, 0)
            const float2 v = A.part_ml[at * MAX_PARTS + p];
            const float mn = fmaxf(m, v.x), u = mn == -INFINITY ? 0.f : mn;
            l = l * fast_exp2(m - u) + v.y * fast_exp2(v.x - u);
            m = mn;
        }
        A.lse[at] = m + log2f(l);
    }
}

// A block takes MIX_GROUPS groups of four rows of a unit; the group's scores of all heads come as one 1 KB bulk copy a head, three
// groups ahead; a warp mixes half a row.  A head's place is 16 bytes longer than its data, so that the four heads a quarter of a
// warp reads together lie in different banks.
constexpr int MIX_ROWS = 4, MIX_GROUPS = 8, MIX_STAGES = 3, MIX_PLANE = MIX_ROWS * BN * 4 + 16;
template <int MT>
__global__ void __launch_bounds__(256, MT == 1 ? 3 : MT == 2 ? 2 : 1) mix_weights_kernel(const MixArgs A) {
    extern __shared__ __align__(16) unsigned char msm[];
    __shared__ uint64_t bar[MIX_STAGES];
    __shared__ int abort_shared;
    volatile int* abort_flag = &abort_shared;
    const int unit = A.n_units - 1 - blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int4 tl = A.tiles[A.unit_tile[unit]];
    const int b = tl.x, key0 = (unit - tl.z) * BN, r0 = blockIdx.y * (MIX_ROWS * MIX_GROUPS);
    const int qs = A.q_start[b], qlen = A.q_start[b + 1] - qs, sp = A.start_pos[b];
    const int n = lane >> 2, c = lane & 3, row_in = warp >> 1, half = warp & 1;
    const int rows = min(MIX_ROWS * MIX_GROUPS, qlen - tl.y * BM - r0), groups = rows > 0 ? (rows + MIX_ROWS - 1) / MIX_ROWS : 0;
    const uint32_t stage_bytes = (uint32_t)A.nq * MIX_PLANE;
    const float* src = A.scores + (size_t)unit * A.nq * (BM * BN) + r0 * BN;
    auto fetch = [&](int gq) {                               // by warp 0: group gq's rows of every head
        uint64_t* br = bar + gq % MIX_STAGES;
        if (lane == 0) mbar_expect_tx(br, (uint32_t)A.nq * (MIX_ROWS * BN * 4));
        __syncwarp();
        for (int h = lane; h < A.nq; h += 32)
            bulk_load(smem_addr(msm) + (gq % MIX_STAGES) * stage_bytes + h * MIX_PLANE, src + (size_t)h * (BM * BN) + gq * (MIX_ROWS * BN), MIX_ROWS * BN * 4, br);
    };
    if (threadIdx.x == 0) {
        for (int i = 0; i < MIX_STAGES; ++i) mbar_init(bar + i, 1);
        abort_shared = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    if (warp == 0)
        for (int gq = 0; gq < MIX_STAGES && gq < groups; ++gq) fetch(gq);
    bool ok = true;
    float L[MT][4], L_next[MT][4];                           // the next group's while this one is worked on
    auto fetch_lse = [&](int gq) {
        const int R = tl.y * BM + r0 + gq * MIX_ROWS + row_in;
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int g = mix_head(t, k, c);
                L_next[t][k] = g < A.nq && R < qlen ? A.lse[(size_t)(qs + R) * A.nq + g] : 0.f;
            }
    };
    fetch_lse(0);
#pragma unroll 1
    for (int gq = 0; gq < MIX_GROUPS; ++gq) {
        const int r = r0 + gq * MIX_ROWS + row_in, R = tl.y * BM + r;
        const int live = R < qlen ? sp + R - (key0 + half * 32) + 1 : 0;             // keys of this half that the row sees
        float acc[MT][4][4];
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
            for (int k = 0; k < 4; ++k) L[t][k] = L_next[t][k];
        if (gq + 1 < groups) fetch_lse(gq + 1);
        if (gq < groups && ok) ok = __all_sync(0xffffffffu, mbar_wait(bar + gq % MIX_STAGES, (gq / MIX_STAGES) & 1, abort_flag, A.status, 51));
        if (live > 0 && ok) {
            const unsigned char* st = msm + (size_t)(gq % MIX_STAGES) * stage_bytes + row_in * (BN * 4) + (((half * 8 + n) ^ (r & 7)) << 4);
            mix_row<MT>(acc, A.mix, A.hp, A.nq, lane, live, L, [&](int g) { return *reinterpret_cast<const float4*>(st + (size_t)g * MIX_PLANE); });
        } else {
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int e = 0; e < 4; ++e)
#pragma unroll
                    for (int q = 0; q < 4; ++q) acc[m][e][q] = 0.f;
        }
        bf16* dst = A.mixed + (size_t)unit * A.nq * (BM * BN) + r * BN + (((half * 4 + c) ^ (r & 7)) << 3);
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int h = m * 16 + u * 8 + n;
                if (h < A.nq) {
                    uint4 v;
                    v.x = pack_bf16(acc[m][0][2 * u], acc[m][1][2 * u]);         v.y = pack_bf16(acc[m][2][2 * u], acc[m][3][2 * u]);
                    v.z = pack_bf16(acc[m][0][2 * u + 1], acc[m][1][2 * u + 1]); v.w = pack_bf16(acc[m][2][2 * u + 1], acc[m][3][2 * u + 1]);
                    *reinterpret_cast<uint4*>(dst + (size_t)h * (BM * BN)) = v;
                }
            }
        if (gq + MIX_STAGES < groups) {                      // uniform over the block: the stage has been read by every warp
            __syncthreads();
            if (warp == 0) fetch(gq + MIX_STAGES);
        }
    }
    // a block that gave up on a wait leaves only when its own copies have had their (bounded) time
    if (!ok) {
        const long long t0 = clock64();
        while (clock64() - t0 < 2000000LL) { }
    }
}

// ------------------------------------------------------------------------------------------------ prompts: values
// Warps 0..3: V by asynchronous copies (pages under 8 tokens), then the epilogue (one row a thread); warp 4: MMA issue; warp 5: P'
// tiles by bulk copies and V by TMA.
constexpr int V_STAGES = D <= 128 ? 3 : 2;                    // two blocks an SM (one block of six stages was slower)
constexpr int V_THREADS = 192;
constexpr int SV_TILES = V_STAGES * (P_BYTES + K_BYTES);
constexpr int SV_SMEM = SV_TILES + 1024 + 256;
static_assert(SV_SMEM <= 227 * 1024 && V_STAGES <= 8, "shared memory");

template <bool TMA>
__global__ void __launch_bounds__(V_THREADS, 2) mix_values_kernel(const __grid_constant__ CUtensorMap map_v, const MixArgs A) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const uint32_t sP = smem_addr(base), sV = sP + V_STAGES * P_BYTES;
    uint64_t* bars = reinterpret_cast<uint64_t*>(base + SV_TILES);
    uint64_t* bar_p = bars;              // [stage] P' has landed (bytes)
    uint64_t* bar_v = bars + 8;          // [stage] V has landed
    uint64_t* bar_free = bars + 16;      // [stage] the product that read the stage is complete (commit)
    uint64_t* bar_o = bars + 24;         // O is complete
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 25);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x % A.nq, kh = h / (A.nq / A.nkv);
    const int4 tl = A.tiles[blockIdx.x / A.nq];
    const int b = tl.x, row0 = tl.y * BM, n_kt = tl.w;
    const int qs = A.q_start[b], qlen = A.q_start[b + 1] - qs, sp = A.start_pos[b];
    const int pos_hi = sp + min(row0 + BM, qlen) - 1;
    const int* tab = A.table + (size_t)tl_checked(A.slots[b], A.lim.table_rows, A.lim, TL_K_TC_PREFILL) * A.max_pages;
    tl_checked(pos_hi / A.page_size, A.max_pages, A.lim, TL_K_TC_PREFILL);

    if (tid == 0) {
        for (int i = 0; i < V_STAGES; ++i) { mbar_init(bar_p + i, 1); mbar_init(bar_v + i, BM); mbar_init(bar_free + i, 1); }
        mbar_init(bar_o, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 4) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(tmem_slot)), "r"(O_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;

    if (warp < 4) {
        const int ps_shift = shift_of(A.page_size);
        const size_t page_stride = (size_t)A.nkv * A.page_size * D;
        const bf16* pages = A.v_pages + (size_t)kh * A.page_size * D;
        bool ok = true;
        for (int j = 0; !TMA && j < n_kt && ok; ++j) {       // tile j is on its way while tile j - 1 is waited for
            const int st = j % V_STAGES;
            if (j >= V_STAGES) ok = mbar_wait(bar_free + st, (j / V_STAGES - 1) & 1, abort_flag, A.status, 46, true);
            if (!ok) break;
            copy_keys<BM>(sV + st * K_BYTES, pages, tab, ps_shift, page_stride, j * BN, pos_hi, tid, A.lim);
            asm volatile("cp.async.commit_group;" ::: "memory");
            if (j >= 1) {
                asm volatile("cp.async.wait_group 1;" ::: "memory");
                fence_async_proxy();
                mbar_arrive(bar_v + (j - 1) % V_STAGES);
            }
        }
        if (!TMA) {
            cp_async_wait_all();
            fence_async_proxy();
            if (ok) mbar_arrive(bar_v + (n_kt - 1) % V_STAGES);
        }
        if (ok) ok = mbar_wait(bar_o, 0, abort_flag, A.status, 47, true);
        if (__all_sync(0xffffffffu, ok)) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int R = row0 + tid;
            bf16* dst = R < qlen ? A.out + ((size_t)(qs + R) * A.nq + h) * D : nullptr;
            const uint32_t lane_addr = tmem + ((uint32_t)(warp * 32) << 16);
#pragma unroll 1
            for (int c0 = 0; c0 < D; c0 += 32) {
                float o[32];
                tmem_ld32(lane_addr + c0, o);
                tmem_ld_wait();
                if (dst) {
#pragma unroll
                    for (int c = 0; c < 32; c += 8) {
                        uint4 v;
                        v.x = pack_bf16(o[c], o[c + 1]); v.y = pack_bf16(o[c + 2], o[c + 3]);
                        v.z = pack_bf16(o[c + 4], o[c + 5]); v.w = pack_bf16(o[c + 6], o[c + 7]);
                        *reinterpret_cast<uint4*>(dst + c0 + c) = v;
                    }
                }
            }
        }
    } else if (warp == 4) {
        if (lane == 0) {
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(D >> 3) << 17) | ((uint32_t)(BM >> 4) << 24);
            bool ok = true;
            for (int j = 0; j < n_kt && ok; ++j) {
                const int st = j % V_STAGES, ph = (j / V_STAGES) & 1;
                ok = mbar_wait(bar_p + st, ph, abort_flag, A.status, 48, true) && (TMA || mbar_wait(bar_v + st, ph, abort_flag, A.status, 49, true));
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
                for (int k = 0; k < BN / 16; ++k)
                    umma(tmem, desc_kmajor(sP + st * P_BYTES + k * 32), desc_mnmajor(sV + st * K_BYTES + k * 16 * 128, BN * 128), idesc,
                         (j > 0 || k > 0) ? 1u : 0u);
                umma_commit(bar_free + st);
            }
            if (ok) umma_commit(bar_o);
        }
    } else {
        if (lane == 0) {
            bool ok = true;
            int issued = 0;
            const int ps_shift = shift_of(A.page_size);
            if (TMA) asm volatile("prefetch.tensormap [%0];" ::"l"(&map_v) : "memory");
            for (int j = 0; j < n_kt && ok; ++j) {
                const int st = j % V_STAGES;
                int page[8];
                if (TMA) pages_of(page, tab, A.max_pages, ps_shift, j * BN, A.lim);
                if (j >= V_STAGES) ok = mbar_wait(bar_free + st, (j / V_STAGES - 1) & 1, abort_flag, A.status, 50, true);
                if (!ok) break;
                mbar_expect_tx(bar_p + st, P_BYTES + (TMA ? K_BYTES : 0));
                if (TMA) fetch_keys(sV + st * K_BYTES, &map_v, bar_p + st, page, ps_shift, A.nkv, kh);
                bulk_load(sP + st * P_BYTES, A.mixed + ((size_t)(tl.z + j) * A.nq + h) * (BM * BN), P_BYTES, bar_p + st);
                issued = j + 1;
            }
            // a block that gives up waits (bounded) for its own copies before it leaves
            if (!ok) {
                for (int j = max(0, issued - V_STAGES); j < issued; ++j) {
                    const long long t0 = clock64();
                    while (!mbar_try_wait(bar_p + j % V_STAGES, (j / V_STAGES) & 1) && clock64() - t0 < 2000000LL) { }
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (*abort_flag) {
        const long long t0 = clock64();
        while (clock64() - t0 < 2000000LL) { }
    }
    if (warp == 4) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(O_COLS) : "memory");
    }
}

// ------------------------------------------------------------------------------------------------ decoding
struct MixDecodeArgs {
    const bf16* q; int q_stride;
    bf16* out;
    const bf16* k_pages; const bf16* v_pages;
    const int* table; int max_pages; int page_size;
    const int* rows; const int* start_pos; const int* slots;     // per request: its row in q and out, its position, its slot
    int nq, nkv;
    float scale_log2;
    int range, splits;                   // keys a block (a multiple of 64), ranges
    float* scores;                       // [n][nq][splits * range]
    float* ml;                           // [n][splits][nq][2]
    float* part;                         // [n][splits][nq][D]; one range: unused
    const bf16* mix; int hp;
    int units, gc;                       // mix and values: 16-byte pieces of the KV heads' rows a block, heads of a group a block
    TlLimits lim;
};

constexpr int MIX_MAX_RANGE = 512;
// The page numbers of keys [k_lo, k_hi) into shared memory, by `parts` threads.
__device__ __forceinline__ void range_pages(int* page_of, const int* tab, int max_pages, int ps_shift, int k_lo, int k_hi, int part, int parts,
                                            const TlLimits& L) {
    const int first = k_lo >> ps_shift, last = (k_hi - 1) >> ps_shift;
    for (int i = part; i <= last - first; i += parts)
        page_of[i] = tl_checked(tab[tl_checked(first + i, max_pages, L, TL_K_DECODE)], L.total_pages, L, TL_K_DECODE);
}

// grid (ranges, KV heads x tiles of 16 heads of the group, requests), 4 warps; a warp takes 16 keys at a time.  The lanes of
// a quad hold a key's row in 16-byte pieces, and Q in the same order of dimensions, so K goes from memory to the product.
__global__ void __launch_bounds__(128) mix_decode_scores_kernel(const MixDecodeArgs A) {
    __shared__ float sm_m[4][16], sm_l[4][16];
    grid_dependency_wait();
    grid_dependency_trigger();
    const int n = blockIdx.z, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = A.nq / A.nkv, gt = (g + 15) / 16, kh = blockIdx.y / gt, h0 = kh * g + (blockIdx.y % gt) * 16, hn = min(16, (kh + 1) * g - h0);
    const int p = A.start_pos[n], k_lo = blockIdx.x * A.range, k_hi = min(k_lo + A.range, p + 1);
    if (k_lo > p) return;
    const int r = lane >> 2, c = lane & 3, ps_shift = shift_of(A.page_size), ps_mask = A.page_size - 1;
    const int* tab = A.table + (size_t)tl_checked(A.slots[n], A.lim.table_rows, A.lim, TL_K_DECODE) * A.max_pages;
    const bf16* pages = A.k_pages + (size_t)kh * A.page_size * D;
    const size_t page_stride = (size_t)A.nkv * A.page_size * D;
    __shared__ int page_of[MIX_MAX_RANGE];
    range_pages(page_of, tab, A.max_pages, ps_shift, k_lo, k_hi, threadIdx.x, 128, A.lim);
    __syncthreads();
    uint4 qa[D / 32], qb[D / 32];
    {
        const bf16* q = A.q + (size_t)A.rows[n] * A.q_stride + (size_t)h0 * D + 8 * c;
#pragma unroll
        for (int s = 0; s < D / 32; ++s) {
            qa[s] = r < hn ? *reinterpret_cast<const uint4*>(q + (size_t)r * D + 32 * s) : make_uint4(0, 0, 0, 0);
            qb[s] = r + 8 < hn ? *reinterpret_cast<const uint4*>(q + (size_t)(r + 8) * D + 32 * s) : make_uint4(0, 0, 0, 0);
        }
    }
    const size_t span = (size_t)A.splits * A.range;
    float* out = A.scores + ((size_t)n * A.nq + h0) * span;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    for (int k0 = k_lo + warp * 16; k0 < k_hi; k0 += 64) {
        uint4 kv[2][D / 32];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int j = k0 + u * 8 + r;
            const bool live = j <= p;
            const int page = live ? page_of[(j >> ps_shift) - (k_lo >> ps_shift)] : 0;
            const bf16* src = pages + (size_t)page * page_stride + (size_t)(j & ps_mask) * D + 8 * c;
#pragma unroll
            for (int s = 0; s < D / 32; ++s) kv[u][s] = live ? *reinterpret_cast<const uint4*>(src + 32 * s) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            float d[4] = {0.f, 0.f, 0.f, 0.f}, d1[4] = {0.f, 0.f, 0.f, 0.f};          // two chains
#pragma unroll
            for (int s = 0; s < D / 32; ++s) {
                const uint32_t a0[4] = {qa[s].x, qb[s].x, qa[s].y, qb[s].y}, a1[4] = {qa[s].z, qb[s].z, qa[s].w, qb[s].w};
                mma16816(d, a0, kv[u][s].x, kv[u][s].y);
                mma16816(d1, a1, kv[u][s].z, kv[u][s].w);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) d[e] += d1[e];
            const int j = k0 + u * 8 + 2 * c;
#pragma unroll
            for (int e = 0; e < 4; ++e) d[e] = j + (e & 1) <= p ? d[e] * A.scale_log2 : -INFINITY;
            if (r < hn) *reinterpret_cast<float2*>(out + (size_t)r * span + j) = make_float2(d[0], d[1]);
            if (r + 8 < hn) *reinterpret_cast<float2*>(out + (size_t)(r + 8) * span + j) = make_float2(d[2], d[3]);
            const float n0 = fmaxf(m0, fmaxf(d[0], d[1])), n1 = fmaxf(m1, fmaxf(d[2], d[3]));
            const float u0 = n0 == -INFINITY ? 0.f : n0, u1 = n1 == -INFINITY ? 0.f : n1;
            l0 = l0 * fast_exp2(m0 - u0) + fast_exp2(d[0] - u0) + fast_exp2(d[1] - u0);
            l1 = l1 * fast_exp2(m1 - u1) + fast_exp2(d[2] - u1) + fast_exp2(d[3] - u1);
            m0 = n0; m1 = n1;
        }
    }
    auto join = [](float& m, float& l, float mo, float lo) {
        const float mn = fmaxf(m, mo), u = mn == -INFINITY ? 0.f : mn;
        l = l * fast_exp2(m - u) + lo * fast_exp2(mo - u);
        m = mn;
    };
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
        join(m0, l0, __shfl_xor_sync(0xffffffffu, m0, o), __shfl_xor_sync(0xffffffffu, l0, o));
        join(m1, l1, __shfl_xor_sync(0xffffffffu, m1, o), __shfl_xor_sync(0xffffffffu, l1, o));
    }
    if (c == 0) { sm_m[warp][r] = m0; sm_l[warp][r] = l0; sm_m[warp][r + 8] = m1; sm_l[warp][r + 8] = l1; }
    __syncthreads();
    if (threadIdx.x < hn) {
        float m = -INFINITY, l = 0.f;
        for (int w = 0; w < 4; ++w) join(m, l, sm_m[w][threadIdx.x], sm_l[w][threadIdx.x]);
        *reinterpret_cast<float2*>(A.ml + (((size_t)n * A.splits + blockIdx.x) * A.nq + h0 + threadIdx.x) * 2) = make_float2(m, l);
    }
}

// grid (ranges, requests, unit groups x group chunks), 256 threads.  The range's P' for all heads into shared memory (a warp a
// run of 32 keys), then a thread owns one 16-byte piece of one KV head's values for GC heads of its group and every KS-th key.
template <int MT, int GC>
__global__ void __launch_bounds__(256) mix_decode_values_kernel(const MixDecodeArgs A) {
    extern __shared__ float dsm[];
    const int n = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, tid = threadIdx.x;
    float* lse = dsm;                                        // [nq]
    float* pm = dsm + ((A.nq + 3) & ~3);                     // [nq][range + 4]; later the key slots' shares
    const int pstride = A.range + 4;
    grid_dependency_wait();
    grid_dependency_trigger();
    const int p = A.start_pos[n], k_lo = blockIdx.x * A.range, k_hi = min(k_lo + A.range, p + 1), keys = k_hi - k_lo;
    if (k_lo > p) return;
    const int used = p / A.range + 1;                        // ranges that hold keys
    const int g = A.nq / A.nkv, all_units = A.nkv * CH, chunks = (g + GC - 1) / GC;
    const int u0 = (blockIdx.z / chunks) * A.units, gi0 = (blockIdx.z % chunks) * GC, un = min(A.units, all_units - u0);
    // this thread's piece of the values and its first keys, on their way while the weights are made
    const int ks_n = 256 / un, ks = tid / un, unit = u0 + tid - ks * un, kh = unit / CH, piece = unit - kh * CH;
    const bool live = ks < ks_n;
    const int ps_shift = shift_of(A.page_size), ps_mask = A.page_size - 1;
    const int* tab = A.table + (size_t)tl_checked(A.slots[n], A.lim.table_rows, A.lim, TL_K_DECODE) * A.max_pages;
    const bf16* pages = A.v_pages + (size_t)kh * A.page_size * D + piece * 8;
    const size_t page_stride = (size_t)A.nkv * A.page_size * D;
    __shared__ int page_of[MIX_MAX_RANGE];                   // the range's pages
    range_pages(page_of, tab, A.max_pages, ps_shift, k_lo, k_hi, tid, 256, A.lim);
    __syncthreads();
    constexpr int UN = 8;
    uint4 v[UN];
    auto fetch = [&](int k0) {
#pragma unroll
        for (int u = 0; u < UN; ++u) {
            const int k = k0 + u * ks_n, j = k_lo + k;
            v[u] = make_uint4(0, 0, 0, 0);
            if (live && k < keys)
                v[u] = *reinterpret_cast<const uint4*>(pages + (size_t)page_of[(j >> ps_shift) - (k_lo >> ps_shift)] * page_stride + (size_t)(j & ps_mask) * D);
        }
    };
    fetch(ks);
    for (int h = warp; h < A.nq; h += 8) {                   // a warp a head, a lane a range
        float m = -INFINITY, l = 0.f;
        for (int s = lane; s < used; s += 32) {
            const float2 x = *reinterpret_cast<const float2*>(A.ml + (((size_t)n * A.splits + s) * A.nq + h) * 2);
            const float mn = fmaxf(m, x.x);
            l = l * fast_exp2(m - mn) + x.y * fast_exp2(x.x - mn);
            m = mn;
        }
        const float top = warp_max(m);
        l = warp_sum(m == -INFINITY ? 0.f : l * fast_exp2(m - top));
        if (lane == 0) lse[h] = top + log2f(l);
    }
    __syncthreads();
    const size_t span = (size_t)A.splits * A.range;
    for (int k0 = warp * 32; k0 < keys; k0 += 256) {
        const int nr = lane >> 2, c = lane & 3;
        float acc[MT][4][4], L[MT][4];
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
            for (int k = 0; k < 4; ++k) { const int gg = mix_head(t, k, c); L[t][k] = gg < A.nq ? lse[gg] : 0.f; }
        const float* src = A.scores + (size_t)n * A.nq * span + k_lo + k0 + 4 * nr;
        mix_row<MT>(acc, A.mix, A.hp, A.nq, lane, keys - k0, L, [&](int gg) { return *reinterpret_cast<const float4*>(src + (size_t)gg * span); });
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int h = m * 16 + u * 8 + nr;
                if (h < A.nq) {
                    float* dst = pm + (size_t)h * pstride + k0 + 8 * c;
                    *reinterpret_cast<float4*>(dst) = make_float4(acc[m][0][2 * u], acc[m][1][2 * u], acc[m][2][2 * u], acc[m][3][2 * u]);
                    *reinterpret_cast<float4*>(dst + 4) = make_float4(acc[m][0][2 * u + 1], acc[m][1][2 * u + 1], acc[m][2][2 * u + 1], acc[m][3][2 * u + 1]);
                }
            }
    }
    __syncthreads();
    const int gn = min(GC, g - gi0);
    float o[GC][8];
#pragma unroll
    for (int i = 0; i < GC; ++i)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[i][e] = 0.f;
    if (live) {
        const float* pw = pm + (size_t)(kh * g + gi0) * pstride;
        for (int k0 = ks; k0 < keys; k0 += UN * ks_n) {
            if (k0 != ks) fetch(k0);
#pragma unroll
            for (int u = 0; u < UN; ++u) {
                const int k = k0 + u * ks_n;
                if (k < keys) {
                    const __nv_bfloat162* v2 = reinterpret_cast<const __nv_bfloat162*>(&v[u]);
                    float f[8];
#pragma unroll
                    for (int e = 0; e < 4; ++e) { f[2 * e] = __low2float(v2[e]); f[2 * e + 1] = __high2float(v2[e]); }
#pragma unroll
                    for (int i = 0; i < GC; ++i) {
                        if (i < gn) {
                            const float w = pw[(size_t)i * pstride + k];
#pragma unroll
                            for (int e = 0; e < 8; ++e) o[i][e] = fmaf(w, f[e], o[i][e]);
                        }
                    }
                }
            }
        }
    }
    // the key slots' shares, summed in their order; [GC * 8][thread] takes the place of the weights
    __syncthreads();
    if (live) {
#pragma unroll
        for (int i = 0; i < GC; ++i)
#pragma unroll
            for (int e = 0; e < 8; ++e) pm[(i * 8 + e) * 256 + tid] = o[i][e];
    }
    __syncthreads();
    for (int idx = tid; idx < un * GC * 8; idx += 256) {
        const int uu = idx % un, ie = idx / un, i = ie >> 3, e = ie & 7;
        if (i >= gn) continue;
        float v = 0.f;
        for (int s = 0; s < ks_n; ++s) v += pm[ie * 256 + s * un + uu];
        const int k2 = (u0 + uu) / CH, pc = (u0 + uu) - k2 * CH, h = k2 * g + gi0 + i;
        if (A.splits == 1) A.out[((size_t)A.rows[n] * A.nq + h) * D + pc * 8 + e] = __float2bfloat16_rn(v);
        else A.part[(((size_t)n * A.splits + blockIdx.x) * A.nq + h) * D + pc * 8 + e] = v;
    }
}

// grid (pieces of nq * D, requests): the ranges' shares in their order
__global__ void __launch_bounds__(128) mix_decode_sum_kernel(const MixDecodeArgs A) {
    grid_dependency_wait();
    grid_dependency_trigger();
    const int n = blockIdx.y, width = A.nq * D, i = (blockIdx.x * 128 + threadIdx.x) * 4;
    if (i >= width) return;
    const int used = A.start_pos[n] / A.range + 1;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < used; ++s) {
        const float4 x = *reinterpret_cast<const float4*>(A.part + ((size_t)n * A.splits + s) * width + i);
        v.x += x.x; v.y += x.y; v.z += x.z; v.w += x.w;
    }
    uint2 o;
    o.x = pack_bf16(v.x, v.y); o.y = pack_bf16(v.z, v.w);
    *reinterpret_cast<uint2*>(A.out + (size_t)A.rows[n] * width + i) = o;
}

// ------------------------------------------------------------------------------------------------ decoding in a cluster
// One launch for the three above: the blocks of a request form a thread-block cluster, each with an equal run of its keys and all
// heads.  A block scores its run into shared memory; the runs' (m, l) meet through distributed shared memory; the block mixes
// its run in place, applies it to the values and leaves its share of O in shared memory, where the cluster adds the shares up,
// a slice of the columns a block.  grid (cluster size, requests).
constexpr int MC_THREADS = D <= 128 ? 512 : 256;
constexpr int MC_WARPS = MC_THREADS / 32;

struct MixClusterShape { int pstride, pages; };              // floats a head's row of weights, page numbers of a run

__device__ __forceinline__ void mc_barrier() {
    asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ uint32_t mc_peer(const void* p, int rank) {
    uint32_t out;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(out) : "r"(smem_addr(p)), "r"(rank));
    return out;
}
__device__ __forceinline__ float2 mc_load2(uint32_t at) {
    float2 v;
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(at) : "memory");
    return v;
}
__device__ __forceinline__ float4 mc_load4(uint32_t at) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(at) : "memory");
    return v;
}
// floats of shared memory in front of the weights: (m, l) and L of every head; and behind them: O of every slice of the keys
__host__ __device__ __forceinline__ int mc_heads_floats(int nq) { return (3 * nq + 3) & ~3; }
__host__ __device__ __forceinline__ int mc_slices(int nq, int tiles) {
    const int every = tiles < MC_WARPS ? MC_WARPS / tiles : 1, most = nq < 64 ? 64 / nq : 1;
    return every < most ? every : most;
}
__host__ __device__ __forceinline__ int mc_bytes(int nq, int tiles, MixClusterShape S) {
    return 4 * (mc_heads_floats(nq) + nq * S.pstride + mc_slices(nq, tiles) * nq * D + ((S.pages + 3) & ~3));
}

template <int MT>
__global__ void __launch_bounds__(MC_THREADS, 1) mix_decode_cluster_kernel(const MixDecodeArgs A, const MixClusterShape Sh) {
    extern __shared__ __align__(16) float dsm[];
    const int C = gridDim.x, rank = blockIdx.x, n = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* ml = dsm;                                         // [nq][2]
    float* lse = dsm + 2 * A.nq;                             // [nq]
    float* pm = dsm + mc_heads_floats(A.nq);                 // [nq][pstride]  scores, then weights
    float* os = pm + (size_t)A.nq * Sh.pstride;              // [slices][nq][D]
    const int g = A.nq / A.nkv, gt = (g + 15) / 16, nt = A.nkv * gt, slices = mc_slices(A.nq, nt);
    int* page_of = reinterpret_cast<int*>(os + (size_t)slices * A.nq * D);
    grid_dependency_wait();
    grid_dependency_trigger();
    const int p = A.start_pos[n], rng = ((p + C) / C + 31) & ~31, k_lo = rank * rng, k_hi = min(k_lo + rng, p + 1), keys = max(0, k_hi - k_lo);
    const int ps_shift = shift_of(A.page_size), ps_mask = A.page_size - 1;
    const size_t page_stride = (size_t)A.nkv * A.page_size * D, row = A.rows[n];
    if (keys > 0) {
        const int* tab = A.table + (size_t)tl_checked(A.slots[n], A.lim.table_rows, A.lim, TL_K_DECODE) * A.max_pages;
        range_pages(page_of, tab, A.max_pages, ps_shift, k_lo, k_hi, tid, MC_THREADS, A.lim);
    }
    __syncthreads();
    {   // scores: a warp keeps the queries of one tile of heads and takes 16 keys at a time
        const int groups = min(nt, MC_WARPS), every = MC_WARPS / groups, r = lane >> 2, c = lane & 3;
        for (int t = warp % groups; t < nt && warp < groups * every; t += groups) {
            const int kh = t / gt, h0 = kh * g + (t % gt) * 16, hn = min(16, (kh + 1) * g - h0);
            const bf16* pages = A.k_pages + (size_t)kh * A.page_size * D + 8 * c;
            const bf16* q = A.q + row * A.q_stride + (size_t)h0 * D + 8 * c;
            uint4 qa[D / 32], qb[D / 32], kv[2][D / 32];
#pragma unroll
            for (int s = 0; s < D / 32; ++s) {
                qa[s] = r < hn ? *reinterpret_cast<const uint4*>(q + (size_t)r * D + 32 * s) : make_uint4(0, 0, 0, 0);
                qb[s] = r + 8 < hn ? *reinterpret_cast<const uint4*>(q + (size_t)(r + 8) * D + 32 * s) : make_uint4(0, 0, 0, 0);
            }
            for (int k0 = warp / groups * 16; k0 < keys; k0 += every * 16) {
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int k = k0 + u * 8 + r, j = k_lo + k;
                    const bf16* src = pages + (size_t)(k < keys ? page_of[(j >> ps_shift) - (k_lo >> ps_shift)] : 0) * page_stride + (size_t)(j & ps_mask) * D;
#pragma unroll
                    for (int s = 0; s < D / 32; ++s) kv[u][s] = k < keys ? *reinterpret_cast<const uint4*>(src + 32 * s) : make_uint4(0, 0, 0, 0);
                }
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    float d[4] = {0.f, 0.f, 0.f, 0.f}, d1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                    for (int s = 0; s < D / 32; ++s) {
                        const uint32_t a0[4] = {qa[s].x, qb[s].x, qa[s].y, qb[s].y}, a1[4] = {qa[s].z, qb[s].z, qa[s].w, qb[s].w};
                        mma16816(d, a0, kv[u][s].x, kv[u][s].y);
                        mma16816(d1, a1, kv[u][s].z, kv[u][s].w);
                    }
                    const int k = k0 + u * 8 + 2 * c;
#pragma unroll
                    for (int e = 0; e < 4; ++e) d[e] = k + (e & 1) < keys ? (d[e] + d1[e]) * A.scale_log2 : -INFINITY;
                    if (r < hn) *reinterpret_cast<float2*>(pm + (size_t)(h0 + r) * Sh.pstride + k) = make_float2(d[0], d[1]);
                    if (r + 8 < hn) *reinterpret_cast<float2*>(pm + (size_t)(h0 + r + 8) * Sh.pstride + k) = make_float2(d[2], d[3]);
                }
            }
        }
    }
    __syncthreads();
    for (int h = warp; h < A.nq; h += MC_WARPS) {            // the run's maximum and sum, a warp a head
        float m = -INFINITY, l = 0.f;
        for (int k = lane; k < keys; k += 32) m = fmaxf(m, pm[(size_t)h * Sh.pstride + k]);
        m = warp_max(m);
        for (int k = lane; k < keys; k += 32) l += fast_exp2(pm[(size_t)h * Sh.pstride + k] - m);
        l = warp_sum(l);
        if (lane == 0) { ml[2 * h] = m; ml[2 * h + 1] = l; }
    }
    mc_barrier();
    for (int h = warp; h < A.nq; h += MC_WARPS) {            // over all runs, a lane a run
        float2 x = make_float2(-INFINITY, 0.f);
        if (lane < C) x = mc_load2(mc_peer(ml + 2 * h, lane));
        const float top = warp_max(x.x);
        const float l = warp_sum(x.x == -INFINITY ? 0.f : x.y * fast_exp2(x.x - top));
        if (lane == 0) lse[h] = top + log2f(l);
    }
    __syncthreads();
    for (int k0 = warp * 32; k0 < keys; k0 += MC_THREADS) {  // the mix, 32 keys a warp, in place: nobody else touches these keys
        const int nr = lane >> 2, c = lane & 3;
        float acc[MT][4][4], L[MT][4];
#pragma unroll
        for (int t = 0; t < MT; ++t)
#pragma unroll
            for (int k = 0; k < 4; ++k) { const int gg = mix_head(t, k, c); L[t][k] = gg < A.nq ? lse[gg] : 0.f; }
        mix_row<MT>(acc, A.mix, A.hp, A.nq, lane, keys - k0, L,
                    [&](int gg) { return *reinterpret_cast<const float4*>(pm + (size_t)gg * Sh.pstride + k0 + 4 * nr); });
        __syncwarp();
        // P' rounded for the product with the values: a row's 32 keys as packed pairs in the first half of their 32 floats
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int h = m * 16 + u * 8 + nr;
                if (h < A.nq) {
                    uint4 v;
                    v.x = pack_bf16(acc[m][0][2 * u], acc[m][1][2 * u]);         v.y = pack_bf16(acc[m][2][2 * u], acc[m][3][2 * u]);
                    v.z = pack_bf16(acc[m][0][2 * u + 1], acc[m][1][2 * u + 1]); v.w = pack_bf16(acc[m][2][2 * u + 1], acc[m][3][2 * u + 1]);
                    *reinterpret_cast<uint4*>(pm + (size_t)h * Sh.pstride + k0 + 4 * c) = v;
                }
            }
    }
    __syncthreads();
    {   // values: a warp takes one tile of heads and every slices-th 16 keys.  Lane (r, c) fetches 16-byte pieces of the rows of keys
        // 2c, 2c + 1, 2c + 8, 2c + 9, dimensions 64 s + 8 r ..; product i of a piece takes dimension 64 s + 8 n + i as its column n
        const int groups = min(nt, MC_WARPS / slices), r = lane >> 2, c = lane & 3, slice = warp / groups;
        for (int t = warp % groups; t < nt && slice < slices; t += groups) {
            const int kh = t / gt, h0 = kh * g + (t % gt) * 16, hn = min(16, (kh + 1) * g - h0);
            const bf16* pages = A.v_pages + (size_t)kh * A.page_size * D + 8 * r;
            float o[D / 8][4];
#pragma unroll
            for (int i = 0; i < D / 8; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
            for (int k0 = slice * 16; k0 < keys; k0 += slices * 16) {
                uint4 v[4][D / 64];
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const int k = k0 + 2 * c + (q & 1) + (q >> 1) * 8, j = k_lo + k;
                    const bf16* src = pages + (size_t)(k < keys ? page_of[(j >> ps_shift) - (k_lo >> ps_shift)] : 0) * page_stride + (size_t)(j & ps_mask) * D;
#pragma unroll
                    for (int s = 0; s < D / 64; ++s) v[q][s] = k < keys ? *reinterpret_cast<const uint4*>(src + 64 * s) : make_uint4(0, 0, 0, 0);
                }
                uint32_t a[4];
                const float* w = pm + (size_t)(h0 + r) * Sh.pstride + (k0 & ~31) + ((k0 & 31) >> 1) + c;
                a[0] = r < hn ? __float_as_uint(w[0]) : 0u;     a[1] = r + 8 < hn ? __float_as_uint(w[8 * (size_t)Sh.pstride]) : 0u;
                a[2] = r < hn ? __float_as_uint(w[4]) : 0u;     a[3] = r + 8 < hn ? __float_as_uint(w[8 * (size_t)Sh.pstride + 4]) : 0u;
#pragma unroll
                for (int s = 0; s < D / 64; ++s) {
                    const uint32_t x[4][4] = {{v[0][s].x, v[0][s].y, v[0][s].z, v[0][s].w}, {v[1][s].x, v[1][s].y, v[1][s].z, v[1][s].w},
                                              {v[2][s].x, v[2][s].y, v[2][s].z, v[2][s].w}, {v[3][s].x, v[3][s].y, v[3][s].z, v[3][s].w}};
#pragma unroll
                    for (int i = 0; i < 8; ++i)
                        mma16816(o[s * 8 + i], a, __byte_perm(x[0][i >> 1], x[1][i >> 1], i & 1 ? 0x7632 : 0x5410),
                                 __byte_perm(x[2][i >> 1], x[3][i >> 1], i & 1 ? 0x7632 : 0x5410));
                }
            }
#pragma unroll
            for (int s = 0; s < D / 64; ++s)
#pragma unroll
                for (int i = 0; i < 8; ++i)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int hr = r + (e >> 1) * 8;
                        if (hr < hn) os[((size_t)slice * A.nq + h0 + hr) * D + 64 * s + 8 * (2 * c + (e & 1)) + i] = o[s * 8 + i][e];
                    }
        }
    }
    __syncthreads();
    for (int i = tid; slices > 1 && i < A.nq * D; i += MC_THREADS) {
        float x = os[i];
        for (int s = 1; s < slices; ++s) x += os[(size_t)s * A.nq * D + i];
        os[i] = x;
    }
    mc_barrier();
    const int width = A.nq * D, slice = ((width + C - 1) / C + 3) & ~3;
    for (int i = rank * slice + 4 * tid; i < min(width, (rank + 1) * slice); i += 4 * MC_THREADS) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        float4 x[16];                                        // every block's share on its way before the first addition
#pragma unroll
        for (int s = 0; s < 16; ++s) if (s < C) x[s] = mc_load4(mc_peer(os + i, s));
#pragma unroll
        for (int s = 0; s < 16; ++s) if (s < C) { v.x += x[s].x; v.y += x[s].y; v.z += x[s].z; v.w += x[s].w; }
        uint2 o;
        o.x = pack_bf16(v.x, v.y); o.y = pack_bf16(v.z, v.w);
        *reinterpret_cast<uint2*>(A.out + row * width + i) = o;
    }
    mc_barrier();                                            // nobody leaves while its shared memory is still read
}

template <typename K>
int raise_smem(K kernel, int bytes, bool (&done)[TL_MAX_DEVICES]) {
    const int dev = tl_device_index();
    if (dev < 0) return 1;
    if (!done[dev]) {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
        if (e != cudaSuccess) return (int)e;
        done[dev] = true;
    }
    return 0;
}

}  // namespace

template <int MT>
static int launch_mix(const MixArgs& A, cudaStream_t stream) {
    const int most = MIX_STAGES * 16 * MT * MIX_PLANE, smem = MIX_STAGES * A.nq * MIX_PLANE;
    static bool done[TL_MAX_DEVICES] = {};
    const int e = raise_smem(mix_weights_kernel<MT>, most, done);
    if (e) return e;
    mix_weights_kernel<MT><<<dim3(A.n_units, BM / (MIX_ROWS * MIX_GROUPS)), 256, smem, stream>>>(A);
    return tl_launch_status();
}

// Runs a row tile of n_kt key tiles is cut into.
TL_EXPORT int tl_mix_parts(int n_kt) { return (n_kt + part_tiles(n_kt) - 1) / part_tiles(n_kt); }
TL_EXPORT int tl_mix_max_parts() { return MAX_PARTS; }

// Prompt portions: four launches over `n_tiles` row tiles.  The caller sizes the scratch: scores n_units * nq * 32 KB, mixed
// half of it, part_ml [T, nq, MAX_PARTS, 2], lse [T, nq].  Pages of 2 to 64 tokens, a power of two; up to 64 query heads.
TL_EXPORT int tl_mix_prefill(const void* q, int q_stride, void* out, const void* k_pages, const void* v_pages, const int* table, int max_pages,
                             int page_size, const int* q_start, const int* start_pos, const int* slots, int nq, int nkv, float scale,
                             const int* tiles, int n_tiles, const int* parts, int n_parts, const int* unit_tile, int n_units, float* scores,
                             float* part_ml, float* lse, void* mixed, const void* mix, int hp, int* status, int table_rows, int total_pages,
                             int* fault, cudaStream_t stream) {
    if (n_tiles <= 0) return 0;
    if (nq < 1 || nq > 64 || nq % nkv || hp < nq || hp % 16 || page_size < 2 || page_size > 64 || (page_size & (page_size - 1)) || (q_stride & 7)) return 1;
    const MixArgs A{(const bf16*)q, q_stride, (bf16*)out, (const bf16*)k_pages, (const bf16*)v_pages, table, max_pages, page_size, q_start,
                    start_pos, slots, nq, nkv, scale * 1.4426950408889634f, (const int4*)tiles, n_tiles, (const int2*)parts, n_parts, unit_tile, n_units, scores, (float2*)part_ml, lse,
                    (bf16*)mixed, (const bf16*)mix, hp, status, TlLimits{table_rows, total_pages, fault}};
    static bool done_s[TL_MAX_DEVICES] = {}, done_v[TL_MAX_DEVICES] = {}, done_st[TL_MAX_DEVICES] = {}, done_vt[TL_MAX_DEVICES] = {};
    int e = raise_smem(mix_scores_kernel<false>, SS_SMEM, done_s);
    if (!e) e = raise_smem(mix_scores_kernel<true>, SS_SMEM, done_st);
    if (!e) e = raise_smem(mix_values_kernel<false>, SV_SMEM, done_v);
    if (!e) e = raise_smem(mix_values_kernel<true>, SV_SMEM, done_vt);
    if (e) return e;
    const bool tma = page_size >= 8 && (((uintptr_t)k_pages | (uintptr_t)v_pages) & 127) == 0 && total_pages > 0;
    CUtensorMap mk{}, mv{};
    if (tma) {
        const long long rows = (long long)total_pages * nkv * page_size;
        if ((e = load_encode()) || (e = make_pages_map(&mk, k_pages, rows, D, page_size)) || (e = make_pages_map(&mv, v_pages, rows, D, page_size))) return e;
    }
    if (tma) mix_scores_kernel<true><<<n_parts * nq, S_THREADS, SS_SMEM, stream>>>(mk, A);
    else mix_scores_kernel<false><<<n_parts * nq, S_THREADS, SS_SMEM, stream>>>(mk, A);
    if ((e = tl_launch_status())) return e;
    mix_lse_kernel<<<dim3(n_tiles, (BM * nq + 255) / 256), 256, 0, stream>>>(A);
    if ((e = tl_launch_status())) return e;
    switch ((nq + 15) / 16) {
        case 1: e = launch_mix<1>(A, stream); break;
        case 2: e = launch_mix<2>(A, stream); break;
        case 3: e = launch_mix<3>(A, stream); break;
        default: e = launch_mix<4>(A, stream);
    }
    if (e) return e;
    if (tma) mix_values_kernel<true><<<n_tiles * nq, V_THREADS, SV_SMEM, stream>>>(mv, A);
    else mix_values_kernel<false><<<n_tiles * nq, V_THREADS, SV_SMEM, stream>>>(mv, A);
    return tl_launch_status();
}

template <int MT, int GC>
static int launch_decode_values(const MixDecodeArgs& A, int n, cudaStream_t stream) {
    const int g = A.nq / A.nkv, groups = (A.nkv * CH + A.units - 1) / A.units * ((g + GC - 1) / GC);
    const size_t weights = (size_t)A.nq * (A.range + 4), shares = (size_t)256 * GC * 8;
    const int smem = (int)((((A.nq + 3) & ~3) + (weights > shares ? weights : shares)) * sizeof(float));
    if (smem > 200 * 1024) return 1;
    static bool done[TL_MAX_DEVICES] = {};
    const int e = raise_smem(mix_decode_values_kernel<MT, GC>, 200 * 1024, done);
    if (e) return e;
    return launch_after_wait(mix_decode_values_kernel<MT, GC>, dim3(A.splits, n, groups), dim3(256), smem, stream, A);
}

// Single tokens of n requests.  part: float [n, splits, nq, D] (splits > 1), scores [n, nq, splits * range], ml [n, splits, nq, 2].
TL_EXPORT int tl_mix_decode(const void* q, int q_stride, void* out, const void* k_pages, const void* v_pages, const int* table, int max_pages,
                            int page_size, const int* rows, const int* start_pos, const int* slots, int n, int nq, int nkv, float scale,
                            int range, int splits, float* scores, float* ml, float* part, const void* mix, int hp, int table_rows,
                            int total_pages, int* fault, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (nq < 1 || nq > 64 || nq % nkv || hp < nq || hp % 16 || page_size < 1 || page_size > 64 || (page_size & (page_size - 1)) ||
        (q_stride & 7) || range < 64 || range % 64 || range > MIX_MAX_RANGE || splits < 1 || (splits > 1 && !part) || n > 65535) return 1;
    const int g = nq / nkv, gc = g == 1 ? 1 : g == 2 ? 2 : g <= 4 ? 4 : 8;
    const int units = nkv * CH < 64 ? nkv * CH : 64;
    const MixDecodeArgs A{(const bf16*)q, q_stride, (bf16*)out, (const bf16*)k_pages, (const bf16*)v_pages, table, max_pages, page_size, rows,
                          start_pos, slots, nq, nkv, scale * 1.4426950408889634f, range, splits, scores, ml, part, (const bf16*)mix, hp,
                          units, gc, TlLimits{table_rows, total_pages, fault}};
    int e = launch_after_wait(mix_decode_scores_kernel, dim3(splits, nkv * ((g + 15) / 16), n), dim3(128), 0, stream, A);
    if (e) return e;
#define MDV(MT) (gc == 1 ? launch_decode_values<MT, 1>(A, n, stream) : gc == 2 ? launch_decode_values<MT, 2>(A, n, stream) : \
                 gc == 4 ? launch_decode_values<MT, 4>(A, n, stream) : launch_decode_values<MT, 8>(A, n, stream))
    switch ((nq + 15) / 16) {
        case 1: e = MDV(1); break;
        case 2: e = MDV(2); break;
        case 3: e = MDV(3); break;
        default: e = MDV(4);
    }
#undef MDV
    if (e || splits == 1) return e;
    return launch_after_wait(mix_decode_sum_kernel, dim3((nq * D / 4 + 127) / 128, n), dim3(128), 0, stream, A);
}

template <int MT>
static int launch_decode_cluster(const MixDecodeArgs& A, const MixClusterShape& Sh, int n, int clusters, cudaStream_t stream) {
    constexpr int most = 220 * 1024;
    const int g = A.nq / A.nkv, smem = mc_bytes(A.nq, A.nkv * ((g + 15) / 16), Sh);
    if (smem > most) return 2;
    static bool done[TL_MAX_DEVICES] = {}, wide[TL_MAX_DEVICES] = {};
    int e = raise_smem(mix_decode_cluster_kernel<MT>, most, done);
    if (e) return e;
    const int dev = tl_device_index();
    if (clusters > 8 && !wide[dev]) {                        // clusters of 9 to 16 blocks
        const cudaError_t ce = cudaFuncSetAttribute(mix_decode_cluster_kernel<MT>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        if (ce != cudaSuccess) return (int)ce;
        wide[dev] = true;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(clusters, n); cfg.blockDim = dim3(MC_THREADS); cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = (unsigned)clusters; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = tl_dependent_launch_enabled() ? 2 : 1;
    const cudaError_t ce = cudaLaunchKernelEx(&cfg, mix_decode_cluster_kernel<MT>, A, Sh);
    return ce != cudaSuccess ? (int)ce : (int)cudaGetLastError();
}

// The same in one launch: `clusters` (1 to 16) blocks a request form a cluster, none reads more than `most_keys` keys (a multiple of
// 32, clusters * most_keys >= the longest context).  Returns 2 if the weights of that many keys do not fit the shared memory.
TL_EXPORT int tl_mix_decode_cluster(const void* q, int q_stride, void* out, const void* k_pages, const void* v_pages, const int* table,
                                    int max_pages, int page_size, const int* rows, const int* start_pos, const int* slots, int n, int nq,
                                    int nkv, float scale, int clusters, int most_keys, const void* mix, int hp, int table_rows,
                                    int total_pages, int* fault, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (nq < 1 || nq > 64 || nq % nkv || hp < nq || hp % 16 || page_size < 1 || page_size > 64 || (page_size & (page_size - 1)) ||
        (q_stride & 7) || clusters < 1 || clusters > 16 || most_keys < 32 || most_keys % 32 || n > 65535) return 1;
    const MixDecodeArgs A{(const bf16*)q, q_stride, (bf16*)out, (const bf16*)k_pages, (const bf16*)v_pages, table, max_pages, page_size, rows,
                          start_pos, slots, nq, nkv, scale * 1.4426950408889634f, 0, 0, nullptr, nullptr, nullptr, (const bf16*)mix, hp,
                          0, 0, TlLimits{table_rows, total_pages, fault}};
    const MixClusterShape Sh{most_keys + 4, most_keys / page_size + 2};
    switch ((nq + 15) / 16) {
        case 1: return launch_decode_cluster<1>(A, Sh, n, clusters, stream);
        case 2: return launch_decode_cluster<2>(A, Sh, n, clusters, stream);
        case 3: return launch_decode_cluster<3>(A, Sh, n, clusters, stream);
        default: return launch_decode_cluster<4>(A, Sh, n, clusters, stream);
    }
}
