// The recurrence with channel gates (HGRN2) for steps of many tokens: chunks of a request's tokens side by side.
//
//   S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,  o_t = S_t^T q_t       f_t = lower + (1 - lower) sigmoid(x_f + bias), q_t = silu(x_q)
//
// The recurrence is linear in S, so a chunk of CS_L tokens takes a start state S to F S + E with F the product of its gates (per
// row) and E its end state from zero:
//   gates    x_q and x_f in the projection's rows become q and f, once for all that read them
//   local    every chunk but a request's last: E and F, all chunks at once
//   carry    per state element, chunk after chunk: the chunk's start state takes the place of its E
//   outputs  every chunk from its start state, all at once; the last one leaves the request's state in its slot
// All arithmetic is float.  The state in the slots has the layout of the scan kernel of recurrent.cu (R rows in each of IS threads
// a column, slices of 16 columns), so both kernels may take turns on one request.  A request of one chunk reads and writes its
// slot in one block and skips the first two.
//
// A thread owns 8 rows and 4 columns of S: a token costs it 64 operations for the state and 32 for the outputs against five
// 16-byte reads of shared memory.  Rows lie across the lanes; the outputs of four tokens and four columns are summed over the
// lanes together, every step of the exchange halving what a lane still holds.
#include "common.cuh"

constexpr int CS_L = 128;                // tokens a chunk
constexpr int CS_COLS = 16;              // columns a slice of the state's layout

struct ChannelScanArgs {
    float* proj; int stride; int q_off, f_off, v_off; int T;
    const float* lower; const float* bias;
    float* state; long long slot_stride;
    const int* q_start; const int* slots;
    const int4* chunks;                  // (request, number of the chunk, the request's chunks, first chunk of the request in the list)
    const int* carried;                  // first chunks of the requests that have several
    float* carry;                        // [chunks][H * state floats a head]
    float* decay;                        // [chunks][H][DP]
    float* out;
    int H, d, dv, nz;
};

__device__ __forceinline__ float cs_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

// x_q -> silu(x_q), x_f -> f in place; grid (column groups, rows)
__global__ void __launch_bounds__(256) channel_gates_kernel(const ChannelScanArgs A) {
    const int i = blockIdx.x * 256 + threadIdx.x, width = A.H * A.d;
    if (i >= width) return;
    const float lo = A.lower[i], bias = A.bias[i];
    for (int t = blockIdx.y; t < A.T; t += gridDim.y) {
        float* row = A.proj + (size_t)t * A.stride + i;
        const float x = row[A.q_off], z = row[A.f_off];
        row[A.q_off] = x * cs_sigmoid(x);
        row[A.f_off] = fmaf(1.0f - lo, cs_sigmoid(z + bias), lo);
    }
}

__device__ __forceinline__ void cs_copy(float* dst, const float* src, bool four) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if (four) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}

// Shared memory of the chunk kernel: two stages of f, (q,) v.
template <int DP, bool OUT> struct ChannelShape {
    static constexpr int RG = DP / 8, CB = 256 / RG * 4;     // row groups across the lanes, columns a block
    static constexpr int STAGE = DP == 256 ? 8 : 16;         // tokens a stage
    static constexpr int RS = 12;                            // a row group's place: 8 floats and a pad against bank conflicts
    static constexpr int FLOATS = STAGE * ((OUT ? 2 : 1) * RG * RS + CB);
};

// DP: rows a head, padded (32, 64, 128, 256); OUT: outputs, else the local end state.
template <int DP, bool OUT>
__global__ void __launch_bounds__(256, 2) channel_chunk_kernel(const ChannelScanArgs A) {
    using Sh = ChannelShape<DP, OUT>;
    constexpr int RG = Sh::RG, CB = Sh::CB, CS_STAGE = Sh::STAGE, RS = Sh::RS;
    constexpr int R = DP == 32 ? 4 : 8, IS = DP / R, NT = IS * CS_COLS, PB = R * NT;
    extern __shared__ __align__(16) float csm[];
    const int4 ck = A.chunks[blockIdx.x];
    const int b = ck.x, c = ck.y, nc = ck.z;
    if (!OUT && c == nc - 1) return;
    const int h = blockIdx.y, col0 = blockIdx.z * CB;
    const int tid = threadIdx.x, rg = tid % RG, cg = tid / RG;
    const int base = A.q_start[b], t0 = base + c * CS_L, t1 = min(t0 + CS_L, A.q_start[b + 1]);
    const size_t head_floats = (size_t)A.nz * PB;
    float* slot = A.state + (size_t)A.slots[b] * A.slot_stride + h * head_floats;
    float* mine = A.carry + ((size_t)(ck.w + c) * A.H + h) * head_floats;
    auto at = [&](int r, int cc) {                           // row rg * 8 + r, column cg * 4 + cc of this block
        const int row = rg * 8 + r, col = col0 + cg * 4 + cc;
        return ((size_t)(col / CS_COLS) * R + row % R) * NT + (col % CS_COLS) * IS + row / R;
    };
    const bool owns = col0 + cg * 4 < A.nz * CS_COLS;
    float S[8][4], F[8];
    const float* from = nc == 1 ? slot : mine;
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        F[r] = 1.0f;
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) S[r][cc] = OUT && owns ? from[at(r, cc)] : 0.f;
    }
    // a stage's rows on their way into buffer `buf`: f, q, v; rows that do not exist and tokens behind the chunk change nothing
    const bool four = ((A.stride | A.q_off | A.f_off | A.v_off | A.d | A.dv) & 3) == 0 && ((uintptr_t)A.proj & 15) == 0;
    auto fetch = [&](int s0, int buf) {
        float* f_s = csm + buf * Sh::FLOATS;
        float* q_s = f_s + CS_STAGE * RG * RS;
        float* v_s = f_s + (OUT ? 2 : 1) * CS_STAGE * RG * RS;
        const int n = min(CS_STAGE, t1 - s0), w = four ? 4 : 1;
        for (int i = tid * w; i < CS_STAGE * DP; i += 256 * w) {
            const int t = i / DP, e = i - t * DP, place = t * RG * RS + (e >> 3) * RS + (e & 7);
            if (t < n && e < A.d) {
                const float* row = A.proj + (size_t)(s0 + t) * A.stride + h * A.d + e;
                cs_copy(f_s + place, row + A.f_off, four);
                if (OUT) cs_copy(q_s + place, row + A.q_off, four);
            } else {
                for (int k = 0; k < w; ++k) { f_s[place + k] = 1.0f; if (OUT) q_s[place + k] = 0.f; }
            }
        }
        for (int i = tid * w; i < CS_STAGE * CB; i += 256 * w) {
            const int t = i / CB, e = i - t * CB;
            if (t < n && col0 + e < A.dv) cs_copy(v_s + i, A.proj + (size_t)(s0 + t) * A.stride + A.v_off + h * A.dv + col0 + e, four);
            else for (int k = 0; k < w; ++k) v_s[i + k] = 0.f;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (t0 < t1) fetch(t0, 0);
    int buf = 0;
    for (int s0 = t0; s0 < t1; s0 += CS_STAGE, buf ^= 1) {
        const int n = min(CS_STAGE, t1 - s0);
        if (s0 + CS_STAGE < t1) {
            fetch(s0 + CS_STAGE, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const float* f_s = csm + buf * Sh::FLOATS + rg * RS;
        const float* q_s = f_s + CS_STAGE * RG * RS;
        const float* v_s = csm + buf * Sh::FLOATS + (OUT ? 2 : 1) * CS_STAGE * RG * RS + cg * 4;
#pragma unroll 1
        for (int u = 0; u < n; u += 4) {
            float po[16];                                    // [token][column]
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int t = u + k;                         // tokens behind the chunk hold f = 1, q = v = 0
                const float4 v = *reinterpret_cast<const float4*>(v_s + t * CB);
                float f[8], q[8];
                *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(f_s + t * RG * RS);
                *reinterpret_cast<float4*>(f + 4) = *reinterpret_cast<const float4*>(f_s + t * RG * RS + 4);
                if (OUT) {
                    *reinterpret_cast<float4*>(q) = *reinterpret_cast<const float4*>(q_s + t * RG * RS);
                    *reinterpret_cast<float4*>(q + 4) = *reinterpret_cast<const float4*>(q_s + t * RG * RS + 4);
                }
                float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    S[r][0] = fmaf(f[r], S[r][0] - v.x, v.x); S[r][1] = fmaf(f[r], S[r][1] - v.y, v.y);
                    S[r][2] = fmaf(f[r], S[r][2] - v.z, v.z); S[r][3] = fmaf(f[r], S[r][3] - v.w, v.w);
                    if (OUT) { o0 = fmaf(S[r][0], q[r], o0); o1 = fmaf(S[r][1], q[r], o1); o2 = fmaf(S[r][2], q[r], o2); o3 = fmaf(S[r][3], q[r], o3); }
                    else F[r] *= f[r];
                }
                po[k * 4] = o0; po[k * 4 + 1] = o1; po[k * 4 + 2] = o2; po[k * 4 + 3] = o3;
            }
            if (OUT) {
                // halve what a lane holds while the lanes of a row group's set add up: lane bit i picks the upper half at step i
                int first = 0, held = 16;
#pragma unroll
                for (int o = 1; o < RG; o <<= 1) {
                    const bool upper = rg & o;
                    if (held > 1) {
                        held >>= 1;
#pragma unroll
                        for (int i = 0; i < 8; ++i)
                            if (i < held) {
                                const float give = upper ? po[i] : po[i + held], keep = upper ? po[i + held] : po[i];
                                po[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                            }
                        if (upper) first += held;
                    } else po[0] += __shfl_xor_sync(0xffffffffu, po[0], o);
                }
                if (RG <= 16 || rg < 16) {
#pragma unroll
                    for (int i = 0; i < (RG >= 16 ? 1 : 16 / RG); ++i) {
                        const int k = (first + i) >> 2, col = col0 + cg * 4 + ((first + i) & 3);
                        if (u + k < n && col < A.dv) A.out[(size_t)(s0 + u + k) * A.H * A.dv + (size_t)h * A.dv + col] = po[i];
                    }
                }
            }
        }
        __syncthreads();                                     // everyone has read the stage that the next fetch overwrites
    }
    if (OUT) {
        if (c == nc - 1 && owns)
#pragma unroll
            for (int r = 0; r < 8; ++r)
#pragma unroll
                for (int cc = 0; cc < 4; ++cc) slot[at(r, cc)] = S[r][cc];
    } else {
        if (owns)
#pragma unroll
            for (int r = 0; r < 8; ++r)
#pragma unroll
                for (int cc = 0; cc < 4; ++cc) mine[at(r, cc)] = S[r][cc];
        if (cg == 0 && blockIdx.z == 0)
#pragma unroll
            for (int r = 0; r < 8; ++r) A.decay[((size_t)(ck.w + c) * A.H + h) * DP + rg * 8 + r] = F[r];
    }
}

template <int DP>
__global__ void __launch_bounds__(256) channel_carry_kernel(const ChannelScanArgs A) {
    constexpr int R = DP == 32 ? 4 : 8, IS = DP / R, NT = IS * CS_COLS, PB = R * NT;
    const int first = A.carried[blockIdx.y];
    const int4 ck = A.chunks[first];
    const size_t per = (size_t)A.H * A.nz * PB, i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= per) return;
    const int h = (int)(i / ((size_t)A.nz * PB)), in = (int)(i % PB), row = (in % NT) % IS * R + in / NT;
    float* e = A.carry + (size_t)first * per + i;
    const float* f = A.decay + ((size_t)first * A.H + h) * DP + row;
    float S = A.state[(size_t)A.slots[ck.x] * A.slot_stride + i];
    float next = e[0], fn = f[0];
    for (int c = 0; c < ck.z - 1; ++c) {
        const float E = next, Fc = fn;
        if (c + 2 < ck.z) { next = e[(size_t)(c + 1) * per]; fn = f[(size_t)(c + 1) * A.H * DP]; }
        e[(size_t)c * per] = S;
        S = fmaf(Fc, S, E);
    }
    e[(size_t)(ck.z - 1) * per] = S;
}

template <int DP>
static int launch_channel_scan(const ChannelScanArgs& A, int n_chunks, int n_carried, cudaStream_t stream) {
    constexpr int R = DP == 32 ? 4 : 8, PB = R * (DP / R) * CS_COLS, CB = ChannelShape<DP, true>::CB;
    constexpr int smem_out = 2 * ChannelShape<DP, true>::FLOATS * 4, smem_local = 2 * ChannelShape<DP, false>::FLOATS * 4;
    static bool raised[TL_MAX_DEVICES] = {};
    const int dev = tl_device_index();
    if (dev < 0) return 1;
    if (!raised[dev]) {
        cudaError_t e = cudaFuncSetAttribute(channel_chunk_kernel<DP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_out);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(channel_chunk_kernel<DP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_local);
        if (e != cudaSuccess) return (int)e;
        raised[dev] = true;
    }
    const dim3 grid(n_chunks, A.H, (A.dv + CB - 1) / CB);
    int e;
    if (n_carried > 0) {
        channel_chunk_kernel<DP, false><<<grid, 256, smem_local, stream>>>(A);
        if ((e = tl_launch_status())) return e;
        channel_carry_kernel<DP><<<dim3((unsigned)(((size_t)A.H * A.nz * PB + 255) / 256), n_carried), 256, 0, stream>>>(A);
        if ((e = tl_launch_status())) return e;
    }
    channel_chunk_kernel<DP, true><<<grid, 256, smem_out, stream>>>(A);
    return tl_launch_status();
}

TL_EXPORT int tl_channel_chunk() { return CS_L; }

// The gates take the place of x_q and x_f in `proj`.  carry: float [n_chunks, H * state floats a head], decay: float [n_chunks, H, d padded to 32, 64, 128 or 256]; neither is touched
// where no request has several chunks.
TL_EXPORT int tl_channel_scan(float* proj, int T, int stride, int q_off, int f_off, int v_off, const float* lower, const float* bias,
                              float* state, long long slot_stride, const int* q_start, const int* slots, const int* chunks, int n_chunks,
                              const int* carried, int n_carried, float* carry, float* decay, float* out, int H, int d, int dv,
                              cudaStream_t stream) {
    if (n_chunks <= 0 || H <= 0) return 0;
    if (H > 65535 || d < 1 || d > 256 || n_carried > 65535) return 1;
    const ChannelScanArgs A{proj, stride, q_off, f_off, v_off, T, lower, bias, state, slot_stride, q_start, slots, (const int4*)chunks, carried,
                            carry, decay, out, H, d, dv, (dv + CS_COLS - 1) / CS_COLS};
    channel_gates_kernel<<<dim3((H * d + 255) / 256, T < 1024 ? T : 1024), 256, 0, stream>>>(A);
    const int e = tl_launch_status();
    if (e) return e;
    if (d <= 32) return launch_channel_scan<32>(A, n_chunks, n_carried, stream);
    if (d <= 64) return launch_channel_scan<64>(A, n_chunks, n_carried, stream);
    if (d <= 128) return launch_channel_scan<128>(A, n_chunks, n_carried, stream);
    return launch_channel_scan<256>(A, n_chunks, n_carried, stream);
}
