// The state-space recurrence of Mamba-2 (one decay per head and token, input and output vectors shared by a group of
// heads), over a per-request state in float:
//
//     S_t = exp(-exp(A_log_h) dt_t) S_(t-1) + dt_t B_t x_t^T          S [N, vdim] per head, zero before the first token
//     y_t = S_t^T C_t + D_h x_t                                       dt_t = softplus(dt_raw_t + dt_bias_h)
//
// x, B and C are column ranges of one tensor (what a short convolution left, float or bf16), dt_raw a column range of the
// projection; head h uses group h / (heads / groups).  y is float.  Three kernels:
//
//   walk    token by token, any sizes, float or bf16 inputs: a column of S belongs to DG neighbouring threads that keep NR
//           of its rows each in registers (as the retention kernel does);
//   step    spans of one token each (decoding): a block takes one request's head, the state goes through registers once as
//           16-byte pieces;
//   chunks  bf16 inputs, on tensor cores (mma.sync): with L_t the running sum of the log decays inside a chunk of 64
//           tokens and S_0 the state before it,
//               y_t = e^{L_t} S_0^T C_t + sum_{s<=t} (C_t . B_s) e^{L_t - L_s} dt_s x_s + D x_t
//               S_n = e^{L_n} S_0 + sum_s B_s (e^{L_n - L_s} dt_s x_s)^T
//           Every exponent is <= 0.  B, C and x enter the products as the bf16 numbers they are; what is float (the state,
//           the weighted x of the state's update, the weighted scores) enters as the sum of two bf16 numbers, one product
//           each (16 bits of mantissa in the operand, float sums; the state itself is carried in float).
//           A long span is cut into pieces that run side by side: a local pass (every piece but the last from a zero state,
//           leaving its contribution and its decay), a scan over the pieces, and the output pass.
#include <math.h>

#include "common.cuh"
#include "warp_mma.cuh"

namespace {

using namespace wm;

struct SsmParams {
    const void* xbc;            // [T, stride]: x [H, vdim] at x_off, B [G, N] at b_off, C [G, N] at c_off
    long long stride;
    int x_off, b_off, c_off;
    const void* dt;             // [T, dt_stride]: H numbers from column dt_off on, before the bias and the softplus
    long long dt_stride;
    int dt_off, dt_dtype;
    const float* dt_bias;       // [H]
    const float* rate;          // [H] exp(A_log)
    const float* skip;          // [H] D
    const int* span_row;
    const int* span_len;
    const int* span_pos;
    const int* span_slot;
    float* state;               // a slot's S [H, N, vdim] begins at slot * state_stride + state_off
    long long state_stride, state_off;
    float* out;                 // [T, H, vdim]
    int H, G, N, vdim, EV;
    // chunks: pieces of `chunk` tokens (a multiple of 64)
    const int* item_span;
    const int* item_c;
    int chunk;
    const int* span_first;
    float* scratch;             // [items, H, N, vdim]
    float* piece_keep;          // [items, H]: the decay over the whole of the piece before
};

__device__ __forceinline__ float ssm_softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float ssm_dt(const SsmParams& p, size_t row, int h) {
    const size_t at = row * p.dt_stride + p.dt_off + h;
    const float raw = p.dt_dtype == LLB_F32 ? ((const float*)p.dt)[at] : __bfloat162float(((const __nv_bfloat16*)p.dt)[at]);
    return ssm_softplus(raw + p.dt_bias[h]);
}

// ---- walk -----------------------------------------------------------------------------------------------------------
constexpr int WALK_STAGE = 16;

template <typename T, int NR, int DG>
__global__ void __launch_bounds__(256) ssm_walk_kernel(SsmParams p) {
    extern __shared__ __align__(16) float sm[];
    constexpr int PADF = DG > 1 ? 4 : 0;
    constexpr int DPAD = DG * (NR + PADF);
    const int span = blockIdx.x, h = blockIdx.y;
    const int N = p.N, vdim = p.vdim;
    const int len = p.span_len[span], row0 = p.span_row[span], pos0 = p.span_pos[span];
    const int g = h / (p.H / p.G);
    float* bs = sm;                              // [STAGE][DPAD]
    float* cs = bs + WALK_STAGE * DPAD;          // [STAGE][DPAD]
    float* xs = cs + WALK_STAGE * DPAD;          // [STAGE][EV]
    float* gs = xs + WALK_STAGE * p.EV;          // [STAGE][2]: keep, dt
    const int dg = threadIdx.x % DG, el = threadIdx.x / DG;
    const int e = blockIdx.z * p.EV + el;
    const bool live = el < p.EV && e < vdim;
    const float rate = p.rate[h], skip = p.skip[h];
    float* slot = p.state + (long long)p.span_slot[span] * p.state_stride + p.state_off + (size_t)h * N * vdim;
    const T* src = (const T*)p.xbc;

    float S[NR];
#pragma unroll
    for (int j = 0; j < NR; ++j) {
        const int n = dg * NR + j;
        S[j] = (pos0 > 0 && live && n < N) ? slot[(size_t)n * vdim + e] : 0.0f;
    }
    for (int i = threadIdx.x; i < 2 * WALK_STAGE * DPAD; i += blockDim.x) sm[i] = 0.0f;     // the padding stays zero
    auto at = [](int n) { return (n / NR) * (NR + PADF) + n % NR; };
    for (int c0 = 0; c0 < len; c0 += WALK_STAGE) {
        const int cnt = min(WALK_STAGE, len - c0);
        __syncthreads();
        for (int it = threadIdx.x; it < cnt * N; it += blockDim.x) {
            const int tl = it / N, n = it - tl * N;
            const T* row = src + (size_t)(row0 + c0 + tl) * p.stride + (size_t)g * N + n;
            bs[tl * DPAD + at(n)] = llb_to_float(row[p.b_off]);
            cs[tl * DPAD + at(n)] = llb_to_float(row[p.c_off]);
        }
        for (int it = threadIdx.x; it < cnt * p.EV; it += blockDim.x) {
            const int tl = it / p.EV, cc = it - tl * p.EV;
            const int ee = blockIdx.z * p.EV + cc;
            xs[it] = ee < vdim ? llb_to_float(src[(size_t)(row0 + c0 + tl) * p.stride + p.x_off + (size_t)h * vdim + ee]) : 0.0f;
        }
        for (int it = threadIdx.x; it < cnt; it += blockDim.x) {
            const float dt = ssm_dt(p, (size_t)(row0 + c0 + it), h);
            gs[2 * it] = expf(-rate * dt);
            gs[2 * it + 1] = dt;
        }
        __syncthreads();
        for (int tl = 0; tl < cnt; ++tl) {
            const float keep = gs[2 * tl];
            const float xv = el < p.EV ? xs[tl * p.EV + el] : 0.0f;
            const float take = xv * gs[2 * tl + 1];
            const float4* b4p = reinterpret_cast<const float4*>(bs + tl * DPAD + dg * (NR + PADF));
            const float4* c4p = reinterpret_cast<const float4*>(cs + tl * DPAD + dg * (NR + PADF));
            float a0 = 0.0f, a1 = 0.0f, a2 = 0.0f, a3 = 0.0f;
#pragma unroll
            for (int j = 0; j < NR; j += 4) {
                const float4 b4 = b4p[j >> 2], c4 = c4p[j >> 2];
                S[j] = fmaf(keep, S[j], b4.x * take);
                S[j + 1] = fmaf(keep, S[j + 1], b4.y * take);
                S[j + 2] = fmaf(keep, S[j + 2], b4.z * take);
                S[j + 3] = fmaf(keep, S[j + 3], b4.w * take);
                a0 = fmaf(S[j], c4.x, a0);
                a1 = fmaf(S[j + 1], c4.y, a1);
                a2 = fmaf(S[j + 2], c4.z, a2);
                a3 = fmaf(S[j + 3], c4.w, a3);
            }
            float acc = (a0 + a1) + (a2 + a3);
#pragma unroll
            for (int o = 1; o < DG; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            if (live && dg == 0) p.out[((size_t)(row0 + c0 + tl) * p.H + h) * vdim + e] = fmaf(skip, xv, acc);
        }
    }
    if (!live) return;
#pragma unroll
    for (int j = 0; j < NR; ++j) {
        const int n = dg * NR + j;
        if (n < N) slot[(size_t)n * vdim + e] = S[j];
    }
}

template <typename T, int NR, int DG>
int launch_walk_as(SsmParams p, int num_spans, cudaStream_t stream) {
    constexpr int PADF = DG > 1 ? 4 : 0;
    const int per_block = 256 / DG;
    p.EV = p.vdim < per_block ? p.vdim : per_block;
    const dim3 grid(num_spans, p.H, llb_ceil_div(p.vdim, p.EV));
    const int threads = ((p.EV * DG + 31) / 32) * 32;
    const size_t smem = ((size_t)2 * WALK_STAGE * DG * (NR + PADF) + (size_t)WALK_STAGE * p.EV + 2 * WALK_STAGE) * sizeof(float);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(ssm_walk_kernel<T, NR, DG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return llb_fail("state_space: %s", cudaGetErrorString(e));
    }
    ssm_walk_kernel<T, NR, DG><<<grid, threads, smem, stream>>>(p);
    return llb_check_launch("state_space_walk");
}

template <typename T>
int launch_walk(const SsmParams& p, int num_spans, cudaStream_t stream) {
    if (p.N <= 16) return launch_walk_as<T, 16, 1>(p, num_spans, stream);
    if (p.N <= 32) return launch_walk_as<T, 32, 1>(p, num_spans, stream);
    if (p.N <= 64) return launch_walk_as<T, 32, 2>(p, num_spans, stream);
    if (p.N <= 128) return launch_walk_as<T, 32, 4>(p, num_spans, stream);
    if (p.N <= 256) return launch_walk_as<T, 32, 8>(p, num_spans, stream);
    return launch_walk_as<T, 64, 8>(p, num_spans, stream);
}

// ---- step -----------------------------------------------------------------------------------------------------------
// One token a span.  A block takes (span, head) and all columns in pieces of four; thread (r, c) owns rows r, r + RT, ...
// of column piece c.  All of a thread's 16-byte loads of the state are in flight at once (ROWS of them).
constexpr int STEP_THREADS = 128;

template <typename T, int ROWS>
__global__ void __launch_bounds__(STEP_THREADS) ssm_step_kernel(SsmParams p) {
    extern __shared__ __align__(16) float sm[];       // B [N], C [N], then (16-byte aligned) the partial sums [RT][vdim]
    const int span = blockIdx.x, h = blockIdx.y;
    const int N = p.N, vdim = p.vdim, CP = vdim >> 2, RT = STEP_THREADS / CP;
    const int row = p.span_row[span];
    const int g = h / (p.H / p.G);
    const bool fresh = p.span_pos[span] == 0;
    float4* slot = reinterpret_cast<float4*>(p.state + (long long)p.span_slot[span] * p.state_stride + p.state_off + (size_t)h * N * vdim);
    const int c = threadIdx.x % CP, r = threadIdx.x / CP;
    const bool live = r < RT;
    float4 S[ROWS];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = r + j * RT;
        S[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (live && !fresh && n < N) S[j] = slot[(size_t)n * CP + c];
    }
    float* bs = sm;
    float* cs = sm + N;
    float* part = sm + ((2 * N + 3) & ~3);
    const T* src = (const T*)p.xbc + (size_t)row * p.stride;
    for (int n = threadIdx.x; n < N; n += STEP_THREADS) {
        bs[n] = llb_to_float(src[p.b_off + (size_t)g * N + n]);
        cs[n] = llb_to_float(src[p.c_off + (size_t)g * N + n]);
    }
    const float dt = ssm_dt(p, (size_t)row, h);
    const float keep = expf(-p.rate[h] * dt);
    float x4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (live) {
#pragma unroll
        for (int i = 0; i < 4; ++i) x4[i] = llb_to_float(src[p.x_off + (size_t)h * vdim + 4 * c + i]);
    }
    __syncthreads();
    float4 acc = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = r + j * RT;
        if (live && n < N) {
            const float b = bs[n] * dt, cc = cs[n];
            S[j].x = fmaf(keep, S[j].x, b * x4[0]);
            S[j].y = fmaf(keep, S[j].y, b * x4[1]);
            S[j].z = fmaf(keep, S[j].z, b * x4[2]);
            S[j].w = fmaf(keep, S[j].w, b * x4[3]);
            slot[(size_t)n * CP + c] = S[j];
            acc.x = fmaf(cc, S[j].x, acc.x);
            acc.y = fmaf(cc, S[j].y, acc.y);
            acc.z = fmaf(cc, S[j].z, acc.z);
            acc.w = fmaf(cc, S[j].w, acc.w);
        }
    }
    if (live) *reinterpret_cast<float4*>(part + (size_t)r * vdim + 4 * c) = acc;
    __syncthreads();
    const float skip = p.skip[h];
    for (int e = threadIdx.x; e < vdim; e += STEP_THREADS) {
        float y = 0.0f;
        for (int i = 0; i < RT; ++i) y += part[(size_t)i * vdim + e];
        p.out[((size_t)row * p.H + h) * vdim + e] = fmaf(skip, llb_to_float(src[p.x_off + (size_t)h * vdim + e]), y);
    }
}

// Whether the step kernel takes the shape: columns in whole pieces of four that divide the block's threads evenly enough
// and at most 16 rows a thread.
inline bool step_supports(const SsmParams& p) {
    if (p.vdim % 4 != 0 || p.vdim > 4 * STEP_THREADS || p.state_stride % 4 != 0 || p.state_off % 4 != 0 || (uintptr_t)p.state % 16 != 0) return false;
    const int RT = STEP_THREADS / (p.vdim / 4);
    return (p.N + RT - 1) / RT <= 16;
}

template <typename T>
int launch_step(const SsmParams& p, int num_spans, cudaStream_t stream) {
    const int RT = STEP_THREADS / (p.vdim / 4), rows = (p.N + RT - 1) / RT;
    const size_t smem = ((size_t)((2 * p.N + 3) & ~3) + (size_t)RT * p.vdim) * sizeof(float);
    const dim3 grid(num_spans, p.H);
    if (rows <= 4) ssm_step_kernel<T, 4><<<grid, STEP_THREADS, smem, stream>>>(p);
    else if (rows <= 8) ssm_step_kernel<T, 8><<<grid, STEP_THREADS, smem, stream>>>(p);
    else ssm_step_kernel<T, 16><<<grid, STEP_THREADS, smem, stream>>>(p);
    return llb_check_launch("state_space_step");
}

// ---- chunks ---------------------------------------------------------------------------------------------------------
constexpr int CL = 64;                 // tokens a chunk
enum { SSM_LOCAL = 1, SSM_OUT = 3 };

// two floats as (hi, lo) pairs of bf16: v = hi + lo up to 2^-17 of v
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = pack_bf16(a - __bfloat162float(h.x), b - __bfloat162float(h.y));
}

// Shared memory of the chunk kernel.  Rows are padded by 16 bytes, so that the eight rows an ldmatrix touches lie on
// different banks.  NP: N rounded up to 64 * MT; EV columns of x and S.
// NST stages: with one, a block's copies wait for its work, and two blocks an SM hide each other's; with two a block alone
// overlaps them (measured: one stage where two would leave room for a single block).
template <int MT, int EV>
struct ChunkShape {
    static constexpr int NST = (MT >= 2 && EV == 64) || MT == 4 ? 1 : 2;
    static constexpr int NP = 64 * MT;
    static constexpr int NB = NP * 2 + 16;            // bytes a row of B and C
    static constexpr int XB = EV * 2 + 16;            // bytes a row of x, of its weighted halves and of S's halves
    static constexpr int STAGE = 2 * CL * NB + CL * XB;
    static constexpr int OFF_XW = NST * STAGE;          // weighted x: hi, lo [CL]
    static constexpr int OFF_S = OFF_XW + 2 * CL * XB;        // S before the chunk: hi, lo [NP]
    static constexpr int OFF_G = OFF_S + 2 * NP * XB;         // per stage: L [CL], dt [CL]
    static constexpr int BYTES = OFF_G + 2 * 2 * CL * 4;
};

template <int MT, int EV, int MODE>
__global__ void __launch_bounds__(128) ssm_chunk_kernel(SsmParams p) {
    using Sh = ChunkShape<MT, EV>;
    constexpr int NP = Sh::NP, NB = Sh::NB, XB = Sh::XB, NE = EV / 8, KS = NP / 16, NST = Sh::NST;
    extern __shared__ __align__(16) uint8_t smem[];
    const int item = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * EV;
    const int span = p.item_span[item], pc = p.item_c[item];
    const int slen = p.span_len[span];
    const int pieces = (slen + p.chunk - 1) / p.chunk;
    const bool last = pc == pieces - 1;
    if (MODE == SSM_LOCAL && last) return;               // the last piece's contribution is never needed
    const int t0 = pc * p.chunk;
    const int len = min(p.chunk, slen - t0);
    const int row0 = p.span_row[span] + t0, pos0 = p.span_pos[span] + t0;
    const int N = p.N, vdim = p.vdim;
    const int g = h / (p.H / p.G);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t base = smem_addr(smem);
    const float rate = p.rate[h];
    const size_t plane = (size_t)N * vdim;
    float* slot = p.state + (long long)p.span_slot[span] * p.state_stride + p.state_off + (size_t)h * plane;
    const __nv_bfloat16* src = (const __nv_bfloat16*)p.xbc;

    // Copies of one chunk into a stage (rows past the piece's end and columns past N or vdim: zeros).
    auto fetch = [&](int c0, int stage) {
        const uint32_t sb = base + stage * Sh::STAGE;
        constexpr int BCH = NP / 8;
        for (int i = threadIdx.x; i < CL * BCH; i += 128) {
            const int r = i / BCH, ch = i - r * BCH;
            const bool ok = c0 + r < len && ch * 8 < N;
            const __nv_bfloat16* row = src + (size_t)(row0 + (c0 + r < len ? c0 + r : 0)) * p.stride + (size_t)g * N + (ok ? ch * 8 : 0);
            cp_async16(sb + r * NB + ch * 16, row + p.b_off, ok);
            if (MODE == SSM_OUT) cp_async16(sb + CL * NB + r * NB + ch * 16, row + p.c_off, ok);
        }
        constexpr int XCH = EV / 8;
        for (int i = threadIdx.x; i < CL * XCH; i += 128) {
            const int r = i / XCH, ch = i - r * XCH;
            const bool ok = c0 + r < len && e0 + ch * 8 < vdim;
            const __nv_bfloat16* row = src + (size_t)(row0 + (c0 + r < len ? c0 + r : 0)) * p.stride + p.x_off + (size_t)h * vdim + (ok ? e0 + ch * 8 : 0);
            cp_async16(sb + 2 * CL * NB + r * XB + ch * 16, row, ok);
        }
        cp_async_commit();
    };
    // dt and the running sum of the log decays of one chunk (warp 0; two tokens a lane).  Rows past the end: dt = 0.
    auto gates = [&](int c0, int stage) {
        if (warp != 0) return;
        float* L = reinterpret_cast<float*>(smem + Sh::OFF_G) + stage * 2 * CL;
        float* D = L + CL;
        const int a = 2 * lane, b = 2 * lane + 1;
        const float da = c0 + a < len ? ssm_dt(p, (size_t)(row0 + c0 + a), h) : 0.0f;
        const float db = c0 + b < len ? ssm_dt(p, (size_t)(row0 + c0 + b), h) : 0.0f;
        float run = da + db;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += up;
        }
        D[a] = da;
        D[b] = db;
        L[b] = -rate * run;
        L[a] = -rate * (run - db);
    };

    fetch(0, 0);
    gates(0, 0);
    // The state: warp w owns rows w * 16 * MT .. + 16 * MT of it, as accumulator fragments.
    float S[MT][NE][4];
    const float* from = nullptr;
    if (MODE == SSM_OUT) {
        if (pieces > 1) from = p.scratch + ((size_t)item * p.H + h) * plane;
        else if (pos0 > 0) from = slot;
    }
    const int fr = lane >> 2, fc = (lane & 3) * 2;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NE; ++i)
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int n = (warp * MT + m) * 16 + fr + (q >> 1) * 8, e = e0 + i * 8 + fc + (q & 1);
                S[m][i][q] = (from != nullptr && n < N && e < vdim) ? from[(size_t)n * vdim + e] : 0.0f;
            }
    float total = 0.0f;          // log decay over the whole piece
    const float skip = MODE == SSM_OUT ? p.skip[h] : 0.0f;
    int turn = 0;
    for (int c0 = 0; c0 < len; c0 += CL, turn ^= 1) {
        const bool more = c0 + CL < len;
        const int stage = NST == 2 ? turn : 0;
        if (more && NST == 2) {
            fetch(c0 + CL, stage ^ 1);          // (last read before the barrier that ended the chunk before)
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        if (more) gates(c0 + CL, turn ^ 1);
        __syncthreads();
        const uint32_t sB = base + stage * Sh::STAGE, sC = sB + CL * NB, sX = sC + CL * NB;
        const uint8_t* gX = smem + stage * Sh::STAGE + 2 * CL * NB;
        const float* L = reinterpret_cast<const float*>(smem + Sh::OFF_G) + turn * 2 * CL;
        const float* D = L + CL;
        const float Ln = L[CL - 1];
        // the weighted x of the state's update, as halves; S before the chunk, as halves
        for (int i = threadIdx.x; i < CL * (EV / 2); i += 128) {
            const int r = i / (EV / 2), c2 = i - r * (EV / 2);
            const float w = expf(Ln - L[r]) * D[r];
            const float2 x2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gX + r * XB + c2 * 4));
            uint32_t hi, lo;
            split_pair(w * x2.x, w * x2.y, hi, lo);
            *reinterpret_cast<uint32_t*>(smem + Sh::OFF_XW + r * XB + c2 * 4) = hi;
            *reinterpret_cast<uint32_t*>(smem + Sh::OFF_XW + (CL + r) * XB + c2 * 4) = lo;
        }
        if (MODE == SSM_OUT) {
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < NE; ++i)
#pragma unroll
                    for (int q = 0; q < 4; q += 2) {
                        const int n = (warp * MT + m) * 16 + fr + (q >> 1) * 8;
                        uint32_t hi, lo;
                        split_pair(S[m][i][q], S[m][i][q + 1], hi, lo);
                        uint8_t* dst = smem + Sh::OFF_S + n * XB + (i * 8 + fc) * 2;
                        *reinterpret_cast<uint32_t*>(dst) = hi;
                        *reinterpret_cast<uint32_t*>(dst + NP * XB) = lo;
                    }
        }
        __syncthreads();
        if (MODE == SSM_OUT) {
            // Warp w: tokens 16 w .. 16 w + 15 of the chunk.
            const int tr = warp * 16;
            const uint32_t a_row = (uint32_t)(tr + (lane & 7) + ((lane >> 3) & 1) * 8), a_ch = lane >> 4;
            float y[NE][4], G[8][4];
#pragma unroll
            for (int i = 0; i < NE; ++i) y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.0f;
#pragma unroll
            for (int i = 0; i < 8; ++i) G[i][0] = G[i][1] = G[i][2] = G[i][3] = 0.0f;
#pragma unroll 2
            for (int ks = 0; ks < KS; ks += 2) {
                if (ks * 16 >= N) break;          // (columns past N are zeros; uniform)
                uint32_t ca[4], cb[4];
                ldmatrix_x4(sC + a_row * NB + (ks * 2 + a_ch) * 16, ca);
                ldmatrix_x4(sC + a_row * NB + (ks * 2 + 2 + a_ch) * 16, cb);
                // G = C B^T: columns (tokens s) up to the diagonal
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    if (i * 8 <= tr + 15) {          // uniform over the warp
                        uint32_t b[4];
                        ldmatrix_x4(sB + (i * 8 + (lane & 7)) * NB + (ks * 2 + (lane >> 3)) * 16, b);
                        mma_bf16(G[i], ca, b[0], b[1]);
                        mma_bf16(G[i], cb, b[2], b[3]);
                    }
                }
                // y = C S_0 (both halves of S)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const uint32_t sS = base + Sh::OFF_S + half * NP * XB;
#pragma unroll
                    for (int i = 0; i < NE; i += 2) {
                        const uint32_t at = (lane & 7) + ((lane >> 3) & 1) * 8, ch = i + (lane >> 4);
                        uint32_t b[4];
                        ldmatrix_x4_trans(sS + (ks * 16 + at) * XB + ch * 16, b);
                        mma_bf16(y[i], ca, b[0], b[1]);
                        mma_bf16(y[i + 1], ca, b[2], b[3]);
                        ldmatrix_x4_trans(sS + (ks * 16 + 16 + at) * XB + ch * 16, b);
                        mma_bf16(y[i], cb, b[0], b[1]);
                        mma_bf16(y[i + 1], cb, b[2], b[3]);
                    }
                }
            }
            const int ta = tr + fr, tb = ta + 8;
            const float La = L[ta], Lb = L[tb];
            const float ea = expf(La), eb = expf(Lb);
#pragma unroll
            for (int i = 0; i < NE; ++i) {
                y[i][0] *= ea; y[i][1] *= ea;
                y[i][2] *= eb; y[i][3] *= eb;
            }
            // the weighted scores as A fragments (halves), times x
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (j > warp) break;          // tokens 16 j .. past the diagonal of every row of this warp
                uint32_t mh[4], ml[4];
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int i = 2 * j + u, s = i * 8 + fc;
                    const float L0 = L[s], L1 = L[s + 1], d0 = D[s], d1 = D[s + 1];
                    const float w0 = s <= ta ? G[i][0] * expf(La - L0) * d0 : 0.0f;
                    const float w1 = s + 1 <= ta ? G[i][1] * expf(La - L1) * d1 : 0.0f;
                    const float w2 = s <= tb ? G[i][2] * expf(Lb - L0) * d0 : 0.0f;
                    const float w3 = s + 1 <= tb ? G[i][3] * expf(Lb - L1) * d1 : 0.0f;
                    split_pair(w0, w1, mh[u * 2], ml[u * 2]);
                    split_pair(w2, w3, mh[u * 2 + 1], ml[u * 2 + 1]);
                }
#pragma unroll
                for (int i = 0; i < NE; i += 2) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(sX + (j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * XB + (i + (lane >> 4)) * 16, b);
                    mma_bf16(y[i], mh, b[0], b[1]);
                    mma_bf16(y[i + 1], mh, b[2], b[3]);
                    mma_bf16(y[i], ml, b[0], b[1]);
                    mma_bf16(y[i + 1], ml, b[2], b[3]);
                }
            }
#pragma unroll
            for (int i = 0; i < NE; ++i) {
                const int el = i * 8 + fc, e = e0 + el;
                if (e >= vdim) continue;          // vdim is even
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int t = u ? tb : ta;
                    if (c0 + t >= len) continue;
                    const float2 x2 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gX + t * XB + el * 2));
                    float* o = p.out + ((size_t)(row0 + c0 + t) * p.H + h) * vdim + e;
                    *reinterpret_cast<float2*>(o) = make_float2(fmaf(skip, x2.x, y[i][u * 2]), fmaf(skip, x2.y, y[i][u * 2 + 1]));
                }
            }
        }
        // S = e^{L_n} S + B^T x'
        const float eN = expf(Ln);
        total += Ln;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int i = 0; i < NE; ++i) {
                S[m][i][0] *= eN; S[m][i][1] *= eN; S[m][i][2] *= eN; S[m][i][3] *= eN;
            }
#pragma unroll
        for (int j = 0; j < 4; ++j) {             // 16 tokens a step
            uint32_t a[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m)
                ldmatrix_x4_trans(sB + (j * 16 + (lane & 7) + (lane >> 4) * 8) * NB + ((warp * MT + m) * 2 + ((lane >> 3) & 1)) * 16, a[m]);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
#pragma unroll
                for (int i = 0; i < NE; i += 2) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(base + Sh::OFF_XW + (half * CL + j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * XB + (i + (lane >> 4)) * 16, b);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_bf16(S[m][i], a[m], b[0], b[1]);
                        mma_bf16(S[m][i + 1], a[m], b[2], b[3]);
                    }
                }
            }
        }
        __syncthreads();          // every warp has read this stage, the weighted x and S's halves
        if (more && NST == 1) fetch(c0 + CL, 0);
    }
    float* to = nullptr;
    if (MODE == SSM_LOCAL) {
        to = p.scratch + ((size_t)(item + 1) * p.H + h) * plane;     // the next piece's place
        if (threadIdx.x == 0 && blockIdx.z == 0) p.piece_keep[(size_t)(item + 1) * p.H + h] = expf(total);
    } else if (last) {
        to = slot;
    }
    if (to == nullptr) return;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NE; ++i)
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const int n = (warp * MT + m) * 16 + fr + (q >> 1) * 8, e = e0 + i * 8 + fc + (q & 1);
                if (n < N && e < vdim) to[(size_t)n * vdim + e] = S[m][i][q];
            }
}

// start_0 = the request's state (zero at position 0); start_c = keep_(c-1) * start_(c-1) + contribution_(c-1).
__global__ void __launch_bounds__(256) ssm_scan_kernel(SsmParams p) {
    const int span = blockIdx.x, h = blockIdx.y;
    const int slen = p.span_len[span];
    const int pieces = (slen + p.chunk - 1) / p.chunk;
    if (pieces <= 1) return;
    const size_t plane = (size_t)p.N * p.vdim;
    const float* slot = p.state + (long long)p.span_slot[span] * p.state_stride + p.state_off + (size_t)h * plane;
    const bool fresh = p.span_pos[span] == 0;
    const size_t first = (size_t)p.span_first[span];
    const size_t stride = (size_t)p.H * plane;
    const float* pk = p.piece_keep + first * p.H + h;
    for (size_t i = (size_t)blockIdx.z * blockDim.x + threadIdx.x; i < plane; i += (size_t)gridDim.z * blockDim.x) {
        float s = fresh ? 0.0f : slot[i];
        float* at = p.scratch + (first * p.H + h) * plane + i;
        at[0] = s;
        for (int c = 1; c < pieces; c += 8) {          // eight pieces' contributions are requested together
            float a[8], k[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                a[u] = c + u < pieces ? at[(size_t)(c + u) * stride] : 0.0f;
                k[u] = c + u < pieces ? pk[(size_t)(c + u) * p.H] : 1.0f;
            }
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                s = fmaf(k[u], s, a[u]);
                a[u] = s;
            }
#pragma unroll
            for (int u = 0; u < 8; ++u)
                if (c + u < pieces) at[(size_t)(c + u) * stride] = a[u];
        }
    }
}

inline bool chunks_support(const SsmParams& p) {
    return p.N % 8 == 0 && p.N <= 256 && p.vdim % 8 == 0 && p.stride % 8 == 0 && p.x_off % 8 == 0 && p.b_off % 8 == 0 &&
           p.c_off % 8 == 0 && (uintptr_t)p.xbc % 16 == 0;
}

template <int MT, int EV, int MODE>
int launch_chunk(const SsmParams& p, int num_items, cudaStream_t stream) {
    constexpr int bytes = ChunkShape<MT, EV>::BYTES;
    static bool configured = false;
    if (!configured && bytes > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(ssm_chunk_kernel<MT, EV, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
        if (e != cudaSuccess) return llb_fail("state_space: %s", cudaGetErrorString(e));
        configured = true;
    }
    ssm_chunk_kernel<MT, EV, MODE><<<dim3(num_items, p.H, llb_ceil_div(p.vdim, EV)), 128, bytes, stream>>>(p);
    return llb_check_launch("state_space_chunks");
}

template <int EV>
int launch_chunks(const SsmParams& p, int num_items, int mode, cudaStream_t stream) {
    const int mt = p.N <= 64 ? 1 : p.N <= 128 ? 2 : 4;
    if (mode == SSM_LOCAL) {
        if (mt == 1) return launch_chunk<1, EV, SSM_LOCAL>(p, num_items, stream);
        if (mt == 2) return launch_chunk<2, EV, SSM_LOCAL>(p, num_items, stream);
        return launch_chunk<4, EV, SSM_LOCAL>(p, num_items, stream);
    }
    if (mt == 1) return launch_chunk<1, EV, SSM_OUT>(p, num_items, stream);
    if (mt == 2) return launch_chunk<2, EV, SSM_OUT>(p, num_items, stream);
    return launch_chunk<4, EV, SSM_OUT>(p, num_items, stream);
}

// ---- the gated norm behind the recurrence ---------------------------------------------------------------------------
// out[t, :] = norm_parts(y[t, :] * silu(z[t, :])) * w: one block a (token, part), float statistics.
template <typename TZ, int V>
__global__ void __launch_bounds__(256) gated_group_norm_kernel(const float* __restrict__ y, const TZ* __restrict__ z,
                                                               long long z_stride, const float* __restrict__ w,
                                                               TZ* __restrict__ out, int size, int parts, float eps) {
    const int t = blockIdx.x, part = blockIdx.y;
    const int n = size * parts;
    const float* yr = y + (size_t)t * n + (size_t)part * size;
    const TZ* zr = z + (size_t)t * z_stride + (size_t)part * size;
    const float* wr = w + (size_t)part * size;
    TZ* o = out + (size_t)t * n + (size_t)part * size;
    constexpr int HOLD = 4;                       // pieces of V numbers a thread keeps between the passes
    float v[HOLD][V];
    float ss = 0.0f;
    auto product = [&](int d, float (&q)[V]) {
        if (V == 4) {
            const float4 y4 = *reinterpret_cast<const float4*>(yr + d);
            q[0] = y4.x; q[1 % V] = y4.y; q[2 % V] = y4.z; q[3 % V] = y4.w;
        } else {
            q[0] = yr[d];
        }
#pragma unroll
        for (int i = 0; i < V; ++i) q[i] *= llb_silu(llb_to_float(zr[d + i]));
    };
    for (int k = 0, d = threadIdx.x * V; d < size; d += blockDim.x * V, ++k) {
        float q[V];
        product(d, q);
#pragma unroll
        for (int i = 0; i < V; ++i) ss = fmaf(q[i], q[i], ss);
#pragma unroll
        for (int u = 0; u < HOLD; ++u)
            if (u == k)
#pragma unroll
                for (int i = 0; i < V; ++i) v[u][i] = q[i];
    }
    __shared__ float warp_part[8];
    ss = llb_warp_sum(ss);
    if ((threadIdx.x & 31) == 0) warp_part[threadIdx.x >> 5] = ss;
    __syncthreads();
    float total = 0.0f;
    for (int i = 0; i < (int)(blockDim.x >> 5); ++i) total += warp_part[i];
    const float inv = 1.0f / sqrtf(total / (float)size + eps);
    for (int k = 0, d = threadIdx.x * V; d < size; d += blockDim.x * V, ++k) {
        float q[V];
        if (k < HOLD) {
#pragma unroll
            for (int u = 0; u < HOLD; ++u)
                if (u == k)
#pragma unroll
                    for (int i = 0; i < V; ++i) q[i] = v[u][i];
        } else {
            product(d, q);
        }
        TZ r[V];
#pragma unroll
        for (int i = 0; i < V; ++i) r[i] = llb_from_float<TZ>(q[i] * inv * wr[d + i]);
        if (V == 4 && sizeof(TZ) == 2) *reinterpret_cast<uint2*>(o + d) = *reinterpret_cast<const uint2*>(r);
        else
#pragma unroll
            for (int i = 0; i < V; ++i) o[d + i] = r[i];
    }
}

template <typename TZ>
int launch_group_norm(const float* y, const void* z, long long z_stride, const float* w, void* out, int T, int size, int parts,
                      float eps, cudaStream_t stream) {
    const dim3 grid(T, parts);
    const bool vec = size % 4 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)out % 8 == 0;
    const int per = vec ? 4 : 1;
    int threads = 32 * ((size / per + 31) / 32);
    threads = threads > 256 ? 256 : threads < 32 ? 32 : threads;
    if (vec) gated_group_norm_kernel<TZ, 4><<<grid, threads, 0, stream>>>(y, (const TZ*)z, z_stride, w, (TZ*)out, size, parts, eps);
    else gated_group_norm_kernel<TZ, 1><<<grid, threads, 0, stream>>>(y, (const TZ*)z, z_stride, w, (TZ*)out, size, parts, eps);
    return llb_check_launch("gated_group_norm");
}

}  // namespace

// xbc [T, stride] (dtype): x [H, vdim] at column x_off, B [G, N] at b_off, C [G, N] at c_off; dt [T, dt_stride] (dt_dtype): H
// columns from dt_off on, before dt_bias [H] and the softplus; rate [H] = exp(A_log); skip [H] = D; the spans as in every
// kernel of a step; state: float base of the requests' state plane, `state_stride` floats a slot, a request's S [H, N,
// vdim] at `state_off` inside its slot (read where a span continues a request, written at its end); out float [T, H, vdim].
// single != 0 (every span is one token): the step kernel where the sizes allow.  Otherwise num_items > 0 asks for the chunk
// kernels (bf16, N and vdim multiples of 8, N <= 256, aligned columns; else the call fails): item_span, item_c
// [num_items], span_first [num_spans] name the pieces of `chunk` tokens (a multiple of 64) that the spans are cut into;
// multi != 0: some span has several pieces, scratch float [num_items, H, N, vdim] and piece_keep float [num_items, H] are
// needed.  num_items == 0: token by token.
LLB_EXPORT int llb_state_space(const void* xbc, int dtype, long long stride, int x_off, int b_off, int c_off, const void* dt,
                               int dt_dtype, long long dt_stride, int dt_off, const float* dt_bias, const float* rate,
                               const float* skip, const int* span_row, const int* span_len, const int* span_pos,
                               const int* span_slot, int num_spans, int H, int G, int N, int vdim, float* state,
                               long long state_stride, long long state_off, float* out, int single, const int* item_span,
                               const int* item_c, const int* span_first, int num_items, int chunk, int multi, float* scratch,
                               float* piece_keep, cudaStream_t stream) {
    if (num_spans == 0) return 0;
    LLB_REQUIRE(num_spans > 0 && H > 0 && G > 0 && N > 0 && vdim > 0 && xbc && dt && dt_bias && rate && skip && state && out &&
                span_row && span_len && span_pos && span_slot, "state_space: bad arguments");
    LLB_REQUIRE(H % G == 0 && H <= 65535 && N <= 512, "state_space: %d heads in %d groups, states of %d (at most 512)", H, G, N);
    LLB_REQUIRE(dtype == LLB_F32 || dtype == LLB_BF16, "state_space: unknown dtype %d", dtype);
    SsmParams p = {};
    p.xbc = xbc; p.stride = stride; p.x_off = x_off; p.b_off = b_off; p.c_off = c_off;
    p.dt = dt; p.dt_stride = dt_stride; p.dt_off = dt_off; p.dt_dtype = dt_dtype; p.dt_bias = dt_bias; p.rate = rate; p.skip = skip;
    p.span_row = span_row; p.span_len = span_len; p.span_pos = span_pos; p.span_slot = span_slot;
    p.state = state; p.state_stride = state_stride; p.state_off = state_off; p.out = out;
    p.H = H; p.G = G; p.N = N; p.vdim = vdim;
    if (single && step_supports(p)) {
        if (dtype == LLB_F32) return launch_step<float>(p, num_spans, stream);
        return launch_step<__nv_bfloat16>(p, num_spans, stream);
    }
    if (!single && num_items > 0) {
        LLB_REQUIRE(dtype == LLB_BF16 && chunks_support(p), "state_space: the chunk kernels take bf16, N and vdim multiples of 8, "
                    "N <= 256 and aligned columns (N %d, vdim %d)", N, vdim);
        LLB_REQUIRE(item_span && item_c && span_first && chunk > 0 && (!multi || (scratch && piece_keep && chunk % CL == 0)),
                    "state_space: the pieces are not described");
        p.item_span = item_span; p.item_c = item_c; p.span_first = span_first; p.chunk = chunk;
        p.scratch = scratch; p.piece_keep = piece_keep;
        int rc = 0;
        for (int pass = multi ? 0 : 2; pass < 3 && rc == 0; ++pass) {
            if (pass == 1) {
                int z = (N * vdim + 255) / 256;
                if (z > 64) z = 64;
                ssm_scan_kernel<<<dim3(num_spans, H, z), 256, 0, stream>>>(p);
                rc = llb_check_launch("state_space_scan");
                continue;
            }
            const int mode = pass == 0 ? SSM_LOCAL : SSM_OUT;
            // few heads: narrow column blocks, so that a lone prompt's pieces still fill the multiprocessors
            if (vdim <= 16) rc = launch_chunks<16>(p, num_items, mode, stream);
            else if (vdim <= 32 || N > 128) rc = launch_chunks<32>(p, num_items, mode, stream);
            else rc = launch_chunks<64>(p, num_items, mode, stream);
        }
        return rc;
    }
    if (dtype == LLB_F32) return launch_walk<float>(p, num_spans, stream);
    return launch_walk<__nv_bfloat16>(p, num_spans, stream);
}

// Whether the chunk kernels take these sizes (columns at multiples of 8, 16-byte aligned rows).
LLB_EXPORT int llb_state_space_chunks_support(int N, int vdim, int stride, int x_off, int b_off, int c_off) {
    SsmParams p = {};
    p.N = N; p.vdim = vdim; p.stride = stride; p.x_off = x_off; p.b_off = b_off; p.c_off = c_off;
    return chunks_support(p) ? 1 : 0;
}

// y float [T, parts * size]; z [T, z_stride] (dtype, the first parts * size columns from the pointer on); w float [parts *
// size]; out [T, parts * size] (dtype): y * silu(z), every part divided by its own root mean square (eps inside), times w.
LLB_EXPORT int llb_gated_group_norm(const float* y, const void* z, int dtype, long long z_stride, const float* w, void* out,
                                    int T, int size, int parts, float eps, cudaStream_t stream) {
    if (T == 0) return 0;
    LLB_REQUIRE(T > 0 && size > 0 && parts > 0 && parts <= 65535 && y && z && w && out, "gated_group_norm: bad arguments");
    if (dtype == LLB_F32) return launch_group_norm<float>(y, z, z_stride, w, out, T, size, parts, eps, stream);
    if (dtype == LLB_BF16) return launch_group_norm<__nv_bfloat16>(y, z, z_stride, w, out, T, size, parts, eps, stream);
    return llb_fail("gated_group_norm: unknown dtype %d", dtype);
}
