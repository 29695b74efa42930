// A contraction per head: out[t, h, o] = sum_i x[t, h, i] * w[h, o, i], for projections that differ from head to head
// (the up-projections of a shared latent folded onto the query and the output).  Float accumulation; x, w and out
// float or bf16.  The heads' numbers may lie anywhere in a row of x and of out (a stride from head to head), and a range
// of a head's numbers may be rotated by position and laid behind the result (the rotated part of a query whose other part
// goes through the contraction).
//
// Two kernels: CUDA cores for any sizes and float, and mma.sync tiles for bf16 with inputs in multiples of 8.
#include "common.cuh"
#include "warp_mma.cuh"

namespace {

using namespace wm;

struct HeadLinearParams {
    const void* x;              // row t, head h: x + t * x_stride + x_off + h * x_head, `in` numbers
    long long x_stride, x_head;
    int x_off;
    const void* w;              // [H, on, in]
    void* out;                  // row t, head h: out + t * out_stride + h * out_head, `on` numbers
    long long out_stride, out_head;
    int T, H, in, on;
    // rotation: numbers rot_src .. + rot_dim of a head of x turn by position and go to rot_dst of the head of out
    int rot_dim, rot_src, rot_dst, interleaved;
    const int* positions;       // [T]
    const float* inv_freq;      // [rot_dim / 2]
};

// rotates the heads' rotated ranges of rows t0 .. t0 + rows - 1 of head h
template <typename T>
__device__ __forceinline__ void rotate_rows(const HeadLinearParams& p, int t0, int rows, int h) {
    const int half = p.rot_dim >> 1;
    for (int i = threadIdx.x; i < rows * half; i += blockDim.x) {
        const int r = i / half, j = i - r * half;
        const T* src = (const T*)p.x + (size_t)(t0 + r) * p.x_stride + p.x_off + (size_t)h * p.x_head + p.rot_src;
        T* dst = (T*)p.out + (size_t)(t0 + r) * p.out_stride + (size_t)h * p.out_head + p.rot_dst;
        const int a = p.interleaved ? 2 * j : j, b = p.interleaved ? 2 * j + 1 : j + half;
        const float angle = (float)p.positions[t0 + r] * p.inv_freq[j];
        const float cs = cosf(angle), sn = sinf(angle);
        const float u = llb_to_float(src[a]), v = llb_to_float(src[b]);
        dst[a] = llb_from_float<T>(u * cs - v * sn);
        dst[b] = llb_from_float<T>(v * cs + u * sn);
    }
}

constexpr int HL_ROWS = 16;     // tokens per block

template <typename T>
__global__ void __launch_bounds__(256) head_linear_kernel(HeadLinearParams p) {
    extern __shared__ float xs[];          // [HL_ROWS][in]
    const int in = p.in, on = p.on;
    const int t0 = blockIdx.x * HL_ROWS, h = blockIdx.y;
    const int rows = min(HL_ROWS, p.T - t0);
    const T* x = (const T*)p.x + p.x_off + (size_t)h * p.x_head;
    for (int i = threadIdx.x; i < rows * in; i += blockDim.x) {
        const int r = i / in, c = i - r * in;
        xs[i] = llb_to_float(x[(size_t)(t0 + r) * p.x_stride + c]);
    }
    __syncthreads();
    const T* wh = (const T*)p.w + (size_t)h * on * in;
    T* out = (T*)p.out + (size_t)h * p.out_head;
    // a thread owns output column o for all rows of the tile: its weight row is read once
    for (int o = threadIdx.x; o < on; o += blockDim.x) {
        float acc[HL_ROWS];
#pragma unroll
        for (int r = 0; r < HL_ROWS; ++r) acc[r] = 0.0f;
        const T* wr = wh + (size_t)o * in;
        for (int i = 0; i < in; ++i) {
            const float wv = llb_to_float(wr[i]);
#pragma unroll
            for (int r = 0; r < HL_ROWS; ++r) acc[r] = fmaf(xs[r * in + i], wv, acc[r]);
        }
#pragma unroll
        for (int r = 0; r < HL_ROWS; ++r)
            if (r < rows) out[(size_t)(t0 + r) * p.out_stride + o] = llb_from_float<T>(acc[r]);
    }
    if (p.rot_dim) rotate_rows<T>(p, t0, rows, h);
}

// Tiles of 16 * RG rows x 64 outputs of one head; four warps, RG of them along the rows and 4 / RG along the outputs.
// Inputs come 64 at a time through two buffers.  Rows of shared memory are padded by 16 bytes (ldmatrix without conflicts).
constexpr int HL_OT = 64, HL_KB = 64, HL_PITCH = HL_KB * 2 + 16;

template <int RG>
__global__ void __launch_bounds__(128) head_linear_mma_kernel(HeadLinearParams p) {
    constexpr int MR = 16 * RG, CW = 4 / RG, NT = HL_OT / CW / 8;          // n-tiles of 8 outputs a warp
    __shared__ __align__(16) uint8_t xs[2][MR * HL_PITCH];
    __shared__ __align__(16) uint8_t ws[2][HL_OT * HL_PITCH];
    const int t0 = blockIdx.x * MR, h = blockIdx.y, o0 = blockIdx.z * HL_OT;
    const int rows = min(MR, p.T - t0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rg = warp % RG, cw = warp / RG;
    const __nv_bfloat16* x = (const __nv_bfloat16*)p.x + p.x_off + (size_t)h * p.x_head + (size_t)t0 * p.x_stride;
    const __nv_bfloat16* w = (const __nv_bfloat16*)p.w + ((size_t)h * p.on + o0) * p.in;
    const uint32_t xb = smem_addr(xs), wb = smem_addr(ws);
    auto fetch = [&](int k0, int buf) {
        for (int i = threadIdx.x; i < (MR + HL_OT) * (HL_KB / 8); i += 128) {
            const int r = i / (HL_KB / 8), ch = i % (HL_KB / 8);
            const bool kin = k0 + ch * 8 < p.in;
            if (r < MR) {
                const bool ok = kin && r < rows;
                cp_async16(xb + buf * MR * HL_PITCH + r * HL_PITCH + ch * 16, x + (ok ? (size_t)r * p.x_stride + k0 + ch * 8 : 0), ok);
            } else {
                const int o = r - MR;
                const bool ok = kin && o0 + o < p.on;
                cp_async16(wb + buf * HL_OT * HL_PITCH + o * HL_PITCH + ch * 16, w + (ok ? (size_t)o * p.in + k0 + ch * 8 : 0), ok);
            }
        }
        cp_async_commit();
    };
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
    fetch(0, 0);
    int buf = 0;
    for (int k0 = 0; k0 < p.in; k0 += HL_KB, buf ^= 1) {
        if (k0 + HL_KB < p.in) {
            fetch(k0 + HL_KB, buf ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t xa = xb + buf * MR * HL_PITCH + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * HL_PITCH;
        const uint32_t wa = wb + buf * HL_OT * HL_PITCH;
#pragma unroll
        for (int ks = 0; ks < HL_KB / 16; ks += 2) {
            if (k0 + ks * 16 >= p.in) break;
            uint32_t a0[4], a1[4];
            ldmatrix_x4(xa + (ks * 2 + (lane >> 4)) * 16, a0);
            ldmatrix_x4(xa + (ks * 2 + 2 + (lane >> 4)) * 16, a1);
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                uint32_t b[4];
                ldmatrix_x4(wa + (cw * NT * 8 + i * 8 + (lane & 7)) * HL_PITCH + (ks * 2 + (lane >> 3)) * 16, b);
                mma_bf16(acc[i], a0, b[0], b[1]);
                mma_bf16(acc[i], a1, b[2], b[3]);
            }
        }
        __syncthreads();
    }
    __nv_bfloat16* out = (__nv_bfloat16*)p.out + (size_t)h * p.out_head;
    const bool pairs = p.on % 2 == 0 && p.out_stride % 2 == 0 && p.out_head % 2 == 0;          // 4-byte stores (out is 16-byte aligned)
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int o = o0 + cw * NT * 8 + i * 8 + (lane & 3) * 2;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int r = rg * 16 + (lane >> 2) + u * 8;
            if (r >= rows || o >= p.on) continue;
            __nv_bfloat16* d = out + (size_t)(t0 + r) * p.out_stride + o;
            if (pairs) {
                *reinterpret_cast<uint32_t*>(d) = pack_bf16(acc[i][2 * u], acc[i][2 * u + 1]);
            } else {
                d[0] = __float2bfloat16_rn(acc[i][2 * u]);
                if (o + 1 < p.on) d[1] = __float2bfloat16_rn(acc[i][2 * u + 1]);
            }
        }
    }
    if (p.rot_dim && blockIdx.z == 0) rotate_rows<__nv_bfloat16>(p, t0, rows, h);
}

}  // namespace

// x: row t, head h at x + t * x_stride + x_off + h * x_head, `in` numbers; w [H, on, in]; out: row t, head h at out + t *
// out_stride + h * out_head, `on` numbers (all of one dtype).  rot_dim > 0: the rot_dim numbers from rot_src on of a head of
// x are rotated (pairs (i, i + rot_dim / 2), or neighbours with `interleaved`; angle = positions[t] * inv_freq[i]) and
// written from rot_dst on into the head of out.
LLB_EXPORT int llb_head_linear_rotated(const void* x, long long x_stride, int x_off, long long x_head, const void* w, void* out,
                                       long long out_stride, long long out_head, int dtype, int T, int H, int in, int on,
                                       int rot_dim, int rot_src, int rot_dst, int interleaved, const int* positions,
                                       const float* inv_freq, cudaStream_t stream) {
    if (T == 0) return 0;
    LLB_REQUIRE(T > 0 && H > 0 && in > 0 && on > 0 && x && w && out, "head_linear: bad arguments");
    LLB_REQUIRE(rot_dim >= 0 && rot_dim % 2 == 0 && (rot_dim == 0 || (positions && inv_freq)), "head_linear: rotation of %d numbers", rot_dim);
    LLB_REQUIRE(H <= 65535, "head_linear: too many heads");
    HeadLinearParams p;
    p.x = x; p.x_stride = x_stride; p.x_off = x_off; p.x_head = x_head; p.w = w; p.out = out; p.out_stride = out_stride;
    p.out_head = out_head; p.T = T; p.H = H; p.in = in; p.on = on; p.rot_dim = rot_dim; p.rot_src = rot_src; p.rot_dst = rot_dst;
    p.interleaved = interleaved ? 1 : 0; p.positions = positions; p.inv_freq = inv_freq;
    if (dtype == LLB_BF16 && in % 8 == 0 && x_stride % 8 == 0 && x_off % 8 == 0 && x_head % 8 == 0 && (uintptr_t)x % 16 == 0 &&
        (uintptr_t)w % 16 == 0 && (uintptr_t)out % 16 == 0) {
        const int oz = (on + HL_OT - 1) / HL_OT;
        if (T <= 16) head_linear_mma_kernel<1><<<dim3((T + 15) / 16, H, oz), 128, 0, stream>>>(p);
        else head_linear_mma_kernel<4><<<dim3((T + 63) / 64, H, oz), 128, 0, stream>>>(p);
        return llb_check_launch("head_linear_mma");
    }
    const size_t smem = (size_t)HL_ROWS * in * sizeof(float);
    LLB_REQUIRE(smem <= 48 * 1024, "head_linear: %d input features per head need %zu bytes of shared memory", in, smem);
    const dim3 grid((T + HL_ROWS - 1) / HL_ROWS, H);
    // zero rows beyond the tile's end are never read: acc of such rows is dropped
    if (dtype == LLB_F32) head_linear_kernel<float><<<grid, 256, smem, stream>>>(p);
    else if (dtype == LLB_BF16) head_linear_kernel<__nv_bfloat16><<<grid, 256, smem, stream>>>(p);
    else return llb_fail("head_linear: unknown dtype %d", dtype);
    return llb_check_launch("head_linear");
}

// x: row t starts at x + t * x_stride + x_off and holds H*in values; w [H, on, in]; out [T, H*on].
LLB_EXPORT int llb_head_linear(const void* x, long long x_stride, int x_off, const void* w, void* out, int dtype, int T,
                               int H, int in, int on, cudaStream_t stream) {
    return llb_head_linear_rotated(x, x_stride, x_off, in, w, out, (long long)H * on, on, dtype, T, H, in, on, 0, 0, 0, 0,
                                   nullptr, nullptr, stream);
}
