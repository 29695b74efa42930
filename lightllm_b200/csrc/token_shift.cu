// Norms of one stream read by the branches of a parallel layer, in one pass over the rows, the first of them followed by a
// token shift:
//
//     h_t  = x_t / sqrt(mean(x_t^2) + eps) * w1
//     out1 = h_t + (h_(t-1) - h_t) * mix            h before a sequence's first token is zero
//     out2 = x_t / sqrt(mean(x_t^2) + eps) * w2     (optional: the other branch's norm; the statistics are the same)
//
// A request's last h lives in its state slot (float, D numbers).  The block of a span's first row is the only one that reads
// it, and that block also writes the new one (it norms the span's last row once more), so no two blocks of a launch touch
// the same slot.  Optionally the rows of a buffer are cleared (the float sum that the layer's branches add into).
// Everything is float; the outputs are rounded once.
#include "common.cuh"

namespace {

struct ShiftParams {
    const float* x;             // [T, D]
    const float* w1;            // [D]
    const float* mix;           // [D]
    const float* w2;            // [D] or null
    void* out1;                 // [T, D]
    void* out2;
    float* clear;               // [T, D] or null
    const int* span_row;
    const int* span_len;
    const int* span_pos;
    const int* span_slot;
    int num_spans, D;
    float* state;
    long long state_stride, state_off;
    float eps;
};

template <int V> __device__ __forceinline__ void load_row(const float* p, float (&v)[V]) {
    if (V == 4) {
        const float4 q = *reinterpret_cast<const float4*>(p);
        v[0] = q.x; v[1 % V] = q.y; v[2 % V] = q.z; v[3 % V] = q.w;
    } else {
        v[0] = *p;
    }
}
template <typename TO, int V> __device__ __forceinline__ void store_row(TO* p, const float (&v)[V]) {
    TO r[V];
#pragma unroll
    for (int i = 0; i < V; ++i) r[i] = llb_from_float<TO>(v[i]);
    if (V == 4 && sizeof(TO) == 4) *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(r);
    else if (V == 4) *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(r);
    else *p = r[0];
}

// One block a row: the row and the one before it are read once for the sums of squares and again (from cache) for the result.
template <typename TO, int V>
__global__ void __launch_bounds__(256) norm_shift_kernel(ShiftParams p) {
    const int t = blockIdx.x, D = p.D;
    int lo = 0, hi = p.num_spans - 1;          // the last span whose first row is <= t
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (p.span_row[mid] <= t) lo = mid;
        else hi = mid - 1;
    }
    const int row0 = p.span_row[lo], len = p.span_len[lo];
    const bool first = t == row0, fresh = p.span_pos[lo] == 0;
    const int last = row0 + len - 1;
    float* kept = p.state + (long long)p.span_slot[lo] * p.state_stride + p.state_off;
    const float* xt = p.x + (size_t)t * D;
    const float* xo = first ? p.x + (size_t)last * D : xt - D;          // the row before, or (first row) the span's last
    float ss = 0.0f, so = 0.0f;
    for (int d = threadIdx.x * V; d < D; d += blockDim.x * V) {
        float a[V], b[V];
        load_row<V>(xt + d, a);
        load_row<V>(xo + d, b);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            ss = fmaf(a[i], a[i], ss);
            so = fmaf(b[i], b[i], so);
        }
    }
    __shared__ float part[2][8];
    ss = llb_warp_sum(ss);
    so = llb_warp_sum(so);
    if ((threadIdx.x & 31) == 0) {
        part[0][threadIdx.x >> 5] = ss;
        part[1][threadIdx.x >> 5] = so;
    }
    __syncthreads();
    ss = so = 0.0f;
    for (int i = 0; i < (int)(blockDim.x >> 5); ++i) {
        ss += part[0][i];
        so += part[1][i];
    }
    const float inv = 1.0f / sqrtf(ss / (float)D + p.eps), invo = 1.0f / sqrtf(so / (float)D + p.eps);
    TO* o1 = (TO*)p.out1 + (size_t)t * D;
    TO* o2 = (TO*)p.out2 + (size_t)t * D;
    for (int d = threadIdx.x * V; d < D; d += blockDim.x * V) {
        float a[V], b[V], w[V], m[V], h[V], o[V];
        load_row<V>(xt + d, a);
        load_row<V>(p.w1 + d, w);
        load_row<V>(p.mix + d, m);
        load_row<V>(xo + d, b);
        if (first) {
            float k[V];
#pragma unroll
            for (int i = 0; i < V; ++i) k[i] = 0.0f;
            if (!fresh) load_row<V>(kept + d, k);
            float keep[V];
#pragma unroll
            for (int i = 0; i < V; ++i) {
                keep[i] = b[i] * invo * w[i];          // the span's last h: the request's new record
                b[i] = k[i];
            }
            store_row<float, V>(kept + d, keep);
        } else {
#pragma unroll
            for (int i = 0; i < V; ++i) b[i] = b[i] * invo * w[i];
        }
#pragma unroll
        for (int i = 0; i < V; ++i) {
            h[i] = a[i] * inv * w[i];
            o[i] = fmaf(b[i] - h[i], m[i], h[i]);
        }
        store_row<TO, V>(o1 + d, o);
        if (p.w2) {
            load_row<V>(p.w2 + d, w);
#pragma unroll
            for (int i = 0; i < V; ++i) o[i] = a[i] * inv * w[i];
            store_row<TO, V>(o2 + d, o);
        }
        if (p.clear) {
#pragma unroll
            for (int i = 0; i < V; ++i) o[i] = 0.0f;
            store_row<float, V>(p.clear + (size_t)t * D + d, o);
        }
    }
}

template <typename TO>
int launch_norm_shift(const ShiftParams& p, int T, cudaStream_t stream) {
    const bool vec = p.D % 4 == 0 && p.state_stride % 4 == 0 && p.state_off % 4 == 0 && (uintptr_t)p.state % 16 == 0 &&
                     (uintptr_t)p.x % 16 == 0 && (uintptr_t)p.w1 % 16 == 0 && (uintptr_t)p.w2 % 16 == 0 && (uintptr_t)p.mix % 16 == 0 &&
                     (uintptr_t)p.out1 % 16 == 0 && (uintptr_t)p.out2 % 16 == 0 && (uintptr_t)p.clear % 16 == 0;
    const int per = vec ? 4 : 1;
    int threads = 32 * ((p.D / per + 31) / 32);
    threads = threads > 256 ? 256 : threads < 32 ? 32 : threads;
    if (vec) norm_shift_kernel<TO, 4><<<T, threads, 0, stream>>>(p);
    else norm_shift_kernel<TO, 1><<<T, threads, 0, stream>>>(p);
    return llb_check_launch("norm_shift");
}

}  // namespace

// x float [T, D]; w1, mix float [D], w2 float [D] or null; out1 (and out2 with w2) [T, D] float or bf16; clear float [T, D]
// or null; spans as in every kernel of a step; state: float base of the state plane, `state_stride` floats a slot, a
// request's last h [D] at `state_off` inside its slot.
LLB_EXPORT int llb_norm_shift(const float* x, const float* w1, const float* mix, const float* w2, void* out1, void* out2,
                              int out_dtype, float* clear, int T, int D, float eps, const int* span_row, const int* span_len,
                              const int* span_pos, const int* span_slot, int num_spans, float* state, long long state_stride,
                              long long state_off, cudaStream_t stream) {
    if (T == 0) return 0;
    LLB_REQUIRE(T > 0 && D > 0 && x && w1 && mix && out1 && (!w2 || out2) && span_row && span_len && span_pos && span_slot &&
                num_spans > 0 && state, "norm_shift: bad arguments");
    ShiftParams p;
    p.x = x; p.w1 = w1; p.mix = mix; p.w2 = w2; p.out1 = out1; p.out2 = out2; p.clear = clear; p.span_row = span_row;
    p.span_len = span_len; p.span_pos = span_pos; p.span_slot = span_slot; p.num_spans = num_spans; p.D = D;
    p.state = state; p.state_stride = state_stride; p.state_off = state_off; p.eps = eps;
    if (out_dtype == LLB_F32) return launch_norm_shift<float>(p, T, stream);
    if (out_dtype == LLB_BF16) return launch_norm_shift<__nv_bfloat16>(p, T, stream);
    return llb_fail("norm_shift: unknown dtype %d", out_dtype);
}
