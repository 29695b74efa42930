// Attention over a cached latent (see latent_attention.cu) for prompt portions on the 5th-generation tensor cores, bf16.
//
// All heads share the key rows, so the rows of a tile are (token, head) pairs: 128 consecutive pairs f = token * H + head of
// one span, which lie one behind the other in q [T * H, W] and in out [T * H, r].  A block takes one tile over all keys that
// any of its pairs sees, 64 at a time (tiles begin at multiples of 64 positions, so a row's arithmetic does not depend on
// how the tokens were cut).  Three roles:
//   loader     TMA: the pairs' q once, then the key tiles page by page, as many stages ahead as the shared memory holds
//   MMA warp   S = Q K^T of the next tile (64 columns of tensor memory, two buffers), then O += P V of this one; V is the
//              key tile itself, its first r columns as the MN-major operand, so a key row is copied once
//   softmax    four warps, a thread a row: scores from tensor memory, masks, P (bf16) into the swizzled A-operand tile.  The
//              output stays in tensor memory; a row's reference maximum moves (and its output is rescaled there) only when
//              the maximum has grown by more than 2^8 since, which leaves the result exact: probabilities and their sum share
//              the reference
// S of tile j + 1 is computed while the softmax warps work on tile j.  Two commits a tile: behind S and behind P V.
// Every wait is bounded in time; when one runs out the block raises the error flag, walks through the rest without work,
// frees its tensor memory and returns.
//
// W and r multiples of 8, r at most 256, page sizes 8, 16, 32 and 64.
#include <math.h>

#include "tcgen05_common.cuh"
#include "warp_mma.cuh"

namespace {

using namespace t5;
using wm::fast_exp2;

constexpr int MR = 128;                     // pairs a block = TMEM lanes
constexpr int BK = 64;                      // keys a tile
constexpr int THREADS = 192;
constexpr int MMA_WARP = 4, LOAD_WARP = 5;
constexpr int MAX_STAGES = 4;
constexpr uint32_t QBLK = MR * 128, KBLK = BK * 128;          // bytes of a 64-column block of q and of a key tile
constexpr float LAZY = 8.0f;                // a row's reference maximum moves when the maximum has grown by more than this (base 2)

struct LatentTcParams {
    __nv_bfloat16* out;                     // [T * H, r]
    const int* span_row;
    const int* span_len;
    const int* span_pos;
    const int* block_table;                 // [S, max_pages]
    int num_spans, max_pages, page_size, H, W, r, window, num_slots, kblocks, stages, vcols, tmem_cols;
    float scale_log2e;
    const float* sinks;                     // [H] or null
    uint32_t dynamic_smem_bytes;
    int* error_flag;
};

__device__ __forceinline__ void tmem_st32(uint32_t taddr, const float (&v)[32]) {
    const uint32_t* u = reinterpret_cast<const uint32_t*>(v);
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%32], "
        "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
        "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31};"
        ::"r"(u[0]), "r"(u[1]), "r"(u[2]), "r"(u[3]), "r"(u[4]), "r"(u[5]), "r"(u[6]), "r"(u[7]),
          "r"(u[8]), "r"(u[9]), "r"(u[10]), "r"(u[11]), "r"(u[12]), "r"(u[13]), "r"(u[14]), "r"(u[15]),
          "r"(u[16]), "r"(u[17]), "r"(u[18]), "r"(u[19]), "r"(u[20]), "r"(u[21]), "r"(u[22]), "r"(u[23]),
          "r"(u[24]), "r"(u[25]), "r"(u[26]), "r"(u[27]), "r"(u[28]), "r"(u[29]), "r"(u[30]), "r"(u[31]), "r"(taddr)
        : "memory");
}
__device__ __forceinline__ void tmem_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

__global__ void __launch_bounds__(THREADS, 1)
latent_attention_tcgen05_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const LatentTcParams p) {
    __shared__ __align__(8) uint64_t bars[5 + 2 * MAX_STAGES];
    __shared__ uint32_t tmem_slot;
    __shared__ int abort_s;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    const int KB = p.kblocks, ST = p.stages, H = p.H;
    uint8_t* q_s = smem;                              // KB blocks
    uint8_t* k_s = q_s + KB * QBLK;                   // ST x KB blocks
    uint8_t* p_s = k_s + ST * KB * KBLK;              // [128][64] bf16, swizzled
    uint64_t* q_full = &bars[0];
    uint64_t* s_full = &bars[1];                      // [2]
    uint64_t* p_full = &bars[3];                      // the four softmax warps have written P (and read S)
    uint64_t* pv_done = &bars[4];                     // P V of a tile has been computed
    uint64_t* k_full = &bars[5];                      // [ST]
    uint64_t* k_free = &bars[5 + MAX_STAGES];         // [ST]
    volatile int* abort_flag = &abort_s;

    // which pairs (the grid is an upper bound of the spans' tiles)
    int span = 0, fb = blockIdx.x;
    while (span < p.num_spans) {
        const int n = (p.span_len[span] * H + MR - 1) / MR;
        if (fb < n) break;
        fb -= n;
        ++span;
    }
    if (span >= p.num_spans) return;                  // uniform over the block, before anything is allocated
    if (p_s + QBLK > smem_raw + p.dynamic_smem_bytes) {
        if (threadIdx.x == 0 && p.error_flag) atomicExch(p.error_flag, 3);
        return;
    }
    const int f0 = fb * MR, pairs = min(MR, p.span_len[span] * H - f0);
    const int row0 = p.span_row[span], pos0 = p.span_pos[span];
    const int first_pos = pos0 + f0 / H, hi = pos0 + (f0 + pairs - 1) / H + 1;          // keys [lo, hi) can be visible
    const int lo = llb_first_visible(first_pos, p.window);
    const int inner_lo = llb_first_visible(hi - 1, p.window);                          // every pair sees [inner_lo, first_pos]
    const int kt0 = lo / BK * BK, n = (hi - kt0 + BK - 1) / BK;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        mbar_init(&s_full[0], 1);
        mbar_init(&s_full[1], 1);
        mbar_init(p_full, 4);
        mbar_init(pv_done, 1);
        for (int i = 0; i < MAX_STAGES; ++i) {
            mbar_init(&k_full[i], 1);
            mbar_init(&k_free[i], 1);
        }
        *abort_flag = 0;
        mbar_init_fence();
    }
    if (warp == 0) tmem_alloc(&tmem_slot, p.tmem_cols);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;

    if (warp == LOAD_WARP) {
        // ---- loader ------------------------------------------------------------------------------
        bool ok = true;
        if (lane == 0) {
            mbar_expect_tx(q_full, KB * QBLK);
            for (int kb = 0; kb < KB; ++kb) tma_load_2d(q_s + kb * QBLK, &map_q, kb * 64, row0 * H + f0, q_full);
        }
        __syncwarp();
        const int* bt = p.block_table + (size_t)span * p.max_pages;
        const int ppt = BK / p.page_size;
        int st = 0, round = 0;
        for (int j = 0; j < n; ++j) {
            // page numbers first: their latency lies under the wait for the stage; only pages that hold keys of [lo, hi)
            const int lp = (kt0 + j * BK) / p.page_size + lane;
            const bool holds = lp * p.page_size < hi && (lp + 1) * p.page_size > lo;
            const int page = (lane < ppt && lp < p.max_pages && holds) ? bt[lp] : -1;
            if (round > 0) ok = mbar_wait(&k_free[st], (round - 1) & 1, abort_flag) && ok;
            ok = __all_sync(0xffffffffu, ok);
            if (ok) {
                if (lane == 0) mbar_expect_tx(&k_full[st], KB * KBLK);
                __syncwarp();
                if (lane < ppt) {
                    const int y = page >= 0 ? page * p.page_size : p.num_slots;          // out of range: the box is zero-filled
                    uint8_t* dst = k_s + (size_t)st * KB * KBLK + lane * p.page_size * 128;
                    for (int kb = 0; kb < KB; ++kb) tma_load_2d(dst + kb * KBLK, &map_k, kb * 64, y, &k_full[st]);
                }
                __syncwarp();
            }
            if (++st == ST) {
                st = 0;
                ++round;
            }
        }
    } else if (warp == MMA_WARP) {
        // ---- tensor-core instructions ----------------------------------------------------------------
        const uint32_t idesc_s = idesc_bf16(MR, BK, 0), idesc_pv = idesc_bf16(MR, p.vcols, 1);
        const int ksteps = (p.W + 15) / 16;
        const uint32_t qa = smem_u32(q_s), ka = smem_u32(k_s), pa = smem_u32(p_s);
        bool ok = mbar_wait(q_full, 0, abort_flag);
        auto issue_s = [&](int st, int buf) {
            tc_fence_after();
            const uint32_t kst = ka + st * KB * KBLK, d = tmem + buf * BK;
            for (int ks = 0; ks < ksteps; ++ks)
                umma_bf16(d, desc_kmajor(qa + (ks >> 2) * QBLK + (ks & 3) * 32), desc_kmajor(kst + (ks >> 2) * KBLK + (ks & 3) * 32), idesc_s,
                          ks > 0 ? 1u : 0u);
        };
        int st = 0, next = 0, next_round = 0;          // stage of tile j, of tile j + 1
        ok = mbar_wait(&k_full[0], 0, abort_flag) && ok;
        ok = __all_sync(0xffffffffu, ok);
        if (lane == 0 && ok) {
            issue_s(0, 0);
            umma_commit(&s_full[0]);
        }
        __syncwarp();
        for (int j = 0; j < n; ++j) {
            if (++next == ST) {
                next = 0;
                ++next_round;
            }
            if (j + 1 < n) {
                ok = mbar_wait(&k_full[next], next_round & 1, abort_flag) && ok;
                ok = __all_sync(0xffffffffu, ok);
                if (lane == 0 && ok) {
                    issue_s(next, (j + 1) & 1);
                    umma_commit(&s_full[(j + 1) & 1]);
                }
                __syncwarp();
            }
            ok = mbar_wait(p_full, j & 1, abort_flag) && ok;
            ok = __all_sync(0xffffffffu, ok);
            if (lane == 0 && ok) {
                tc_fence_after();
                const uint32_t vst = ka + st * KB * KBLK;
#pragma unroll
                for (int k = 0; k < BK / 16; ++k)
                    umma_bf16(tmem + 2 * BK, desc_kmajor(pa + k * 32), desc_mnmajor(vst + k * 16 * 128, KBLK), idesc_pv, (j > 0 || k > 0) ? 1u : 0u);
                umma_commit(pv_done);
            }
            __syncwarp();
            st = next;
        }
    } else {
        // ---- softmax ---------------------------------------------------------------------------------
        const int m = threadIdx.x;                                    // pair of this thread = TMEM lane
        const uint32_t lanes = tmem + ((uint32_t)(warp * 32) << 16), t_o = lanes + 2 * BK;
        const int qpos = m < pairs ? pos0 + (f0 + m) / H : -1;          // (a row beyond the pairs sees nothing)
        const int qlo = m < pairs ? llb_first_visible(qpos, p.window) : 0;
        uint8_t* prow = p_s + m * 128;
        float m_run = -INFINITY, l_run = 0.0f;
        bool ok = true;
        int st = 0;                                                   // stage of tile j
        for (int j = 0; j < n; ++j) {
            const int kt = kt0 + j * BK;
            ok = mbar_wait(&s_full[j & 1], (j >> 1) & 1, abort_flag) && ok;
            __syncwarp();
            tc_fence_after();
            if (kt + BK > hi && m < BK && kt + m >= hi) {
                // rows that no token has written yet (what an earlier owner of the page left): their probabilities are exact
                // zeros, and zero times anything must stay zero.  S is complete, so the tile has landed.
                for (int kb = 0; kb < KB; ++kb) {
                    uint4* v = reinterpret_cast<uint4*>(k_s + ((size_t)st * KB + kb) * KBLK + m * 128);
#pragma unroll
                    for (int q = 0; q < 8; ++q) v[q] = make_uint4(0u, 0u, 0u, 0u);
                }
            }
            float s[64];
            tmem_ld32_nowait(lanes + (j & 1) * BK, *reinterpret_cast<uint32_t(*)[32]>(&s[0]));
            tmem_ld32_nowait(lanes + (j & 1) * BK + 32, *reinterpret_cast<uint32_t(*)[32]>(&s[32]));
            tmem_wait_ld();
            const bool interior = kt >= inner_lo && kt + BK - 1 <= first_pos;          // uniform over the block
            float t0 = -INFINITY, t1 = -INFINITY, t2 = -INFINITY, t3 = -INFINITY;
            if (interior) {
#pragma unroll
                for (int i = 0; i < 64; ++i) s[i] *= p.scale_log2e;
            } else {
                const int c_lo = qlo - kt, c_hi = qpos - kt;
#pragma unroll
                for (int i = 0; i < 64; ++i) s[i] = (i >= c_lo && i <= c_hi) ? s[i] * p.scale_log2e : -INFINITY;
            }
#pragma unroll
            for (int i = 0; i < 64; i += 4) {
                t0 = fmaxf(t0, s[i]); t1 = fmaxf(t1, s[i + 1]); t2 = fmaxf(t2, s[i + 2]); t3 = fmaxf(t3, s[i + 3]);
            }
            const float m_tile = fmaxf(fmaxf(t0, t1), fmaxf(t2, t3));
            float factor = 1.0f;
            if (m_run == -INFINITY) {
                m_run = m_tile;                                       // nothing accumulated yet
            } else if (m_tile > m_run + LAZY) {
                factor = fast_exp2(m_run - m_tile);
                m_run = m_tile;
            }
            const float m_use = m_run == -INFINITY ? 0.0f : m_run;
            l_run *= factor;
            float l0 = 0.0f, l1 = 0.0f;
            uint32_t w[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                const float p0 = fast_exp2(s[2 * i] - m_use), p1 = fast_exp2(s[2 * i + 1] - m_use);
                l0 += p0;
                l1 += p1;
                w[i] = wm::pack_bf16(p0, p1);
            }
            l_run += l0 + l1;
            if (j > 0) {                                              // P is free and O stands still
                ok = mbar_wait(pv_done, (j - 1) & 1, abort_flag) && ok;
                __syncwarp();
                tc_fence_after();
                if (threadIdx.x == 0) mbar_arrive(&k_free[st == 0 ? ST - 1 : st - 1]);
                if (__any_sync(0xffffffffu, factor != 1.0f)) {
                    for (int c = 0; c < p.vcols; c += 32) {
                        float o[32];
                        tmem_ld32(t_o + c, o);
#pragma unroll
                        for (int i = 0; i < 32; ++i) o[i] *= factor;
                        tmem_st32(t_o + c, o);
                    }
                    tmem_wait_st();
                }
            }
#pragma unroll
            for (int q = 0; q < 8; ++q)
                *reinterpret_cast<uint4*>(prow + ((q ^ (m & 7)) * 16)) = make_uint4(w[4 * q], w[4 * q + 1], w[4 * q + 2], w[4 * q + 3]);
            fence_async_smem();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
            if (++st == ST) st = 0;
        }
        ok = mbar_wait(pv_done, (n - 1) & 1, abort_flag) && ok;
        __syncwarp();
        tc_fence_after();
        float den = l_run;
        if (p.sinks && m < pairs) den += exp2f(p.sinks[(f0 + m) % H] * 1.4426950408889634f - m_run);
        const float inv = 1.0f / den;
        __nv_bfloat16* dst = p.out + ((size_t)row0 * H + f0 + m) * p.r;
        for (int c = 0; c < p.vcols; c += 32) {
            float o[32];
            tmem_ld32(t_o + c, o);
            if (ok && m < pairs) {
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (c + q * 8 < p.r)
                        *reinterpret_cast<uint4*>(dst + c + q * 8) =
                            make_uint4(wm::pack_bf16(o[8 * q] * inv, o[8 * q + 1] * inv), wm::pack_bf16(o[8 * q + 2] * inv, o[8 * q + 3] * inv),
                                       wm::pack_bf16(o[8 * q + 4] * inv, o[8 * q + 5] * inv), wm::pack_bf16(o[8 * q + 6] * inv, o[8 * q + 7] * inv));
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag && threadIdx.x == 0 && p.error_flag) atomicExch(p.error_flag, 2);
    if (warp == 0) {
        tc_fence_after();
        tmem_dealloc(tmem, p.tmem_cols);
    }
}

// Stages of key tiles that fit beside q and P, or 0.
inline int latent_stages(int W) {
    const int kb = (W + 63) / 64;
    const long long left = 227ll * 1024 - 1024 - 256 - (long long)kb * QBLK - QBLK;
    const int st = (int)(left / ((long long)kb * KBLK));
    return left <= 0 ? 0 : st > MAX_STAGES ? MAX_STAGES : st;
}

}  // namespace

// Whether the kernel takes key rows of W numbers whose first r are the values, in pages of page_size rows.
LLB_EXPORT int llb_latent_attention_tcgen05_supports(int W, int r, int page_size) {
    return W % 8 == 0 && r % 8 == 0 && r > 0 && r <= W && r <= 256 && (page_size == 8 || page_size == 16 || page_size == 32 || page_size == 64) &&
           latent_stages(W) >= 2;
}

// q [T, H, W], cache [num_slots, W], out [T, H, r], all bf16; spans, block tables, window and sinks as llb_latent_attention.
LLB_EXPORT int llb_latent_attention_tcgen05(const void* q, const void* cache, void* out, int T, const int* span_row,
                                            const int* span_len, const int* span_pos, int num_spans, const int* block_table,
                                            int max_pages, int page_size, int num_slots, int H, int W, int r, int window,
                                            float scale, const float* sinks, int* error_flag, cudaStream_t stream) {
    if (T == 0) return 0;
    LLB_REQUIRE(T > 0 && num_spans > 0 && H > 0 && q && cache && out && span_row && span_len && span_pos && block_table &&
                max_pages > 0 && num_slots > 0, "latent_attention_tcgen05: bad arguments");
    LLB_REQUIRE(llb_latent_attention_tcgen05_supports(W, r, page_size), "latent_attention_tcgen05: key rows of %d with values of %d in "
                "pages of %d are not supported", W, r, page_size);
    LLB_REQUIRE(((uintptr_t)q % 16 == 0) && ((uintptr_t)cache % 16 == 0) && ((uintptr_t)out % 16 == 0), "latent_attention_tcgen05: alignment");
    const long long tiles = (long long)T * H / MR + num_spans;
    LLB_REQUIRE((long long)T * H < (1ll << 31), "latent_attention_tcgen05: too many rows");
    CUtensorMap mq, mk;
    int rc;
    if ((rc = make_map_bf16(q, (long long)T * H, W, MR, &mq))) return rc;
    if ((rc = make_map_bf16(cache, num_slots, W, page_size, &mk))) return rc;
    LatentTcParams p;
    p.out = (__nv_bfloat16*)out; p.span_row = span_row; p.span_len = span_len; p.span_pos = span_pos; p.block_table = block_table;
    p.num_spans = num_spans; p.max_pages = max_pages; p.page_size = page_size; p.H = H; p.W = W; p.r = r; p.window = window;
    p.num_slots = num_slots; p.kblocks = (W + 63) / 64; p.stages = latent_stages(W); p.vcols = (r + 63) / 64 * 64;
    p.tmem_cols = 2 * BK + p.vcols <= 256 ? 256 : 512; p.scale_log2e = scale * 1.4426950408889634f; p.sinks = sinks;
    p.error_flag = error_flag;
    const size_t smem = (size_t)p.kblocks * QBLK + (size_t)p.stages * p.kblocks * KBLK + QBLK + 1024;
    p.dynamic_smem_bytes = (uint32_t)smem;
    static size_t configured = 0;
    if (smem > configured) {
        const cudaError_t e = cudaFuncSetAttribute(latent_attention_tcgen05_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return llb_fail("latent_attention_tcgen05: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured = smem;
    }
    latent_attention_tcgen05_kernel<<<(unsigned)tiles, THREADS, smem, stream>>>(mq, mk, p);
    return llb_check_launch("latent_attention_tcgen05");
}
