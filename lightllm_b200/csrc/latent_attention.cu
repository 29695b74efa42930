// Attention over a cached low-rank latent with a rotated key part shared by all heads: every query head reads ONE key row a
// token, [latent (r) | rotated part], and its value row is the first r numbers of it, so only that row is cached.
//
// `llb_latent_prepare`: the norms, the rotation and the cache write between the layer's projections.
//
// `llb_latent_attention`: the attention itself for bf16 on tensor cores (mma.sync over cp.async tiles), prompt portions and
// single tokens alike.  All heads share the keys, so the rows of a tile are (token, head) pairs: pair f of a span is token
// f / H, head f % H, and a block takes 16 * RG consecutive pairs (RG = 1, 2 or 4) of one span over all keys that any of
// them sees, 64 at a time (tiles begin at multiples of 64 positions, so a row's arithmetic does not depend on how the
// tokens were cut).  Eight warps: RG along the rows, 8 / RG along the columns.
//     S = Q K^T     a warp takes its 16 rows and 64 * RG / 8 of the tile's keys; Q and K from shared memory by ldmatrix
//     softmax       the column warps of a row group agree on the row maxima through shared memory; P (bf16) goes back to
//                   shared memory; a column warp sums its own keys' probabilities
//     O += P V      a warp takes its 16 rows and r * RG / 8 of the value columns; V is the K tile itself, read transposed
// A key tile is copied once for scores and values.  Two tile buffers: the next tile arrives while one is computed.  With
// few rows the key range is cut into up to 8 pieces, the blocks of one thread-block cluster, which merge through
// distributed shared memory.  Scores, maxima, sums and the accumulated output are float.
#include <math.h>

#include "common.cuh"
#include "warp_mma.cuh"

namespace {

using namespace wm;

// ---------------------------------------------------------------------------------------------------------------------
struct LatentPrepareParams {
    const void* src;            // [T, stride]: query latent (q_rank) at q_off, latent (r) at c_off, rotated part (rd) at rot_off
    long long stride;
    int q_off, c_off, rot_off, q_rank, r, rd, interleaved;
    const float* q_w;           // [q_rank]
    const float* c_w;           // [r]
    const float* inv_freq;      // [rd / 2]
    const int* positions;       // [T]
    const int* slots;           // [T] cache row of each token (negative: not written)
    void* q_out;                // [T, q_rank] or null
    void* cache;                // [slots, r + rd] or null
    float eps;
};

// One block a token: RMS norms of both latents (float), the rotation, the cache row.
template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(LatentPrepareParams p) {
    const int t = blockIdx.x;
    const T* row = (const T*)p.src + (size_t)t * p.stride;
    float sq = 0.0f, sc = 0.0f;
    for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) {
        const float v = llb_to_float(row[p.q_off + i]);
        sq = fmaf(v, v, sq);
    }
    for (int i = threadIdx.x; i < p.r; i += blockDim.x) {
        const float v = llb_to_float(row[p.c_off + i]);
        sc = fmaf(v, v, sc);
    }
    __shared__ float part[2][4];
    sq = llb_warp_sum(sq);
    sc = llb_warp_sum(sc);
    if ((threadIdx.x & 31) == 0) {
        part[0][threadIdx.x >> 5] = sq;
        part[1][threadIdx.x >> 5] = sc;
    }
    __syncthreads();
    sq = (part[0][0] + part[0][1]) + (part[0][2] + part[0][3]);
    sc = (part[1][0] + part[1][1]) + (part[1][2] + part[1][3]);
    if (p.q_out) {
        const float inv = 1.0f / sqrtf(sq / (float)p.q_rank + p.eps);
        T* o = (T*)p.q_out + (size_t)t * p.q_rank;
        for (int i = threadIdx.x; i < p.q_rank; i += blockDim.x) o[i] = llb_from_float<T>(llb_to_float(row[p.q_off + i]) * inv * p.q_w[i]);
    }
    if (!p.cache || p.slots[t] < 0) return;
    T* c = (T*)p.cache + (size_t)p.slots[t] * (p.r + p.rd);
    const float inv = 1.0f / sqrtf(sc / (float)p.r + p.eps);
    for (int i = threadIdx.x; i < p.r; i += blockDim.x) c[i] = llb_from_float<T>(llb_to_float(row[p.c_off + i]) * inv * p.c_w[i]);
    const int half = p.rd >> 1;
    for (int j = threadIdx.x; j < half; j += blockDim.x) {
        const int a = p.interleaved ? 2 * j : j, b = p.interleaved ? 2 * j + 1 : j + half;
        const float angle = (float)p.positions[t] * p.inv_freq[j];
        const float cs = cosf(angle), sn = sinf(angle);
        const float u = llb_to_float(row[p.rot_off + a]), v = llb_to_float(row[p.rot_off + b]);
        c[p.r + a] = llb_from_float<T>(u * cs - v * sn);
        c[p.r + b] = llb_from_float<T>(v * cs + u * sn);
    }
}

// ---------------------------------------------------------------------------------------------------------------------
constexpr int LBK = 64;                     // keys a tile
constexpr int LPP = LBK * 2 + 16;           // bytes a row of P
constexpr int LTHREADS = 256;
constexpr int LMAX_SPLITS = 8;

struct LatentParams {
    const __nv_bfloat16* q;                 // [T, H, W]
    const __nv_bfloat16* cache;             // [slots, W]
    __nv_bfloat16* out;                     // [T, H, r]
    const int* span_row;
    const int* span_len;
    const int* span_pos;
    const int* block_table;                 // [S, max_pages]
    int T, num_spans, max_pages, page_size, H, W, r, window, nsplit, blocks_per_span;
    float scale_log2e;
    const float* sinks;                     // [H] or null
    int pitch;                              // bytes a row of Q and K in shared memory: W rounded up to 32, plus 8, times 2
};

__device__ __forceinline__ float l_ld_cluster(uint32_t local, uint32_t rank) {
    uint32_t remote;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(rank));
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
    return v;
}
__device__ __forceinline__ void l_cluster_sync() {          // a hardware barrier: every block passes both on every path
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

// RG: row groups of 16 pairs; NTW: the most value n-tiles (8 columns each) a warp owns (even); CLUSTER: the key range is cut.
template <int RG, int NTW, bool CLUSTER>
__global__ void __launch_bounds__(LTHREADS) latent_attention_kernel(LatentParams p) {
    constexpr int CW = 8 / RG, MR = 16 * RG, NK = 8 / CW;          // NK: key n-tiles (8 keys each) a warp scores
    extern __shared__ __align__(16) uint8_t smem[];
    const int pitch = p.pitch, H = p.H, W = p.W;
    // which pairs: blocks_per_span > 0: every span has as many blocks; else walk the spans
    int span = 0, fb;
    if (p.blocks_per_span > 0) {
        span = blockIdx.x / p.blocks_per_span;
        fb = blockIdx.x - span * p.blocks_per_span;
    } else {
        fb = blockIdx.x;
        while (span < p.num_spans) {
            const int n = (p.span_len[span] * H + MR - 1) / MR;
            if (fb < n) break;
            fb -= n;
            ++span;
        }
        if (span >= p.num_spans) return;          // (the grid is an upper bound; no cluster in this case)
    }
    const int f0 = fb * MR, pairs = min(MR, p.span_len[span] * H - f0);
    const int row0 = p.span_row[span], pos0 = p.span_pos[span];
    const int* bt = p.block_table + (size_t)span * p.max_pages;
    const int hi = pos0 + (f0 + pairs - 1) / H + 1;                // keys [lo, hi) can be visible
    const int first_pos = pos0 + f0 / H;
    const int lo = llb_first_visible(first_pos, p.window);
    const int inner_lo = llb_first_visible(hi - 1, p.window);      // every pair sees the keys [inner_lo, first_pos]
    int kt0 = lo / LBK * LBK, kend = hi;
    if (CLUSTER) {          // whole tiles a piece; a piece may be empty
        const int tiles = (hi - kt0 + LBK - 1) / LBK, per = (tiles + p.nsplit - 1) / p.nsplit;
        kt0 += (int)blockIdx.y * per * LBK;
        kend = min(hi, kt0 + per * LBK);
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rg = warp % RG, cw = warp / RG;
    uint8_t* q_s = smem;                                           // [MR][pitch]
    uint8_t* k_s = q_s + MR * pitch;                               // 2 x [LBK][pitch]
    uint8_t* p_s = k_s + 2 * LBK * pitch;                          // [MR][LPP]
    float* mx = reinterpret_cast<float*>(p_s + MR * LPP);          // [CW][MR]
    const uint32_t qb = smem_addr(q_s), kb = smem_addr(k_s), pb = smem_addr(p_s);
    const int chunks = W >> 3, padded = (pitch >> 4) - 1;          // 16-byte pieces of a row, and with the zero columns

    // Q rows (zeros beyond the pairs and beyond W)
    for (int i = threadIdx.x; i < MR * padded; i += LTHREADS) {
        const int m = i / padded, ch = i - m * padded;
        const int f = f0 + m, tok = f / H, h = f - tok * H;
        const bool ok = m < pairs && ch < chunks;
        cp_async16(qb + m * pitch + ch * 16, p.q + (ok ? ((size_t)(row0 + tok) * H + h) * W + ch * 8 : 0), ok);
    }
    // Key rows: four threads a row
    const int krow = threadIdx.x >> 2, kch = threadIdx.x & 3;
    auto slot_of = [&](int kt) -> int {
        const int kpos = kt + krow;
        if (kpos < lo || kpos >= hi || kt >= kend) return -1;      // outside the visible range: zeros, never read
        return bt[kpos / p.page_size] * p.page_size + kpos % p.page_size;
    };
    auto issue = [&](int buf, int slot) {
        const bool ok = slot >= 0;
        const __nv_bfloat16* src = p.cache + (size_t)(ok ? slot : 0) * W;
        const uint32_t dst = kb + (buf * LBK + krow) * pitch;
        for (int ch = kch; ch < padded; ch += 4) cp_async16(dst + ch * 16, src + (ch < chunks ? ch * 8 : 0), ok && ch < chunks);
        cp_async_commit();
    };
    issue(0, slot_of(kt0));
    int slot_next = slot_of(kt0 + LBK);

    // this thread's two rows of the row group: pair -> query position
    const int r0 = lane >> 2, c0 = (lane & 3) * 2;
    int qlo[2], qpos[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int m = rg * 16 + r0 + u * 8;
        qpos[u] = m < pairs ? pos0 + (f0 + m) / H : -1;            // (a row beyond the pairs sees nothing)
        qlo[u] = m < pairs ? llb_first_visible(qpos[u], p.window) : 0;
    }
    float o[NTW][4];
#pragma unroll
    for (int i = 0; i < NTW; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};          // l: over this warp's keys only
    const int col0 = cw * NTW * 8;                                 // first value column of this warp
    const int ksteps = (W + 15) / 16;
    int buf = 0;
    for (int kt = kt0; kt < kend; kt += LBK, buf ^= 1) {
        if (kt + LBK < kend) {
            issue(buf ^ 1, slot_next);          // (last read before the barrier that ended the tile before)
            slot_next = slot_of(kt + 2 * LBK);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint32_t kbuf = kb + buf * LBK * pitch;
        float s[NK][4];
#pragma unroll
        for (int i = 0; i < NK; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
        {
            const uint32_t qa = qb + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (lane >> 4) * 16;
            const uint32_t ka = kbuf + (cw * NK * 8 + (lane & 7)) * pitch + (lane >> 3) * 16;
#pragma unroll 2
            for (int ks = 0; ks < ksteps; ks += 2) {
                uint32_t a0[4], a1[4];
                ldmatrix_x4(qa + ks * 32, a0);
                ldmatrix_x4(qa + ks * 32 + 32, a1);
#pragma unroll
                for (int i = 0; i < NK; ++i) {
                    uint32_t b[4];
                    ldmatrix_x4(ka + i * 8 * pitch + ks * 32, b);
                    mma_bf16(s[i], a0, b[0], b[1]);
                    mma_bf16(s[i], a1, b[2], b[3]);
                }
            }
        }
        const bool interior = kt >= inner_lo && kt + LBK - 1 <= first_pos;          // uniform over the block
        float mt[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < NK; ++i) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int u = e >> 1;
                float v = s[i][e] * p.scale_log2e;
                if (!interior) {
                    const int key = kt + (cw * NK + i) * 8 + c0 + (e & 1);
                    if (key > qpos[u] || key < qlo[u] || key >= kend) v = -INFINITY;
                }
                s[i][e] = v;
                mt[u] = fmaxf(mt[u], v);
            }
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            mt[u] = fmaxf(mt[u], __shfl_xor_sync(0xffffffffu, mt[u], 1));
            mt[u] = fmaxf(mt[u], __shfl_xor_sync(0xffffffffu, mt[u], 2));
            if ((lane & 3) == 0) mx[cw * MR + rg * 16 + r0 + u * 8] = mt[u];
        }
        __syncthreads();
        float corr[2], m_use[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            float m_new = m_run[u];
#pragma unroll
            for (int w = 0; w < CW; ++w) m_new = fmaxf(m_new, mx[w * MR + rg * 16 + r0 + u * 8]);
            m_use[u] = m_new == -INFINITY ? 0.0f : m_new;          // nothing visible yet: all probabilities are 0
            corr[u] = m_run[u] == -INFINITY ? 0.0f : fast_exp2(m_run[u] - m_use[u]);
            m_run[u] = m_new;
        }
        float lt[2] = {0.0f, 0.0f};
#pragma unroll
        for (int i = 0; i < NK; ++i) {
            const float p0 = fast_exp2(s[i][0] - m_use[0]), p1 = fast_exp2(s[i][1] - m_use[0]);
            const float p2 = fast_exp2(s[i][2] - m_use[1]), p3 = fast_exp2(s[i][3] - m_use[1]);
            lt[0] += p0 + p1;
            lt[1] += p2 + p3;
            uint8_t* dst = p_s + (rg * 16 + r0) * LPP + ((cw * NK + i) * 8 + c0) * 2;
            *reinterpret_cast<uint32_t*>(dst) = pack_bf16(p0, p1);
            *reinterpret_cast<uint32_t*>(dst + 8 * LPP) = pack_bf16(p2, p3);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            lt[u] += __shfl_xor_sync(0xffffffffu, lt[u], 1);
            lt[u] += __shfl_xor_sync(0xffffffffu, lt[u], 2);
            l_run[u] = l_run[u] * corr[u] + lt[u];
        }
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            o[i][0] *= corr[0]; o[i][1] *= corr[0];
            o[i][2] *= corr[1]; o[i][3] *= corr[1];
        }
        __syncthreads();
#pragma unroll
        for (int j = 0; j < LBK / 16; ++j) {
            uint32_t a[4];
            ldmatrix_x4(pb + (rg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LPP + (j * 2 + (lane >> 4)) * 16, a);
            const uint32_t va = kbuf + (j * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + col0 * 2 + (lane >> 4) * 16;
#pragma unroll
            for (int i = 0; i < NTW; i += 2) {
                if (col0 + i * 8 < p.r) {          // uniform over the warp
                    uint32_t b[4];
                    ldmatrix_x4_trans(va + i * 16, b);
                    mma_bf16(o[i], a, b[0], b[1]);
                    mma_bf16(o[i + 1], a, b[2], b[3]);
                }
            }
        }
        __syncthreads();          // every warp has read this tile, P and the maxima
    }
    cp_async_wait<0>();
    // the column warps' sums of a row meet; then every warp normalises its columns
    if ((lane & 3) == 0) {
        mx[cw * MR + rg * 16 + r0] = l_run[0];
        mx[cw * MR + rg * 16 + r0 + 8] = l_run[1];
    }
    __syncthreads();
    float l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int w = 0; w < CW; ++w) l[u] += mx[w * MR + rg * 16 + r0 + u * 8];
    if (!CLUSTER) {
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int m = rg * 16 + r0 + u * 8;
            if (m >= pairs) continue;
            const int f = f0 + m, tok = f / H, h = f - tok * H;
            float den = l[u];
            if (p.sinks) den += exp2f(p.sinks[h] * 1.4426950408889634f - m_run[u]);
            const float inv = 1.0f / den;
            __nv_bfloat16* dst = p.out + ((size_t)(row0 + tok) * H + h) * p.r;
#pragma unroll
            for (int i = 0; i < NTW; ++i) {
                const int d = col0 + i * 8 + c0;
                if (d < p.r) *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(o[i][2 * u] * inv, o[i][2 * u + 1] * inv);
            }
        }
        return;
    }
    // Pieces: this block's (o, m, l) to its shared memory, then every block of the cluster takes a share of the outputs.
    float* pacc = reinterpret_cast<float*>(smem);                  // [MR][r]   (the tiles are free now)
    __syncthreads();
    float* pml = pacc + MR * p.r;                                  // [MR][2]
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int m = rg * 16 + r0 + u * 8;
#pragma unroll
        for (int i = 0; i < NTW; ++i) {
            const int d = col0 + i * 8 + c0;
            if (d < p.r) {
                pacc[m * p.r + d] = o[i][2 * u];
                pacc[m * p.r + d + 1] = o[i][2 * u + 1];
            }
        }
        if ((lane & 3) == 0 && cw == 0) {
            pml[m * 2] = m_run[u];
            pml[m * 2 + 1] = l[u];
        }
    }
    l_cluster_sync();
    const uint32_t acc_addr = smem_addr(pacc), ml_addr = smem_addr(pml);
    for (int i = blockIdx.y * LTHREADS + threadIdx.x; i < pairs * p.r; i += p.nsplit * LTHREADS) {
        const int m = i / p.r, d = i - m * p.r;
        const int f = f0 + m, tok = f / H, h = f - tok * H;
        float ms[LMAX_SPLITS], M = -INFINITY;
#pragma unroll
        for (int sp = 0; sp < LMAX_SPLITS; ++sp) {
            ms[sp] = sp < p.nsplit ? l_ld_cluster(ml_addr + m * 8, sp) : -INFINITY;
            M = fmaxf(M, ms[sp]);
        }
        float den = 0.0f, acc = 0.0f;
#pragma unroll
        for (int sp = 0; sp < LMAX_SPLITS; ++sp) {
            if (ms[sp] != -INFINITY) {
                const float e = fast_exp2(ms[sp] - M);
                den += e * l_ld_cluster(ml_addr + m * 8 + 4, sp);
                acc += e * l_ld_cluster(acc_addr + (m * p.r + d) * 4, sp);
            }
        }
        if (p.sinks) den += exp2f(p.sinks[h] * 1.4426950408889634f - M);
        p.out[((size_t)(row0 + tok) * H + h) * p.r + d] = __float2bfloat16_rn(acc / den);
    }
    l_cluster_sync();          // no block leaves while another may still read its shared memory
}

inline int latent_pitch(int W) { return ((W + 31) / 32 * 32 + 8) * 2; }
inline size_t latent_smem(int rg, int W) {
    const size_t pitch = latent_pitch(W), mr = 16 * rg;
    return mr * pitch + 2 * LBK * pitch + mr * LPP + (size_t)(8 / rg) * mr * sizeof(float);
}
constexpr size_t LATENT_SMEM_MAX = 227 * 1024;

template <int RG, int NTW, bool CLUSTER>
int launch_latent_as(const LatentParams& p, int blocks, cudaStream_t stream) {
    size_t smem = latent_smem(RG, p.W);
    if (CLUSTER) {
        const size_t merge = (size_t)16 * RG * (p.r + 2) * sizeof(float);
        if (merge > smem) smem = merge;
    }
    static size_t configured = 0;
    if (smem > 48 * 1024 && smem > configured) {
        const cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<RG, NTW, CLUSTER>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return llb_fail("latent_attention: %zu bytes of shared memory: %s", smem, cudaGetErrorString(e));
        configured = smem;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(blocks, CLUSTER ? p.nsplit : 1);
    cfg.blockDim = dim3(LTHREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1;
    attr[0].val.clusterDim.y = CLUSTER ? p.nsplit : 1;
    attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = CLUSTER ? 1 : 0;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, latent_attention_kernel<RG, NTW, CLUSTER>, p);
    if (e != cudaSuccess) return llb_fail("latent_attention: launch failed: %s", cudaGetErrorString(e));
    return llb_check_launch("latent_attention");
}

template <int RG, bool CLUSTER>
int launch_latent(const LatentParams& p, int blocks, cudaStream_t stream) {
    const int need = (p.r / 8 + 8 / RG - 1) / (8 / RG);          // value n-tiles a warp, rounded up to the next instantiation
    if (need <= 2) return launch_latent_as<RG, 2, CLUSTER>(p, blocks, stream);
    if (need <= 4) return launch_latent_as<RG, 4, CLUSTER>(p, blocks, stream);
    if (need <= 8) return launch_latent_as<RG, 8, CLUSTER>(p, blocks, stream);
    if constexpr (RG >= 2) {
        if (need <= 16) return launch_latent_as<RG, 16, CLUSTER>(p, blocks, stream);
    }
    if constexpr (RG >= 4) {
        if (need <= 32) return launch_latent_as<RG, 32, CLUSTER>(p, blocks, stream);
    }
    return llb_fail("latent_attention: a latent of %d", p.r);
}

}  // namespace

// src [T, stride] (dtype): the query's latent (q_rank) at column q_off, the latent (r) at c_off, the shared rotated part (rd,
// even) at rot_off.  q_out [T, q_rank] = rms norm of the first times q_w; cache rows slots[t] of cache [slots, r + rd] =
// [rms norm of the second times c_w | the third rotated by positions[t] * inv_freq[i], pairs (i, i + rd / 2) or neighbours].
// q_out or cache may be null.
LLB_EXPORT int llb_latent_prepare(const void* src, int dtype, long long stride, int q_off, int c_off, int rot_off, int T,
                                  int q_rank, int r, int rd, int interleaved, const float* q_w, const float* c_w,
                                  const float* inv_freq, const int* positions, const int* slots, void* q_out, void* cache,
                                  float eps, cudaStream_t stream) {
    if (T == 0) return 0;
    LLB_REQUIRE(T > 0 && q_rank >= 0 && r > 0 && rd >= 0 && rd % 2 == 0 && src && c_w && (!q_out || (q_rank > 0 && q_w)) &&
                (!cache || slots) && (rd == 0 || (inv_freq && positions)), "latent_prepare: bad arguments");
    LatentPrepareParams p;
    p.src = src; p.stride = stride; p.q_off = q_off; p.c_off = c_off; p.rot_off = rot_off; p.q_rank = q_rank; p.r = r; p.rd = rd;
    p.interleaved = interleaved ? 1 : 0; p.q_w = q_w; p.c_w = c_w; p.inv_freq = inv_freq; p.positions = positions; p.slots = slots;
    p.q_out = q_out; p.cache = cache; p.eps = eps;
    if (dtype == LLB_F32) latent_prepare_kernel<float><<<T, 128, 0, stream>>>(p);
    else if (dtype == LLB_BF16) latent_prepare_kernel<__nv_bfloat16><<<T, 128, 0, stream>>>(p);
    else return llb_fail("latent_prepare: unknown dtype %d", dtype);
    return llb_check_launch("latent_prepare");
}

// Whether the kernel takes key rows of W numbers whose first r are the values.
LLB_EXPORT int llb_latent_attention_supports(int W, int r) {
    return W % 8 == 0 && r % 8 == 0 && r > 0 && r <= W && r <= 512 && latent_smem(1, W) <= LATENT_SMEM_MAX &&
           (size_t)16 * (r + 2) * sizeof(float) <= LATENT_SMEM_MAX;
}

// q [T, H, W], cache [slots, W], out [T, H, r], all bf16; spans and block tables as in every kernel of a step; window as
// llb_first_visible; sinks float [H] or null (exp(sinks[h]) joins head h's denominator once).  single != 0: every span is
// one token; nsplit > 1 (at most 8, single only): the keys are cut into that many pieces merged inside the kernel.
LLB_EXPORT int llb_latent_attention(const void* q, const void* cache, void* out, int T, const int* span_row, const int* span_len,
                                    const int* span_pos, int num_spans, const int* block_table, int max_pages, int page_size,
                                    int H, int W, int r, int window, float scale, int single, int nsplit, const float* sinks,
                                    cudaStream_t stream) {
    if (T == 0) return 0;
    LLB_REQUIRE(T > 0 && num_spans > 0 && H > 0 && q && cache && out && span_row && span_len && span_pos && block_table &&
                max_pages > 0 && page_size > 0, "latent_attention: bad arguments");
    LLB_REQUIRE(llb_latent_attention_supports(W, r), "latent_attention: key rows of %d with values of %d are not supported", W, r);
    LLB_REQUIRE(((uintptr_t)q % 16 == 0) && ((uintptr_t)cache % 16 == 0) && ((uintptr_t)out % 16 == 0), "latent_attention: alignment");
    LLB_REQUIRE(nsplit >= 1 && nsplit <= LMAX_SPLITS && (nsplit == 1 || single), "latent_attention: %d pieces", nsplit);
    LLB_REQUIRE(!single || T == num_spans, "latent_attention: %d tokens in %d spans are not single tokens", T, num_spans);
    LatentParams p;
    p.q = (const __nv_bfloat16*)q; p.cache = (const __nv_bfloat16*)cache; p.out = (__nv_bfloat16*)out;
    p.span_row = span_row; p.span_len = span_len; p.span_pos = span_pos; p.block_table = block_table; p.T = T;
    p.num_spans = num_spans; p.max_pages = max_pages; p.page_size = page_size; p.H = H; p.W = W; p.r = r; p.window = window;
    p.nsplit = nsplit; p.scale_log2e = scale * 1.4426950408889634f; p.sinks = sinks; p.pitch = latent_pitch(W);
    // pairs a block: as many row groups as the shared memory holds; single tokens no more than their heads fill
    int rg = 4;
    while (rg > 1 && (latent_smem(rg, W) > LATENT_SMEM_MAX || (single && 16 * (rg / 2) >= H))) rg /= 2;
    const int mr = 16 * rg;
    p.blocks_per_span = single ? (H + mr - 1) / mr : 0;
    const long long blocks = single ? (long long)num_spans * p.blocks_per_span : (long long)T * H / mr + num_spans;
    LLB_REQUIRE(blocks < (1ll << 31), "latent_attention: too many rows");
    if (nsplit > 1) {
        if (rg == 1) return launch_latent<1, true>(p, (int)blocks, stream);
        if (rg == 2) return launch_latent<2, true>(p, (int)blocks, stream);
        return launch_latent<4, true>(p, (int)blocks, stream);
    }
    if (rg == 1) return launch_latent<1, false>(p, (int)blocks, stream);
    if (rg == 2) return launch_latent<2, false>(p, (int)blocks, stream);
    return launch_latent<4, false>(p, (int)blocks, stream);
}
