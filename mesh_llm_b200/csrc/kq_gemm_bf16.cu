// Prefill products with bf16 weights, y[m][n] = sum_k W[n][k] x[m][k]: the tensor-core form (tcgen05.mma
// kind::f16 on bf16 operands, f32 accumulators in TMEM) and the f32 form on CUDA cores of the 32-bit mode.
//
// Tensor cores: a persistent CTA per SM walks tiles of 128 tokens (TMEM lanes) x 256, 128 or 64 weight rows (columns), token
// tiles innermost, so that the CTAs at work share the weight rows they read.  K runs in slices of 64 (one
// 128-byte-swizzled row per operand row); a producer thread brings the slices in by tiled TMA copies through a ring
// of stages, one thread issues the MMAs into one of two accumulators in TMEM, four warps drain the other one meanwhile,
// through a transpose in shared memory: stores of one row per lane would run at a fifth of the rate.
// A gate / up pair shares a tile half and half, so that the GLU happens where both values are.
// An f32 operand can come as several bf16 parts (x = hi + mid + lo exactly): the K loop then passes over the
// same weights once per part.  Block-diagonal products offset the K coordinate of x and the row of W by group.  Products
// with experts take the row of W from the expert of the token tile; how many tiles there are is read on the device.
// Every wait is bounded; on a time-out the kernel records an error, lets its copies land, frees its TMEM and
// returns.
#include "kq_dense.cuh"
#include "kq_tc.cuh"

#include <string.h>

#include <algorithm>

namespace {

constexpr int TM = 128, BK = 64, A_BYTES = TM * BK * 2;
constexpr int EC = 32, EP = EC + 4, EPI_BYTES = 4 * 32 * EP * 4; // columns an epilogue warp turns round at a time, floats per staged row
template <int TN>
struct Tile {
    static constexpr int B_BYTES = TN * BK * 2, STAGE_BYTES = A_BYTES + B_BYTES, STAGES = 192 * 1024 / STAGE_BYTES;
    static constexpr int SMEM_TOTAL = STAGES * STAGE_BYTES + EPI_BYTES + 1024;
    static constexpr uint32_t TMEM_COLS = 2 * TN; // two accumulators
};
constexpr int NTHREADS = 192, NEPI = 128; // producer warp, MMA warp, four epilogue warps
constexpr uint64_t LIMIT = 5 * KQ_WAIT_LIMIT_NS;

__device__ int g_gemm_bf16_error;

struct GemmParams {
    CUtensorMap a, b[3];
    KqDense c;
    int32_t nk, parts;      // 64-element K slices per part
    int32_t tile_end[3];    // cumulative N tiles of the segments
    int32_t mt, nt;         // tiles of tokens and of weight rows (all segments)
};

// four consecutive output columns n .. n + 3 (over all groups), for a number of rows
struct Col4 {
    float bias[4];
    int64_t col, n;
    int32_t valid, n_mul; // columns to write; those of them that have a factor in row_mul
    bool vec; // all four next to one another and aligned in every row
    __device__ __forceinline__ Col4(const KqDense &c, const KqDenseSeg &s, int64_t n_, int n_valid) : n(n_), valid(n_valid), n_mul((int)min((int64_t)n_valid, s.n_rows - n_)) {
        vec = valid == 4 && ((s.ldy | n | s.head_in | s.head_out) & 3) == 0 && ((uintptr_t)s.y & 15) == 0;
        col = kq_dense_col(s, n);
#pragma unroll
        for (int e = 0; e < 4; e++) bias[e] = s.bias && e < valid && (c.groups > 1 || n + e < s.n_rows) ? s.bias[n + e] : 0.f;
    }
    // the factors of row m: eight bytes where the row allows it
    __device__ __forceinline__ uint2 factors(const KqDense &c, int64_t m) const {
        const uint16_t *f = c.row_mul + m * c.ld_mul + n;
        if (n_mul >= 4 && ((uintptr_t)f & 7) == 0) return *reinterpret_cast<const uint2 *>(f);
        uint32_t w[4];
#pragma unroll
        for (int e = 0; e < 4; e++) w[e] = e < n_mul ? f[e] : 0;
        return make_uint2(w[0] | (w[1] << 16), w[2] | (w[3] << 16));
    }
    __device__ __forceinline__ void store(const KqDense &c, const KqDenseSeg &s, int64_t m, int g, const float4 &v, const uint2 f = make_uint2(0, 0)) const {
        float o[4] = {v.x + bias[0], v.y + bias[1], v.z + bias[2], v.w + bias[3]};
        if (s.act == KQ_ACT_GELU_TANH) {
#pragma unroll
            for (int e = 0; e < 4; e++) o[e] = kq_gelu_tanh(o[e]);
        }
        if (s.act == KQ_ACT_SOFT_CAP) {
#pragma unroll
            for (int e = 0; e < 4; e++) o[e] = c.cap * tanhf(o[e] / c.cap);
        }
        if (c.head_gate) {
            const float f = kq_sigmoid(c.head_gate[m * c.ld_gate + g]);
#pragma unroll
            for (int e = 0; e < 4; e++) o[e] *= f;
        }
        if (c.row_mul) {
            o[0] *= kq_bf2f((uint16_t)f.x), o[1] *= kq_bf2f((uint16_t)(f.x >> 16));
            o[2] *= kq_bf2f((uint16_t)f.y), o[3] *= kq_bf2f((uint16_t)(f.y >> 16));
        }
        if (vec) {
            const int64_t i = m * s.ldy + col;
            if (s.out == KQ_OUT_F32) {
                *reinterpret_cast<float4 *>((float *)s.y + i) = make_float4(o[0], o[1], o[2], o[3]);
            } else {
                uint32_t w[2];
#pragma unroll
                for (int e = 0; e < 2; e++)
                    w[e] = s.out == KQ_OUT_BF16 ? (uint32_t)kq_f2bf(o[2 * e]) | ((uint32_t)kq_f2bf(o[2 * e + 1]) << 16)
                                                : (uint32_t)kq_f2h_sat(o[2 * e]) | ((uint32_t)kq_f2h_sat(o[2 * e + 1]) << 16);
                *reinterpret_cast<uint2 *>((uint16_t *)s.y + i) = make_uint2(w[0], w[1]);
            }
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++)
                if (e < valid) kq_dense_put(s, m, n + e, o[e]);
        }
    }
};

template <int TN>
__global__ void __launch_bounds__(NTHREADS, 1) gemm_bf16_kernel(const __grid_constant__ GemmParams p) {
    using S = Tile<TN>;
    constexpr uint32_t IDESC = tc_idesc(TM, TN, true, false);
    extern __shared__ uint8_t sm_raw[];
    __shared__ uint64_t full[S::STAGES], empty[S::STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort;
    // the wait comes before the TMEM allocation: a CTA that started early must not hold columns its predecessor needs
    KQ_PDL_ENTER();
    uint8_t *sm = (uint8_t *)(((uintptr_t)sm_raw + 1023) & ~(uintptr_t)1023);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(S::TMEM_COLS)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    if (tid == 0) {
        for (int i = 0; i < S::STAGES; i++) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(&full[i])), "r"(1));
            asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(&empty[i])), "r"(1));
        }
        for (int i = 0; i < 2; i++) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(&acc_full[i])), "r"(1));
            asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(&acc_empty[i])), "r"(NEPI));
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        s_abort = 0;
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = s_tmem;
    const int mt = p.c.experts ? min(p.mt, *p.c.n_tiles) : p.mt;
    const int n_it = p.nk * p.parts, n_tiles = mt * p.nt * p.c.groups;

    struct Where {
        int m0, g, seg, n0, n_rows;
    };
    auto locate = [&](int tile) {
        Where w;
        const int i = tile % mt, rest = tile / mt;
        w.m0 = i * TM;
        int nt = rest % p.nt;
        w.g = p.c.experts ? p.c.tile_expert[i] : rest / p.nt;
        w.seg = 0;
        if (!p.c.glu) {
            if (nt >= p.tile_end[1]) w.seg = 2, nt -= p.tile_end[1];
            else if (nt >= p.tile_end[0]) w.seg = 1, nt -= p.tile_end[0];
        }
        w.n_rows = kq_dense_rows(p.c, w.seg);
        w.n0 = nt * (p.c.glu ? TN / 2 : TN); // first row of the tile inside the group
        return w;
    };
    auto wait = [&](uint64_t *bar, uint32_t parity, int code) { // a warp gives up as a whole
        return __all_sync(0xffffffffu, tc_wait(smem_u32(bar), parity, &s_abort, &g_gemm_bf16_error, code, LIMIT)) != 0;
    };
    // The producer and the MMA warp run their loops with all lanes, so that addresses and descriptors stay in uniform
    // registers; one lane posts and issues.
    if (warp == 0) {
        const bool lead = tc_elect();
        int it = 0, s = 0; // slices over all tiles, stage
        uint32_t round = 0; // uses of the ring so far
        bool ok = true;
        for (int tile = blockIdx.x; ok && tile < n_tiles; tile += gridDim.x) {
            const Where w = locate(tile);
            const int row = w.g * w.n_rows + w.n0, xk = (int)(w.g * p.c.xg);
            const CUtensorMap *map0 = p.b + (p.c.glu ? 0 : w.seg), *map1 = p.b + (p.c.glu ? 1 : w.seg); // half a tile of rows each
            const int row1 = row + (p.c.glu ? 0 : TN / 2);
            int part = 0, kk = 0;
            for (int i = 0; i < n_it; i++, it++) {
                if (round > 0 && !(ok = wait(&empty[s], (round - 1) & 1, 1))) break;
                if (lead) {
                    const uint32_t bar = smem_u32(&full[s]), dst = smem_u32(sm + s * S::STAGE_BYTES);
                    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(S::STAGE_BYTES) : "memory");
                    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(dst),
                                 "l"(&p.a), "r"(xk + kk), "r"(w.m0), "r"(part), "r"(bar)
                                 : "memory");
                    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst + A_BYTES),
                                 "l"(map0), "r"(kk), "r"(row), "r"(bar)
                                 : "memory");
                    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(
                                     dst + A_BYTES + S::B_BYTES / 2),
                                 "l"(map1), "r"(kk), "r"(row1), "r"(bar)
                                 : "memory");
                }
                __syncwarp();
                kk += BK;
                if (kk == p.nk * BK) kk = 0, part++;
                if (++s == S::STAGES) s = 0, round++;
            }
        }
        if (!ok && lead) // copies that were posted must land before the CTA goes away
            for (int i = std::max(0, it - S::STAGES); i < it; i++)
                kq_mbar_wait(smem_u32(&full[i % S::STAGES]), (uint32_t)((i / S::STAGES) & 1), KQ_WAIT_LIMIT_NS);
        __syncwarp();
    } else if (warp == 1) {
        const bool lead = tc_elect();
        int s = 0, t = 0;
        uint32_t round = 0;
        bool ok = true;
        for (int tile = blockIdx.x; ok && tile < n_tiles; tile += gridDim.x, t++) {
            const int buf = t & 1;
            if (t >= 2 && !(ok = wait(&acc_empty[buf], (uint32_t)((t / 2 - 1) & 1), 4))) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            for (int i = 0; i < n_it; i++) {
                if (!(ok = wait(&full[s], round & 1, 2))) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (lead) {
                    const uint32_t a = smem_u32(sm + s * S::STAGE_BYTES), b = a + A_BYTES;
                    const uint64_t da = tc_desc_k(a, 0), db = tc_desc_k(b, 0);
#pragma unroll
                    for (int k = 0; k < BK / 16; k++) // 32 bytes further per step: 2 in the descriptor's address field
                        tc_mma_ss(tmem + buf * TN, da + 2 * k, db + 2 * k, IDESC, (i > 0 || k > 0) ? 1u : 0u);
                    tc_commit(smem_u32(&empty[s]));
                }
                __syncwarp();
                if (++s == S::STAGES) s = 0, round++;
            }
            if (lead) tc_commit(smem_u32(&acc_full[buf]));
            __syncwarp();
        }
        if (!ok && lead) // MMAs in flight end before TMEM is freed
            for (int i = std::max(0, t - 2); i < t; i++) kq_mbar_wait(smem_u32(&acc_full[i & 1]), (uint32_t)((i / 2) & 1), KQ_WAIT_LIMIT_NS);
        __syncwarp();
    } else {
        const int q = warp & 3; // a warp reaches the TMEM lanes of its quarter
        float *stage = reinterpret_cast<float *>(sm + S::STAGES * S::STAGE_BYTES) + q * 32 * EP;
        int t = 0;
        for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, t++) {
            const int buf = t & 1;
            const bool ok = wait(&acc_full[buf], (uint32_t)((t / 2) & 1), 3);
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            if (!ok) break;
            const Where w = locate(tile);
            const int n0 = w.n0, n_rows = w.n_rows, m0 = w.m0 + q * 32, m_end = std::min(p.c.M, m0 + 32);
            const uint32_t tl = tmem + ((uint32_t)(q * 32) << 16) + buf * TN;
            const KqDenseSeg s = kq_dense_seg(p.c, w.seg);
            // EC columns at a time: a lane takes its row out of TMEM into shared memory, then eight lanes write a row's columns, four
            // rows per store.  The loops stay loops: unrolled, the four warps would spend their time fetching code.
            const int lim = p.c.groups == 1 ? std::max(n_rows, s.pad_cols) : n_rows; // the padding of a staging row is written too
            const int n_cols = std::min(p.c.glu ? TN / 2 : TN, lim - n0);
            const int r4 = lane >> 3, c4 = (lane & 7) * 4;
#pragma unroll 1
            for (int j = 0; j < n_cols; j += EC) {
#pragma unroll
                for (int h = 0; h < EC; h += 16) {
                    uint32_t a[16], b[16];
                    TMEM_LD16(tl + j + h, a);
                    if (p.c.glu) TMEM_LD16(tl + TN / 2 + j + h, b);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    if (p.c.glu) {
#pragma unroll
                        for (int e = 0; e < 16; e++)
                            a[e] = n0 + j + h + e < n_rows ? __float_as_uint(kq_glu(p.c, __uint_as_float(a[e]), __uint_as_float(b[e]))) : 0u;
                    }
#pragma unroll
                    for (int e = 0; e < 16; e += 4)
                        *reinterpret_cast<uint4 *>(stage + lane * EP + h + e) = make_uint4(a[e], a[e + 1], a[e + 2], a[e + 3]);
                }
                __syncwarp();
                const int n = n0 + j + c4, n_valid = std::min(4, lim - n);
                if (n_valid > 0) {
                    const Col4 col(p.c, s, (p.c.experts ? 0 : (int64_t)w.g * n_rows) + n, n_valid);
                    if (p.c.row_mul) { // the factors of all of a lane's rows are requested together
                        uint2 f[8];
#pragma unroll
                        for (int i = 0; i < 8; i++) f[i] = m0 + r4 + 4 * i < m_end ? col.factors(p.c, m0 + r4 + 4 * i) : make_uint2(0, 0);
#pragma unroll
                        for (int i = 0; i < 8; i++)
                            if (m0 + r4 + 4 * i < m_end)
                                col.store(p.c, s, m0 + r4 + 4 * i, w.g, *reinterpret_cast<const float4 *>(stage + (r4 + 4 * i) * EP + c4), f[i]);
                    } else {
#pragma unroll 2
                        for (int r = r4; m0 + r < m_end; r += 4) {
                            const float4 v = *reinterpret_cast<const float4 *>(stage + r * EP + c4);
                            col.store(p.c, s, m0 + r, w.g, v);
                        }
                    }
                }
                __syncwarp();
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&acc_empty[buf])) : "memory");
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(S::TMEM_COLS) : "memory");
}

// ---- f32 form ------------------------------------------------------------------------------------
constexpr int FT = 64, FK = 16;
struct F32Params {
    KqDense c;
    const float *x;
    int64_t ldx;
    int32_t tile_end[3];
};

template <bool GLU>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const __grid_constant__ F32Params p) {
    KQ_PDL_ENTER();
    __shared__ float sa[FK][FT + 4], sb[GLU ? 2 : 1][FK][FT + 4];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    int seg = 0, nt = blockIdx.y, g = blockIdx.z;
    if (p.c.experts) {
        const int t = blockIdx.x * FT / KQ_TILE_M;
        if (t >= *p.c.n_tiles) return;
        g = p.c.tile_expert[t];
    }
    const int64_t row0 = p.c.experts ? 0 : g; // column groups of the output
    if (!GLU) {
        if (nt >= p.tile_end[1]) seg = 2, nt -= p.tile_end[1];
        else if (nt >= p.tile_end[0]) seg = 1, nt -= p.tile_end[0];
    }
    const KqDenseSeg s = kq_dense_seg(p.c, seg);
    const int m0 = blockIdx.x * FT, n0 = nt * FT, n_rows = s.n_rows, K = p.c.K;
    float acc[GLU ? 2 : 1][4][4] = {};
    for (int k0 = 0; k0 < K; k0 += FK) {
        for (int i = tid; i < FT * FK; i += 256) {
            const int r = i / FK, k = i % FK;
            sa[k][r] = m0 + r < p.c.M && k0 + k < K ? p.x[(m0 + r) * p.ldx + g * p.c.xg + k0 + k] : 0.f;
#pragma unroll
            for (int h = 0; h < (GLU ? 2 : 1); h++)
                sb[h][k][r] = n0 + r < n_rows && k0 + k < K
                                  ? kq_bf2f(kq_dense_w(p.c, GLU ? h : seg)[((int64_t)g * n_rows + n0 + r) * p.c.ldw + k0 + k])
                                  : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < FK; k++) {
            const float4 a = *reinterpret_cast<const float4 *>(&sa[k][ty * 4]);
            const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
            for (int h = 0; h < (GLU ? 2 : 1); h++) {
                const float4 b = *reinterpret_cast<const float4 *>(&sb[h][k][tx * 4]);
                const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                for (int i = 0; i < 4; i++)
#pragma unroll
                    for (int j = 0; j < 4; j++) acc[h][i][j] = fmaf(av[i], bv[j], acc[h][i][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (m >= p.c.M || n >= n_rows) continue;
            if (GLU) kq_dense_put(s, m, n, kq_glu(p.c, acc[0][i][j], acc[GLU ? 1 : 0][i][j]));
            else kq_dense_store(p.c, s, m, row0 * n_rows + n, g, acc[0][i][j]);
        }
}

} // namespace

int kq_gemm_bf16_error_fetch() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_gemm_bf16_error, sizeof(int)) != cudaSuccess) return -1;
    if (v) cudaMemcpyToSymbol(g_gemm_bf16_error, &zero, sizeof(int));
    return v;
}

b200_status kq_gemm_bf16(const KqDense &c, const uint16_t *a, int64_t lda, int parts, cudaStream_t st) {
    KQ_REQUIRE(c.M >= 1 && c.nseg >= 1 && c.nseg <= 3 && c.groups >= 1 && c.K >= 1 && parts >= 1, "gemm_bf16: bad call");
    KQ_REQUIRE(c.ldw % 64 == 0 && c.ldw >= c.K && lda % 64 == 0 && (c.groups == 1 || c.xg % 64 == 0),
               "gemm_bf16: rows must be padded to 64 elements");
    KQ_REQUIRE(!c.experts || (c.groups == 1 && c.tile_expert && c.n_tiles && c.M % TM == 0), "gemm_bf16: products with experts");
    KQ_REQUIRE(!c.glu || (c.nseg == 2 && c.groups == 1 && c.seg[0].n_rows == c.seg[1].n_rows), "gemm_bf16: a GLU has two equal segments");
    GemmParams p;
    p.c = c;
    p.parts = parts;
    p.nk = (int)kq_div_up(c.K, BK);
    p.mt = (int)kq_div_up(c.M, TM);
    // larger tiles read less per product, smaller ones fill the last wave of CTAs better
    auto n_tiles = [&](int tn) {
        int t = 0;
        if (c.glu) t = (int)kq_div_up(std::max(c.seg[0].n_rows, c.seg[0].pad_cols), tn / 2);
        else
            for (int i = 0; i < c.nseg; i++) t += (int)kq_div_up(std::max(c.seg[i].n_rows, c.groups == 1 ? c.seg[i].pad_cols : 0), tn);
        return t;
    };
    const int64_t sms = kq_sm_count();
    const int64_t w256 = kq_div_up((int64_t)p.mt * n_tiles(256) * c.groups, sms) * 20, w128 = kq_div_up((int64_t)p.mt * n_tiles(128) * c.groups, sms) * 13,
                  w64 = kq_div_up((int64_t)p.mt * n_tiles(64) * c.groups, sms) * 9;
    const int tn = w256 <= w128 && w256 <= w64 ? 256 : w128 <= w64 ? 128 : 64;
    p.nt = n_tiles(tn);
    {
        const uint64_t dims[3] = {(uint64_t)lda, (uint64_t)c.M, (uint64_t)parts};
        const uint64_t str[2] = {(uint64_t)lda * 2, (uint64_t)lda * 2 * c.M};
        const uint32_t box[3] = {BK, TM, 1};
        const b200_status rc = kq_tmap_encode(&p.a, 2, 3, a, dims, str, box, 1);
        if (rc != B200_OK) return rc;
    }
    int tiles = 0;
    for (int i = 0; i < 3; i++) {
        const KqDenseSeg &s = c.seg[std::min(i, c.nseg - 1)];
        const uint64_t dims[2] = {(uint64_t)c.ldw, (uint64_t)s.n_rows * std::max(c.groups, c.experts)}, str[1] = {(uint64_t)c.ldw * 2};
        const uint32_t box[2] = {BK, (uint32_t)tn / 2};
        const b200_status rc = kq_tmap_encode(&p.b[i], 2, 2, s.W, dims, str, box, 1);
        if (rc != B200_OK) return rc;
        if (i < c.nseg) tiles += (int)kq_div_up(std::max(s.n_rows, c.groups == 1 ? s.pad_cols : 0), tn);
        p.tile_end[i] = tiles;
    }
    const unsigned grid = (unsigned)std::min<int64_t>((int64_t)p.mt * p.nt * c.groups, sms);
    static bool attr[16];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 16 || !attr[dev]) {
        KQ_CUDA(cudaFuncSetAttribute(gemm_bf16_kernel<256>, cudaFuncAttributeMaxDynamicSharedMemorySize, Tile<256>::SMEM_TOTAL));
        KQ_CUDA(cudaFuncSetAttribute(gemm_bf16_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, Tile<128>::SMEM_TOTAL));
        KQ_CUDA(cudaFuncSetAttribute(gemm_bf16_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, Tile<64>::SMEM_TOTAL));
        if (dev >= 0 && dev < 16) attr[dev] = true;
    }
    if (tn == 256) kq_launch(gemm_bf16_kernel<256>, grid, NTHREADS, Tile<256>::SMEM_TOTAL, st, p);
    else if (tn == 64) kq_launch(gemm_bf16_kernel<64>, grid, NTHREADS, Tile<64>::SMEM_TOTAL, st, p);
    else kq_launch(gemm_bf16_kernel<128>, grid, NTHREADS, Tile<128>::SMEM_TOTAL, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_gemm_f32(const KqDense &c, const float *x, int64_t ldx, cudaStream_t st) {
    KQ_REQUIRE(c.M >= 1 && c.nseg >= 1 && c.nseg <= 3 && c.groups >= 1 && c.K >= 1, "gemm_f32: bad call");
    F32Params p;
    p.c = c;
    p.x = x;
    p.ldx = ldx;
    int tiles = 0;
    for (int i = 0; i < 3; i++) {
        if (i < c.nseg) tiles += (int)kq_div_up(c.seg[i].n_rows, FT);
        p.tile_end[i] = tiles;
    }
    if (c.glu) tiles = (int)kq_div_up(c.seg[0].n_rows, FT);
    const dim3 grid((unsigned)kq_div_up(c.M, FT), (unsigned)tiles, (unsigned)c.groups);
    if (c.glu) kq_launch(gemm_f32_kernel<true>, grid, 256, 0, st, p);
    else kq_launch(gemm_f32_kernel<false>, grid, 256, 0, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
