// Experts with bf16 weights (SiLU GLU, softmax over the chosen logits, a shared expert): the decode form, and the work
// around the matrix products of a prompt.
//
// Decode, 1 .. 8 rows: the router's logits come out of the same launch as the shared expert's gate and up products; the
// experts' gate / up launch chooses for itself in every CTA (a warp over the row's logits) and reads only the chosen
// experts' rows; the down launch forms the weighted sum over the chosen and the shared expert in one go.
// Prompts: choice and shared GLU, a counting sort that gives every expert whole tiles of KQ_TILE_M rows, a gather, two
// products with experts (kq_gemm_bf16.cu), and the weighted sum.
#include "kq_gemv_grouped.cuh"

#include <algorithm>

namespace {

constexpr int NT = 256, NW = NT / 32;

// The choice for one row by one warp.  lr: the row's logits in shared memory, overwritten.  ids / wts in shared memory.
__device__ __forceinline__ void choose(float *lr, int E, int top, int32_t *ids, float *wts, int lane) {
    float first = 0.f, sum = 0.f;
    for (int s = 0; s < top; s++) {
        float best = -INFINITY;
        int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32)
            if (lr[e] > best) best = lr[e], bi = e;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float v = __shfl_xor_sync(0xffffffffu, best, o);
            const int i = __shfl_xor_sync(0xffffffffu, bi, o);
            if (v > best || (v == best && i < bi)) best = v, bi = i;
        }
        bi = min(bi, E - 1); // all left are -inf or no numbers
        if (s == 0) first = best;
        const float w = expf(best - first);
        sum += w;
        if (lane == 0) {
            ids[s] = bi;
            wts[s] = w;
            lr[bi] = -INFINITY;
        }
        __syncwarp();
    }
    for (int s = lane; s < top; s += 32) wts[s] /= sum;
    __syncwarp();
}

// grid (slices of the rows of an expert, rows * top); a warp takes two gate and two up rows at a time
constexpr int FEW_ROWS = 4 * NW; // GLU rows per CTA
__global__ void __launch_bounds__(NT) moe_few_gate_up_kernel(const __grid_constant__ KqMoe m, const float *x, int64_t ldx, const uint16_t *gate, const uint16_t *up,
                                                             float *act, int64_t ld_act, int32_t *ids, float *wts, int xs) {
    extern __shared__ __align__(16) float sm[]; // x of the row as two planes of float4, then the logits
    __shared__ int32_t s_id[KQ_MOE_MAX_TOP];
    __shared__ float s_w[KQ_MOE_MAX_TOP];
    KQ_PDL_ENTER();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, pair = blockIdx.y, row = pair / m.top, slot = pair % m.top;
    const int nck = (m.h + 7) / 8;
    float4 *pl = reinterpret_cast<float4 *>(sm);
    float *lr = sm + xs;
    if (warp == 0) {
        for (int e = lane; e < m.experts; e += 32) lr[e] = m.z[row * m.ldz + e];
        __syncwarp();
        choose(lr, m.experts, m.top, s_id, s_w, lane);
        if (blockIdx.x == 0 && lane == 0) ids[pair] = s_id[slot], wts[pair] = s_w[slot];
    } else {
        const float *xr = x + row * ldx;
        const bool vec = (ldx & 3) == 0 && ((uintptr_t)x & 15) == 0;
        for (int i = tid - 32; i < 2 * nck; i += NT - 32) pl[(i & 1) * nck + (i >> 1)] = kq_load4(xr, 4 * i, m.h, vec);
    }
    __syncthreads();
    const int64_t ldw = kq_bf16_ld(m.h), base = (int64_t)s_id[slot] * m.ff;
    const int j1 = min(m.ff, ((int)blockIdx.x + 1) * FEW_ROWS);
    for (int j = blockIdx.x * FEW_ROWS + warp * 2; j < j1; j += NW * 2) {
        const uint4 *w[4];
#pragma unroll
        for (int r = 0; r < 4; r++) w[r] = reinterpret_cast<const uint4 *>((r & 1 ? up : gate) + (base + min(j + r / 2, m.ff - 1)) * ldw);
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (int c0 = lane; c0 < nck; c0 += 128) { // four chunks of each row in flight
            uint4 q[4][4];
#pragma unroll
            for (int u = 0; u < 4; u++)
#pragma unroll
                for (int r = 0; r < 4; r++) q[u][r] = c0 + 32 * u < nck ? kq_ld_stream(w[r] + c0 + 32 * u) : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const int c = c0 + 32 * u;
                if (c < nck) {
                    const float4 a = pl[c], b = pl[nck + c];
#pragma unroll
                    for (int r = 0; r < 4; r++) acc[r] = kq_dot8(q[u][r], a, b, acc[r]);
                }
            }
        }
#pragma unroll
        for (int r = 0; r < 4; r++) acc[r] = kq_warp_sum(acc[r]);
        if (lane < 2 && j + lane < m.ff) act[pair * ld_act + j + lane] = lane ? kq_silu(acc[2]) * acc[3] : kq_silu(acc[0]) * acc[1];
    }
}

// grid (slices of output rows, rows).  The chosen experts' and the shared one's hidden values are one long row, in chunks of eight;
// warps split the chunks, every warp for all of the CTA's output rows, so that a lane makes its activations once and has
// many weights in flight.
constexpr int DOWN_ROWS = 8;
__global__ void __launch_bounds__(NT) moe_few_down_kernel(const __grid_constant__ KqMoe m, const float *act, int64_t ld_act, const int32_t *ids, const float *wts,
                                                          const uint16_t *down, const uint16_t *sh_down, float *out, int64_t ldo) {
    __shared__ float part[NW][DOWN_ROWS];
    KQ_PDL_ENTER();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.y, n0 = blockIdx.x * DOWN_ROWS;
    const int per = (m.ff + 7) / 8, n_ck = m.top * per, all = n_ck + (m.ff_shared + 7) / 8;
    const int64_t ldw = kq_bf16_ld(m.ff), lds = kq_bf16_ld(m.ff_shared);
    const bool vec = (m.ldz & 3) == 0 && ((((uintptr_t)m.sh_gate | (uintptr_t)m.sh_up) & 15) == 0);
    float acc[DOWN_ROWS] = {};
#pragma unroll 2
    for (int c = tid; c < all; c += NT) {
        const bool shared = c >= n_ck;
        const int s = shared ? 0 : c / per, k = 8 * (shared ? c - n_ck : c - s * per);
        const int64_t step = shared ? lds : ldw;
        const uint16_t *w = (shared ? sh_down + n0 * lds : down + ((int64_t)ids[row * m.top + s] * m.h + n0) * ldw) + k;
        uint4 q[DOWN_ROWS];
#pragma unroll
        for (int r = 0; r < DOWN_ROWS; r++) q[r] = kq_ld_stream(w + min(r, m.h - 1 - n0) * step);
        float4 a, b;
        if (shared) {
            const float4 g0 = kq_load4(m.sh_gate + row * m.ldz, k, m.ff_shared, vec), g1 = kq_load4(m.sh_gate + row * m.ldz, k + 4, m.ff_shared, vec);
            a = kq_load4(m.sh_up + row * m.ldz, k, m.ff_shared, vec), b = kq_load4(m.sh_up + row * m.ldz, k + 4, m.ff_shared, vec);
            a.x *= kq_silu(g0.x), a.y *= kq_silu(g0.y), a.z *= kq_silu(g0.z), a.w *= kq_silu(g0.w);
            b.x *= kq_silu(g1.x), b.y *= kq_silu(g1.y), b.z *= kq_silu(g1.z), b.w *= kq_silu(g1.w);
        } else {
            const float *x = act + ((int64_t)row * m.top + s) * ld_act, wt = wts[row * m.top + s];
            a = kq_load4(x, k, m.ff, true), b = kq_load4(x, k + 4, m.ff, true);
            a.x *= wt, a.y *= wt, a.z *= wt, a.w *= wt, b.x *= wt, b.y *= wt, b.z *= wt, b.w *= wt;
        }
#pragma unroll
        for (int r = 0; r < DOWN_ROWS; r++) acc[r] = kq_dot8(q[r], a, b, acc[r]);
    }
#pragma unroll
    for (int r = 0; r < DOWN_ROWS; r++) {
        const float v = kq_warp_sum(acc[r]);
        if (lane == 0) part[warp][r] = v;
    }
    __syncthreads();
    if (tid < DOWN_ROWS && n0 + tid < m.h) {
        float v = 0.f;
#pragma unroll
        for (int i = 0; i < NW; i++) v += part[i][tid];
        out[row * ldo + n0 + tid] = v;
    }
}

// the first CTAs: a warp per row chooses; the others form the shared GLU, a row and GLU_COLS columns each
constexpr int GLU_COLS = 4 * NT;
__global__ void __launch_bounds__(NT) moe_route_kernel(const __grid_constant__ KqMoe m, int rows, int route_ctas, int slices, KqMoeOrder o, float *sh32, int64_t ld32,
                                                       uint16_t *sh16, int64_t ld16) {
    extern __shared__ __align__(16) float sm[]; // [NW][experts]
    __shared__ int32_t s_id[NW][KQ_MOE_MAX_TOP];
    __shared__ float s_w[NW][KQ_MOE_MAX_TOP];
    KQ_PDL_ENTER();
    if ((int)blockIdx.x >= route_ctas) {
        const int64_t i = blockIdx.x - route_ctas, r = i / slices;
        const int j = (int)(i % slices) * GLU_COLS + threadIdx.x * 4, w = sh16 ? (int)ld16 : m.ff_shared;
        const float *g = m.sh_gate + r * m.ldz, *u = m.sh_up + r * m.ldz;
        if (j >= w) return;
        float v[4];
        if (j + 4 <= m.ff_shared && ((m.ldz & 3) == 0) && ((((uintptr_t)m.sh_gate | (uintptr_t)m.sh_up) & 15) == 0)) {
            const float4 a = *reinterpret_cast<const float4 *>(g + j), b = *reinterpret_cast<const float4 *>(u + j);
            v[0] = kq_silu(a.x) * b.x, v[1] = kq_silu(a.y) * b.y, v[2] = kq_silu(a.z) * b.z, v[3] = kq_silu(a.w) * b.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; e++) v[e] = j + e < m.ff_shared ? kq_silu(g[j + e]) * u[j + e] : 0.f;
        }
        if (sh16) // rows of a multiple of 64 elements, padded with zeros
            *reinterpret_cast<uint2 *>(sh16 + r * ld16 + j) = make_uint2((uint32_t)kq_f2bf(v[0]) | ((uint32_t)kq_f2bf(v[1]) << 16),
                                                                         (uint32_t)kq_f2bf(v[2]) | ((uint32_t)kq_f2bf(v[3]) << 16));
        else
            for (int e = 0; e < 4 && j + e < w; e++) sh32[r * ld32 + j + e] = v[e];
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int64_t row = (int64_t)blockIdx.x * NW + warp;
    if (row < rows) {
        float *lr = sm + (int64_t)warp * m.experts;
        for (int e = lane; e < m.experts; e += 32) lr[e] = m.z[row * m.ldz + e];
        __syncwarp();
        choose(lr, m.experts, m.top, s_id[warp], s_w[warp], lane);
        for (int s = lane; s < m.top; s += 32) {
            o.ids[row * m.top + s] = s_id[warp][s];
            o.wts[row * m.top + s] = s_w[warp][s];
        }
    }
}

// one CTA: how many pairs every expert has, whole tiles for each, a place for every pair
constexpr int ORDER_NT = 1024;
__global__ void __launch_bounds__(ORDER_NT) moe_order_kernel(int E, int pairs, KqMoeOrder o) {
    __shared__ int count[KQ_MOE_MAX_EXPERTS], first[KQ_MOE_MAX_EXPERTS + 1];
    KQ_PDL_ENTER();
    const int tid = threadIdx.x;
    for (int e = tid; e < E; e += ORDER_NT) count[e] = 0;
    __syncthreads();
    for (int i = tid; i < pairs; i += ORDER_NT) atomicAdd(&count[o.ids[i]], 1);
    __syncthreads();
    if (tid < 32) { // tiles in front of every expert
        int run = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + tid, t = e < E ? (count[e] + KQ_TILE_M - 1) / KQ_TILE_M : 0;
            int s = t;
#pragma unroll
            for (int d = 1; d < 32; d *= 2) {
                const int v = __shfl_up_sync(0xffffffffu, s, d);
                if (tid >= d) s += v;
            }
            if (e < E) first[e] = run + s - t;
            run += __shfl_sync(0xffffffffu, s, 31);
        }
        if (tid == 0) {
            first[E] = run;
            *o.n_tiles = run;
        }
    }
    __syncthreads();
    for (int e = tid; e < E; e += ORDER_NT) {
        for (int t = first[e]; t < first[e + 1]; t++) o.tile_expert[t] = e;
        count[e] = 0;
    }
    __syncthreads();
    for (int i = tid; i < pairs; i += ORDER_NT) {
        const int e = o.ids[i];
        o.pos[i] = first[e] * KQ_TILE_M + atomicAdd(&count[e], 1);
    }
}

// a warp per pair
template <typename T>
__global__ void __launch_bounds__(NT) moe_gather_kernel(int top, int64_t pairs, const int32_t *pos, const uint8_t *x, uint8_t *y, int64_t row_bytes) {
    KQ_PDL_ENTER();
    const int64_t i = (int64_t)blockIdx.x * NW + (threadIdx.x >> 5);
    if (i >= pairs) return;
    const T *s = reinterpret_cast<const T *>(x + i / top * row_bytes);
    T *d = reinterpret_cast<T *>(y + (int64_t)pos[i] * row_bytes);
#pragma unroll 4
    for (int c = threadIdx.x & 31; c < row_bytes / (int)sizeof(T); c += 32) d[c] = s[c];
}

// grid (columns, rows)
__global__ void __launch_bounds__(NT) moe_combine_kernel(int top, int h, const int32_t *pos, const float *wts, const float *y, int64_t ldy, float *out, int64_t ldo,
                                                         int first) {
    KQ_PDL_ENTER();
    const int64_t r = blockIdx.y;
    const int c = (blockIdx.x * NT + threadIdx.x) * 4; // ldy and ldo are multiples of four, the padding is writable
    if (c >= h) return;
    float4 a = first ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4 *>(out + r * ldo + c);
#pragma unroll 4
    for (int s = 0; s < top; s++) {
        const float w = wts[r * top + s];
        const float4 v = *reinterpret_cast<const float4 *>(y + (int64_t)pos[r * top + s] * ldy + c);
        a.x = fmaf(w, v.x, a.x), a.y = fmaf(w, v.y, a.y), a.z = fmaf(w, v.z, a.z), a.w = fmaf(w, v.w, a.w);
    }
    *reinterpret_cast<float4 *>(out + r * ldo + c) = a;
}

b200_status check_moe(const KqMoe &m, int rows) {
    KQ_REQUIRE(m.experts >= 1 && m.experts <= KQ_MOE_MAX_EXPERTS && m.top >= 1 && m.top <= KQ_MOE_MAX_TOP && m.top <= m.experts && m.h >= 1 && m.ff >= 1 &&
                   m.ff_shared >= 0 && rows >= 1 && (int64_t)rows * m.top <= INT32_MAX / 2,
               "experts: %d of %d", m.top, m.experts);
    return B200_OK;
}
template <typename K>
b200_status allow_smem(K kern, size_t smem, size_t (&have)[16]) {
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (smem > 48 * 1024 && (dev < 0 || dev >= 16 || have[dev] < smem)) {
        KQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        if (dev >= 0 && dev < 16) have[dev] = smem;
    }
    return B200_OK;
}
constexpr size_t MAX_SMEM = 220 * 1024;

} // namespace

b200_status kq_moe_few_gate_up(const KqMoe &m, const float *x, int64_t ldx, int rows, const uint16_t *gate, const uint16_t *up, float *act,
                               int64_t ld_act, int32_t *ids, float *wts, cudaStream_t st) {
    KQ_TRY(check_moe(m, rows));
    const int xs = (int)kq_pad(m.h, 8);
    const size_t smem = ((size_t)xs + m.experts) * 4;
    KQ_REQUIRE(smem <= MAX_SMEM && rows * m.top <= 65535, "experts: rows of %d values", m.h);
    static size_t have[16];
    KQ_TRY(allow_smem(moe_few_gate_up_kernel, smem, have));
    kq_launch(moe_few_gate_up_kernel, dim3((unsigned)kq_div_up(m.ff, FEW_ROWS), (unsigned)(rows * m.top)), NT, smem, st, m, x, ldx, gate, up, act, ld_act, ids,
              wts, xs);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_moe_few_down(const KqMoe &m, const float *act, int64_t ld_act, const int32_t *ids, const float *wts, int rows, const uint16_t *down,
                            const uint16_t *sh_down, float *out, int64_t ldo, cudaStream_t st) {
    KQ_TRY(check_moe(m, rows));
    KQ_REQUIRE(ld_act % 4 == 0 && ((uintptr_t)act & 15) == 0, "experts: activations");
    kq_launch(moe_few_down_kernel, dim3((unsigned)kq_div_up(m.h, DOWN_ROWS), (unsigned)rows), NT, 0, st, m, act, ld_act, ids, wts, down, sh_down, out, ldo);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

int64_t kq_moe_max_tiles(int64_t pairs, int experts) { return pairs / KQ_TILE_M + std::min<int64_t>(pairs, experts); }

b200_status kq_moe_route(const KqMoe &m, int rows, const KqMoeOrder &o, float *sh32, int64_t ld32, uint16_t *sh16, int64_t ld16, cudaStream_t st) {
    KQ_TRY(check_moe(m, rows));
    const size_t smem = (size_t)NW * m.experts * 4;
    static size_t have[16];
    KQ_TRY(allow_smem(moe_route_kernel, smem + 8192, have));
    const int route_ctas = (int)kq_div_up(rows, NW), slices = m.ff_shared ? (int)kq_div_up(sh16 ? ld16 : m.ff_shared, GLU_COLS) : 0;
    kq_launch(moe_route_kernel, (unsigned)(route_ctas + rows * slices), NT, smem, st, m, rows, route_ctas, slices, o, sh32, ld32, sh16, ld16);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_moe_order(const KqMoe &m, int rows, const KqMoeOrder &o, cudaStream_t st) {
    KQ_TRY(check_moe(m, rows));
    kq_launch(moe_order_kernel, 1, ORDER_NT, 0, st, m.experts, rows * m.top, o);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_moe_gather(const KqMoe &m, int rows, const KqMoeOrder &o, const void *x, void *y, int64_t ld, int elem_bytes, cudaStream_t st) {
    KQ_TRY(check_moe(m, rows));
    const int64_t pairs = (int64_t)rows * m.top;
    KQ_REQUIRE(ld * elem_bytes % 16 == 0 && (((uintptr_t)x | (uintptr_t)y) & 15) == 0, "experts: rows of %lld elements", (long long)ld);
    kq_launch(moe_gather_kernel<uint4>, (unsigned)kq_div_up(pairs, NW), NT, 0, st, m.top, pairs, o.pos, (const uint8_t *)x, (uint8_t *)y, ld * elem_bytes);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_moe_combine(const KqMoe &m, int rows, const KqMoeOrder &o, const float *y, int64_t ldy, float *out, int64_t ldo, bool first, cudaStream_t st) {
    KQ_TRY(check_moe(m, rows));
    KQ_REQUIRE(((ldy | ldo) & 3) == 0 && ldo >= kq_pad(m.h, 4) && ldy >= kq_pad(m.h, 4) && rows <= 65535, "experts: combine");
    kq_launch(moe_combine_kernel, dim3((unsigned)kq_div_up(m.h, 4 * NT), (unsigned)rows), NT, 0, st, m.top, m.h, o.pos, o.wts, y, ldy, out, ldo, first ? 1 : 0);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
