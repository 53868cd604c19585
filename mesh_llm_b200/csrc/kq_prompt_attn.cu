// Attention of a prompt on the 5th-generation tensor cores over f16 keys and values: S = Q K^T and O += P V are
// tcgen05.mma kind::f16 with the accumulators in TMEM, K and V tiles come by TMA, P goes back into TMEM as the A operand
// of the second product, online softmax in base 2 and f32 (as in kq_attn_prefill_tc.cu, whose shapes are fixed).
//
// One CTA serves 128 positions of one query head; any number of them may share a key / value head.  Key and value sizes
// are independent (boxes of 64 dims of [row][head][64-padded dims]), a key may have a second part that all heads share
// ([row][64-padded dims]).  Keys lie one after the other from position `lo`, or in a ring.  What a query sees is causal and may
// begin at the start of a sliding window or of the query's own chunk of positions; both edges are masked, tiles start at
// the first key the CTA's first query sees.  An output gate per head can be applied to the finished rows, which leave as
// bf16, ready for the output projection's GEMM.
#include "kq_dense.cuh"
#include "kq_tc.cuh"

#include <math.h>

#include <algorithm>

namespace {

constexpr int QBOX = 128 * 64 * 2; // bytes of a box of 128 query rows x 64 dims
constexpr uint32_t COL_S = 0;
constexpr int NSOFT = 256, NTHREADS = NSOFT + 32; // eight softmax warps and the issuing warp
constexpr uint64_t LIMIT = 5 * KQ_WAIT_LIMIT_NS;
constexpr int MAX_SMEM = 13 * QBOX; // operands in shared memory

__device__ int g_prompt_attn_error;

struct AttnParams {
    CUtensorMap ku, kr, v;
    const float *q, *gate;
    uint16_t *out;
    int64_t ldq, ldg, ldo;
    int32_t T, pos0, lo, ring;                  // lo: position of row 0; ring > 0: position p in row p % ring instead
    int32_t window, chunk, rep;                 // rep: query heads per key / value head
    int32_t dim, rot, vdim, nu, nr, nv;         // nu, nr, nv: boxes of the own key part, the shared part, the values
    uint32_t tmem_cols;
    float scale_log2;
    int32_t vec, vec_out;
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint32_t pack_h2(float a, float b) {
    const __half2 h = __floats2half2_rn(a, b);
    return *reinterpret_cast<const uint32_t *>(&h);
}
__device__ __forceinline__ uint32_t pack_h2_sat(float a, float b) { return (uint32_t)kq_f2h_sat(a) | ((uint32_t)kq_f2h_sat(b) << 16); }
__device__ __forceinline__ void softmax_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(NSOFT) : "memory"); }

// grid (query tiles, heads); BK keys per tile: 128, or 64 where the operands would leave room for one CTA per SM only
template <int BK>
__global__ void __launch_bounds__(NTHREADS, 2) prompt_attn_kernel(const __grid_constant__ AttnParams p) {
    constexpr int BOX = BK * 128, HK = BK / 2; // bytes of a box of BK rows x 64 dims, keys of a half row
    constexpr uint32_t COL_O = BK;
    KQ_PDL_ENTER();
    extern __shared__ uint8_t sm_raw[];
    __shared__ uint64_t full_k, full_v, s_ready, p_ready, pv_done;
    __shared__ float red[2][2][128], lsum[128];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort_word;
    volatile int &s_abort = *(volatile int *)&s_abort_word;
    uint8_t *sm = (uint8_t *)(((uintptr_t)sm_raw + 1023) & ~(uintptr_t)1023);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int head = blockIdx.y, kv_head = head / p.rep, nk = p.nu + p.nr;
    const int t_base = blockIdx.x * 128, p_base = p.pos0 + t_base, p_last = min(p.pos0 + p.T, p_base + 128) - 1;
    int first = max(p.lo, kq_first_key(p_base, p.window, p.chunk)); // first key (absolute) any row sees
    if (p.ring) first = first / BK * BK;                            // a tile of the ring does not wrap
    const int n_tiles = (p_last - first) / BK + 1;
    uint8_t *sm_q = sm, *sm_k = sm + nk * QBOX, *sm_v = sm_k + nk * BOX;
    const uint32_t bar_k = smem_u32(&full_k), bar_v = smem_u32(&full_v), bar_s = smem_u32(&s_ready), bar_p = smem_u32(&p_ready),
                   bar_pv = smem_u32(&pv_done);
    if (warp == 8) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(p.tmem_cols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    if (tid == 0) {
        asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_k), "r"(1));
        asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_v), "r"(1));
        asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_s), "r"(1));
        asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_p), "r"(NSOFT));
        asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_pv), "r"(1));
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        s_abort = 0;
    }
    const int row = tid & 127, half = (tid >> 7) & 1;
    const bool row_ok = warp < 8 && t_base + row < p.T;
    const int hi = row_ok ? p_base + row : -1;                                    // last visible key of this row
    const int lo = row_ok ? kq_first_key(hi, p.window, p.chunk) : 0;              // first one
    if (warp < 8) { // Q to f16 (scaled), K-major, swizzled
        const float *qr = p.q + (int64_t)(row_ok ? t_base + row : 0) * p.ldq + (int64_t)head * (p.dim + p.rot);
        for (int b = half; b < nk; b += 2) {
            const float *src = b < p.nu ? qr + b * 64 : qr + p.dim + (b - p.nu) * 64;
            const int n = b < p.nu ? p.dim - b * 64 : p.rot - (b - p.nu) * 64;
            uint8_t *dst = sm_q + b * QBOX + row * 128;
#pragma unroll 2
            for (int c = 0; c < 8; c++) {
                float v[8];
                if (row_ok && p.vec && 8 * c + 8 <= n) {
                    const float4 x = *reinterpret_cast<const float4 *>(src + 8 * c), y = *reinterpret_cast<const float4 *>(src + 8 * c + 4);
                    v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w, v[4] = y.x, v[5] = y.y, v[6] = y.z, v[7] = y.w;
                } else {
#pragma unroll
                    for (int e = 0; e < 8; e++) v[e] = row_ok && 8 * c + e < n ? src[8 * c + e] : 0.f;
                }
                uint4 w;
                w.x = pack_h2_sat(v[0] * p.scale_log2, v[1] * p.scale_log2);
                w.y = pack_h2_sat(v[2] * p.scale_log2, v[3] * p.scale_log2);
                w.z = pack_h2_sat(v[4] * p.scale_log2, v[5] * p.scale_log2);
                w.w = pack_h2_sat(v[6] * p.scale_log2, v[7] * p.scale_log2);
                *reinterpret_cast<uint4 *>(dst + ((c ^ (row & 7)) << 4)) = w;
            }
        }
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = s_tmem;
    const int ncol = p.nv * 64, nh = ncol / 2; // columns of O, and of one thread's half

    if (warp == 8) { // all lanes run the loop, so that descriptors stay in uniform registers; one posts and issues
        const bool lead = tc_elect();
        {
            auto row_of = [&](int tile) { return p.ring ? (first + tile * BK) % p.ring : first - p.lo + tile * BK; };
            auto load_k = [&](int tile) {
                const int r0 = row_of(tile);
                asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar_k), "r"(nk * BOX) : "memory");
                for (int b = 0; b < p.nu; b++)
                    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(
                                     smem_u32(sm_k + b * BOX)),
                                 "l"(&p.ku), "r"(b * 64), "r"(kv_head), "r"(r0), "r"(bar_k)
                                 : "memory");
                for (int b = 0; b < p.nr; b++)
                    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(
                                     smem_u32(sm_k + (p.nu + b) * BOX)),
                                 "l"(&p.kr), "r"(b * 64), "r"(r0), "r"(bar_k)
                                 : "memory");
            };
            auto load_v = [&](int tile) {
                const int r0 = row_of(tile);
                asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar_v), "r"(p.nv * BOX) : "memory");
                for (int b = 0; b < p.nv; b++)
                    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(
                                     smem_u32(sm_v + b * BOX)),
                                 "l"(&p.v), "r"(b * 64), "r"(kv_head), "r"(r0), "r"(bar_v)
                                 : "memory");
            };
            if (lead) {
                load_k(0);
                load_v(0);
            }
            __syncwarp();
            const uint32_t q_addr = smem_u32(sm_q), k_addr = smem_u32(sm_k), v_addr = smem_u32(sm_v);
            const uint32_t id_s = tc_idesc(128, BK, false, false), id_o = tc_idesc(128, ncol, false, true);
            const int su = (p.dim + 15) / 16, sr = (p.rot + 15) / 16; // K steps of the two key parts
            auto wait = [&](uint32_t bar, uint32_t parity, int code) {
                return __all_sync(0xffffffffu, tc_wait(bar, parity, &s_abort_word, &g_prompt_attn_error, code, LIMIT)) != 0; // a warp gives up as a whole
            };
            bool go = true;
            for (int i = 0; i < n_tiles; i++) {
                const uint32_t ph = (uint32_t)(i & 1);
                go = go && wait(bar_k, ph, 1);
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (lead) {
                    if (go) {
                        for (int s = 0; s < su; s++)
                            tc_mma_ss(tmem + COL_S, tc_desc_k(q_addr + (s >> 2) * QBOX, s & 3), tc_desc_k(k_addr + (s >> 2) * BOX, s & 3), id_s, s > 0);
                        for (int s = 0; s < sr; s++)
                            tc_mma_ss(tmem + COL_S, tc_desc_k(q_addr + (p.nu + (s >> 2)) * QBOX, s & 3),
                                      tc_desc_k(k_addr + (p.nu + (s >> 2)) * BOX, s & 3), id_s, 1);
                    }
                    tc_commit(bar_s);
                }
                __syncwarp();
                go = wait(bar_s, ph, 2) && go; // K has been read: the next tile's K can come in
                if (lead && go && i + 1 < n_tiles) load_k(i + 1);
                __syncwarp();
                go = go && wait(bar_p, ph, 3);
                go = go && wait(bar_v, ph, 4);
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                if (lead) {
                    if (go) {
#pragma unroll
                        for (int s = 0; s < BK / 16; s++) // 16 keys per instruction: eight packed columns of P at the start of each half's columns of S
                            tc_mma_ts(tmem + COL_O, tmem + COL_S + HK * (s / (HK / 16)) + 8 * (s % (HK / 16)), tc_desc_mn(v_addr, BOX, s), id_o,
                                      (i > 0 || s > 0) ? 1u : 0u);
                    }
                    tc_commit(bar_pv);
                }
                __syncwarp();
                go = wait(bar_pv, ph, 5) && go; // P (over S) and V have been read, O is complete up to this tile
                if (lead && go && i + 1 < n_tiles) load_v(i + 1);
                __syncwarp();
            }
            if (!go) s_abort = 1;
        }
        __syncwarp();
    } else {
        // online softmax, half a row per thread
        const uint32_t tl = tmem + ((uint32_t)((warp & 3) * 32) << 16);
        const int c0 = HK * half, last_lo = kq_first_key(p_last, p.window, p.chunk);
        float m = -INFINITY, l = 0.f;
        for (int i = 0; i < n_tiles; i++) {
            tc_wait(bar_s, (uint32_t)(i & 1), &s_abort_word, &g_prompt_attn_error, 6, LIMIT);
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int t0 = first + i * BK, k0 = t0 + c0;
            // some row of the tile sees only part of these keys: past the diagonal, or in front of what the last row sees
            const bool edge = t0 + BK - 1 > p_base || t0 < last_lo;
            float t4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int c = 0; c < HK / 32; c++) {
                uint32_t s[32];
                TMEM_LD32(tl + COL_S + c0 + 32 * c, s);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (!edge) {
#pragma unroll
                    for (int j = 0; j < 32; j++) t4[j & 3] = fmaxf(t4[j & 3], __uint_as_float(s[j]));
                } else {
#pragma unroll
                    for (int j = 0; j < 32; j++) {
                        const int key = k0 + 32 * c + j;
                        if (key <= hi && key >= lo) t4[j & 3] = fmaxf(t4[j & 3], __uint_as_float(s[j]));
                    }
                }
            }
            red[i & 1][half][row] = row_ok ? fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3])) : -INFINITY;
            softmax_barrier();
            const float m_new = fmaxf(m, fmaxf(red[i & 1][0][row], red[i & 1][1][row]));
            const float alpha = (m_new == -INFINITY || m == m_new) ? 1.f : ex2(m - m_new);
            const float sub = m_new == -INFINITY ? 0.f : m_new;
            // S was issued after the P V of the tile before had completed, so O is at rest here
            if (i > 0 && !s_abort && __any_sync(0xffffffffu, alpha != 1.f)) {
                for (int c = 0; c < nh; c += 32) {
                    uint32_t o[32];
                    TMEM_LD32(tl + COL_O + half * nh + c, o);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int j = 0; j < 32; j++) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
                    TMEM_ST32(tl + COL_O + half * nh + c, o);
                }
            }
            l *= alpha;
            m = m_new;
            float l4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int c = 0; c < HK / 32; c++) {
                uint32_t s[32], pk[16];
                TMEM_LD32(tl + COL_S + c0 + 32 * c, s);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                for (int j = 0; j < 32; j += 2) {
                    float e0 = ex2(__uint_as_float(s[j]) - sub), e1 = ex2(__uint_as_float(s[j + 1]) - sub);
                    if (edge) {
                        const int key = k0 + 32 * c + j;
                        e0 = key <= hi && key >= lo ? e0 : 0.f;
                        e1 = key + 1 <= hi && key + 1 >= lo ? e1 : 0.f;
                    }
                    l4[(j >> 1) & 3] += e0 + e1;
                    pk[j >> 1] = pack_h2(e0, e1);
                }
                if (!s_abort) TMEM_ST16(tl + COL_S + c0 + 16 * c, pk);
            }
            if (row_ok) l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar_p) : "memory");
        }
        // O / l, gated -> out
        if (half == 1) lsum[row] = l;
        softmax_barrier();
        if (half == 0) lsum[row] = l + lsum[row];
        softmax_barrier();
        l = lsum[row];
        tc_wait(bar_pv, (uint32_t)((n_tiles - 1) & 1), &s_abort_word, &g_prompt_attn_error, 7, LIMIT);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const bool go = __all_sync(0xffffffffu, !s_abort);
        if (go) {
            const int t = row_ok ? t_base + row : 0;
            const float f = (l > 0.f ? 1.f / l : 0.f) * (p.gate ? kq_sigmoid(p.gate[t * p.ldg + head]) : 1.f);
            uint16_t *orow = p.out + (int64_t)t * p.ldo + (int64_t)head * p.vdim;
            for (int c = half * nh; c < half * nh + nh; c += 32) {
                uint32_t o[32];
                TMEM_LD32(tl + COL_O + c, o);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (!row_ok) continue;
#pragma unroll
                for (int j = 0; j < 32; j += 8) {
                    if (c + j >= p.vdim) break;
                    if (p.vec_out) {
                        uint32_t w[4];
#pragma unroll
                        for (int e = 0; e < 4; e++)
                            w[e] = (uint32_t)kq_f2bf(__uint_as_float(o[j + 2 * e]) * f) | ((uint32_t)kq_f2bf(__uint_as_float(o[j + 2 * e + 1]) * f) << 16);
                        *reinterpret_cast<uint4 *>(orow + c + j) = make_uint4(w[0], w[1], w[2], w[3]);
                    } else {
#pragma unroll
                        for (int e = 0; e < 8; e++)
                            if (c + j + e < p.vdim) orow[c + j + e] = kq_f2bf(__uint_as_float(o[j + e]) * f);
                    }
                }
            }
        }
    }
    if (s_abort && warp == 8 && lane == 0) { // copies and MMAs that were posted must end before the CTA goes away
        kq_mbar_wait(bar_k, 0u, KQ_WAIT_LIMIT_NS);
        kq_mbar_wait(bar_k, 1u, KQ_WAIT_LIMIT_NS);
        kq_mbar_wait(bar_v, 0u, KQ_WAIT_LIMIT_NS);
        kq_mbar_wait(bar_v, 1u, KQ_WAIT_LIMIT_NS);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 8) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(p.tmem_cols) : "memory");
}

} // namespace

int kq_prompt_attn_error_fetch() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_prompt_attn_error, sizeof(int)) != cudaSuccess) return -1;
    if (v) cudaMemcpyToSymbol(g_prompt_attn_error, &zero, sizeof(int));
    return v;
}

bool kq_prompt_attention_fits(int dim, int rot, int vdim) {
    const int nk = (int)(kq_pad(dim, 64) + kq_pad(rot, 64)) / 64, nv = (int)kq_pad(vdim, 64) / 64;
    return nk * QBOX + (nk + nv) * QBOX / 2 <= MAX_SMEM && nv <= 4; // with 64 keys per tile
}

b200_status kq_prompt_attention(const KqPromptAttn &a, cudaStream_t st) {
    if (!kq_prompt_attention_fits(a.dim, a.rot, a.vdim)) return B200_ERR_UNSUPPORTED;
    KQ_REQUIRE(a.n_head >= 1 && a.kv_heads >= 1 && a.n_head % a.kv_heads == 0 && a.T >= 1 && a.rows >= 1, "prompt_attention: bad call");
    KQ_REQUIRE(a.ring ? a.ring % 128 == 0 && a.ring == a.rows && a.lo == 0 : a.pos0 + a.T - a.lo <= a.rows, "prompt_attention: %lld rows of keys", (long long)a.rows);
    AttnParams p = {};
    const int nk = (int)(kq_pad(a.dim, 64) + kq_pad(a.rot, 64)) / 64, nv = (int)kq_pad(a.vdim, 64) / 64;
    const int bk = 2 * nk + nv <= 6 ? 128 : 64; // two CTAs per SM where that is possible
    const uint64_t G = (uint64_t)a.kv_heads, up = (uint64_t)kq_pad(a.dim, 64), rp = (uint64_t)kq_pad(a.rot, 64), vp = (uint64_t)kq_pad(a.vdim, 64);
    b200_status rc;
    {
        const uint64_t dims[3] = {up, G, (uint64_t)a.rows}, str[2] = {up * 2, G * up * 2};
        const uint32_t box[3] = {64, 1, (uint32_t)bk};
        if ((rc = kq_tmap_encode(&p.ku, 2, 3, a.k, dims, str, box, 1)) != B200_OK) return rc;
    }
    {
        const uint64_t dims[3] = {vp, G, (uint64_t)a.rows}, str[2] = {vp * 2, G * vp * 2};
        const uint32_t box[3] = {64, 1, (uint32_t)bk};
        if ((rc = kq_tmap_encode(&p.v, 2, 3, a.v, dims, str, box, 1)) != B200_OK) return rc;
    }
    if (rp) {
        const uint64_t dims[2] = {rp, (uint64_t)a.rows}, str[1] = {rp * 2};
        const uint32_t box[2] = {64, (uint32_t)bk};
        if ((rc = kq_tmap_encode(&p.kr, 2, 2, a.kr, dims, str, box, 1)) != B200_OK) return rc;
    }
    p.q = a.q, p.gate = a.gate, p.out = a.out, p.ldq = a.ldq, p.ldg = a.ldg, p.ldo = a.ldo;
    p.T = a.T, p.pos0 = a.pos0, p.lo = a.lo, p.ring = a.ring, p.window = a.window, p.chunk = a.chunk, p.rep = a.n_head / a.kv_heads;
    p.dim = a.dim, p.rot = a.rot, p.vdim = a.vdim;
    p.nu = (int)(up / 64), p.nr = (int)(rp / 64), p.nv = (int)(vp / 64);
    p.tmem_cols = bk + p.nv * 64 <= 256 ? 256 : 512;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.vec = a.dim % 4 == 0 && a.rot % 4 == 0 && a.ldq % 4 == 0 && ((uintptr_t)a.q & 15) == 0;
    p.vec_out = a.vdim % 8 == 0 && a.ldo % 8 == 0 && ((uintptr_t)a.out & 15) == 0;
    const size_t smem = (size_t)nk * QBOX + (size_t)(nk + nv) * bk * 128 + 1024;
    static size_t attr[16][2];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    auto kern = bk == 128 ? prompt_attn_kernel<128> : prompt_attn_kernel<64>;
    if (dev < 0 || dev >= 16 || attr[dev][bk == 128] < smem) {
        KQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        if (dev >= 0 && dev < 16) attr[dev][bk == 128] = smem;
    }
    kq_launch(kern, dim3((unsigned)kq_div_up(a.T, 128), (unsigned)a.n_head), NTHREADS, smem, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
