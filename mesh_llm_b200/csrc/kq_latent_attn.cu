// Latent attention over a ring cache: a position keeps one normed latent (kv_rank values) and one rotated key
// part shared by all heads; the per-head keys and values are linear maps of the latent.  Decode folds the key
// map into the query ("absorbed" form): score = q_lat . c + q_rot . k_rot with q_lat = W_uk^T q, and the value
// map into the output: o = W_uv (sum_j p_j c_j), so that a step reads each visible row once for all heads.
//
// A decode step (up to 8 rows) is three launches around the cache: kq_latent_query (norm of the latent, rotations,
// cache store, and in other CTAs of the same launch the absorbed queries), kq_latent_attention (a CTA takes 16
// heads of one row and a range of keys and leaves an unnormalised partial result), kq_latent_output (merges the
// ranges of a head, applies W_uv and the output gate).  With a bf16 cache the products of the attention run on
// mma.m16n8k16, 16 heads being the rows of a tile; queries and probabilities enter as hi + lo pairs of bf16, so that
// the result is that of f32 operands.  The f32 form serves f32 caches and calls with more rows.
#include "kq_gemv_grouped.cuh"

#include <algorithm>
#include <math.h>

namespace {

constexpr int NT = 256, NW = NT / 32, NH = 2, HG = NW * NH, KT = 32; // heads per warp and CTA, keys per tile
constexpr int MAX_SPLIT = 64;

__device__ __forceinline__ float block_sum(float v, float *red) {
    v = kq_warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < NW; i++) t += red[i];
    return t;
}

// sine and cosine of pos * freq; the product and its reduction to one turn are exact to well below f32 rounding
__device__ __forceinline__ void rot_angle(int pos, double freq, float *s, float *c) {
    const double a = (double)pos * freq, turn = 6.283185307179586;
    sincosf((float)(a - turn * rint(a / turn)), s, c);
}

__device__ __forceinline__ void put(const KqLatent &l, int64_t i, float v) {
    if (l.f32) ((float *)l.cache)[i] = v;
    else ((uint16_t *)l.cache)[i] = kq_f2bf(v);
}

struct StoreParams {
    const float *norm_w;
    float eps;
    float *q;
    int64_t ldq;
    const float *kv;
    int64_t ldkv;
    int32_t T, pos0;
    const int32_t *pos0_dev;
    float *q_lat;
    int64_t ldql;
};

// one CTA per row; cs: shared memory for cos and sin of every pair
__device__ __forceinline__ void store_row(const KqLatent &l, const StoreParams &p, int64_t row, float *cs, float *red) {
    const int tid = threadIdx.x, T = p.T, pos0_val = p.pos0;
    const int32_t *pos0_dev = p.pos0_dev;
    const float *norm_w = p.norm_w, *kv = p.kv;
    const float eps = p.eps;
    float *q = p.q, *q_lat = p.q_lat;
    const int64_t ldq = p.ldq, ldkv = p.ldkv, ldql = p.ldql;
    const int seq = (int)(row / T), pos = (pos0_dev ? *pos0_dev : pos0_val) + (int)(row % T);
    const int64_t dst = seq * l.seq_stride + (int64_t)(pos % l.cap) * l.ld;
    const int half = l.rot_dims / 2;
    for (int i = tid; i < half; i += NT) rot_angle(pos, l.freq[i], &cs[half + i], &cs[i]);
    const float *c = kv + row * ldkv;
    float ss = 0.f;
    for (int i = tid; i < l.kv_rank; i += NT) ss += c[i] * c[i];
    const float sc = 1.0f / sqrtf(block_sum(ss, red) / (float)l.kv_rank + eps); // the barrier inside also publishes cs
    for (int i = tid; i < l.kv_rank; i += NT) put(l, dst + i, c[i] * sc * norm_w[i]);
    const float *kr = c + l.kv_rank;
    for (int i = tid; i < l.rot_dim; i += NT) {
        float v = kr[i];
        if (i < 2 * half) {
            const float co = cs[i >> 1], si = cs[half + (i >> 1)];
            v = (i & 1) ? v * co + kr[i - 1] * si : v * co - kr[i + 1] * si;
        }
        put(l, dst + l.rot_at + i, v);
    }
    const int hd = l.qk_dim + l.rot_dim;
    const int np = (l.rot_dim + 1) / 2; // pairs per head, the last one possibly a single value
    for (int i = tid; i < l.n_head * np; i += NT) {
        const int h = i / np, j = i % np;
        float *qr = q + row * ldq + (int64_t)h * hd + l.qk_dim + 2 * j;
        float u = qr[0], v = 2 * j + 1 < l.rot_dim ? qr[1] : 0.f;
        if (j < half) {
            const float co = cs[j], si = cs[half + j], u0 = u;
            u = u0 * co - v * si;
            v = v * co + u0 * si;
        }
        qr[0] = u;
        if (2 * j + 1 < l.rot_dim) qr[1] = v;
        if (q_lat) {
            float *o = q_lat + row * ldql + (int64_t)h * l.ld + l.rot_at + 2 * j;
            o[0] = u;
            if (2 * j + 1 < l.rot_dim) o[1] = v;
        }
    }
    if (q_lat) // padding of the query rows
        for (int i = tid; i < l.n_head * 16; i += NT) {
            const int h = i >> 4, j = i & 15;
            float *o = q_lat + row * ldql + (int64_t)h * l.ld;
            const int k = j < 8 ? l.kv_rank + j : l.rot_at + l.rot_dim + j - 8;
            if (j < 8 ? k < l.rot_at : k < l.ld) o[k] = 0.f;
        }
}

__global__ void __launch_bounds__(NT) latent_store_kernel(const __grid_constant__ KqLatent l, const __grid_constant__ StoreParams p) {
    KQ_PDL_ENTER();
    __shared__ float red[NW];
    extern __shared__ float cs[];
    store_row(l, p, blockIdx.x, cs, red);
}

// the first `rows` CTAs store, the others absorb the unrotated part of the queries
template <int M>
__global__ void __launch_bounds__(NT) latent_query_kernel(const __grid_constant__ KqLatent l, const __grid_constant__ StoreParams p,
                                                          const __grid_constant__ KqGrouped a, int rows) {
    KQ_PDL_TRIGGER();
    __shared__ float red[NW];
    extern __shared__ float cs[];
    if ((int)blockIdx.x < rows) {
        KQ_PDL_WAIT();
        store_row(l, p, blockIdx.x, cs, red);
    } else {
        kq_grouped_rows<M>(a, (int64_t)(blockIdx.x - rows) * NW + (threadIdx.x >> 5), threadIdx.x & 31);
    }
}

// eight consecutive cache values from shared memory as floats
template <typename E>
__device__ __forceinline__ void row8(const E *p, float (&v)[8]) {
    if (sizeof(E) == 2) {
        const uint4 q = *reinterpret_cast<const uint4 *>(p);
        const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
        for (int i = 0; i < 4; i++) {
            v[2 * i] = __uint_as_float(w[i] << 16);
            v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    } else {
        const float4 a = reinterpret_cast<const float4 *>(p)[0], b = reinterpret_cast<const float4 *>(p)[1];
        v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
    }
}

// grid (key ranges, head groups, rows).  E: cache element; NC: 256-value chunks of the latent
template <typename E, int NC>
__global__ void __launch_bounds__(NT) latent_attn_kernel(const __grid_constant__ KqLatent l, const float *q_lat, int T,
                                                         const int32_t *pos0_dev, int pos0_val, int keys_per_split, float *o_lat,
                                                         int64_t ldo, float *scratch, int pitch) {
    KQ_PDL_ENTER();
    extern __shared__ __align__(16) uint8_t sm[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int split = blockIdx.x, hg = blockIdx.y;
    const int64_t row = blockIdx.z;
    const int seq = (int)(row / T), pos = (pos0_dev ? *pos0_dev : pos0_val) + (int)(row % T);
    const int lo = l.window > 0 ? max(0, pos - l.window + 1) : 0, vis = pos + 1 - lo;
    const int n_split = (vis + keys_per_split - 1) / keys_per_split;
    if (split >= n_split) return;
    const int k0 = lo + split * keys_per_split, k1 = min(pos + 1, k0 + keys_per_split);
    float *sq = reinterpret_cast<float *>(sm);            // [HG][ld]
    uint8_t *tile = sm + (size_t)HG * l.ld * sizeof(float); // [KT] rows of `pitch` bytes
    const E *cache = (const E *)l.cache + seq * l.seq_stride;
    for (int i = tid; i < HG * l.ld; i += NT) {
        const int h = hg * HG + i / l.ld;
        sq[i] = h < l.n_head ? q_lat[(row * l.n_head + h) * l.ld + i % l.ld] * (l.scale * 1.4426950408889634f) : 0.f;
    }
    float m[NH], sum[NH], o[NH][NC][8];
#pragma unroll
    for (int a = 0; a < NH; a++) {
        m[a] = -INFINITY;
        sum[a] = 0.f;
#pragma unroll
        for (int c = 0; c < NC; c++)
#pragma unroll
            for (int e = 0; e < 8; e++) o[a][c][e] = 0.f;
    }
    const int n16 = l.ld * (int)sizeof(E) / 16, nck = l.ld / 8, nlat = (l.kv_rank + 7) / 8;
    const bool active = hg * HG + warp * NH < l.n_head;
    for (int kb = k0; kb < k1; kb += KT) {
        __syncthreads(); // everybody is done with the tile before (and, the first time, q is in)
        for (int i = tid; i < KT * n16; i += NT) {
            const int r = i / n16, c = i % n16, key = kb + r;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (key < k1) v = *reinterpret_cast<const uint4 *>((const uint8_t *)(cache + (int64_t)(key % l.cap) * l.ld) + 16 * c);
            *reinterpret_cast<uint4 *>(tile + (size_t)r * pitch + 16 * c) = v;
        }
        __syncthreads();
        if (!active) continue;
        // scores, lane = key
        float s[NH] = {};
        const E *kr = reinterpret_cast<const E *>(tile + (size_t)lane * pitch);
        for (int c = 0; c < nck; c++) {
            float v[8];
            row8(kr + 8 * c, v);
#pragma unroll
            for (int a = 0; a < NH; a++) {
                const float4 x = *reinterpret_cast<const float4 *>(sq + (warp * NH + a) * l.ld + 8 * c);
                const float4 y = *reinterpret_cast<const float4 *>(sq + (warp * NH + a) * l.ld + 8 * c + 4);
                s[a] = fmaf(x.x, v[0], s[a]), s[a] = fmaf(x.y, v[1], s[a]), s[a] = fmaf(x.z, v[2], s[a]), s[a] = fmaf(x.w, v[3], s[a]);
                s[a] = fmaf(y.x, v[4], s[a]), s[a] = fmaf(y.y, v[5], s[a]), s[a] = fmaf(y.z, v[6], s[a]), s[a] = fmaf(y.w, v[7], s[a]);
            }
        }
        float p[NH];
#pragma unroll
        for (int a = 0; a < NH; a++) {
            const float sv = kb + lane < k1 ? s[a] : -INFINITY;
            const float mn = fmaxf(m[a], kq_warp_max(sv)); // the tile has at least one key
            const float al = exp2f(m[a] - mn);
            p[a] = exp2f(sv - mn);
            sum[a] = sum[a] * al + kq_warp_sum(p[a]);
            m[a] = mn;
#pragma unroll
            for (int c = 0; c < NC; c++)
#pragma unroll
                for (int e = 0; e < 8; e++) o[a][c][e] *= al;
        }
        // values, lane = latent dimensions 8 lane + 256 c ..
        const int nk = min(KT, k1 - kb);
        for (int j = 0; j < nk; j++) {
            float pj[NH];
#pragma unroll
            for (int a = 0; a < NH; a++) pj[a] = __shfl_sync(0xffffffffu, p[a], j);
#pragma unroll
            for (int c = 0; c < NC; c++)
                if (lane + 32 * c < nlat) {
                    float v[8];
                    row8(reinterpret_cast<const E *>(tile + (size_t)j * pitch) + 8 * (lane + 32 * c), v);
#pragma unroll
                    for (int a = 0; a < NH; a++)
#pragma unroll
                        for (int e = 0; e < 8; e++) o[a][c][e] = fmaf(pj[a], v[e], o[a][c][e]);
                }
        }
    }
    const int64_t rp = kq_f32_ld(l.kv_rank);
    if (o_lat) {
#pragma unroll
        for (int a = 0; a < NH; a++) {
            const int h = hg * HG + warp * NH + a;
            if (h >= l.n_head) break;
            const float inv = 1.f / sum[a];
#pragma unroll
            for (int c = 0; c < NC; c++)
#pragma unroll
                for (int e = 0; e < 8; e++) {
                    const int d = 8 * (lane + 32 * c) + e;
                    if (d < l.kv_rank) o_lat[row * ldo + h * rp + d] = o[a][c][e] * inv;
                }
        }
        return;
    }
    // partial results: [row][head][range] of (rp values, max, sum)
    const int64_t ps = rp + 2;
#pragma unroll
    for (int a = 0; a < NH; a++) {
        const int h = hg * HG + warp * NH + a;
        if (h >= l.n_head) break;
        float *d = scratch + ((row * l.n_head + h) * gridDim.x + split) * ps;
#pragma unroll
        for (int c = 0; c < NC; c++)
            if (lane + 32 * c < nlat) {
                float2 *d2 = reinterpret_cast<float2 *>(d + 8 * (lane + 32 * c));
#pragma unroll
                for (int e = 0; e < 4; e++) d2[e] = make_float2(o[a][c][2 * e], o[a][c][2 * e + 1]);
            }
        if (lane == 0) {
            d[rp] = m[a];
            d[rp + 1] = sum[a];
        }
    }
}

// ---- bf16 cache, few rows: tensor-core form ------------------------------------------------------------
constexpr int MK = 64, SP = MK + 4, PP = MK * 2 + 16; // keys per tile, floats per score row, bytes per probability row

__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(addr));
}
__device__ __forceinline__ void ldsm2(uint32_t addr, uint32_t (&r)[2]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// grid (key ranges, head groups, rows).  Warp w owns keys 8w .. 8w+7 of a tile in S = Q C^T, heads 2w and 2w+1 in the
// softmax, and latent dimensions 16w, 16w + 128, ... in O = P C.  NP: pairs of 8-dimension tiles per warp.
template <int NP>
__global__ void __launch_bounds__(NT) latent_attn_mma_kernel(const __grid_constant__ KqLatent l, const float *q_lat, int T,
                                                             const int32_t *pos0_dev, int pos0_val, int keys_per_split, float *scratch,
                                                             int pitch) {
    KQ_PDL_ENTER();
    extern __shared__ __align__(16) uint8_t sm[];
    __shared__ float ss[HG][SP], s_alpha[HG];
    __shared__ __align__(16) uint8_t sp_hi[HG * PP], sp_lo[HG * PP];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int split = blockIdx.x, hg = blockIdx.y;
    const int64_t row = blockIdx.z;
    const int seq = (int)(row / T), pos = (pos0_dev ? *pos0_dev : pos0_val) + (int)(row % T);
    const int lo = l.window > 0 ? max(0, pos - l.window + 1) : 0, vis = pos + 1 - lo;
    const int n_split = (vis + keys_per_split - 1) / keys_per_split;
    if (split >= n_split) return;
    const int k0 = lo + split * keys_per_split, k1 = min(pos + 1, k0 + keys_per_split);
    uint8_t *q_hi = sm, *q_lo = sm + HG * pitch, *tile = sm + 2 * HG * pitch;
    const uint16_t *cache = (const uint16_t *)l.cache + seq * l.seq_stride;
    const int ks = (l.ld + 15) / 16, ld16 = ks * 16, n16 = ks * 2; // K steps of the scores, row length padded to them, 16-byte chunks
    auto load_tile = [&](int kb) {
        const int slot0 = kb % l.cap;
#pragma unroll 2
        for (int r = warp; r < MK; r += NW) { // a warp per row
            const int key = kb + r, slot = slot0 + r < l.cap ? slot0 + r : slot0 + r - l.cap; // visible rows never wrap twice
            const uint8_t *src = (const uint8_t *)(cache + (int64_t)slot * l.ld);
            uint8_t *dst = tile + (size_t)r * pitch;
            for (int c = lane; c < n16; c += 32) {
                if (key < k1 && 8 * c < l.ld)
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst + 16 * c)), "l"(src + 16 * c)
                                 : "memory");
                else
                    *reinterpret_cast<uint4 *>(dst + 16 * c) = make_uint4(0, 0, 0, 0);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load_tile(k0);
    constexpr int QB = 9; // loads per head in flight
    for (int d0 = 2 * lane; d0 < ld16; d0 += 64 * QB) { // queries of the warp's two heads, scaled, as hi + lo
        float2 v[QB][NH];
#pragma unroll
        for (int e = 0; e < QB; e++)
#pragma unroll
            for (int a = 0; a < NH; a++) {
                const int h = hg * HG + warp * NH + a, d = d0 + 64 * e;
                v[e][a] = h < l.n_head && d < l.ld ? *reinterpret_cast<const float2 *>(q_lat + (row * l.n_head + h) * l.ld + d) : make_float2(0.f, 0.f);
            }
#pragma unroll
        for (int e = 0; e < QB; e++)
#pragma unroll
            for (int a = 0; a < NH; a++) {
                const int d = d0 + 64 * e;
                if (d >= ld16) break;
                const float f = l.scale * 1.4426950408889634f, x = v[e][a].x * f, y = v[e][a].y * f;
                const uint16_t hx = kq_f2bf(x), hy = kq_f2bf(y);
                *reinterpret_cast<uint32_t *>(q_hi + (warp * NH + a) * pitch + 2 * d) = (uint32_t)hx | ((uint32_t)hy << 16);
                *reinterpret_cast<uint32_t *>(q_lo + (warp * NH + a) * pitch + 2 * d) =
                    (uint32_t)kq_f2bf(x - kq_bf2f(hx)) | ((uint32_t)kq_f2bf(y - kq_bf2f(hy)) << 16);
            }
    }
    float m[NH] = {-INFINITY, -INFINITY}, sum[NH] = {}, o[NP][2][4];
#pragma unroll
    for (int a = 0; a < NP; a++)
#pragma unroll
        for (int b = 0; b < 2; b++)
#pragma unroll
            for (int e = 0; e < 4; e++) o[a][b][e] = 0.f;
    const uint32_t t_addr = (uint32_t)__cvta_generic_to_shared(tile), qh = (uint32_t)__cvta_generic_to_shared(q_hi),
                   ql = (uint32_t)__cvta_generic_to_shared(q_lo), ph = (uint32_t)__cvta_generic_to_shared(sp_hi),
                   pl = (uint32_t)__cvta_generic_to_shared(sp_lo);
    for (int kb = k0; kb < k1; kb += MK) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        { // S: 16 heads x 8 keys
            float sa[2][4] = {}, sb[2][4] = {};
            const uint32_t aoff = (uint32_t)((lane & 15) * pitch + (lane >> 4) * 16);
            const uint32_t boff = t_addr + (uint32_t)((8 * warp + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16);
            for (int k0 = 0; k0 < ks; k0 += 4) { // the fragments of four steps, then their products in four chains
                uint32_t ah[4][4], al[4][4], b[4][2];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int k = min(k0 + e, ks - 1);
                    ldsm2(boff + 32 * k, b[e]);
                    ldsm4(qh + aoff + 32 * k, ah[e]);
                    ldsm4(ql + aoff + 32 * k, al[e]);
                }
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (k0 + e < ks) {
                        mma16816(sa[e & 1], ah[e], b[e][0], b[e][1]);
                        mma16816(sb[e & 1], al[e], b[e][0], b[e][1]);
                    }
            }
#pragma unroll
            for (int e = 0; e < 4; e++) sa[0][e] += sa[1][e] + (sb[0][e] + sb[1][e]);
            const int r = lane >> 2, c = 8 * warp + (lane & 3) * 2;
            ss[r][c] = sa[0][0], ss[r][c + 1] = sa[0][1];
            ss[r + 8][c] = sa[0][2], ss[r + 8][c + 1] = sa[0][3];
        }
        __syncthreads();
#pragma unroll
        for (int a = 0; a < NH; a++) { // softmax of two heads
            const int hl = warp * NH + a;
            const float s0 = kb + 2 * lane < k1 ? ss[hl][2 * lane] : -INFINITY, s1 = kb + 2 * lane + 1 < k1 ? ss[hl][2 * lane + 1] : -INFINITY;
            const float mn = fmaxf(m[a], kq_warp_max(fmaxf(s0, s1))); // the tile has at least one key
            const float al = exp2f(m[a] - mn), p0 = exp2f(s0 - mn), p1 = exp2f(s1 - mn);
            sum[a] = sum[a] * al + kq_warp_sum(p0 + p1);
            m[a] = mn;
            const uint16_t h0 = kq_f2bf(p0), h1 = kq_f2bf(p1);
            *reinterpret_cast<uint32_t *>(sp_hi + hl * PP + 4 * lane) = (uint32_t)h0 | ((uint32_t)h1 << 16);
            *reinterpret_cast<uint32_t *>(sp_lo + hl * PP + 4 * lane) =
                (uint32_t)kq_f2bf(p0 - kq_bf2f(h0)) | ((uint32_t)kq_f2bf(p1 - kq_bf2f(h1)) << 16);
            if (lane == 0) s_alpha[hl] = al;
        }
        __syncthreads();
        const float a0 = s_alpha[lane >> 2], a1 = s_alpha[(lane >> 2) + 8];
        uint32_t fh[4][4], fl[4][4];
#pragma unroll
        for (int k = 0; k < 4; k++) {
            const uint32_t off = (uint32_t)((lane & 15) * PP + (lane >> 4) * 16 + 32 * k);
            ldsm4(ph + off, fh[k]);
            ldsm4(pl + off, fl[k]);
        }
#pragma unroll
        for (int t = 0; t < NP; t++) {
            const int d0 = 16 * (warp + NW * t);
            if (d0 >= l.kv_rank) break;
#pragma unroll
            for (int b = 0; b < 2; b++) o[t][b][0] *= a0, o[t][b][1] *= a0, o[t][b][2] *= a1, o[t][b][3] *= a1;
            uint32_t v[4][4];
#pragma unroll
            for (int k = 0; k < 4; k++) // 16 keys per step; lanes 0-15: keys, lanes 16-31: the next eight dimensions
                ldsm4t(t_addr + (uint32_t)((16 * k + (lane & 15)) * pitch + 2 * d0 + (lane >> 4) * 16), v[k]);
#pragma unroll
            for (int k = 0; k < 4; k++) {
                mma16816(o[t][0], fh[k], v[k][0], v[k][1]);
                mma16816(o[t][1], fh[k], v[k][2], v[k][3]);
                mma16816(o[t][0], fl[k], v[k][0], v[k][1]);
                mma16816(o[t][1], fl[k], v[k][2], v[k][3]);
            }
        }
        if (kb + MK < k1) {
            __syncthreads(); // everybody is done with the tile
            load_tile(kb + MK);
        }
    }
    const int64_t rp = kq_f32_ld(l.kv_rank), ps = rp + 2;
    auto part = [&](int hl) { return scratch + ((row * l.n_head + hg * HG + hl) * gridDim.x + split) * ps; };
#pragma unroll
    for (int t = 0; t < NP; t++)
#pragma unroll
        for (int b = 0; b < 2; b++) {
            const int d = 16 * (warp + NW * t) + 8 * b + (lane & 3) * 2;
            if (d >= l.kv_rank) break; // rp is a multiple of 8: d + 1 stays inside the row
            const int r = lane >> 2;
            if (hg * HG + r < l.n_head) *reinterpret_cast<float2 *>(part(r) + d) = make_float2(o[t][b][0], o[t][b][1]);
            if (hg * HG + r + 8 < l.n_head) *reinterpret_cast<float2 *>(part(r + 8) + d) = make_float2(o[t][b][2], o[t][b][3]);
        }
#pragma unroll
    for (int a = 0; a < NH; a++)
        if (lane == 0 && hg * HG + warp * NH + a < l.n_head) {
            float *d = part(warp * NH + a);
            d[rp] = m[a];
            d[rp + 1] = sum[a];
        }
}

// ---- merge of the key ranges, values, output gate: grid (row slices of all heads, rows)
constexpr int OROWS = 32; // output rows per CTA, four per warp
__global__ void __launch_bounds__(NT) latent_output_kernel(const __grid_constant__ KqLatent l, const float *scratch, int n_part, int keys_per_split,
                                                           int T, const int32_t *pos0_dev, int pos0_val, const uint16_t *uv, int64_t ldw,
                                                           const float *gate, int64_t ldg, float *out, int64_t ldo, int slices) {
    extern __shared__ __align__(16) float so[]; // the head's merged latent, zero-padded to 8
    __shared__ float s_w[MAX_SPLIT];
    KQ_PDL_TRIGGER();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.x / slices, r0 = (blockIdx.x % slices) * OROWS + warp * 4;
    const int64_t row = blockIdx.y;
    const int nck = (l.kv_rank + 7) / 8;
    const uint4 *wp[4];
    uint4 w[4][2];
#pragma unroll
    for (int r = 0; r < 4; r++) {
        wp[r] = reinterpret_cast<const uint4 *>(uv + ((int64_t)h * l.v_dim + min(r0 + r, l.v_dim - 1)) * ldw);
#pragma unroll
        for (int j = 0; j < 2; j++) w[r][j] = lane + 32 * j < nck ? kq_ld_stream(wp[r] + lane + 32 * j) : make_uint4(0, 0, 0, 0);
    }
    KQ_PDL_WAIT();
    const int pos = (pos0_dev ? *pos0_dev : pos0_val) + (int)(row % T);
    const int vis = l.window > 0 ? min(pos + 1, l.window) : pos + 1;
    const int n_split = (vis + keys_per_split - 1) / keys_per_split;
    const int64_t rp = kq_f32_ld(l.kv_rank), ps = rp + 2;
    const float *src = scratch + (row * l.n_head + h) * n_part * ps;
    if (warp == 0) {
        float m0 = lane < n_split ? src[lane * ps + rp] : -INFINITY, m1 = lane + 32 < n_split ? src[(lane + 32) * ps + rp] : -INFINITY;
        const float l0 = lane < n_split ? src[lane * ps + rp + 1] : 0.f, l1 = lane + 32 < n_split ? src[(lane + 32) * ps + rp + 1] : 0.f;
        const float mx = kq_warp_max(fmaxf(m0, m1));
        m0 = exp2f(m0 - mx), m1 = exp2f(m1 - mx);
        const float inv = 1.f / kq_warp_sum(m0 * l0 + m1 * l1);
        s_w[lane] = m0 * inv;
        s_w[lane + 32] = m1 * inv;
    }
    __syncthreads();
    for (int d = 2 * tid; d < 8 * nck; d += 2 * NT) {
        float2 acc = make_float2(0.f, 0.f);
        for (int s0 = 0; s0 < n_split; s0 += 16) { // sixteen ranges in flight
            float2 v[16];
#pragma unroll
            for (int e = 0; e < 16; e++)
                v[e] = s0 + e < n_split ? *reinterpret_cast<const float2 *>(src + (s0 + e) * ps + d) : make_float2(0.f, 0.f);
#pragma unroll
            for (int e = 0; e < 16; e++) { // weights past n_split are zero
                acc.x = fmaf(s_w[s0 + e], v[e].x, acc.x);
                acc.y = fmaf(s_w[s0 + e], v[e].y, acc.y);
            }
        }
        so[d] = d < l.kv_rank ? acc.x : 0.f;
        so[d + 1] = d + 1 < l.kv_rank ? acc.y : 0.f;
    }
    __syncthreads();
    if (r0 >= l.v_dim) return;
    float acc[4] = {};
    for (int c = lane; c < nck; c += 32) {
        const float4 a = *reinterpret_cast<const float4 *>(so + 8 * c), b = *reinterpret_cast<const float4 *>(so + 8 * c + 4);
#pragma unroll
        for (int r = 0; r < 4; r++) acc[r] = kq_dot8(c == lane ? w[r][0] : c == lane + 32 ? w[r][1] : kq_ld_stream(wp[r] + c), a, b, acc[r]);
    }
    const float g = gate ? kq_sigmoid(gate[row * ldg + h]) : 1.f;
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const float v = kq_warp_sum(acc[r]);
        if (lane == 0 && r0 + r < l.v_dim) out[row * ldo + (int64_t)h * l.v_dim + r0 + r] = v * g;
    }
}

// key ranges of a call with few rows: enough CTAs to fill the GPU about once
struct Plan {
    int n_split, kps;
};
Plan plan(int n_head, int rows, int max_keys, int tile) {
    const int tiles = (int)kq_div_up(max_keys, tile);
    const int want = (int)std::max<int64_t>(1, kq_sm_count() / (rows * kq_div_up(n_head, HG)));
    Plan p;
    p.n_split = std::min(std::min(MAX_SPLIT, tiles), want);
    p.kps = tile * (int)kq_div_up(tiles, p.n_split);
    p.n_split = (int)kq_div_up(max_keys, p.kps);
    return p;
}
bool use_mma(const KqLatent &l) { // the tile and the queries must fit in shared memory
    return !l.f32 && (int64_t)(MK + 2 * HG) * (kq_pad(l.ld, 16) * 2 + 144) <= 200 * 1024;
}

template <typename E, int NC>
b200_status launch(const KqLatent &l, const float *q_lat, int rows, int T, const int32_t *pos0_dev, int pos0, int n_split,
                   int kps, float *o_lat, float *scratch, cudaStream_t st) {
    int pitch = l.ld * (int)sizeof(E);
    while (pitch % 128 != 16) pitch += 16;
    const size_t smem = (size_t)HG * l.ld * 4 + (size_t)KT * pitch;
    static size_t attr[16];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (smem > 220 * 1024) {
        kq_set_error("latent attention: latent rows of %d values do not fit in shared memory", l.ld);
        return B200_ERR_UNSUPPORTED;
    }
    if (dev < 0 || dev >= 16 || attr[dev] < smem) {
        KQ_CUDA(cudaFuncSetAttribute(latent_attn_kernel<E, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        if (dev >= 0 && dev < 16) attr[dev] = smem;
    }
    kq_launch(latent_attn_kernel<E, NC>, dim3((unsigned)n_split, (unsigned)kq_div_up(l.n_head, HG), (unsigned)rows), NT, smem, st, l, q_lat, T, pos0_dev,
              pos0, kps, o_lat, (int64_t)l.n_head * kq_f32_ld(l.kv_rank), scratch, pitch);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

template <int NP>
b200_status launch_mma(const KqLatent &l, const float *q_lat, int rows, int T, const int32_t *pos0_dev, int pos0, const Plan &pl, float *scratch,
                       cudaStream_t st) {
    int pitch = (int)kq_pad(l.ld, 16) * 2;
    while (pitch % 128 != 16) pitch += 16;
    const size_t smem = (size_t)(MK + 2 * HG) * pitch;
    static size_t attr[16];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 16 || attr[dev] < smem) {
        KQ_CUDA(cudaFuncSetAttribute(latent_attn_mma_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        if (dev >= 0 && dev < 16) attr[dev] = smem;
    }
    kq_launch(latent_attn_mma_kernel<NP>, dim3((unsigned)pl.n_split, (unsigned)kq_div_up(l.n_head, HG), (unsigned)rows), NT, smem, st, l, q_lat, T,
              pos0_dev, pos0, pl.kps, scratch, pitch);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status check_store(const KqLatent &l, int n_seq, int T) {
    KQ_REQUIRE(l.kv_rank >= 1 && l.rot_dim >= 0 && l.rot_dims % 2 == 0 && l.rot_dims <= l.rot_dim && l.cap >= 1 && n_seq >= 1 && T >= 1,
               "latent attention: bad shape");
    KQ_REQUIRE(l.ld == kq_latent_ld(l.kv_rank, l.rot_dim) && l.rot_at == kq_latent_rot_at(l.kv_rank), "latent attention: row layout");
    KQ_REQUIRE(l.rot_dims <= 4096, "latent attention: rotated dimensions");
    return B200_OK;
}

} // namespace

b200_status kq_latent_store(const KqLatent &l, const float *norm_w, float eps, float *q, int64_t ldq, const float *kv,
                            int64_t ldkv, int n_seq, int T, const int32_t *pos0_dev, int pos0, float *q_lat, int64_t ldql,
                            cudaStream_t st) {
    const b200_status rc = check_store(l, n_seq, T);
    if (rc != B200_OK) return rc;
    const StoreParams p = {norm_w, eps, q, ldq, kv, ldkv, T, pos0, pos0_dev, q_lat, ldql};
    kq_launch(latent_store_kernel, (unsigned)(n_seq * T), NT, (size_t)l.rot_dims * 4 + 16, st, l, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_latent_query(const KqLatent &l, const float *norm_w, float eps, float *q, int64_t ldq, const float *kv, int64_t ldkv, int n_seq,
                            int T, const int32_t *pos0_dev, int pos0, float *q_lat, int64_t ldql, const KqDense &absorb, cudaStream_t st) {
    const b200_status rc = check_store(l, n_seq, T);
    if (rc != B200_OK) return rc;
    const int rows = n_seq * T;
    KQ_REQUIRE(rows <= KQ_LATENT_ROWS && absorb.M == rows && q_lat, "latent_query: up to %d rows", KQ_LATENT_ROWS);
    const StoreParams p = {norm_w, eps, q, ldq, kv, ldkv, T, pos0, pos0_dev, q_lat, ldql};
    const KqGrouped a = kq_grouped_params(absorb, q, ldq);
    const unsigned grid = (unsigned)(rows + kq_div_up((int64_t)a.quads * absorb.groups, NW));
    const size_t smem = (size_t)l.rot_dims * 4 + 16;
    if (rows == 1) kq_launch(latent_query_kernel<1>, grid, NT, smem, st, l, p, a, rows);
    else if (rows <= 2) kq_launch(latent_query_kernel<2>, grid, NT, smem, st, l, p, a, rows);
    else if (rows <= 4) kq_launch(latent_query_kernel<4>, grid, NT, smem, st, l, p, a, rows);
    else kq_launch(latent_query_kernel<8>, grid, NT, smem, st, l, p, a, rows);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

size_t kq_latent_scratch_bytes(const KqLatent &l, int max_keys) {
    size_t n = 0;
    for (int rows = 1; rows <= KQ_LATENT_ROWS; rows++)
        n = std::max(n, (size_t)rows * l.n_head * plan(l.n_head, rows, max_keys, use_mma(l) ? MK : KT).n_split * (kq_f32_ld(l.kv_rank) + 2) * 4);
    return n;
}

b200_status kq_latent_attention(const KqLatent &l, const float *q_lat, int n_seq, int T, const int32_t *pos0_dev, int pos0, int max_keys,
                                float *o_lat, float *scratch, size_t scratch_bytes, cudaStream_t st) {
    const int rows = n_seq * T;
    KQ_REQUIRE(rows >= 1 && rows <= 65535 && max_keys >= 1, "latent_attention: bad shape");
    if (l.kv_rank > 1024) {
        kq_set_error("latent attention: latents of up to 1024 values");
        return B200_ERR_UNSUPPORTED;
    }
    Plan pl = {1, max_keys};
    const int nc = (int)kq_div_up(l.kv_rank, 256);
    if (!o_lat) {
        KQ_REQUIRE(rows <= KQ_LATENT_ROWS && scratch && scratch_bytes >= kq_latent_scratch_bytes(l, max_keys), "latent_attention: scratch");
        pl = plan(l.n_head, rows, max_keys, use_mma(l) ? MK : KT);
        if (use_mma(l))
            return nc <= 1   ? launch_mma<2>(l, q_lat, rows, T, pos0_dev, pos0, pl, scratch, st)
                   : nc <= 2 ? launch_mma<4>(l, q_lat, rows, T, pos0_dev, pos0, pl, scratch, st)
                             : launch_mma<8>(l, q_lat, rows, T, pos0_dev, pos0, pl, scratch, st);
    }
#define GO(E)                                                                                               \
    (nc <= 1   ? launch<E, 1>(l, q_lat, rows, T, pos0_dev, pos0, pl.n_split, pl.kps, o_lat, scratch, st)     \
     : nc <= 2 ? launch<E, 2>(l, q_lat, rows, T, pos0_dev, pos0, pl.n_split, pl.kps, o_lat, scratch, st)     \
               : launch<E, 4>(l, q_lat, rows, T, pos0_dev, pos0, pl.n_split, pl.kps, o_lat, scratch, st))
    return l.f32 ? GO(float) : GO(uint16_t);
#undef GO
}

b200_status kq_latent_output(const KqLatent &l, const float *scratch, int n_seq, int T, const int32_t *pos0_dev, int pos0, int max_keys,
                             const uint16_t *uv, const float *gate, int64_t ldg, float *out, int64_t ldo, cudaStream_t st) {
    const int rows = n_seq * T;
    KQ_REQUIRE(rows >= 1 && rows <= KQ_LATENT_ROWS, "latent_output: up to %d rows", KQ_LATENT_ROWS);
    const Plan pl = plan(l.n_head, rows, max_keys, use_mma(l) ? MK : KT);
    const int slices = (int)kq_div_up(l.v_dim, OROWS);
    kq_launch(latent_output_kernel, dim3((unsigned)(l.n_head * slices), (unsigned)rows), NT, (size_t)kq_pad(l.kv_rank, 8) * 4, st, l, scratch,
              pl.n_split, pl.kps, T, pos0_dev, pos0, uv, kq_bf16_ld(l.kv_rank), gate, ldg, out, ldo, slices);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
