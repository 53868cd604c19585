// Latent attention over a ring cache: a position keeps one normed latent (kv_rank values) and one rotated key
// part shared by all heads; the per-head keys and values are linear maps of the latent.  Decode folds the key
// map into the query ("absorbed" form): score = q_lat . c + q_rot . k_rot with q_lat = W_uk^T q, and the value
// map into the output: o = W_uv (sum_j p_j c_j), so that a step reads each visible row once for all heads.
//
// kq_latent_store writes the rows of the new positions, kq_latent_attention is the absorbed attention for any
// number of rows (f32 products, f32 or bf16 cache): a CTA takes 16 heads of one row and a range of keys, tiles of
// 32 rows go through shared memory; scores with lane = key, values with lane = latent dimensions, online
// softmax per head.  Few rows are cut into key ranges, the last CTA of a (row, head group) to finish merges them.
#include "kq_dense.cuh"

#include <algorithm>
#include <math.h>

namespace {

constexpr int NT = 256, NW = NT / 32, NH = 2, HG = NW * NH, KT = 32; // heads per warp and CTA, keys per tile
constexpr int MAX_SPLIT = 64, SPLIT_ROWS = 8;

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

// one CTA per row
__global__ void __launch_bounds__(NT) latent_store_kernel(const __grid_constant__ KqLatent l, const float *norm_w, float eps, float *q,
                                                          int64_t ldq, const float *kv, int64_t ldkv, int T, const int32_t *pos0_dev,
                                                          int pos0_val, float *q_lat, int64_t ldql) {
    KQ_PDL_ENTER();
    __shared__ float red[NW];
    extern __shared__ float cs[]; // cos, sin of every pair
    const int tid = threadIdx.x;
    const int64_t row = blockIdx.x;
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
                                                         int64_t ldo, float *scratch, int *counters, int pitch) {
    KQ_PDL_ENTER();
    extern __shared__ __align__(16) uint8_t sm[];
    __shared__ int s_last;
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
    if (n_split == 1) {
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
    // partial results: [row][head][split] of (rp values, max, sum)
    const int64_t ps = rp + 2, base = (row * l.n_head + hg * HG) * MAX_SPLIT;
#pragma unroll
    for (int a = 0; a < NH; a++) {
        const int hl = warp * NH + a;
        if (hg * HG + hl >= l.n_head) break;
        float *d = scratch + (base + (int64_t)hl * MAX_SPLIT + split) * ps;
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
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        int *ctr = counters + row * gridDim.y + hg;
        s_last = atomicAdd(ctr, 1) == n_split - 1;
        if (s_last) *ctr = 0;
        __threadfence();
    }
    __syncthreads();
    if (!s_last) return;
#pragma unroll
    for (int a = 0; a < NH; a++) {
        const int hl = warp * NH + a, h = hg * HG + hl;
        if (h >= l.n_head) break;
        const float *src = scratch + (base + (int64_t)hl * MAX_SPLIT) * ps;
        float m0 = lane < n_split ? __ldcg(src + lane * ps + rp) : -INFINITY;
        float m1 = lane + 32 < n_split ? __ldcg(src + (lane + 32) * ps + rp) : -INFINITY;
        const float mx = kq_warp_max(fmaxf(m0, m1));
        m0 = exp2f(m0 - mx);
        m1 = exp2f(m1 - mx);
        const float tot = kq_warp_sum((lane < n_split ? m0 * __ldcg(src + lane * ps + rp + 1) : 0.f) +
                                      (lane + 32 < n_split ? m1 * __ldcg(src + (lane + 32) * ps + rp + 1) : 0.f));
        const float inv = 1.f / tot;
        for (int d0 = 0; d0 < l.kv_rank; d0 += 64) {
            const int d = d0 + 2 * lane;
            float2 acc = make_float2(0.f, 0.f);
#pragma unroll 4
            for (int s = 0; s < n_split; s++) {
                const float w = __shfl_sync(0xffffffffu, s < 32 ? m0 : m1, s & 31);
                if (d < l.kv_rank) {
                    const float2 v = __ldcg(reinterpret_cast<const float2 *>(src + s * ps + d));
                    acc.x = fmaf(w, v.x, acc.x);
                    acc.y = fmaf(w, v.y, acc.y);
                }
            }
            if (d < l.kv_rank) o_lat[row * ldo + h * rp + d] = acc.x * inv;
            if (d + 1 < l.kv_rank) o_lat[row * ldo + h * rp + d + 1] = acc.y * inv;
        }
    }
}

template <typename E, int NC>
b200_status launch(const KqLatent &l, const float *q_lat, int rows, int T, const int32_t *pos0_dev, int pos0, int n_split,
                   int kps, float *o_lat, float *scratch, int *counters, cudaStream_t st) {
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
              pos0, kps, o_lat, (int64_t)l.n_head * kq_f32_ld(l.kv_rank), scratch, counters, pitch);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

} // namespace

b200_status kq_latent_store(const KqLatent &l, const float *norm_w, float eps, float *q, int64_t ldq, const float *kv,
                            int64_t ldkv, int n_seq, int T, const int32_t *pos0_dev, int pos0, float *q_lat, int64_t ldql,
                            cudaStream_t st) {
    KQ_REQUIRE(l.kv_rank >= 1 && l.rot_dim >= 0 && l.rot_dims % 2 == 0 && l.rot_dims <= l.rot_dim && l.cap >= 1 && n_seq >= 1 && T >= 1,
               "latent_store: bad shape");
    KQ_REQUIRE(l.ld == kq_latent_ld(l.kv_rank, l.rot_dim) && l.rot_at == kq_latent_rot_at(l.kv_rank), "latent_store: row layout");
    KQ_REQUIRE(l.rot_dims <= 4096, "latent_store: rotated dimensions");
    kq_launch(latent_store_kernel, (unsigned)(n_seq * T), NT, (size_t)l.rot_dims * 4 + 16, st, l, norm_w, eps, q, ldq, kv, ldkv, T, pos0_dev, pos0,
              q_lat, ldql);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

size_t kq_latent_scratch_bytes(int n_head, int kv_rank, int max_keys) {
    (void)max_keys;
    return (size_t)SPLIT_ROWS * kq_pad(n_head, HG) * MAX_SPLIT * (kq_f32_ld(kv_rank) + 2) * 4;
}
size_t kq_latent_counter_bytes(int n_head) { return (size_t)SPLIT_ROWS * kq_div_up(n_head, HG) * 4; }

b200_status kq_latent_attention(const KqLatent &l, const float *q_lat, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                                int max_keys, float *o_lat, float *scratch, size_t scratch_bytes, int *counters, cudaStream_t st) {
    const int rows = n_seq * T;
    KQ_REQUIRE(rows >= 1 && rows <= 65535 && max_keys >= 1, "latent_attention: bad shape");
    if (l.kv_rank > 1024) {
        kq_set_error("latent attention: latents of up to 1024 values");
        return B200_ERR_UNSUPPORTED;
    }
    // few rows: enough key ranges to fill the GPU about twice; many rows: one range each
    int n_split = 1, kps = max_keys;
    if (rows <= SPLIT_ROWS) {
        const int tiles = (int)kq_div_up(max_keys, KT);
        const int want = (int)std::max<int64_t>(1, 2 * kq_sm_count() / (rows * kq_div_up(l.n_head, HG)));
        n_split = std::min(std::min(MAX_SPLIT, tiles), want);
        kps = KT * (int)kq_div_up(tiles, n_split);
        n_split = (int)kq_div_up(max_keys, kps);
        KQ_REQUIRE(scratch && counters && scratch_bytes >= kq_latent_scratch_bytes(l.n_head, l.kv_rank, max_keys), "latent_attention: scratch");
    }
    const int nc = (int)kq_div_up(l.kv_rank, 256);
#define GO(E)                                                                                                               \
    (nc <= 1   ? launch<E, 1>(l, q_lat, rows, T, pos0_dev, pos0, n_split, kps, o_lat, scratch, counters, st)                 \
     : nc <= 2 ? launch<E, 2>(l, q_lat, rows, T, pos0_dev, pos0, n_split, kps, o_lat, scratch, counters, st)                 \
               : launch<E, 4>(l, q_lat, rows, T, pos0_dev, pos0, n_split, kps, o_lat, scratch, counters, st))
    return l.f32 ? GO(float) : GO(uint16_t);
#undef GO
}
