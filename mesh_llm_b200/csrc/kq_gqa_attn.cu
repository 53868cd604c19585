// Grouped-query attention with per-head query / key norms over a ring of keys and values: the cache store, and attention
// of single rows (decode steps, short portions, the 32-bit mode); prompts run on the tensor cores (kq_prompt_attn.cu).
//
// A CTA takes a range of one row's visible keys for up to RT query heads of one key / value head.  Lanes split the
// dimensions two by two, so that a warp reads whole key rows; a warp takes four keys at a time, their scores are reduced
// across the warp together.  Scores of a tile of keys sit in shared memory, the softmax is online over tiles, all in f32.
// The ranges' results (maximum, sum, weighted values) are merged by the last CTA of a row to arrive; ranges without keys
// take no part.  In a decode step the same launch norms the queries and the new key and stores the new row: only the CTA
// whose range ends with the new position reads that row, and it is the one that stores it.  The ranges' rows are prefetched
// into L2 ahead of the dependency wait: they are of earlier steps, and loads see the latest values wherever they lie.
#include "kq_dense.cuh"

#include <algorithm>

namespace {

constexpr int NT = 128, NW = NT / 32, KT = 128; // threads, warps, keys per tile
constexpr int MAX_SPLITS = KT, MIN_RANGE = 64;  // ranges of a row's keys, keys of a range

struct Params {
    KqGqa a;
    const float *q, *k, *v;
    int64_t ldp;
    int32_t T, pos0;
    const int32_t *pos0_dev;
    float *out;
    int64_t ldo;
    uint16_t *out16;
    int64_t ldo16;
    float *part;        // [row][head][split][vdim padded to 4]: weighted values
    float2 *ml;         // [row][head][split]: maximum, sum
    unsigned *counters; // [row][head group], zero between launches
    int32_t splits, groups;
};

template <typename CT>
__device__ __forceinline__ float2 ld2(const CT *p);
template <>
__device__ __forceinline__ float2 ld2<float>(const float *p) { return *reinterpret_cast<const float2 *>(p); }
template <>
__device__ __forceinline__ float2 ld2<uint16_t>(const uint16_t *p) { return __half22float2(*reinterpret_cast<const __half2 *>(p)); }
__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(uint16_t *p, float v) { *p = kq_f2h_sat(v); }

// 1 / rms of a head's values, by one warp
__device__ __forceinline__ float head_scale(const float *x, int dim, float eps, int lane) {
    float s = 0.f;
    for (int d = lane; d < dim; d += 32) s += x[d] * x[d];
    return 1.0f / sqrtf(kq_warp_sum(s) / (float)dim + eps);
}
// one key / value head of one new row, by one warp
template <typename CT>
__device__ __forceinline__ void store_row(const KqGqa &a, const float *k, const float *v, int64_t seq, int pos, int g, int lane) {
    const int64_t ldk = (a.dim + 63) / 64 * 64, ldv = (a.vdim + 63) / 64 * 64, row = seq * a.cap + pos % a.cap;
    CT *kd = (CT *)a.k + (row * a.kv_heads + g) * ldk, *vd = (CT *)a.v + (row * a.kv_heads + g) * ldv;
    const float sc = head_scale(k, a.dim, a.eps, lane);
    for (int d = lane; d < a.dim; d += 32) put(kd + d, k[d] * sc * a.k_norm[d]);
    for (int d = lane; d < a.vdim; d += 32) put(vd + d, v[d]);
}

// grid (rows, quarters of the heads): a warp per query head or per key / value head
template <typename CT>
__global__ void __launch_bounds__(NT) gqa_store_kernel(const __grid_constant__ KqGqa a, float *q, const float *k, const float *v, int64_t ldp, int T,
                                                       const int32_t *pos0_dev, int pos0_val) {
    KQ_PDL_ENTER();
    const int lane = threadIdx.x & 31, h = blockIdx.y * NW + (threadIdx.x >> 5);
    const int64_t r = blockIdx.x;
    if (h < a.n_head) {
        float *x = q + r * ldp + (int64_t)h * a.dim;
        const float sc = head_scale(x, a.dim, a.eps, lane);
        for (int d = lane; d < a.dim; d += 32) x[d] *= sc * a.q_norm[d];
    } else if (a.own_kv && h < a.n_head + a.kv_heads) {
        const int g = h - a.n_head, pos = (pos0_dev ? *pos0_dev : pos0_val) + (int)(r % T);
        store_row<CT>(a, k + r * ldp + (int64_t)g * a.dim, v + r * ldp + (int64_t)g * a.vdim, r / T, pos, g, lane);
    }
}

// N: pairs of dimensions per lane (dims up to 64 N); RT: query heads per CTA
template <typename CT, int N, int RT, bool FUSED>
__global__ void __launch_bounds__(NT) gqa_attn_kernel(const __grid_constant__ Params p) {
    KQ_PDL_TRIGGER();
    const KqGqa &a = p.a;
    __shared__ __align__(16) float s_p[RT][KT];
    __shared__ __align__(16) float2 s_o[NW][RT][N * 32];
    __shared__ __align__(16) float s_q[RT][N * 64];
    __shared__ int s_last;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int split = blockIdx.x, S = p.splits, rep = a.n_head / a.kv_heads, gpk = (rep + RT - 1) / RT;
    const int g = blockIdx.y / gpk, h0 = g * rep + blockIdx.y % gpk * RT, nh = min(RT, (g + 1) * rep - h0);
    const int64_t r = blockIdx.z, seq = r / p.T;
    const int ldk = (a.dim + 63) / 64 * 64, ldv = (a.vdim + 63) / 64 * 64;
    const CT *kc = (const CT *)a.k + (seq * a.cap * a.kv_heads + g) * (int64_t)ldk, *vc = (const CT *)a.v + (seq * a.cap * a.kv_heads + g) * (int64_t)ldv;
    const int64_t rk = (int64_t)a.kv_heads * ldk, rv = (int64_t)a.kv_heads * ldv;
    if (S > 1) { // the position may still be the one before
        int pos = p.pos0;
        if (p.pos0_dev) pos = __ldcg(p.pos0_dev);
        pos = max(0, pos + (int)(r % p.T));
        const int lo = kq_first_key(pos, a.window, a.chunk), n = pos - lo + 1, per = max((n + S - 1) / S, MIN_RANGE);
        const int j0 = min(n, split * per), j1 = min(n, j0 + per), k_lines = (ldk * (int)sizeof(CT) + 127) / 128, v_lines = (ldv * (int)sizeof(CT) + 127) / 128;
        for (int i = tid; i < (j1 - j0) * (k_lines + v_lines); i += NT) {
            const int j = i / (k_lines + v_lines), l = i % (k_lines + v_lines);
            const int64_t row = (lo + j0 + j) % a.cap;
            const uint8_t *line = l < k_lines ? (const uint8_t *)(kc + row * rk) + l * 128 : (const uint8_t *)(vc + row * rv) + (l - k_lines) * 128;
            asm volatile("prefetch.global.L2 [%0];" ::"l"(line));
        }
    }
    KQ_PDL_WAIT();
    const int pos = (p.pos0_dev ? *p.pos0_dev : p.pos0) + (int)(r % p.T);
    const int lo = kq_first_key(pos, a.window, a.chunk), n = pos - lo + 1, per = max((n + S - 1) / S, MIN_RANGE);
    const int j0 = min(n, split * per), j1 = min(n, j0 + per); // keys lo + j0 .. lo + j1 - 1
    const int live = (n + per - 1) / per;                      // ranges that have any
    if (j0 >= j1) return;

    {
        if (FUSED && a.own_kv && j1 == n && warp == NW - 1) // head groups of one key head store the same values
            store_row<CT>(a, p.k + r * p.ldp + (int64_t)g * a.dim, p.v + r * p.ldp + (int64_t)g * a.vdim, seq, pos, g, lane);
        for (int t = warp; t < RT; t += NW) {
            const float *x = p.q + r * p.ldp + (int64_t)(h0 + min(t, nh - 1)) * a.dim;
            const float sc = a.scale * (FUSED ? head_scale(x, a.dim, a.eps, lane) : 1.f);
            for (int d = lane; d < N * 64; d += 32) s_q[t][d] = d < a.dim ? x[d] * sc * (FUSED ? a.q_norm[d] : 1.f) : 0.f;
        }
    }
    __syncthreads();
    float2 q[RT][N];
    float m[RT], l[RT];
    float2 o[RT][N];
#pragma unroll
    for (int t = 0; t < RT; t++) {
        m[t] = -INFINITY, l[t] = 0.f;
#pragma unroll
        for (int i = 0; i < N; i++) o[t][i] = make_float2(0.f, 0.f);
    }
    const int row0 = (lo + j0) % a.cap; // of the first key; a range wraps at most once
    auto row_of = [&](int j) {
        const int x = row0 + j - j0;
        return (int64_t)(x >= a.cap ? x - a.cap : x);
    };
    for (int t0 = j0; t0 < j1; t0 += KT) {
        const int nk = min(KT, j1 - t0);
#pragma unroll
        for (int t = 0; t < RT; t++)
#pragma unroll
            for (int i = 0; i < N; i++) q[t][i] = *reinterpret_cast<const float2 *>(&s_q[t][2 * lane + 64 * i]);
#pragma unroll 2
        for (int j = warp * 4; j < nk; j += NW * 4) {
            float2 kv[4][N];
#pragma unroll
            for (int e = 0; e < 4; e++)
#pragma unroll
                for (int i = 0; i < N; i++)
                    kv[e][i] = 64 * i < ldk ? ld2(kc + row_of(t0 + min(j + e, nk - 1)) * rk + 2 * lane + 64 * i) : make_float2(0.f, 0.f);
#pragma unroll
            for (int t = 0; t < RT; t++) {
                float s[4];
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    s[e] = 0.f;
#pragma unroll
                    for (int i = 0; i < N; i++) s[e] = fmaf(q[t][i].x, kv[e][i].x, fmaf(q[t][i].y, kv[e][i].y, s[e]));
                }
                // four sums across the warp: after two exchanges a lane holds one key's sum over four lanes' worth
                const bool h16 = lane & 16, h8 = lane & 8;
                const float x0 = __shfl_xor_sync(0xffffffffu, h16 ? s[0] : s[2], 16), x1 = __shfl_xor_sync(0xffffffffu, h16 ? s[1] : s[3], 16);
                const float a0 = (h16 ? s[2] : s[0]) + x0, a1 = (h16 ? s[3] : s[1]) + x1;
                float v = (h8 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, h8 ? a0 : a1, 8);
                v += __shfl_xor_sync(0xffffffffu, v, 4);
                v += __shfl_xor_sync(0xffffffffu, v, 2);
                v += __shfl_xor_sync(0xffffffffu, v, 1);
                const int e = ((lane >> 4) & 1) * 2 + ((lane >> 3) & 1);
                if ((lane & 7) == 0 && j + e < nk) s_p[t][j + e] = v;
            }
        }
        __syncthreads();
        // every warp finds the maxima; warp w turns the scores of the heads w, w + NW, ... into weights
        float mn[RT], al[RT];
#pragma unroll
        for (int t = 0; t < RT; t++) {
            float v = -INFINITY;
#pragma unroll
            for (int i = 0; i < KT / 32; i++)
                if (lane + 32 * i < nk) v = fmaxf(v, s_p[t][lane + 32 * i]);
            mn[t] = fmaxf(m[t], kq_warp_max(v));
            al[t] = m[t] == -INFINITY ? 0.f : expf(m[t] - mn[t]);
            m[t] = mn[t];
        }
        __syncthreads();
        for (int i = tid; i < RT * KT; i += NT) {
            const int t = i / KT, j = i % KT;
            float mt = mn[0];
#pragma unroll
            for (int u = 1; u < RT; u++)
                if (t == u) mt = mn[u];
            s_p[t][j] = j < nk ? expf(s_p[t][j] - mt) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int t = 0; t < RT; t++) {
            float v = 0.f;
#pragma unroll
            for (int i = 0; i < KT / 32; i++) v += s_p[t][lane + 32 * i];
            l[t] = l[t] * al[t] + kq_warp_sum(v);
#pragma unroll
            for (int i = 0; i < N; i++) o[t][i].x *= al[t], o[t][i].y *= al[t];
        }
#pragma unroll 2
        for (int j = warp * 4; j < nk; j += NW * 4) {
            float2 vv[4][N];
#pragma unroll
            for (int e = 0; e < 4; e++)
#pragma unroll
                for (int i = 0; i < N; i++)
                    vv[e][i] = 64 * i < ldv ? ld2(vc + row_of(t0 + min(j + e, nk - 1)) * rv + 2 * lane + 64 * i) : make_float2(0.f, 0.f);
#pragma unroll
            for (int t = 0; t < RT; t++) {
                const float4 w = *reinterpret_cast<const float4 *>(&s_p[t][j]); // zero past the tile's keys
                const float we[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int e = 0; e < 4; e++)
#pragma unroll
                    for (int i = 0; i < N; i++) {
                        o[t][i].x = fmaf(we[e], vv[e][i].x, o[t][i].x);
                        o[t][i].y = fmaf(we[e], vv[e][i].y, o[t][i].y);
                    }
            }
        }
        __syncthreads();
    }
    // the warps' shares of the values; then out, or to the merge
#pragma unroll
    for (int t = 0; t < RT; t++)
#pragma unroll
        for (int i = 0; i < N; i++) s_o[warp][t][lane + 32 * i] = o[t][i];
    if (tid < RT) {
        float mt = m[0], lt = l[0];
#pragma unroll
        for (int u = 1; u < RT; u++)
            if (tid == u) mt = m[u], lt = l[u];
        s_p[tid][0] = mt, s_p[tid][1] = lt;
    }
    __syncthreads();
    const int64_t rec = (a.vdim + 3) / 4 * 4;
    auto emit = [&](int h, int d, float v) {
        const int64_t c = (int64_t)h * a.vdim + d;
        if (p.out) p.out[r * p.ldo + c] = v;
        if (p.out16) p.out16[r * p.ldo16 + c] = kq_f2bf(v);
    };
    for (int i = tid; i < nh * a.vdim; i += NT) {
        const int t = i / a.vdim, d = i % a.vdim;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < NW; w++) v += reinterpret_cast<const float *>(s_o[w][t])[d];
        if (live == 1) emit(h0 + t, d, v / s_p[t][1]);
        else __stcg(p.part + ((r * a.n_head + h0 + t) * S + split) * rec + d, v);
    }
    if (live == 1) return;
    if (tid < nh) __stcg(p.ml + (r * a.n_head + h0 + tid) * S + split, make_float2(s_p[tid][0], s_p[tid][1]));
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        unsigned *c = p.counters + r * p.groups + blockIdx.y;
        s_last = atomicAdd(c, 1u) == (unsigned)live - 1;
        if (s_last) *c = 0u;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    for (int t = warp; t < nh; t += NW) { // weights of the ranges, by a warp per head
        const float2 *d = p.ml + (r * a.n_head + h0 + t) * S;
        float2 x[MAX_SPLITS / 32];
        float mx = -INFINITY, sum = 0.f;
#pragma unroll
        for (int i = 0; i < MAX_SPLITS / 32; i++) {
            x[i] = lane + 32 * i < live ? __ldcg(d + lane + 32 * i) : make_float2(-INFINITY, 0.f);
            mx = fmaxf(mx, x[i].x);
        }
        mx = kq_warp_max(mx);
#pragma unroll
        for (int i = 0; i < MAX_SPLITS / 32; i++) sum += x[i].y * expf(x[i].x - mx);
        sum = kq_warp_sum(sum);
#pragma unroll
        for (int i = 0; i < MAX_SPLITS / 32; i++) s_p[t][lane + 32 * i] = expf(x[i].x - mx) / sum;
    }
    __syncthreads();
    const int n4 = (int)rec / 4;
    for (int i = tid; i < nh * n4; i += NT) { // what lies behind vdim is not written out
        const int t = i / n4, d = i % n4 * 4;
        const float4 *src = reinterpret_cast<const float4 *>(p.part + (r * a.n_head + h0 + t) * S * rec + d);
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 16
        for (int s = 0; s < live; s++) {
            const float w = s_p[t][s];
            const float4 x = __ldcg(src + s * n4);
            v.x = fmaf(w, x.x, v.x), v.y = fmaf(w, x.y, v.y), v.z = fmaf(w, x.z, v.z), v.w = fmaf(w, x.w, v.w);
        }
        const float o4[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int e = 0; e < 4; e++)
            if (d + e < a.vdim) emit(h0 + t, d + e, o4[e]);
    }
}

constexpr int SPLIT_ROWS = 8; // up to SPLIT_ROWS rows are split

int splits_of(const KqGqa &a, int rows, int max_keys) {
    if (rows > SPLIT_ROWS) return 1;
    const int64_t ctas = (int64_t)rows * a.kv_heads * kq_div_up(a.n_head / a.kv_heads, 4);
    const int64_t fill = kq_div_up(4 * (int64_t)kq_sm_count(), ctas);
    return (int)std::max<int64_t>(1, std::min<int64_t>({kq_div_up(max_keys, MIN_RANGE), fill, MAX_SPLITS}));
}

template <typename CT, bool FUSED>
b200_status launch(const Params &p, dim3 grid, int n, bool one, cudaStream_t st) {
#define GO(N)                                                                                   \
    do {                                                                                        \
        if (one) kq_launch(gqa_attn_kernel<CT, N, 1, FUSED>, grid, NT, 0, st, p);               \
        else kq_launch(gqa_attn_kernel<CT, N, (N > 4 ? 2 : 4), FUSED>, grid, NT, 0, st, p);     \
    } while (0)
    if (n <= 1) GO(1);
    else if (n <= 2) GO(2);
    else if (n <= 4) GO(4);
    else GO(8);
#undef GO
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

} // namespace

b200_status kq_gqa_store(const KqGqa &a, float *q, const float *k, const float *v, int64_t ldp, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                         cudaStream_t st) {
    KQ_REQUIRE(n_seq >= 1 && T >= 1 && T <= a.cap && (int64_t)n_seq * T <= INT32_MAX, "gqa_store: bad call");
    const dim3 grid((unsigned)(n_seq * T), (unsigned)kq_div_up(a.n_head + (a.own_kv ? a.kv_heads : 0), NW));
    if (a.f32) kq_launch(gqa_store_kernel<float>, grid, NT, 0, st, a, q, k, v, ldp, T, pos0_dev, pos0);
    else kq_launch(gqa_store_kernel<uint16_t>, grid, NT, 0, st, a, q, k, v, ldp, T, pos0_dev, pos0);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

size_t kq_gqa_scratch_bytes(const KqGqa &a, int max_rows, int max_keys) {
    size_t n = 0;
    for (int r = 1; r <= std::min(max_rows, SPLIT_ROWS); r++)
        n = std::max(n, (size_t)r * a.n_head * splits_of(a, r, max_keys) * (2 + (size_t)kq_pad(a.vdim, 4)) * 4);
    return n + 16;
}
int64_t kq_gqa_counters(const KqGqa &a) { return (int64_t)SPLIT_ROWS * a.n_head; }

b200_status kq_gqa_attention(const KqGqa &a, bool fused, const float *q, const float *k, const float *v, int64_t ldp, int n_seq, int T,
                             const int32_t *pos0_dev, int pos0, int max_keys, float *out, int64_t ldo, uint16_t *out16, int64_t ldo16,
                             float *scratch, size_t scratch_bytes, unsigned *counters, cudaStream_t st) {
    const int rows = n_seq * T, rep = a.n_head / a.kv_heads, dmax = std::max(a.dim, a.vdim);
    KQ_REQUIRE(n_seq >= 1 && T >= 1 && rows <= 65535 && (!fused || T == 1), "gqa_attention: bad call");
    KQ_REQUIRE(a.n_head % a.kv_heads == 0 && dmax <= KQ_GQA_MAX_DIM && a.cap >= 1, "gqa_attention: %d heads on %d, %d dimensions", a.n_head, a.kv_heads, dmax);
    Params p;
    p.a = a;
    p.q = q, p.k = k, p.v = v, p.ldp = ldp, p.T = T, p.pos0 = pos0, p.pos0_dev = pos0_dev;
    p.out = out, p.ldo = ldo, p.out16 = out16, p.ldo16 = ldo16;
    const int n = (int)kq_div_up(dmax, 64), rt = rep == 1 ? 1 : n > 4 ? 2 : 4;
    p.splits = splits_of(a, rows, max_keys);
    p.groups = (int)(a.kv_heads * kq_div_up(rep, rt));
    p.counters = counters;
    const int64_t records = (int64_t)rows * a.n_head * p.splits, per = kq_pad(a.vdim, 4);
    p.part = scratch;
    p.ml = (float2 *)(scratch + records * per);
    KQ_REQUIRE(p.splits == 1 || (counters && scratch_bytes >= (size_t)records * (2 + per) * 4), "gqa_attention: scratch");
    const dim3 grid((unsigned)p.splits, (unsigned)p.groups, (unsigned)rows);
    KQ_REQUIRE(p.groups <= 65535, "gqa_attention: %d heads", a.n_head);
    if (a.f32) return fused ? launch<float, true>(p, grid, n, rt == 1, st) : launch<float, false>(p, grid, n, rt == 1, st);
    return fused ? launch<uint16_t, true>(p, grid, n, rt == 1, st) : launch<uint16_t, false>(p, grid, n, rt == 1, st);
}
