// Four rows of a block-diagonal product by one warp, for up to M rows of activations (f32, from L1 / L2): the body of
// gemv_grouped_bf16_kernel, also part of the kernel that prepares a decode step's latent queries.
#pragma once
#include "kq_dense.cuh"

__device__ __forceinline__ float4 kq_load4(const float *p, int k, int K, bool vec) {
    if (vec && k + 3 < K) return *reinterpret_cast<const float4 *>(p + k);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (k < K) v.x = p[k];
    if (k + 1 < K) v.y = p[k + 1];
    if (k + 2 < K) v.z = p[k + 2];
    if (k + 3 < K) v.w = p[k + 3];
    return v;
}
// eight bf16 weights times eight activations
__device__ __forceinline__ float kq_dot8(const uint4 q, const float4 a, const float4 b, float s) {
    s = fmaf(__uint_as_float(q.x << 16), a.x, s);
    s = fmaf(__uint_as_float(q.x & 0xffff0000u), a.y, s);
    s = fmaf(__uint_as_float(q.y << 16), a.z, s);
    s = fmaf(__uint_as_float(q.y & 0xffff0000u), a.w, s);
    s = fmaf(__uint_as_float(q.z << 16), b.x, s);
    s = fmaf(__uint_as_float(q.z & 0xffff0000u), b.y, s);
    s = fmaf(__uint_as_float(q.w << 16), b.z, s);
    return fmaf(__uint_as_float(q.w & 0xffff0000u), b.w, s);
}

struct KqGrouped {
    KqDense c;
    const float *x;
    int64_t ldx;
    int32_t quads; // four-row units per group and segment
    int32_t vec;
};

// unit `id` (a warp index over quads * groups * segments); waits for the kernel before it after requesting the first weights
template <int M>
__device__ __forceinline__ void kq_grouped_rows(const KqGrouped &p, int64_t id, int lane) {
    const int64_t per = (int64_t)p.quads * p.c.groups;
    const bool live = id < per * p.c.nseg;
    const int sg = live ? (int)(id / per) : 0;
    const int g = live ? (int)(id % per / p.quads) : 0, r0 = (int)(id % p.quads) * 4;
    const KqDenseSeg s = kq_dense_seg(p.c, sg);
    const bool ok = live && r0 < s.n_rows;
    const int K = p.c.K, nck = (K + 7) / 8;
    const uint4 *wp[4];
    uint4 w[4];
#pragma unroll
    for (int r = 0; r < 4; r++) {
        wp[r] = reinterpret_cast<const uint4 *>(s.W + ((int64_t)g * s.n_rows + min(r0 + r, s.n_rows - 1)) * p.c.ldw);
        w[r] = ok && lane < nck ? kq_ld_stream(wp[r] + lane) : make_uint4(0, 0, 0, 0);
    }
    KQ_PDL_WAIT();
    if (!ok) return;
    float acc[4][M];
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
        for (int m = 0; m < M; m++) acc[r][m] = 0.f;
    for (int c = lane; c < nck; c += 32) {
        if (c != lane) {
#pragma unroll
            for (int r = 0; r < 4; r++) w[r] = kq_ld_stream(wp[r] + c);
        }
#pragma unroll
        for (int m = 0; m < M; m++) {
            if (m >= p.c.M) break;
            const float *x = p.x + m * p.ldx + g * p.c.xg;
            const float4 a = kq_load4(x, 8 * c, K, p.vec), b = kq_load4(x, 8 * c + 4, K, p.vec);
#pragma unroll
            for (int r = 0; r < 4; r++) acc[r][m] = kq_dot8(w[r], a, b, acc[r][m]);
        }
    }
#pragma unroll
    for (int r = 0; r < 4; r++)
#pragma unroll
        for (int m = 0; m < M; m++) {
            const float v = kq_warp_sum(acc[r][m]);
            if (lane == 0 && m < p.c.M && r0 + r < s.n_rows) kq_dense_store(p.c, s, m, (int64_t)g * s.n_rows + r0 + r, g, v);
        }
}
static inline KqGrouped kq_grouped_params(const KqDense &c, const float *x, int64_t ldx) {
    KqGrouped p;
    p.c = c;
    p.x = x;
    p.ldx = ldx;
    p.quads = 0;
    for (int i = 0; i < c.nseg; i++)
        if ((c.seg[i].n_rows + 3) / 4 > p.quads) p.quads = (c.seg[i].n_rows + 3) / 4;
    p.vec = ldx % 4 == 0 && c.xg % 4 == 0 && ((uintptr_t)x & 15) == 0;
    return p;
}
// the call for rows m0 .. m0 + m - 1 of a larger one
static inline KqDense kq_rows_of(const KqDense &c, int m0, int m) {
    KqDense d = c;
    d.M = m;
    for (int i = 0; i < d.nseg; i++)
        d.seg[i].y = (uint8_t *)c.seg[i].y + m0 * c.seg[i].ldy * (c.seg[i].out == KQ_OUT_F32 ? 4 : 2);
    if (d.head_gate) d.head_gate += m0 * d.ld_gate;
    if (d.row_mul) d.row_mul += m0 * d.ld_mul;
    return d;
}
