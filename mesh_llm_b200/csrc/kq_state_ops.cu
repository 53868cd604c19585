// Recurrences whose state is a matrix per head, all in f32: linear attention under a fixed decay, and the delta rule with a
// decay per key channel behind short convolutions.
//
// Prompts: one launch prepares every token's q, k, v, decay and write strength (convolution, SiLU, unit norms); the token loop
// then keeps the state in registers.  A column of the state (one value dimension) belongs to eight lanes that split the
// key dimension in groups of four, so a token costs two multiply-adds per element for the products with k and q, one
// for the decay and one for the write, and one exchange over eight lanes: the read-out of the new state is the read-out
// of the decayed one plus (q.k) u, so both products wait for the same reduction.  A CTA has 16 columns of one head; tiles of
// tokens come through shared memory by cp.async, two tiles in flight.
// A decode step is one launch: a CTA per head convolves, norms, works out the low-rank decays and gates, updates the
// state and norms and gates the head's output.
#include "kq_gemv_grouped.cuh"

#include <algorithm>

namespace {

constexpr int COLS = 16, SCAN_NT = COLS * 8; // columns and threads of a CTA of the token loop

__device__ __forceinline__ float sum8(float v) { // over the eight lanes of a column
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 1);
}

// the convolution's input at position pos0 + t: this call's rows, the ring, or zero before the start
struct ConvIn {
    const float *x; // column of row 0 of the sequence
    int64_t ld;
    const float *ring; // column of slot 0
    int64_t channels;
    int taps, pos0;
    __device__ __forceinline__ float at(int t) const {
        if (t >= 0) return x[t * ld];
        const int pos = pos0 + t;
        return pos >= 0 ? ring[(int64_t)(pos % taps) * channels] : 0.f;
    }
};

// ---- tokens ------------------------------------------------------------------------------------------
constexpr int TOK_NT = 256, TOK_NW = TOK_NT / 32, RUN = 16; // tokens a warp walks for one head
struct TokParams {
    KqMatState m;
    KqStateIn in;
    KqStateTok t;
    int32_t T, pos0;
    const int32_t *pos0_dev;
    int64_t ldq, ldv, ldg;
};

// SiLU of the convolution of up to 32 C channels of one head for a run of tokens: f(t, values of the lane's channels)
template <int C, typename F>
__device__ __forceinline__ void conv_run(const TokParams &p, const float *x, const float *w, int64_t channel0, int n, int64_t seq, int t0, int t1, int pos0,
                                         int lane, F f) {
    const int taps = p.m.taps;
    const int64_t row0 = seq * p.T, channels = kq_state_channels(p.m);
    if (taps == 4) { // the last inputs and the weights stay in registers
        float cw[C][4], in[C][4];
#pragma unroll
        for (int c = 0; c < C; c++) {
            const int d = lane + 32 * c;
            const ConvIn ci = {x + row0 * p.in.ld + d, p.in.ld, p.m.conv + seq * taps * channels + channel0 + d, channels, taps, pos0};
#pragma unroll
            for (int k = 0; k < 4; k++) {
                cw[c][k] = d < n ? w[d * 4 + k] : 0.f;
                in[c][k] = d < n && k < 3 ? ci.at(t0 - 3 + k) : 0.f;
            }
        }
        for (int t = t0; t < t1; t++) {
            float v[C];
#pragma unroll
            for (int c = 0; c < C; c++) {
                const int d = lane + 32 * c;
                in[c][3] = d < n ? x[(row0 + t) * p.in.ld + d] : 0.f;
                float s = 0.f;
#pragma unroll
                for (int k = 0; k < 4; k++) s = fmaf(cw[c][k], in[c][k], s);
                v[c] = kq_silu(s);
                in[c][0] = in[c][1], in[c][1] = in[c][2], in[c][2] = in[c][3];
            }
            f(t, v);
        }
        return;
    }
    for (int t = t0; t < t1; t++) {
        float v[C];
#pragma unroll
        for (int c = 0; c < C; c++) {
            const int d = lane + 32 * c;
            float s = 0.f;
            if (d < n) {
                if (taps == 0) {
                    s = x[(row0 + t) * p.in.ld + d];
                } else {
                    const ConvIn ci = {x + row0 * p.in.ld + d, p.in.ld, p.m.conv + seq * taps * channels + channel0 + d, channels, taps, pos0};
                    for (int k = 0; k < taps; k++) s = fmaf(w[(int64_t)d * taps + k], ci.at(t - (taps - 1) + k), s);
                }
            }
            v[c] = kq_silu(s);
        }
        f(t, v);
    }
}

// grid (jobs / warps, runs of tokens, sequences); a job is a query / key head pair, 32 C channels of the values, or the decays and
// write strengths of a head
template <int C>
__global__ void __launch_bounds__(TOK_NT) state_tokens_kernel(const __grid_constant__ TokParams p, int v_jobs) {
    KQ_PDL_ENTER();
    const KqMatState &m = p.m;
    const int lane = threadIdx.x & 31, t0 = blockIdx.y * RUN, t1 = min(p.T, t0 + RUN);
    const int64_t seq = blockIdx.z, row0 = seq * p.T;
    const int pos0 = p.pos0_dev ? *p.pos0_dev : p.pos0;
    int job = blockIdx.x * TOK_NW + (threadIdx.x >> 5);
    const int64_t nq = (int64_t)m.kv_heads * m.dim;
    if (job < m.kv_heads) { // q, then k and their product
        const int64_t c0 = (int64_t)job * m.dim;
        conv_run<C>(p, p.in.q + c0, m.taps ? m.conv_q + c0 * m.taps : nullptr, c0, m.dim, seq, t0, t1, pos0, lane, [&](int t, const float (&v)[C]) {
            float ss = 0.f;
#pragma unroll
            for (int c = 0; c < C; c++) ss += v[c] * v[c];
            const float sc = m.delta ? 1.0f / sqrtf(kq_warp_sum(ss) + 1e-6f) / sqrtf((float)m.dim) : 1.f;
#pragma unroll
            for (int c = 0; c < C; c++)
                if (lane + 32 * c < m.dim) p.t.q[(row0 + t) * p.ldq + c0 + lane + 32 * c] = v[c] * sc;
        });
        conv_run<C>(p, p.in.k + c0, m.taps ? m.conv_k + c0 * m.taps : nullptr, nq + c0, m.dim, seq, t0, t1, pos0, lane, [&](int t, const float (&v)[C]) {
            float ss = 0.f, qk = 0.f;
#pragma unroll
            for (int c = 0; c < C; c++) ss += v[c] * v[c];
            const float sc = m.delta ? 1.0f / sqrtf(kq_warp_sum(ss) + 1e-6f) : 1.f;
#pragma unroll
            for (int c = 0; c < C; c++)
                if (lane + 32 * c < m.dim) {
                    const int64_t i = (row0 + t) * p.ldq + c0 + lane + 32 * c;
                    if (m.delta) qk = fmaf(p.t.q[i], v[c] * sc, qk); // this lane's own store
                    p.t.k[i] = v[c] * sc;
                }
            if (m.delta) {
                qk = kq_warp_sum(qk);
                const int rep = m.heads / m.kv_heads;
                for (int h = lane; h < rep; h += 32) p.t.b[((row0 + t) * m.heads + job * rep + h) * 2 + 1] = qk;
            }
        });
        return;
    }
    job -= m.kv_heads;
    if (job < v_jobs) {
        const int64_t c0 = (int64_t)job * 32 * C, nv = (int64_t)m.heads * m.vdim;
        const int n = (int)min((int64_t)32 * C, nv - c0);
        conv_run<C>(p, p.in.v + c0, m.taps ? m.conv_v + c0 * m.taps : nullptr, 2 * nq + c0, n, seq, t0, t1, pos0, lane, [&](int t, const float (&v)[C]) {
#pragma unroll
            for (int c = 0; c < C; c++)
                if (lane + 32 * c < n) p.t.v[(row0 + t) * p.ldv + c0 + lane + 32 * c] = v[c];
        });
        return;
    }
    job -= v_jobs;
    if (!m.delta || job >= m.heads) return;
    const float a = expf(m.a_log[job]);
    const int64_t c0 = (int64_t)job * m.dim;
    float bias[C];
#pragma unroll
    for (int c = 0; c < C; c++) bias[c] = lane + 32 * c < m.dim ? m.dt_bias[c0 + lane + 32 * c] : 0.f;
    for (int t = t0; t < t1; t++) {
#pragma unroll
        for (int c = 0; c < C; c++)
            if (lane + 32 * c < m.dim)
                p.t.g[(row0 + t) * p.ldg + c0 + lane + 32 * c] = expf(-a * kq_softplus(p.in.z[(row0 + t) * p.in.ldz + c0 + lane + 32 * c] + bias[c]));
        if (lane == 0) p.t.b[((row0 + t) * m.heads + job) * 2] = kq_sigmoid(p.in.b[(row0 + t) * p.in.ld + job]);
    }
}

// ---- token loop --------------------------------------------------------------------------------------
template <int DP>
struct Scan {
    static constexpr int R4 = DP / 32;                 // groups of four key dimensions per lane
    static constexpr int TT = DP <= 128 ? 16 : 8;      // tokens per tile
    static constexpr int TILE = TT * (3 * DP + COLS + 2); // floats: q, k, g, values of the CTA's columns, (beta, q.k)
    static constexpr int SMEM = (2 * TILE + TT * COLS) * 4;
};
struct ScanParams {
    KqMatState m;
    KqStateIn in;
    KqStateTok t;
    int32_t T, pos0, vec;
    const int32_t *pos0_dev;
    int64_t ldq, ldv, ldg, ldo;
    float *o;
};

__device__ __forceinline__ void cp4(uint32_t dst, const void *src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void cp16(uint32_t dst, const void *src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }

// the last `taps` inputs of every channel into the ring, shared out over all CTAs of the grid
__device__ __forceinline__ void move_ring(const KqMatState &m, const KqStateIn &in, int64_t n_seq, int T, int pos0, int64_t id, int64_t n_threads) {
    const int64_t channels = kq_state_channels(m), nq = (int64_t)m.kv_heads * m.dim;
    const int keep = min(T, m.taps);
    for (int64_t i = id; i < n_seq * keep * channels; i += n_threads) {
        const int64_t c = i % channels, rest = i / channels, seq = rest / keep;
        const int t = T - keep + (int)(rest % keep);
        const float *x = c < nq ? in.q + c : c < 2 * nq ? in.k + (c - nq) : in.v + (c - 2 * nq);
        m.conv[(seq * m.taps + (pos0 + t) % m.taps) * channels + c] = x[(seq * T + t) * in.ld];
    }
}

// grid (blocks of columns, heads, sequences)
template <int DP, bool DELTA>
__global__ void __launch_bounds__(SCAN_NT) state_scan_kernel(const __grid_constant__ ScanParams p) {
    KQ_PDL_ENTER();
    using S = Scan<DP>;
    constexpr int R4 = S::R4, TT = S::TT;
    extern __shared__ __align__(16) float sm[];
    const KqMatState &m = p.m;
    const int tid = threadIdx.x, part = tid & 7, col = tid >> 3;
    const int h = blockIdx.y, kh = h / (m.heads / m.kv_heads), e0 = blockIdx.x * COLS, ne = min(COLS, m.vdim - e0);
    const int64_t seq = blockIdx.z, row0 = seq * p.T;
    const int pos0 = p.pos0_dev ? *p.pos0_dev : p.pos0;
    if (m.taps)
        move_ring(m, p.in, gridDim.z, p.T, pos0, ((seq * gridDim.y + h) * gridDim.x + blockIdx.x) * SCAN_NT + tid,
                  (int64_t)gridDim.x * gridDim.y * gridDim.z * SCAN_NT);
    for (int i = tid; i < 2 * S::TILE; i += SCAN_NT) sm[i] = 0.f; // what no copy reaches stays zero
    __syncthreads();
    const float *q = p.t.q + row0 * p.ldq + (int64_t)kh * m.dim, *k = p.t.k + row0 * p.ldq + (int64_t)kh * m.dim,
                *g = DELTA ? p.t.g + row0 * p.ldg + (int64_t)h * m.dim : nullptr, *v = p.t.v + row0 * p.ldv + (int64_t)h * m.vdim + e0,
                *b = DELTA ? p.t.b + (row0 * m.heads + h) * 2 : nullptr;
    auto request = [&](int tile) {
        float *dst = sm + (tile & 1) * S::TILE;
        const int t0 = tile * TT, n = min(TT, p.T - t0);
        const uint32_t d0 = (uint32_t)__cvta_generic_to_shared(dst);
        if (p.vec) {
            const int n4 = m.dim / 4, v4 = ne / 4;
            for (int i = tid; i < n * n4; i += SCAN_NT) {
                const int t = i / n4, c = i % n4 * 4;
                const uint32_t d = d0 + (t * DP + c) * 4;
                cp16(d, q + (int64_t)(t0 + t) * p.ldq + c);
                cp16(d + TT * DP * 4, k + (int64_t)(t0 + t) * p.ldq + c);
                if (DELTA) cp16(d + 2 * TT * DP * 4, g + (int64_t)(t0 + t) * p.ldg + c);
            }
            for (int i = tid; i < n * v4; i += SCAN_NT) {
                const int t = i / v4, c = i % v4 * 4;
                cp16(d0 + (3 * TT * DP + t * COLS + c) * 4, v + (int64_t)(t0 + t) * p.ldv + c);
            }
        } else {
            for (int i = tid; i < n * m.dim; i += SCAN_NT) {
                const int t = i / m.dim, c = i % m.dim;
                const uint32_t d = d0 + (t * DP + c) * 4;
                cp4(d, q + (int64_t)(t0 + t) * p.ldq + c);
                cp4(d + TT * DP * 4, k + (int64_t)(t0 + t) * p.ldq + c);
                if (DELTA) cp4(d + 2 * TT * DP * 4, g + (int64_t)(t0 + t) * p.ldg + c);
            }
            for (int i = tid; i < n * ne; i += SCAN_NT) cp4(d0 + (3 * TT * DP + i / ne * COLS + i % ne) * 4, v + (int64_t)(t0 + i / ne) * p.ldv + i % ne);
        }
        if (DELTA)
            for (int i = tid; i < 2 * n; i += SCAN_NT) cp4(d0 + (TT * (3 * DP + COLS) + i) * 4, b + (int64_t)(t0 + i / 2) * 2 * m.heads + (i & 1));
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // the column's state; a lane holds the dimensions 4 (part + 8 i) .. + 3
    const bool live = col < ne;
    float *sp = m.s + ((seq * m.heads + h) * m.vdim + e0 + (live ? col : 0)) * DP;
    float4 s[R4];
#pragma unroll
    for (int i = 0; i < R4; i++) s[i] = pos0 > 0 ? *reinterpret_cast<const float4 *>(sp + 4 * (part + 8 * i)) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float decay = DELTA ? 1.f : m.decay[h];
    const int n_tiles = (p.T + TT - 1) / TT;
    float *so = sm + 2 * S::TILE;
    request(0);
    for (int tile = 0; tile < n_tiles; tile++) {
        if (tile + 1 < n_tiles) {
            request(tile + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float *src = sm + (tile & 1) * S::TILE;
        const int n = min(TT, p.T - tile * TT);
        for (int t = 0; t < n; t++) {
            const float4 *sq = reinterpret_cast<const float4 *>(src + t * DP), *sk = sq + TT * DP / 4, *sg = sk + TT * DP / 4;
            const float vt = src[3 * TT * DP + t * COLS + col];
            if (DELTA) {
                const float beta = src[TT * (3 * DP + COLS) + 2 * t], qk = src[TT * (3 * DP + COLS) + 2 * t + 1];
                float4 kk[R4], dk = make_float4(0.f, 0.f, 0.f, 0.f), dq = dk;
#pragma unroll
                for (int i = 0; i < R4; i++) {
                    const float4 gg = sg[part + 8 * i], qq = sq[part + 8 * i];
                    kk[i] = sk[part + 8 * i];
                    s[i].x *= gg.x, s[i].y *= gg.y, s[i].z *= gg.z, s[i].w *= gg.w;
                    dk.x = fmaf(s[i].x, kk[i].x, dk.x), dk.y = fmaf(s[i].y, kk[i].y, dk.y), dk.z = fmaf(s[i].z, kk[i].z, dk.z), dk.w = fmaf(s[i].w, kk[i].w, dk.w);
                    dq.x = fmaf(s[i].x, qq.x, dq.x), dq.y = fmaf(s[i].y, qq.y, dq.y), dq.z = fmaf(s[i].z, qq.z, dq.z), dq.w = fmaf(s[i].w, qq.w, dq.w);
                }
                const float rk = sum8((dk.x + dk.y) + (dk.z + dk.w)), rq = sum8((dq.x + dq.y) + (dq.z + dq.w));
                const float u = beta * (vt - rk);
#pragma unroll
                for (int i = 0; i < R4; i++) {
                    s[i].x = fmaf(kk[i].x, u, s[i].x), s[i].y = fmaf(kk[i].y, u, s[i].y);
                    s[i].z = fmaf(kk[i].z, u, s[i].z), s[i].w = fmaf(kk[i].w, u, s[i].w);
                }
                if (part == 0) so[t * COLS + col] = fmaf(qk, u, rq);
            } else {
                float4 dq = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int i = 0; i < R4; i++) {
                    const float4 kk = sk[part + 8 * i], qq = sq[part + 8 * i];
                    s[i].x = fmaf(kk.x, vt, decay * s[i].x), s[i].y = fmaf(kk.y, vt, decay * s[i].y);
                    s[i].z = fmaf(kk.z, vt, decay * s[i].z), s[i].w = fmaf(kk.w, vt, decay * s[i].w);
                    dq.x = fmaf(s[i].x, qq.x, dq.x), dq.y = fmaf(s[i].y, qq.y, dq.y), dq.z = fmaf(s[i].z, qq.z, dq.z), dq.w = fmaf(s[i].w, qq.w, dq.w);
                }
                const float rq = sum8((dq.x + dq.y) + (dq.z + dq.w));
                if (part == 0) so[t * COLS + col] = rq;
            }
        }
        __syncthreads(); // the tile's buffer is free, its outputs are complete
        for (int i = tid; i < n * COLS; i += SCAN_NT)
            if (i % COLS < ne) p.o[(row0 + tile * TT + i / COLS) * p.ldo + (int64_t)h * m.vdim + e0 + i % COLS] = so[i];
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < R4; i++) *reinterpret_cast<float4 *>(sp + 4 * (part + 8 * i)) = s[i];
    }
}

// ---- output of a prompt --------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float *o, int64_t ldo, const float *gate, int64_t ldg, const float *w, float eps, int64_t rows,
                                                             int heads, int vdim, float *out32, int64_t ld32, uint16_t *out16, int64_t ld16) {
    KQ_PDL_ENTER();
    const int64_t id = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5), r = id / heads;
    const int h = (int)(id % heads), lane = threadIdx.x & 31;
    if (r >= rows) return;
    const float *x = o + r * ldo + (int64_t)h * vdim, *gt = gate + r * ldg + (int64_t)h * vdim;
    constexpr int KEEP = 8;
    float v[KEEP], ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; i++) {
        v[i] = lane + 32 * i < vdim ? x[lane + 32 * i] : 0.f;
        ss += v[i] * v[i];
    }
    for (int d = lane + 32 * KEEP; d < vdim; d += 32) ss += x[d] * x[d];
    const float sc = 1.0f / sqrtf(kq_warp_sum(ss) / (float)vdim + eps);
    auto emit = [&](int d, float a) {
        a *= sc * w[d] * kq_sigmoid(gt[d]);
        if (out32) out32[r * ld32 + (int64_t)h * vdim + d] = a;
        if (out16) out16[r * ld16 + (int64_t)h * vdim + d] = kq_f2bf(a);
    };
#pragma unroll
    for (int i = 0; i < KEEP; i++)
        if (lane + 32 * i < vdim) emit(lane + 32 * i, v[i]);
    for (int d = lane + 32 * KEEP; d < vdim; d += 32) emit(d, x[d]);
    if (out16 && h == heads - 1)
        for (int64_t d = (int64_t)heads * vdim + lane; d < ld16; d += 32) out16[r * ld16 + d] = 0;
}

// ---- one token -----------------------------------------------------------------------------------------
constexpr int STEP_NT = 256, STEP_NW = STEP_NT / 32;
struct StepParams {
    KqMatState m;
    KqStateIn in;
    KqStateStep x;
    const int32_t *pos_dev;
    int32_t pos;
    float *z;
    int64_t ldz;
};

// y[i] = W[i] . x for n rows of bf16 weights (16-byte chunks of padded rows), x in shared memory; groups of lanes share rows
__device__ __forceinline__ void small_matvec(const uint16_t *W, int64_t ldw, int n, int K, const float *x, float *y, int warp, int lane) {
    const int nck = (K + 7) / 8;
    int w = 1; // lanes per row
    while (w < nck && w < 32) w *= 2;
    const int per = 32 / w, sub = lane / w, l = lane % w;
    for (int r0 = warp * per; r0 < n; r0 += STEP_NW * per) {
        const int r = r0 + sub;
        float s = 0.f;
        if (r < n)
            for (int c = l; c < nck; c += w) {
                const uint4 q = *reinterpret_cast<const uint4 *>(W + (int64_t)r * ldw + 8 * c);
                s = kq_dot8(q, *reinterpret_cast<const float4 *>(x + 8 * c), *reinterpret_cast<const float4 *>(x + 8 * c + 4), s);
            }
        for (int o = w / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if (r < n && l == 0) y[r] = s;
    }
}
// SiLU of the convolution of one head's channels; the CTA that owns them (`owns`) also stores the new input.  The slot of the
// current position is read by nobody in this launch.
__device__ __forceinline__ void conv_step(const KqMatState &m, const float *x, const float *w, float *ring, int64_t channels, int n, int pos, bool owns, float *out) {
    for (int d = threadIdx.x; d < n; d += STEP_NT) {
        float s = x[d];
        if (m.taps) {
            s = 0.f;
            const ConvIn ci = {x + d, 0, ring + d, channels, m.taps, pos};
            for (int k = 0; k < m.taps; k++) s = fmaf(w[(int64_t)d * m.taps + k], ci.at(k - (m.taps - 1)), s);
            if (owns) ring[(int64_t)(pos % m.taps) * channels + d] = x[d];
        }
        out[d] = kq_silu(s);
    }
}

// grid (heads, sequences)
template <int DP, bool DELTA>
__global__ void __launch_bounds__(STEP_NT) state_step_kernel(const __grid_constant__ StepParams p) {
    constexpr int R4 = DP / 32, PC = STEP_NT / 8; // columns of a pass
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_red[4];
    KQ_PDL_TRIGGER();
    const KqMatState &m = p.m;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = tid & 7, col = tid >> 3;
    const int h = blockIdx.x, rep = m.heads / m.kv_heads, kh = h / rep;
    const int64_t seq = blockIdx.y;
    const int ra = (p.x.a_rank + 7) / 8 * 8, rg = (p.x.g_rank + 7) / 8 * 8, vp = (m.vdim + 3) / 4 * 4;
    float *sq = sm, *sk = sq + DP, *sg = sk + DP, *sv = sg + DP, *sgate = sv + vp, *so = sgate + vp, *sa = so + vp, *sg1 = sa + ra;
    if (DELTA) { // the low-rank matrices come towards this SM while the predecessor finishes
        const int64_t lda = kq_bf16_ld(p.x.a_rank), ldg = kq_bf16_ld(p.x.g_rank);
        for (int i = tid * 128; i < m.dim * lda * 2; i += STEP_NT * 128)
            asm volatile("prefetch.global.L2 [%0];" ::"l"((const uint8_t *)(p.x.a2 + (int64_t)h * m.dim * lda) + i));
        for (int i = tid * 128; i < m.vdim * ldg * 2; i += STEP_NT * 128)
            asm volatile("prefetch.global.L2 [%0];" ::"l"((const uint8_t *)(p.x.g2 + (int64_t)h * m.vdim * ldg) + i));
    }
    {
        const uint8_t *s0 = (const uint8_t *)(m.s + (seq * m.heads + h) * (int64_t)m.vdim * DP);
        for (int i = tid * 128; i < m.vdim * DP * 4; i += STEP_NT * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(s0 + i));
    }
    KQ_PDL_WAIT();
    const int pos = p.pos_dev ? *p.pos_dev : p.pos;
    const int64_t channels = kq_state_channels(m), nq = (int64_t)m.kv_heads * m.dim, cq = (int64_t)kh * m.dim, cv = (int64_t)h * m.vdim;
    float *ring = m.taps ? m.conv + seq * m.taps * channels : nullptr;
    const bool owns = h % rep == 0;
    conv_step(m, p.in.q + seq * p.in.ld + cq, m.conv_q + cq * m.taps, ring + cq, channels, m.dim, pos, owns, sq);
    conv_step(m, p.in.k + seq * p.in.ld + cq, m.conv_k + cq * m.taps, ring + nq + cq, channels, m.dim, pos, owns, sk);
    conv_step(m, p.in.v + seq * p.in.ld + cv, m.conv_v + cv * m.taps, ring + 2 * nq + cv, channels, m.vdim, pos, true, sv);
    for (int d = m.dim + tid; d < DP; d += STEP_NT) sq[d] = sk[d] = sg[d] = 0.f;
    if (DELTA) {
        for (int i = tid; i < ra; i += STEP_NT) sa[i] = i < p.x.a_rank ? p.x.a1[seq * p.in.ld + i] : 0.f;
        for (int i = tid; i < rg; i += STEP_NT) sg1[i] = i < p.x.g_rank ? p.x.g1[seq * p.in.ld + i] : 0.f;
    }
    __syncthreads();
    if (DELTA) {
        if (warp < 2) { // unit norms
            float *x = warp ? sk : sq, ss = 0.f;
            for (int d = lane; d < m.dim; d += 32) ss += x[d] * x[d];
            ss = 1.0f / sqrtf(kq_warp_sum(ss) + 1e-6f);
            if (lane == 0) s_red[warp] = warp ? ss : ss / sqrtf((float)m.dim);
        }
        small_matvec(p.x.a2 + (int64_t)h * m.dim * kq_bf16_ld(p.x.a_rank), kq_bf16_ld(p.x.a_rank), m.dim, p.x.a_rank, sa, sg, warp, lane);
        small_matvec(p.x.g2 + (int64_t)h * m.vdim * kq_bf16_ld(p.x.g_rank), kq_bf16_ld(p.x.g_rank), m.vdim, p.x.g_rank, sg1, sgate, warp, lane);
        __syncthreads();
        const float a = expf(m.a_log[h]);
        for (int d = tid; d < m.dim; d += STEP_NT) {
            sq[d] *= s_red[0];
            sk[d] *= s_red[1];
            sg[d] = expf(-a * kq_softplus(sg[d] + m.dt_bias[(int64_t)h * m.dim + d]));
        }
        __syncthreads();
    }
    float4 qq[R4], kk[R4], gg[R4];
#pragma unroll
    for (int i = 0; i < R4; i++) {
        qq[i] = reinterpret_cast<const float4 *>(sq)[part + 8 * i];
        kk[i] = reinterpret_cast<const float4 *>(sk)[part + 8 * i];
        if (DELTA) gg[i] = reinterpret_cast<const float4 *>(sg)[part + 8 * i];
    }
    const float beta = DELTA ? kq_sigmoid(p.in.b[seq * p.in.ld + h]) : 0.f, decay = DELTA ? 1.f : m.decay[h];
    float *base = m.s + (seq * m.heads + h) * (int64_t)m.vdim * DP;
#pragma unroll 2
    for (int e0 = 0; e0 < m.vdim; e0 += PC) {
        const int e = e0 + col;
        const bool live = e < m.vdim;
        float *sp = base + (int64_t)(live ? e : 0) * DP;
        const float vt = live ? sv[e] : 0.f;
        float4 s[R4];
#pragma unroll
        for (int i = 0; i < R4; i++) s[i] = pos > 0 ? *reinterpret_cast<const float4 *>(sp + 4 * (part + 8 * i)) : make_float4(0.f, 0.f, 0.f, 0.f);
        float w = vt;
        if (DELTA) {
            float rk = 0.f;
#pragma unroll
            for (int i = 0; i < R4; i++) {
                s[i].x *= gg[i].x, s[i].y *= gg[i].y, s[i].z *= gg[i].z, s[i].w *= gg[i].w;
                rk = fmaf(s[i].x, kk[i].x, fmaf(s[i].y, kk[i].y, fmaf(s[i].z, kk[i].z, fmaf(s[i].w, kk[i].w, rk))));
            }
            w = beta * (vt - sum8(rk));
        }
        float rq = 0.f;
#pragma unroll
        for (int i = 0; i < R4; i++) {
            s[i].x = fmaf(kk[i].x, w, decay * s[i].x), s[i].y = fmaf(kk[i].y, w, decay * s[i].y);
            s[i].z = fmaf(kk[i].z, w, decay * s[i].z), s[i].w = fmaf(kk[i].w, w, decay * s[i].w);
            rq = fmaf(s[i].x, qq[i].x, fmaf(s[i].y, qq[i].y, fmaf(s[i].z, qq[i].z, fmaf(s[i].w, qq[i].w, rq))));
            if (live) *reinterpret_cast<float4 *>(sp + 4 * (part + 8 * i)) = s[i];
        }
        rq = sum8(rq);
        if (live && part == 0) so[e] = rq;
    }
    __syncthreads();
    float *z = p.z + seq * p.ldz + cv;
    if (DELTA) {
        if (warp == 0) {
            float ss = 0.f;
            for (int e = lane; e < m.vdim; e += 32) ss += so[e] * so[e];
            ss = kq_warp_sum(ss);
            if (lane == 0) s_red[2] = 1.0f / sqrtf(ss / (float)m.vdim + p.x.eps);
        }
        __syncthreads();
        for (int e = tid; e < m.vdim; e += STEP_NT) z[e] = so[e] * s_red[2] * p.x.norm_w[e] * kq_sigmoid(sgate[e]);
    } else {
        for (int e = tid; e < m.vdim; e += STEP_NT) z[e] = so[e];
    }
}

// v = hi + mid + lo exactly
__global__ void __launch_bounds__(256) rank_operands_kernel(const float *a, int n, uint16_t *a16, const float *g, int m, uint16_t *g16, int64_t ld, int64_t rows) {
    KQ_PDL_ENTER();
    const int64_t lda = kq_bf16_ld(n), ldg = kq_bf16_ld(m), r = blockIdx.x, plane = rows * lda;
    for (int64_t i = threadIdx.x; i < lda; i += blockDim.x) {
        float v = i < n ? a[r * ld + i] : 0.f;
#pragma unroll
        for (int q = 0; q < 3; q++) {
            const uint16_t b = kq_f2bf(v);
            a16[q * plane + r * lda + i] = b;
            v -= kq_bf2f(b);
        }
    }
    for (int64_t i = threadIdx.x; i < ldg; i += blockDim.x) g16[r * ldg + i] = i < m ? kq_f2bf(g[r * ld + i]) : 0;
}

b200_status check_state(const KqMatState &m, int n_seq, int T) {
    KQ_REQUIRE(m.heads >= 1 && m.kv_heads >= 1 && m.heads % m.kv_heads == 0 && m.dim >= 1 && m.vdim >= 1 && m.taps >= 0 && n_seq >= 1 && T >= 1 &&
                   m.s && (m.taps == 0 || m.conv),
               "matrix state: bad shape");
    KQ_REQUIRE(m.dim <= KQ_STATE_MAX_DIM && m.heads <= 65535 && n_seq <= 65535, "matrix state: %d heads of %d key dimensions", m.heads, m.dim);
    return B200_OK;
}

template <int DP, bool DELTA>
b200_status launch_scan(const ScanParams &p, int n_seq, cudaStream_t st) {
    static bool attr[16];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 16 || !attr[dev]) {
        KQ_CUDA(cudaFuncSetAttribute(state_scan_kernel<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, Scan<DP>::SMEM));
        if (dev >= 0 && dev < 16) attr[dev] = true;
    }
    kq_launch(state_scan_kernel<DP, DELTA>, dim3((unsigned)kq_div_up(p.m.vdim, COLS), (unsigned)p.m.heads, (unsigned)n_seq), SCAN_NT, Scan<DP>::SMEM, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
template <int DP, bool DELTA>
b200_status launch_step(const StepParams &p, int n_seq, size_t smem, cudaStream_t st) {
    static size_t attr[16];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (smem > 48 * 1024 && (dev < 0 || dev >= 16 || attr[dev] < smem)) {
        KQ_CUDA(cudaFuncSetAttribute(state_step_kernel<DP, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        if (dev >= 0 && dev < 16) attr[dev] = smem;
    }
    kq_launch(state_step_kernel<DP, DELTA>, dim3((unsigned)p.m.heads, (unsigned)n_seq), STEP_NT, smem, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
#define BY_DIM(FN, ...)                                                                              \
    switch (kq_state_ld(m.dim)) {                                                                    \
    case 32: return m.delta ? FN<32, true>(__VA_ARGS__) : FN<32, false>(__VA_ARGS__);                \
    case 64: return m.delta ? FN<64, true>(__VA_ARGS__) : FN<64, false>(__VA_ARGS__);                \
    case 96: return m.delta ? FN<96, true>(__VA_ARGS__) : FN<96, false>(__VA_ARGS__);                \
    case 128: return m.delta ? FN<128, true>(__VA_ARGS__) : FN<128, false>(__VA_ARGS__);             \
    case 192: return m.delta ? FN<192, true>(__VA_ARGS__) : FN<192, false>(__VA_ARGS__);             \
    default: return m.delta ? FN<256, true>(__VA_ARGS__) : FN<256, false>(__VA_ARGS__);              \
    }

} // namespace

b200_status kq_state_tokens(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                            cudaStream_t st) {
    KQ_TRY(check_state(m, n_seq, T));
    TokParams p;
    p.m = m, p.in = in, p.t = t, p.T = T, p.pos0 = pos0, p.pos0_dev = pos0_dev;
    p.ldq = kq_f32_ld((int64_t)m.kv_heads * m.dim), p.ldv = kq_f32_ld((int64_t)m.heads * m.vdim), p.ldg = kq_f32_ld((int64_t)m.heads * m.dim);
    const int c = (int)kq_div_up(m.dim, 32), C = c <= 1 ? 1 : c <= 2 ? 2 : c <= 4 ? 4 : 8;
    const int v_jobs = (int)kq_div_up((int64_t)m.heads * m.vdim, 32 * C);
    const dim3 grid((unsigned)kq_div_up(m.kv_heads + v_jobs + (m.delta ? m.heads : 0), TOK_NW), (unsigned)kq_div_up(T, RUN), (unsigned)n_seq);
    if (C == 1) kq_launch(state_tokens_kernel<1>, grid, TOK_NT, 0, st, p, v_jobs);
    else if (C == 2) kq_launch(state_tokens_kernel<2>, grid, TOK_NT, 0, st, p, v_jobs);
    else if (C == 4) kq_launch(state_tokens_kernel<4>, grid, TOK_NT, 0, st, p, v_jobs);
    else kq_launch(state_tokens_kernel<8>, grid, TOK_NT, 0, st, p, v_jobs);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_state_scan(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                          float *o, int64_t ldo, cudaStream_t st) {
    KQ_TRY(check_state(m, n_seq, T));
    ScanParams p;
    p.m = m, p.in = in, p.t = t, p.T = T, p.pos0 = pos0, p.pos0_dev = pos0_dev, p.o = o, p.ldo = ldo;
    p.ldq = kq_f32_ld((int64_t)m.kv_heads * m.dim), p.ldv = kq_f32_ld((int64_t)m.heads * m.vdim), p.ldg = kq_f32_ld((int64_t)m.heads * m.dim);
    const uintptr_t al = (uintptr_t)t.q | (uintptr_t)t.k | (uintptr_t)t.v | (uintptr_t)t.g;
    p.vec = m.dim % 4 == 0 && m.vdim % 4 == 0 && (al & 15) == 0;
    BY_DIM(launch_scan, p, n_seq, st)
}

b200_status kq_head_norm_gate(const float *o, int64_t ldo, const float *gate, int64_t ldg, const float *norm_w, float eps, int64_t rows, int heads,
                              int vdim, float *out32, int64_t ld32, uint16_t *out16, int64_t ld16, cudaStream_t st) {
    KQ_REQUIRE(o && gate && norm_w && rows >= 1 && heads >= 1 && vdim >= 1, "head_norm_gate: bad call");
    kq_launch(head_norm_gate_kernel, (unsigned)kq_div_up(rows * heads, 8), 256, 0, st, o, ldo, gate, ldg, norm_w, eps, rows, heads, vdim, out32, ld32, out16,
              ld16);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_state_step(const KqMatState &m, const KqStateIn &in, const KqStateStep &x, int n_seq, const int32_t *pos_dev, int pos, float *z,
                          int64_t ldz, cudaStream_t st) {
    KQ_TRY(check_state(m, n_seq, 1));
    StepParams p;
    p.m = m, p.in = in, p.x = x, p.pos_dev = pos_dev, p.pos = pos, p.z = z, p.ldz = ldz;
    const size_t smem = (size_t)(3 * kq_state_ld(m.dim) + 3 * kq_pad(m.vdim, 4) + kq_pad(x.a_rank, 8) + kq_pad(x.g_rank, 8)) * 4;
    KQ_REQUIRE(smem <= 200 * 1024, "matrix state: %d value dimensions", m.vdim);
    BY_DIM(launch_step, p, n_seq, smem, st)
}

b200_status kq_rank_operands(const float *a, int n, uint16_t *a16, const float *g, int m, uint16_t *g16, int64_t ld, int64_t rows, cudaStream_t st) {
    kq_launch(rank_operands_kernel, (unsigned)rows, 256, 0, st, a, n, a16, g, m, g16, ld, rows);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
