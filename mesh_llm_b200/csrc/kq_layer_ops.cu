// Ops of layers with 16-bit weights that are neither projections nor attention: scaled embedding rows, the
// residual / norm prologue as a kernel of its own, the per-channel causal convolution and the gated diagonal
// linear recurrence (prefill as a chunked scan, decode as one launch with the convolution and the gates).
// All arithmetic is f32.
#include "kq_dense.cuh"

#include <algorithm>

namespace {

// a thread per eight values of a row
__global__ void embed_bf16_kernel(const uint16_t *W, int64_t ldw, const int32_t *ids, int64_t rows, int K, float scale, float *y,
                                  int64_t ldy) {
    KQ_PDL_ENTER();
    const int k = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
    const int64_t r = blockIdx.y;
    if (k >= K) return;
    const uint4 q = *reinterpret_cast<const uint4 *>(W + (int64_t)ids[r] * ldw + k);
    const uint32_t w[4] = {q.x, q.y, q.z, q.w};
    float v[8];
#pragma unroll
    for (int e = 0; e < 4; e++) {
        v[2 * e] = __uint_as_float(w[e] << 16) * scale;
        v[2 * e + 1] = __uint_as_float(w[e] & 0xffff0000u) * scale;
    }
    float *o = y + r * ldy + k;
    if (k + 8 <= K && (ldy & 3) == 0) {
        *reinterpret_cast<float4 *>(o) = make_float4(v[0], v[1], v[2], v[3]);
        *reinterpret_cast<float4 *>(o + 4) = make_float4(v[4], v[5], v[6], v[7]);
    } else {
#pragma unroll
        for (int e = 0; e < 8; e++)
            if (k + e < K) o[e] = v[e];
    }
}

// a thread per eight values; rows of a multiple of 64 elements
__global__ void gather_bf16_kernel(const uint16_t *W, const int32_t *ids, uint16_t *y, int64_t ld) {
    KQ_PDL_ENTER();
    const int64_t k = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * 8, r = blockIdx.y;
    if (k < ld) *reinterpret_cast<uint4 *>(y + r * ld + k) = *reinterpret_cast<const uint4 *>(W + (int64_t)ids[r] * ld + k);
}

constexpr int NT = 256;
__device__ __forceinline__ float block_sum(float v, float *red) {
    v = kq_warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < NT / 32; i++) t += red[i];
    return t;
}

// one CTA per row; VEC: four elements per access (K, strides and addresses allow it)
template <bool VEC>
__global__ void __launch_bounds__(NT) norm_prep_kernel(const __grid_constant__ KqNormPrep p, int K, float *h32, int64_t ld32,
                                                       uint16_t *h16, int64_t ld16) {
    KQ_PDL_ENTER();
    constexpr int E = VEC ? 4 : 1, KEEP = 8; // values a thread keeps in registers: rows up to KEEP * E * NT
    __shared__ float red[NT / 32];
    const int64_t r = blockIdx.x;
    const int n = K / E, tid = threadIdx.x;
    const float *x = p.x + r * p.ldx, *sub = p.sub ? p.sub + r * p.ld_sub : nullptr;
    float *xo = p.x_out ? p.x_out + r * p.ld_out : nullptr;
    auto ld = [](const float *q, int i, float (&v)[E]) {
        if (VEC) {
            const float4 f = reinterpret_cast<const float4 *>(q)[i];
            v[0] = f.x, v[E > 1 ? 1 : 0] = f.y, v[E > 2 ? 2 : 0] = f.z, v[E > 3 ? 3 : 0] = f.w;
        } else {
            v[0] = q[i];
        }
    };
    auto stf = [](float *q, int i, const float (&v)[E]) {
        if (VEC) reinterpret_cast<float4 *>(q)[i] = make_float4(v[0], v[E > 1 ? 1 : 0], v[E > 2 ? 2 : 0], v[E > 3 ? 3 : 0]);
        else q[i] = v[0];
    };
    float sc = 1.f;
    if (sub && p.sub_w) {
        float s2 = 0.f;
        for (int i = tid; i < n; i += NT) {
            float v[E];
            ld(sub, i, v);
#pragma unroll
            for (int e = 0; e < E; e++) s2 += v[e] * v[e];
        }
        sc = 1.0f / sqrtf(block_sum(s2, red) / (float)K + p.eps);
    }
    auto value = [&](int i, float (&v)[E]) { // the new residual
        ld(x, i, v);
        if (!sub) return;
        float s[E];
        ld(sub, i, s);
        if (p.sub_w) {
            float g[E];
            ld(p.sub_w, i, g);
#pragma unroll
            for (int e = 0; e < E; e++) v[e] += s[e] * sc * (p.w_off + g[e]);
        } else {
#pragma unroll
            for (int e = 0; e < E; e++) v[e] += s[e];
        }
    };
    float keep[KEEP][E], ss = 0.f;
#pragma unroll
    for (int t = 0; t < KEEP; t++) {
        const int i = tid + t * NT;
        if (i < n) {
            value(i, keep[t]);
#pragma unroll
            for (int e = 0; e < E; e++) ss += keep[t][e] * keep[t][e];
            if (xo) stf(xo, i, keep[t]);
        }
    }
    for (int i = tid + KEEP * NT; i < n; i += NT) {
        float v[E];
        value(i, v);
#pragma unroll
        for (int e = 0; e < E; e++) ss += v[e] * v[e];
        if (xo) stf(xo, i, v);
    }
    if (!h32 && !h16) return;
    const float s2 = p.norm_w ? 1.0f / sqrtf(block_sum(ss, red) / (float)K + p.eps) : 1.f;
    auto emit = [&](int i, float (&v)[E]) {
        if (p.norm_w) {
            float g[E];
            ld(p.norm_w, i, g);
#pragma unroll
            for (int e = 0; e < E; e++) v[e] *= s2 * (p.w_off + g[e]);
        }
        if (p.gate) {
            float g[E];
            ld(p.gate + r * p.ld_gate, i, g);
#pragma unroll
            for (int e = 0; e < E; e++) v[e] *= kq_sigmoid(g[e]);
        }
        if (h32) stf(h32 + r * ld32, i, v);
        if (h16) {
            uint16_t *o = h16 + r * ld16 + i * E;
            if (VEC) {
                *reinterpret_cast<uint2 *>(o) = make_uint2((uint32_t)kq_f2bf(v[0]) | ((uint32_t)kq_f2bf(v[E > 1 ? 1 : 0]) << 16),
                                                           (uint32_t)kq_f2bf(v[E > 2 ? 2 : 0]) | ((uint32_t)kq_f2bf(v[E > 3 ? 3 : 0]) << 16));
            } else {
                o[0] = kq_f2bf(v[0]);
            }
        }
    };
#pragma unroll
    for (int t = 0; t < KEEP; t++) {
        const int i = tid + t * NT;
        if (i < n) emit(i, keep[t]);
    }
    for (int i = tid + KEEP * NT; i < n; i += NT) {
        float v[E];
        value(i, v);
        emit(i, v);
    }
    if (h16)
        for (int i = K + tid; i < ld16; i += NT) h16[r * ld16 + i] = 0;
}

// ---- convolution -----------------------------------------------------------------------------------
// input of the convolution at position pos0 + t of a sequence: this call's rows, the ring, or zero before the start
__device__ __forceinline__ float conv_in(const float *x, int64_t ldx, const float *ring, int width, int taps, int64_t row0, int t, int pos0,
                                         int c) {
    if (t >= 0) return x[(row0 + t) * ldx + c];
    const int pos = pos0 + t;
    return pos >= 0 ? ring[(int64_t)(pos % taps) * width + c] : 0.f;
}

// v = hi + mid + lo exactly
__device__ __forceinline__ void split3(float v, uint16_t *o, int64_t plane) {
    const uint16_t hi = kq_f2bf(v);
    float rest = v - kq_bf2f(hi);
    const uint16_t mid = kq_f2bf(rest);
    rest -= kq_bf2f(mid);
    o[0] = hi;
    o[plane] = mid;
    o[2 * plane] = kq_f2bf(rest);
}

// grid (channels, runs of CT positions, sequences); a thread keeps the last inputs of its channel in registers.  TAPS:
// 0 = any number of taps, read again for every position
constexpr int CT = 16;
template <int TAPS>
__global__ void __launch_bounds__(NT) causal_conv_kernel(const __grid_constant__ KqRecW w, KqRecState st, const float *x, int64_t ldx,
                                                         int T, const int32_t *pos0_dev, int pos0_val, float *u, int64_t ldu,
                                                         uint16_t *u16, int64_t rows, int m, int mp) {
    KQ_PDL_ENTER();
    const int cp = blockIdx.x * NT + threadIdx.x; // channel in the block-padded layout
    if (cp >= w.blocks * mp) return;
    const int seq = blockIdx.z, b = cp / mp, j = cp % mp, c = b * m + j, t0 = blockIdx.y * CT, t1 = min(T, t0 + CT);
    const int64_t row0 = (int64_t)seq * T, ld16 = (int64_t)w.blocks * mp, plane = rows * ld16;
    if (j >= m) {
        for (int t = t0; t < t1; t++)
            for (int q = 0; q < 3; q++) u16[q * plane + (row0 + t) * ld16 + cp] = 0;
        return;
    }
    const int pos0 = pos0_dev ? *pos0_dev : pos0_val, taps = TAPS ? TAPS : w.taps;
    const float *ring = st.conv + (int64_t)seq * w.taps * w.width;
    const float bias = w.conv_b[c];
    if (TAPS) {
        constexpr int N = TAPS ? TAPS : 1;
        float cw[N], in[N + CT - 1];
#pragma unroll
        for (int k = 0; k < N; k++) cw[k] = w.conv_w[(int64_t)c * N + k];
#pragma unroll
        for (int i = 0; i < N + CT - 1; i++) {
            const int t = t0 - (N - 1) + i;
            in[i] = t < t1 ? conv_in(x, ldx, ring, w.width, N, row0, t, pos0, c) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < CT; i++) {
            if (t0 + i >= t1) break;
            float v = 0.f;
#pragma unroll
            for (int k = 0; k < N; k++) v = fmaf(cw[k], in[i + k], v);
            v += bias;
            u[(row0 + t0 + i) * ldu + c] = v;
            if (u16) split3(v, u16 + (row0 + t0 + i) * ld16 + cp, plane);
        }
    } else {
        for (int t = t0; t < t1; t++) {
            float v = 0.f;
            for (int k = 0; k < taps; k++)
                v = fmaf(w.conv_w[(int64_t)c * taps + k], conv_in(x, ldx, ring, w.width, taps, row0, t - (taps - 1) + k, pos0, c), v);
            v += bias;
            u[(row0 + t) * ldu + c] = v;
            if (u16) split3(v, u16 + (row0 + t) * ld16 + cp, plane);
        }
    }
}

// gates and step of one element: log a = -decay sigmoid(r) softplus(lam); (a, sqrt(1 - a^2) sigmoid(i) u)
__device__ __forceinline__ void rec_coeff(float r, float i, float u, float decay_sp, float &a, float &b) {
    const float la = -decay_sp * kq_sigmoid(r);
    a = expf(la);
    b = sqrtf(-expm1f(2.f * la)) * kq_sigmoid(i) * u;
}

// Prefill in two passes over chunks of `chunk` positions, a thread per channel.  First: coefficients (over the gates, in
// place) and each chunk's map of the state, s -> A s + B.  Second: the state in front of a chunk from the maps of the
// chunks before it, then the recurrence inside the chunk.
constexpr int RC = 128, RCHUNK = 64; // channels per CTA, positions per chunk
__global__ void __launch_bounds__(RC) recurrence_chunks_kernel(const __grid_constant__ KqRecW w, KqRecState st, float *r, float *ig, int64_t ldr, const float *u,
                                                               int64_t ldu, int T, const int32_t *pos0_dev, int pos0_val, int chunk, float *maps) {
    KQ_PDL_ENTER();
    const int c = blockIdx.x * RC + threadIdx.x, k = blockIdx.y, seq = blockIdx.z;
    if (c >= w.width) return;
    const int t0 = k * chunk, t1 = min(T, t0 + chunk);
    const int64_t row0 = (int64_t)seq * T;
    const float dsp = w.decay * kq_softplus(w.lam[c]);
    float A = 1.f, B = 0.f;
#pragma unroll 4
    for (int t = t0; t < t1; t++) {
        const int64_t o = (row0 + t) * ldr + c;
        float a, b;
        rec_coeff(r[o], ig[o], u[(row0 + t) * ldu + c], dsp, a, b);
        r[o] = a;
        ig[o] = b;
        A *= a;
        B = fmaf(a, B, b);
    }
    float *d = maps + ((int64_t)seq * (gridDim.y + 1) + k + 1) * 2 * w.width + c;
    d[0] = A;
    d[w.width] = B;
    if (k == 0) { // entry 0: the state in front of the call, which the second pass may already be replacing when others need it
        const int pos0 = pos0_dev ? *pos0_dev : pos0_val;
        maps[(int64_t)seq * (gridDim.y + 1) * 2 * w.width + c] = pos0 > 0 ? st.s[(int64_t)seq * w.width + c] : 0.f;
    }
}

__global__ void __launch_bounds__(RC) recurrence_scan_kernel(const __grid_constant__ KqRecW w, KqRecState st, const float *a, const float *b, int64_t ldr,
                                                             const float *x, int64_t ldx, const float *y, int64_t ldy, int T,
                                                             const int32_t *pos0_dev, int pos0_val, int chunk, const float *maps, float *z32,
                                                             int64_t ld32, uint16_t *z16, int64_t ld16) {
    KQ_PDL_ENTER();
    const int c = blockIdx.x * RC + threadIdx.x, k = blockIdx.y, seq = blockIdx.z;
    const int t0 = k * chunk, t1 = min(T, t0 + chunk);
    const int64_t row0 = (int64_t)seq * T;
    if (c >= w.width) {
        if (z16 && c < ld16)
            for (int t = t0; t < t1; t++) z16[(row0 + t) * ld16 + c] = 0;
        return;
    }
    const int pos0 = pos0_dev ? *pos0_dev : pos0_val;
    const bool last = k == (int)gridDim.y - 1;
    if (last) // the conv ring: its old entries were last read by the convolution of this call
        for (int t = max(0, T - w.taps); t < T; t++)
            st.conv[((int64_t)seq * w.taps + (pos0 + t) % w.taps) * w.width + c] = x[(row0 + t) * ldx + c];
    const float *d = maps + (int64_t)seq * (gridDim.y + 1) * 2 * w.width + c;
    float s = d[0];
#pragma unroll 8
    for (int j = 1; j <= k; j++) s = fmaf(d[(int64_t)j * 2 * w.width], s, d[((int64_t)j * 2 + 1) * w.width]);
#pragma unroll 8
    for (int t = t0; t < t1; t++) {
        const int64_t o = (row0 + t) * ldr + c;
        s = fmaf(a[o], s, b[o]);
        const float v = s * y[(row0 + t) * ldy + c];
        if (z32) z32[(row0 + t) * ld32 + c] = v;
        if (z16) z16[(row0 + t) * ld16 + c] = kq_f2bf(v);
    }
    if (last) st.s[(int64_t)seq * w.width + c] = s;
}

// ---- one token: grid (row slices of all blocks, sequences); a CTA convolves its block's channels, then each warp
// takes rows of the two gate matrices
constexpr int RROWS = 16; // rows per CTA
__global__ void __launch_bounds__(NT) recurrence_step_kernel(const __grid_constant__ KqRecW w, KqRecState st, const float *x, int64_t ldx,
                                                             const float *y, int64_t ldy, const int32_t *pos_dev, int pos_val, float *z,
                                                             int64_t ldz, int m, int64_t ldw, int slices) {
    extern __shared__ __align__(16) float su[]; // u of the block, zero-padded to 8
    KQ_PDL_TRIGGER();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, seq = blockIdx.y;
    const int b = blockIdx.x / slices, r0 = (blockIdx.x % slices) * RROWS, nck = (m + 7) / 8;
    constexpr int PW = RROWS / (NT / 32); // rows per warp
    uint4 wr[PW], wi[PW]; // the first chunk of every row, requested before the dependency wait
#pragma unroll
    for (int j = 0; j < PW; j++) {
        const int rr = min(r0 + warp * PW + j, m - 1);
        wr[j] = wi[j] = make_uint4(0, 0, 0, 0);
        if (lane < nck) {
            wr[j] = kq_ld_stream(w.ra + ((int64_t)b * m + rr) * ldw + lane * 8);
            wi[j] = kq_ld_stream(w.ri + ((int64_t)b * m + rr) * ldw + lane * 8);
        }
    }
    KQ_PDL_WAIT();
    const int pos = pos_dev ? *pos_dev : pos_val;
    float *ring = st.conv + (int64_t)seq * w.taps * w.width;
    for (int j = tid; j < nck * 8; j += NT) {
        float v = 0.f;
        if (j < m) {
            const int c = b * m + j;
            const float xt = x[seq * ldx + c];
            for (int k = 0; k < w.taps; k++) {
                const int q = pos - (w.taps - 1) + k;
                const float in = k == w.taps - 1 ? xt : q >= 0 ? ring[(int64_t)(q % w.taps) * w.width + c] : 0.f;
                v = fmaf(w.conv_w[(int64_t)c * w.taps + k], in, v);
            }
            v += w.conv_b[c];
            // the slot of the current position is read by nobody in this launch
            if (j >= r0 && j < r0 + RROWS) ring[(int64_t)(pos % w.taps) * w.width + c] = xt;
        }
        su[j] = v;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < PW; j++) {
        const int rr = r0 + warp * PW + j;
        if (rr >= m) break;
        float ar = 0.f, ai = 0.f;
        for (int cidx = lane; cidx < nck; cidx += 32) {
            const uint4 p = cidx == lane ? wr[j] : kq_ld_stream(w.ra + ((int64_t)b * m + rr) * ldw + cidx * 8);
            const uint4 q = cidx == lane ? wi[j] : kq_ld_stream(w.ri + ((int64_t)b * m + rr) * ldw + cidx * 8);
            const float4 a = *reinterpret_cast<const float4 *>(su + cidx * 8), d = *reinterpret_cast<const float4 *>(su + cidx * 8 + 4);
            const float f[8] = {a.x, a.y, a.z, a.w, d.x, d.y, d.z, d.w};
            const uint32_t pw[4] = {p.x, p.y, p.z, p.w}, qw[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
            for (int e = 0; e < 4; e++) {
                ar = fmaf(__uint_as_float(pw[e] << 16), f[2 * e], ar);
                ar = fmaf(__uint_as_float(pw[e] & 0xffff0000u), f[2 * e + 1], ar);
                ai = fmaf(__uint_as_float(qw[e] << 16), f[2 * e], ai);
                ai = fmaf(__uint_as_float(qw[e] & 0xffff0000u), f[2 * e + 1], ai);
            }
        }
        ar = kq_warp_sum(ar);
        ai = kq_warp_sum(ai);
        if (lane == 0) {
            const int c = b * m + rr;
            float a, bb;
            rec_coeff(ar + w.ra_b[c], ai + w.ri_b[c], su[rr], w.decay * kq_softplus(w.lam[c]), a, bb);
            float *sp = st.s + (int64_t)seq * w.width + c;
            const float s = fmaf(a, pos > 0 ? *sp : 0.f, bb);
            *sp = s;
            z[seq * ldz + c] = s * y[seq * ldy + c];
        }
    }
}

} // namespace

b200_status kq_embed_bf16(const uint16_t *W, int64_t ldw, const int32_t *ids, int64_t rows, int K, float scale, float *y,
                          int64_t ldy, cudaStream_t st) {
    KQ_REQUIRE(W && ids && y && rows >= 1 && K >= 1, "embed_bf16: bad call");
    KQ_REQUIRE(rows <= 65535 && ((uintptr_t)y & 15) == 0, "embed_bf16: %lld rows", (long long)rows);
    kq_launch(embed_bf16_kernel, dim3((unsigned)kq_div_up(K, 8 * 128), (unsigned)rows), 128, 0, st, W, ldw, ids, rows, K, scale, y, ldy);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_gather_bf16(const uint16_t *W, const int32_t *ids, int64_t rows, uint16_t *y, int64_t ld, cudaStream_t st) {
    KQ_REQUIRE(W && ids && y && rows >= 1 && rows <= 65535 && ld % 64 == 0, "gather_bf16: bad call");
    kq_launch(gather_bf16_kernel, dim3((unsigned)kq_div_up(ld, 8 * 128), (unsigned)rows), 128, 0, st, W, ids, y, ld);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_norm_prep(const KqNormPrep &p, int64_t rows, int K, float *h32, int64_t ld32, uint16_t *h16, int64_t ld16,
                         cudaStream_t st) {
    KQ_REQUIRE(p.x && rows >= 1 && K >= 1, "norm_prep: bad call");
    const uintptr_t al = (uintptr_t)p.x | (uintptr_t)p.sub | (uintptr_t)p.sub_w | (uintptr_t)p.norm_w | (uintptr_t)p.x_out | (uintptr_t)h32 |
                         (uintptr_t)h16 | (uintptr_t)p.gate;
    const bool vec = K % 4 == 0 && (al & 15) == 0 && ((p.ldx | p.ld_sub | p.ld_out | ld32 | ld16 | p.ld_gate) & 3) == 0;
    if (vec) kq_launch(norm_prep_kernel<true>, (unsigned)rows, NT, 0, st, p, K, h32, ld32, h16, ld16);
    else kq_launch(norm_prep_kernel<false>, (unsigned)rows, NT, 0, st, p, K, h32, ld32, h16, ld16);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

static b200_status check_rec(const KqRecW &w, int n_seq, int T) {
    KQ_REQUIRE(w.width >= 1 && w.blocks >= 1 && w.width % w.blocks == 0 && w.taps >= 1 && n_seq >= 1 && T >= 1, "recurrence: bad shape");
    KQ_REQUIRE((int64_t)n_seq * T <= 65535, "recurrence: %d rows in one call", n_seq * T);
    return B200_OK;
}

b200_status kq_causal_conv(const KqRecW &w, const KqRecState &s, const float *x, int64_t ldx, int n_seq, int T,
                           const int32_t *pos0_dev, int pos0, float *u, int64_t ldu, uint16_t *u16, cudaStream_t st) {
    const b200_status rc = check_rec(w, n_seq, T);
    if (rc != B200_OK) return rc;
    const int m = w.width / w.blocks, mp = u16 ? (int)kq_bf16_ld(m) : m;
    const dim3 grid((unsigned)kq_div_up((int64_t)w.blocks * mp, NT), (unsigned)kq_div_up(T, CT), (unsigned)n_seq);
    const int64_t rows = (int64_t)n_seq * T;
#define GO(N) kq_launch(causal_conv_kernel<N>, grid, NT, 0, st, w, s, x, ldx, T, pos0_dev, pos0, u, ldu, u16, rows, m, mp)
    if (w.taps == 4) GO(4);
    else if (w.taps == 3) GO(3);
    else if (w.taps == 2) GO(2);
    else GO(0);
#undef GO
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

size_t kq_recurrence_scratch_bytes(int width, int rows, int n_seq) {
    return (size_t)(rows / RCHUNK + 2 * std::min(n_seq, rows) + 1) * 2 * width * 4;
}

b200_status kq_linear_recurrence(const KqRecW &w, const KqRecState &s, float *r, float *i, int64_t ldr, const float *u,
                                 int64_t ldu, const float *x, int64_t ldx, const float *y, int64_t ldy, int n_seq, int T,
                                 const int32_t *pos0_dev, int pos0, float *z32, int64_t ld32, uint16_t *z16, int64_t ld16,
                                 float *scratch, size_t scratch_bytes, cudaStream_t st) {
    const b200_status rc = check_rec(w, n_seq, T);
    if (rc != B200_OK) return rc;
    const unsigned chunks = (unsigned)kq_div_up(T, RCHUNK);
    KQ_REQUIRE(scratch && scratch_bytes >= (size_t)n_seq * (chunks + 1) * 2 * w.width * 4, "recurrence: scratch");
    const int64_t cols = z16 ? std::max<int64_t>(w.width, ld16) : w.width;
    kq_launch(recurrence_chunks_kernel, dim3((unsigned)kq_div_up(w.width, RC), chunks, (unsigned)n_seq), RC, 0, st, w, s, r, i, ldr, u, ldu, T, pos0_dev,
              pos0, RCHUNK, scratch);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    kq_launch(recurrence_scan_kernel, dim3((unsigned)kq_div_up(cols, RC), chunks, (unsigned)n_seq), RC, 0, st, w, s, r, i, ldr, x, ldx, y, ldy, T,
              pos0_dev, pos0, RCHUNK, scratch, z32, ld32, z16, ld16);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_recurrence_step(const KqRecW &w, const KqRecState &s, const float *x, int64_t ldx, const float *y,
                               int64_t ldy, int n_seq, const int32_t *pos_dev, int pos, float *z, int64_t ldz, cudaStream_t st) {
    const b200_status rc = check_rec(w, n_seq, 1);
    if (rc != B200_OK) return rc;
    const int m = w.width / w.blocks, slices = (int)kq_div_up(m, RROWS);
    const size_t smem = (size_t)kq_pad(m, 8) * 4;
    KQ_REQUIRE(smem <= 48 * 1024, "recurrence: blocks of %d channels", m);
    kq_launch(recurrence_step_kernel, dim3((unsigned)(w.blocks * slices), (unsigned)n_seq), NT, smem, st, w, s, x, ldx, y, ldy, pos_dev, pos, z, ldz,
              m, kq_bf16_ld(m), slices);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
