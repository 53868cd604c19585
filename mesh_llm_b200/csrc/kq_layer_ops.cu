// Ops of layers with 16-bit weights that are neither projections nor attention: scaled embedding rows, the
// residual / norm prologue as a kernel of its own, the per-channel causal convolution and the gated diagonal
// linear recurrence (prefill as a chunked scan, decode as one launch with the convolution and the gates).
// All arithmetic is f32.
#include "kq_dense.cuh"

#include <algorithm>

namespace {

__global__ void embed_bf16_kernel(const uint16_t *W, int64_t ldw, const int32_t *ids, int64_t rows, int K, float scale, float *y,
                                  int64_t ldy) {
    KQ_PDL_ENTER();
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= rows * K) return;
    const int64_t r = i / K;
    const int k = (int)(i % K);
    y[r * ldy + k] = kq_bf2f(W[(int64_t)ids[r] * ldw + k]) * scale;
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

__global__ void __launch_bounds__(NT) causal_conv_kernel(const __grid_constant__ KqRecW w, KqRecState st, const float *x, int64_t ldx,
                                                         int T, const int32_t *pos0_dev, int pos0_val, float *u, int64_t ldu,
                                                         uint16_t *u16, int64_t rows, int m, int mp) {
    KQ_PDL_ENTER();
    const int64_t row = blockIdx.y;
    const int cp = blockIdx.x * NT + threadIdx.x; // channel in the block-padded layout
    if (cp >= w.blocks * mp) return;
    const int b = cp / mp, j = cp % mp, c = b * m + j;
    const int pos0 = pos0_dev ? *pos0_dev : pos0_val, seq = (int)(row / T), t = (int)(row % T);
    float v = 0.f;
    if (j < m) {
        const float *ring = st.conv + (int64_t)seq * w.taps * w.width;
        for (int k = 0; k < w.taps; k++)
            v = fmaf(w.conv_w[(int64_t)c * w.taps + k], conv_in(x, ldx, ring, w.width, w.taps, (int64_t)seq * T, t - (w.taps - 1) + k, pos0, c), v);
        v += w.conv_b[c];
        u[row * ldu + c] = v;
    }
    if (u16) { // v = hi + mid + lo exactly
        const int64_t ld = (int64_t)w.blocks * mp, i = row * ld + cp;
        const uint16_t hi = kq_f2bf(v);
        float rest = v - kq_bf2f(hi);
        const uint16_t mid = kq_f2bf(rest);
        rest -= kq_bf2f(mid);
        u16[i] = hi;
        u16[rows * ld + i] = mid;
        u16[2 * rows * ld + i] = kq_f2bf(rest);
    }
}

// gates and step of one element: log a = -decay sigmoid(r) softplus(lam); (a, sqrt(1 - a^2) sigmoid(i) u)
__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ void rec_coeff(float r, float i, float u, float decay_sp, float &a, float &b) {
    const float la = -decay_sp * kq_sigmoid(r);
    a = expf(la);
    b = sqrtf(-expm1f(2.f * la)) * kq_sigmoid(i) * u;
}

constexpr int SC = 32, SW = 16; // channels per CTA, time chunks (one warp each)
__global__ void __launch_bounds__(SC * SW) linear_recurrence_kernel(const __grid_constant__ KqRecW w, KqRecState st, float *r, float *ig,
                                                                    int64_t ldr, const float *u, int64_t ldu, const float *x,
                                                                    int64_t ldx, const float *y, int64_t ldy, int T,
                                                                    const int32_t *pos0_dev, int pos0_val, float *z32, int64_t ld32,
                                                                    uint16_t *z16, int64_t ld16) {
    KQ_PDL_ENTER();
    __shared__ float sa[SW][SC], sb[SW][SC];
    const int lane = threadIdx.x & 31, k = threadIdx.x >> 5, seq = blockIdx.y;
    const int c = blockIdx.x * SC + lane;
    const int pos0 = pos0_dev ? *pos0_dev : pos0_val;
    const bool ok = c < w.width;
    const int chunk = (T + SW - 1) / SW, t0 = min(T, k * chunk), t1 = min(T, t0 + chunk);
    const int64_t row0 = (int64_t)seq * T;
    const float dsp = ok ? w.decay * softplus(w.lam[c]) : 0.f;
    float A = 1.f, B = 0.f;
    if (ok)
        for (int t = t0; t < t1; t++) {
            const int64_t o = (row0 + t) * ldr + c;
            float a, b;
            rec_coeff(r[o], ig[o], u[(row0 + t) * ldu + c], dsp, a, b);
            r[o] = a;
            ig[o] = b;
            A *= a;
            B = fmaf(a, B, b);
        }
    sa[k][lane] = A;
    sb[k][lane] = B;
    // the conv ring: its old entries were last read by the convolution of this call
    if (ok)
        for (int t = max(0, T - w.taps) + k; t < T; t += SW)
            st.conv[((int64_t)seq * w.taps + (pos0 + t) % w.taps) * w.width + c] = x[(row0 + t) * ldx + c];
    float s = ok && pos0 > 0 ? st.s[(int64_t)seq * w.width + c] : 0.f;
    __syncthreads();
    for (int j = 0; j < k; j++) s = fmaf(sa[j][lane], s, sb[j][lane]);
    if (ok) {
        for (int t = t0; t < t1; t++) {
            const int64_t o = (row0 + t) * ldr + c;
            s = fmaf(r[o], s, ig[o]);
            const float v = s * y[(row0 + t) * ldy + c];
            if (z32) z32[(row0 + t) * ld32 + c] = v;
            if (z16) z16[(row0 + t) * ld16 + c] = kq_f2bf(v);
        }
    } else if (z16 && c < ld16) {
        for (int t = t0; t < t1; t++) z16[(row0 + t) * ld16 + c] = 0;
    }
    if (ok && t1 == T && t0 < T) st.s[(int64_t)seq * w.width + c] = s;
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
            rec_coeff(ar + w.ra_b[c], ai + w.ri_b[c], su[rr], w.decay * softplus(w.lam[c]), a, bb);
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
    kq_launch(embed_bf16_kernel, (unsigned)kq_div_up(rows * K, 256), 256, 0, st, W, ldw, ids, rows, K, scale, y, ldy);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_norm_prep(const KqNormPrep &p, int64_t rows, int K, float *h32, int64_t ld32, uint16_t *h16, int64_t ld16,
                         cudaStream_t st) {
    KQ_REQUIRE(p.x && rows >= 1 && K >= 1, "norm_prep: bad call");
    const uintptr_t al = (uintptr_t)p.x | (uintptr_t)p.sub | (uintptr_t)p.sub_w | (uintptr_t)p.norm_w | (uintptr_t)p.x_out | (uintptr_t)h32 |
                         (uintptr_t)h16;
    const bool vec = K % 4 == 0 && (al & 15) == 0 && ((p.ldx | p.ld_sub | p.ld_out | ld32 | ld16) & 3) == 0;
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
    kq_launch(causal_conv_kernel, dim3((unsigned)kq_div_up((int64_t)w.blocks * mp, NT), (unsigned)(n_seq * T)), NT, 0, st, w, s, x, ldx, T, pos0_dev,
              pos0, u, ldu, u16, (int64_t)n_seq * T, m, mp);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_linear_recurrence(const KqRecW &w, const KqRecState &s, float *r, float *i, int64_t ldr, const float *u,
                                 int64_t ldu, const float *x, int64_t ldx, const float *y, int64_t ldy, int n_seq, int T,
                                 const int32_t *pos0_dev, int pos0, float *z32, int64_t ld32, uint16_t *z16, int64_t ld16,
                                 cudaStream_t st) {
    const b200_status rc = check_rec(w, n_seq, T);
    if (rc != B200_OK) return rc;
    const int64_t cols = z16 ? std::max<int64_t>(w.width, ld16) : w.width;
    kq_launch(linear_recurrence_kernel, dim3((unsigned)kq_div_up(cols, SC), (unsigned)n_seq), SC * SW, 0, st, w, s, r, i, ldr, u, ldu, x, ldx, y, ldy,
              T, pos0_dev, pos0, z32, ld32, z16, ld16);
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
