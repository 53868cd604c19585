// Matrix-vector products for 1..8 rows of f32 activations and bf16 weights: the decode projections of a 16-bit
// model.  The products are f32 throughout (a bf16 weight is exact in f32), so the same kernels serve the 32-bit
// mode.
//
// Every CTA owns an equal share of the output rows (to within one row) and all its warps split K: a thread
// reads the 16-byte chunks tid, tid + 256, ... of four rows at a time straight from global memory, the activations
// sit in shared memory as two planes of float4 (elements 0..3 and 4..7 of each chunk), so that a warp's reads are
// free of bank conflicts.  The four rows' partial sums are reduced across the warp in six shuffles, the eight
// warps' through shared memory once per 64 rows.  The prologue can add a normed sub-layer output to the
// residual and norm the result (every CTA does that for itself; CTA 0 also leaves the new residual), the
// first weights are requested before the dependency wait.
#include "kq_gemv_grouped.cuh"

#include <algorithm>
#include <stdlib.h>

namespace {

constexpr int NT = 256, NW = NT / 32, SB = 64; // threads, warps, rows between two combines
constexpr int MAX_X_BYTES = 192 * 1024;       // activations in shared memory, next to 32 KB of partial sums at 8 rows

struct GemvParams {
    KqDense c;
    KqNormPrep p;
    int32_t V;   // rows in all (a gate / up pair is two), in the order they are walked
    int32_t nck; // 16-byte chunks per weight row
};

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

// walked row v -> (segment, row); gate / up rows alternate
__device__ __forceinline__ void locate(const GemvParams &p, int v, int &seg, int &row) {
    if (p.c.glu) {
        seg = v & 1;
        row = v >> 1;
        return;
    }
    seg = 0;
    row = v;
    if (p.c.nseg > 1 && row >= p.c.seg[0].n_rows) {
        seg = 1;
        row -= p.c.seg[0].n_rows;
        if (p.c.nseg > 2 && row >= p.c.seg[1].n_rows) {
            seg = 2;
            row -= p.c.seg[1].n_rows;
        }
    }
}

// brings n floats into this SM's L1 without waiting for them
__device__ __forceinline__ void touch(const float *p, int n) {
    for (int i = threadIdx.x * 8; i < n; i += NT * 8) asm volatile("{\n\t.reg .f32 t;\n\tld.global.ca.f32 t, [%0];\n\t}" ::"l"(p + i));
}

template <int M>
__global__ void __launch_bounds__(NT, M <= 2 ? 4 : 2) gemv_bf16_kernel(const __grid_constant__ GemvParams p) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float part[2][NW][SB][M];
    __shared__ float red[NW];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int nck = p.nck, K = p.c.K, step = p.c.glu ? 2 : 1;
    const int64_t units = p.V / step;
    const int v0 = (int)(units * blockIdx.x / gridDim.x) * step, v1 = (int)(units * (blockIdx.x + 1) / gridDim.x) * step;
    KQ_PDL_TRIGGER();

    auto row_ptr = [&](int v) {
        int s, r;
        locate(p, min(v, p.V - 1), s, r);
        return reinterpret_cast<const uint4 *>(kq_dense_w(p.c, s) + (int64_t)r * p.c.ldw);
    };
    // first weights of this CTA: they depend on nothing
    uint4 w[4][2];
    const uint4 *wp[4];
    auto load = [&](int i, int n) { // n: rows of the batch that are this CTA's
#pragma unroll
        for (int r = 0; r < 4; r++)
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int c = i + j * NT;
                w[r][j] = c < nck && r < n ? kq_ld_stream(wp[r] + c) : make_uint4(0, 0, 0, 0);
            }
    };
    if (v0 < v1) {
#pragma unroll
        for (int r = 0; r < 4; r++) wp[r] = row_ptr(v0 + r);
        load(tid, v1 - v0);
    }
    if (p.p.sub_w) touch(p.p.sub_w, K);
    if (p.p.norm_w) touch(p.p.norm_w, K);
    KQ_PDL_WAIT();

    // ---- activations
    float4 *pl = reinterpret_cast<float4 *>(sm); // [M][2][nck]
    const bool vec = (p.p.ldx & 3) == 0 && (p.p.ld_sub & 3) == 0 && (p.p.ld_out & 3) == 0 &&
                     (p.p.ld_gate & 3) == 0 && (((uintptr_t)p.p.x | (uintptr_t)p.p.sub | (uintptr_t)p.p.x_out | (uintptr_t)p.p.gate) & 15) == 0;
    const int n4 = nck * 2;
#pragma unroll 1
    for (int m = 0; m < M; m++) {
        float4 *px = pl + (int64_t)m * 2 * nck;
        const float *x = p.p.x + m * p.p.ldx;
        float ss = 0.f;
        if (p.p.sub) {
            const float *sub = p.p.sub + m * p.p.ld_sub;
            float sc = 1.f;
            if (p.p.sub_w) {
                float s2 = 0.f;
                for (int i = tid; i < n4; i += NT) { // x comes along: its round trip is over when it is needed
                    const float4 v = kq_load4(sub, 4 * i, K, vec);
                    px[(i & 1) * nck + (i >> 1)] = kq_load4(x, 4 * i, K, vec);
                    s2 += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                }
                sc = 1.0f / sqrtf(block_sum(s2, red) / (float)K + p.p.eps);
            }
            for (int i = tid; i < n4; i += NT) {
                const float4 a = p.p.sub_w ? px[(i & 1) * nck + (i >> 1)] : kq_load4(x, 4 * i, K, vec), b = kq_load4(sub, 4 * i, K, vec);
                float4 g = make_float4(1.f, 1.f, 1.f, 1.f);
                if (p.p.sub_w) {
                    g = kq_load4(p.p.sub_w, 4 * i, K, true);
                    g.x += p.p.w_off, g.y += p.p.w_off, g.z += p.p.w_off, g.w += p.p.w_off;
                }
                float4 v = make_float4(a.x + b.x * sc * g.x, a.y + b.y * sc * g.y, a.z + b.z * sc * g.z, a.w + b.w * sc * g.w);
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                px[(i & 1) * nck + (i >> 1)] = v;
                if (p.p.x_out && blockIdx.x == 0) {
                    float *o = p.p.x_out + m * p.p.ld_out + 4 * i;
                    if (vec && 4 * i + 3 < K) *reinterpret_cast<float4 *>(o) = v;
                    else {
                        if (4 * i < K) o[0] = v.x;
                        if (4 * i + 1 < K) o[1] = v.y;
                        if (4 * i + 2 < K) o[2] = v.z;
                        if (4 * i + 3 < K) o[3] = v.w;
                    }
                }
            }
        } else {
            for (int i = tid; i < n4; i += NT) {
                const float4 v = kq_load4(x, 4 * i, K, vec);
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                px[(i & 1) * nck + (i >> 1)] = v;
            }
        }
        if (p.p.norm_w) {
            const float sc = 1.0f / sqrtf(block_sum(ss, red) / (float)K + p.p.eps);
            for (int i = tid; i < n4; i += NT) {
                const float4 g = kq_load4(p.p.norm_w, 4 * i, K, true);
                float4 v = px[(i & 1) * nck + (i >> 1)];
                v.x *= sc * (p.p.w_off + g.x), v.y *= sc * (p.p.w_off + g.y);
                v.z *= sc * (p.p.w_off + g.z), v.w *= sc * (p.p.w_off + g.w);
                px[(i & 1) * nck + (i >> 1)] = v;
            }
        }
        if (p.p.gate) {
            const float *gate = p.p.gate + m * p.p.ld_gate;
            for (int i = tid; i < n4; i += NT) { // the elements this thread wrote above
                const float4 g = kq_load4(gate, 4 * i, K, vec);
                float4 v = px[(i & 1) * nck + (i >> 1)];
                v.x *= kq_sigmoid(g.x), v.y *= kq_sigmoid(g.y), v.z *= kq_sigmoid(g.z), v.w *= kq_sigmoid(g.w);
                px[(i & 1) * nck + (i >> 1)] = v;
            }
        }
    }
    __syncthreads();

    // ---- rows; the first weights of the next four are requested before this group's sums are reduced
    int buf = 0;
    for (int vb = v0; vb < v1; vb += SB, buf ^= 1) {
        const int ve = min(v1, vb + SB);
        for (int v = vb; v < ve; v += 4) {
            float acc[4][M];
#pragma unroll
            for (int r = 0; r < 4; r++)
#pragma unroll
                for (int m = 0; m < M; m++) acc[r][m] = 0.f;
            for (int i = tid; i < nck; i += 2 * NT) {
                if (i != tid) load(i, v1 - v);
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    const int c = i + j * NT;
                    if (c < nck) {
#pragma unroll
                        for (int m = 0; m < M; m++) {
                            const float4 a = pl[(m * 2) * nck + c], b = pl[(m * 2 + 1) * nck + c];
#pragma unroll
                            for (int r = 0; r < 4; r++) acc[r][m] = kq_dot8(w[r][j], a, b, acc[r][m]);
                        }
                    }
                }
            }
            if (v + 4 < v1) {
#pragma unroll
                for (int r = 0; r < 4; r++) wp[r] = row_ptr(v + 4 + r);
                load(tid, v1 - v - 4);
            }
            // four rows across the warp: after two exchanges a lane holds one row's sum over four lanes' worth
#pragma unroll
            for (int m = 0; m < M; m++) {
                const bool h16 = lane & 16, h8 = lane & 8;
                const float s0 = __shfl_xor_sync(0xffffffffu, h16 ? acc[0][m] : acc[2][m], 16);
                const float s1 = __shfl_xor_sync(0xffffffffu, h16 ? acc[1][m] : acc[3][m], 16);
                const float a0 = (h16 ? acc[2][m] : acc[0][m]) + s0, a1 = (h16 ? acc[3][m] : acc[1][m]) + s1;
                float t = (h8 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, h8 ? a0 : a1, 8);
                t += __shfl_xor_sync(0xffffffffu, t, 4);
                t += __shfl_xor_sync(0xffffffffu, t, 2);
                t += __shfl_xor_sync(0xffffffffu, t, 1);
                if ((lane & 7) == 0) part[buf][warp][v - vb + ((lane >> 4) & 1) * 2 + ((lane >> 3) & 1)][m] = t;
            }
        }
        __syncthreads();
        const int nout = (ve - vb) / step * M;
        for (int t = tid; t < nout; t += NT) {
            const int u = t / M, m = t % M, vl = u * step;
            float s = 0.f, s2 = 0.f;
#pragma unroll
            for (int i = 0; i < NW; i++) s += part[buf][i][vl][m];
            int sg, r;
            locate(p, vb + vl, sg, r);
            if (p.c.glu) {
#pragma unroll
                for (int i = 0; i < NW; i++) s2 += part[buf][i][vl + 1][m];
                kq_dense_put(p.c.seg[0], m, r, kq_glu(p.c, s, s2));
            } else {
                kq_dense_store(p.c, kq_dense_seg(p.c, sg), m, r, 0, s);
            }
        }
    }
}

template <int M>
__global__ void __launch_bounds__(NT) gemv_grouped_bf16_kernel(const __grid_constant__ KqGrouped p) {
    KQ_PDL_TRIGGER();
    kq_grouped_rows<M>(p, (int64_t)blockIdx.x * NW + (threadIdx.x >> 5), threadIdx.x & 31);
}

template <int M>
b200_status launch_gemv(const GemvParams &p, size_t smem, cudaStream_t st) {
    static bool attr[16];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 16 || !attr[dev]) {
        KQ_CUDA(cudaFuncSetAttribute(gemv_bf16_kernel<M>, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_X_BYTES));
        if (dev >= 0 && dev < 16) attr[dev] = true;
    }
    static int mul = -1; // B200_GEMV16_CTAS: CTAs per SM of the decode projections
    if (mul < 0) {
        const char *v = getenv("B200_GEMV16_CTAS");
        mul = v ? std::max(1, atoi(v)) : 4;
    }
    const int64_t units = p.V / (p.c.glu ? 2 : 1);
    const int64_t want = std::max<int64_t>(1, kq_div_up(units * (p.c.glu ? 2 : 1), 4));
    const unsigned grid = (unsigned)std::min<int64_t>(want, (int64_t)kq_sm_count() * mul);
    kq_launch(gemv_bf16_kernel<M>, grid, NT, smem, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

} // namespace

b200_status kq_gemv_bf16(const KqDense &c, const KqNormPrep &pr, cudaStream_t st) {
    KQ_REQUIRE(c.M >= 1 && c.nseg >= 1 && c.nseg <= 3 && c.groups == 1 && c.K >= 1, "gemv_bf16: bad call");
    KQ_REQUIRE(c.ldw % 64 == 0 && c.ldw >= c.K, "gemv_bf16: weight rows must be padded to 64 elements");
    const int nck = (int)kq_div_up(c.K, 8);
    const int64_t row_smem = (int64_t)nck * 32;
    const int cap = (int)std::min<int64_t>(8, MAX_X_BYTES / row_smem);
    if (cap < 1) {
        kq_set_error("gemv_bf16: rows of %d values do not fit in shared memory", c.K);
        return B200_ERR_UNSUPPORTED;
    }
    for (int m0 = 0; m0 < c.M;) {
        const int left = c.M - m0;
        const int m = left >= 8 && cap >= 8 ? 8 : left >= 4 && cap >= 4 ? 4 : left >= 2 && cap >= 2 ? 2 : 1;
        GemvParams p;
        p.c = kq_rows_of(c, m0, m);
        p.p = pr;
        p.p.x += m0 * pr.ldx;
        if (pr.sub) p.p.sub += m0 * pr.ld_sub;
        if (pr.x_out) p.p.x_out += m0 * pr.ld_out;
        if (pr.gate) p.p.gate += m0 * pr.ld_gate;
        p.nck = nck;
        p.V = 0;
        for (int i = 0; i < c.nseg; i++) p.V += c.seg[i].n_rows;
        b200_status rc;
        const size_t smem = (size_t)(row_smem * m);
        switch (m) {
        case 1: rc = launch_gemv<1>(p, smem, st); break;
        case 2: rc = launch_gemv<2>(p, smem, st); break;
        case 4: rc = launch_gemv<4>(p, smem, st); break;
        default: rc = launch_gemv<8>(p, smem, st); break;
        }
        if (rc != B200_OK) return rc;
        m0 += m;
    }
    return B200_OK;
}

b200_status kq_gemv_grouped_bf16(const KqDense &c, const float *x, int64_t ldx, cudaStream_t st) {
    KQ_REQUIRE(c.M >= 1 && c.nseg >= 1 && c.nseg <= 3 && c.groups >= 1 && !c.glu, "gemv_grouped_bf16: bad call");
    for (int m0 = 0; m0 < c.M;) {
        const int left = c.M - m0, m = left >= 4 ? 4 : left >= 2 ? 2 : 1;
        const KqGrouped p = kq_grouped_params(kq_rows_of(c, m0, m), x + m0 * ldx, ldx);
        const unsigned grid = (unsigned)kq_div_up((int64_t)p.quads * c.groups * c.nseg, NW);
        if (m == 4) kq_launch(gemv_grouped_bf16_kernel<4>, grid, NT, 0, st, p);
        else if (m == 2) kq_launch(gemv_grouped_bf16_kernel<2>, grid, NT, 0, st, p);
        else kq_launch(gemv_grouped_bf16_kernel<1>, grid, NT, 0, st, p);
        KQ_COUNT_LAUNCH();
        KQ_LAUNCH_CHECK();
        m0 += m;
    }
    return B200_OK;
}
