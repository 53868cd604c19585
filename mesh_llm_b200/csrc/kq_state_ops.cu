// Recurrences whose state is a matrix per head, all in f32: linear attention under a fixed decay, and the delta rule with a
// decay per key channel behind short convolutions.
//
// Prompts, in blocks of four tokens.  Written out over a block, with S the state in front of it, G_j the product of the
// block's decays up to token j and P_ij that of the decays behind token i up to token j,
//   u_j = beta_j (v_j - S^T (G_j k_j) - sum_(i<j) A_ji u_i),   A_ji = k_j . (P_ij k_i)
//   o_j = S^T (G_j q_j) + sum_(i<=j) B_ji u_i,                 B_ji = q_j . (P_ij k_i)
//   S  <- G_4 S + sum_i (P_i4 k_i) u_i^T
// with products of decays only, no quotients.  One launch makes every block's vectors and scalars (convolution, SiLU, unit
// norms, decays) and leaves them as one record per block and head; the second walks the blocks with the state in
// registers, so that eight products with the state wait for one reduction and a record is read from shared memory once
// per pair of columns.  A thread holds some key dimensions of two columns (value dimensions).  A warp of its own brings the
// records by bulk copies into a ring, the others walk through it without waiting for one another; every wait is bounded.
// The fixed decay is the same with u = v and scalar products of decays.  (kq_state_chunk.cu has the form on tensor cores.)
// A decode step is one launch: a CTA per head convolves, norms, works out the low-rank decays and gates, updates the
// state and norms and gates the head's output.
#include "kq_gemv_grouped.cuh"
#include "kq_state.cuh"

#include <algorithm>

namespace {

__device__ int g_state_error;

__device__ __forceinline__ float sum8(float v) { // over the eight lanes of a column
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 1);
}
// ---- records of blocks of tokens -----------------------------------------------------------------------
constexpr int BT = 4, TOK_NT = 128, TOK_NW = TOK_NT / 32, RUN = 4; // tokens per block, blocks a warp walks
constexpr int N_SCALAR = 32;                                       // beta (4), A (6, from 4), B (four rows of four, from 12)
// floats of a record: decayed k, decayed q, k towards the block's end (four vectors each) and the block's decay; fixed decay: the
// middle two
__host__ __device__ constexpr int rec_floats(int dp, bool delta) { return (delta ? 13 : 8) * dp + N_SCALAR; }

struct TokParams {
    KqMatState m;
    KqStateIn in;
    float *rec, *val; // [seq][block][head][record], [seq][block][head][vdim][BT]
    int32_t T, pos0, blocks, head_ctas;
    const int32_t *pos0_dev;
};

// The convolution of channels lane + 32 c (< n) at the BT positions from t0 on, with SiLU; zero past the call's rows.  Four taps: what
// is read is requested by the constructor.
template <int C>
struct ConvBlock {
    float in[C][BT + 3];
    __device__ __forceinline__ KqConvIn input(const TokParams &p, const float *x, int64_t channel0, int64_t seq, int pos0, int d) const {
        const int64_t channels = kq_state_channels(p.m);
        return {x + seq * p.T * p.in.ld + d, p.in.ld, p.m.taps ? p.m.conv + seq * p.m.taps * channels + channel0 + d : nullptr, channels, p.m.taps, pos0};
    }
    __device__ __forceinline__ ConvBlock(const TokParams &p, const float *x, int64_t channel0, int n, int64_t seq, int t0, int pos0, int lane) {
        if (p.m.taps != 4) return;
        if (t0 >= 3 && t0 + BT <= p.T) { // all of this call
            const float *r = x + (seq * p.T + t0 - 3) * p.in.ld + lane;
#pragma unroll
            for (int k = 0; k < BT + 3; k++)
#pragma unroll
                for (int c = 0; c < C; c++) in[c][k] = lane + 32 * c < n ? r[k * p.in.ld + 32 * c] : 0.f;
        } else {
#pragma unroll
            for (int c = 0; c < C; c++) {
                const KqConvIn ci = input(p, x, channel0, seq, pos0, lane + 32 * c);
#pragma unroll
                for (int k = 0; k < BT + 3; k++) in[c][k] = lane + 32 * c < n && t0 - 3 + k < p.T ? ci.at(t0 - 3 + k) : 0.f;
            }
        }
    }
    __device__ __forceinline__ void run(const TokParams &p, const float *x, const float *w, int64_t channel0, int n, int64_t seq, int t0, int pos0, int lane,
                                        float (&out)[BT][C]) const {
        const int taps = p.m.taps;
#pragma unroll
        for (int c = 0; c < C; c++) {
            const int d = lane + 32 * c;
            if (taps == 4) {
                const float4 cw = d < n ? *reinterpret_cast<const float4 *>(w + d * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int j = 0; j < BT; j++) out[j][c] = fmaf(cw.w, in[c][j + 3], fmaf(cw.z, in[c][j + 2], fmaf(cw.y, in[c][j + 1], cw.x * in[c][j])));
            } else {
                const KqConvIn ci = input(p, x, channel0, seq, pos0, d);
#pragma unroll
                for (int j = 0; j < BT; j++) {
                    float s = 0.f;
                    if (d < n && t0 + j < p.T) {
                        if (taps == 0) s = ci.at(t0 + j);
                        for (int k = 0; k < taps; k++) s = fmaf(w[(int64_t)d * taps + k], ci.at(t0 + j - (taps - 1) + k), s);
                    }
                    out[j][c] = s;
                }
            }
#pragma unroll
            for (int j = 0; j < BT; j++) out[j][c] = t0 + j < p.T ? kq_silu(out[j][c]) : 0.f;
        }
    }
};

// grid (heads / warps, then values, runs of blocks, sequences)
template <int C, bool DELTA>
__global__ void __launch_bounds__(TOK_NT, C > 4 ? 2 : DELTA ? 3 : 6) state_tokens_kernel(const __grid_constant__ TokParams p) {
    KQ_PDL_ENTER();
    constexpr int DP = 32 * C, REC = rec_floats(DP, DELTA);
    const KqMatState &m = p.m;
    const int lane = threadIdx.x & 31, b0 = blockIdx.y * RUN, b1 = min(p.blocks, b0 + RUN);
    const int64_t seq = blockIdx.z, nq = (int64_t)m.kv_heads * m.dim;
    const int pos0 = p.pos0_dev ? *p.pos0_dev : p.pos0;
    if ((int)blockIdx.x >= p.head_ctas) { // a lane per value channel
        const int64_t c0 = ((int64_t)(blockIdx.x - p.head_ctas) * TOK_NW + (threadIdx.x >> 5)) * 32, nv = (int64_t)m.heads * m.vdim;
        if (c0 >= nv) return;
        const int n = (int)min((int64_t)32, nv - c0);
        for (int b = b0; b < b1; b++) {
            float v[BT][1];
            const ConvBlock<1> cv(p, p.in.v + c0, 2 * nq + c0, n, seq, b * BT, pos0, lane);
            cv.run(p, p.in.v + c0, m.conv_v + c0 * m.taps, 2 * nq + c0, n, seq, b * BT, pos0, lane, v);
            if (lane < n) *reinterpret_cast<float4 *>(p.val + (((seq * p.blocks + b) * nv) + c0 + lane) * BT) = make_float4(v[0][0], v[1][0], v[2][0], v[3][0]);
        }
        return;
    }
    const int h = blockIdx.x * TOK_NW + (threadIdx.x >> 5);
    if (h >= m.heads) return;
    const int kh = h / (m.heads / m.kv_heads);
    const int64_t cq = (int64_t)kh * m.dim, cg = (int64_t)h * m.dim;
    float bias[C];
#pragma unroll
    for (int c = 0; c < C; c++) bias[c] = DELTA && lane + 32 * c < m.dim ? m.dt_bias[cg + lane + 32 * c] : 0.f;
    const float a = DELTA ? expf(m.a_log[h]) : 0.f, decay = DELTA ? 1.f : m.decay[h];
    const float q_scale = DELTA ? 1.0f / sqrtf((float)m.dim) : 1.f;
    for (int b = b0; b < b1; b++) {
        const int t0 = b * BT;
        float *rec = p.rec + ((seq * p.blocks + b) * m.heads + h) * (int64_t)REC;
        float q[BT][C], k[BT][C], g[BT][C];
        {
            const ConvBlock<C> a(p, p.in.q + cq, cq, m.dim, seq, t0, pos0, lane), b(p, p.in.k + cq, nq + cq, m.dim, seq, t0, pos0, lane);
            if (DELTA) {
#pragma unroll
                for (int j = 0; j < BT; j++)
#pragma unroll
                    for (int c = 0; c < C; c++)
                        g[j][c] = lane + 32 * c < m.dim && t0 + j < p.T ? p.in.z[(seq * p.T + t0 + j) * p.in.ldz + cg + lane + 32 * c] : 0.f;
            }
            a.run(p, p.in.q + cq, m.conv_q + cq * m.taps, cq, m.dim, seq, t0, pos0, lane, q);
            b.run(p, p.in.k + cq, m.conv_k + cq * m.taps, nq + cq, m.dim, seq, t0, pos0, lane, k);
        }
        if (DELTA) {
            float ss[2 * BT];
#pragma unroll
            for (int j = 0; j < BT; j++) {
                ss[j] = ss[BT + j] = 0.f;
#pragma unroll
                for (int c = 0; c < C; c++) ss[j] = fmaf(q[j][c], q[j][c], ss[j]), ss[BT + j] = fmaf(k[j][c], k[j][c], ss[BT + j]);
            }
            kq_spread_sum<2 * BT, 32>(ss, lane); // lane holds sum lane / 4
            const float sc = 1.0f / sqrtf(ss[0] + 1e-6f);
#pragma unroll
            for (int j = 0; j < BT; j++) {
                const float sq = __shfl_sync(0xffffffffu, sc, 4 * j) * q_scale, sk = __shfl_sync(0xffffffffu, sc, 4 * (BT + j));
#pragma unroll
                for (int c = 0; c < C; c++) {
                    const int d = lane + 32 * c;
                    q[j][c] *= sq, k[j][c] *= sk;
                    g[j][c] = d < m.dim && t0 + j < p.T ? expf(-a * kq_softplus(g[j][c] + bias[c])) : 1.f;
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < BT; j++)
#pragma unroll
                for (int c = 0; c < C; c++) g[j][c] = t0 + j < p.T ? decay : 1.f;
        }
        float dot[16]; // A21 A31 A32 A41 A42 A43, B11 B21 B22 B31 B32 B33 B41 B42 B43 B44
#pragma unroll
        for (int i = 0; i < 16; i++) dot[i] = 0.f;
#pragma unroll
        for (int c = 0; c < C; c++) {
            const float g2 = g[1][c], g3 = g[2][c], g4 = g[3][c];
            const float k1 = k[0][c], k2 = k[1][c], k3 = k[2][c], k4 = k[3][c], q1 = q[0][c], q2 = q[1][c], q3 = q[2][c], q4 = q[3][c];
            const float p12 = g2 * k1, p13 = g3 * p12, p14 = g4 * p13, p23 = g3 * k2, p24 = g4 * p23, p34 = g4 * k3;
            if (DELTA) {
                dot[0] = fmaf(k2, p12, dot[0]), dot[1] = fmaf(k3, p13, dot[1]), dot[2] = fmaf(k3, p23, dot[2]);
                dot[3] = fmaf(k4, p14, dot[3]), dot[4] = fmaf(k4, p24, dot[4]), dot[5] = fmaf(k4, p34, dot[5]);
            }
            dot[6] = fmaf(q1, k1, dot[6]);
            dot[7] = fmaf(q2, p12, dot[7]), dot[8] = fmaf(q2, k2, dot[8]);
            dot[9] = fmaf(q3, p13, dot[9]), dot[10] = fmaf(q3, p23, dot[10]), dot[11] = fmaf(q3, k3, dot[11]);
            dot[12] = fmaf(q4, p14, dot[12]), dot[13] = fmaf(q4, p24, dot[13]), dot[14] = fmaf(q4, p34, dot[14]), dot[15] = fmaf(q4, k4, dot[15]);
            const float G1 = g[0][c], G2 = G1 * g2, G3 = G2 * g3, G4 = G3 * g4;
            float *o = rec + lane + 32 * c;
            if (DELTA) {
                o[0] = G1 * k1, o[DP] = G2 * k2, o[2 * DP] = G3 * k3, o[3 * DP] = G4 * k4;
                o += 4 * DP;
            }
            o[0] = G1 * q1, o[DP] = G2 * q2, o[2 * DP] = G3 * q3, o[3 * DP] = G4 * q4;
            o[4 * DP] = p14, o[5 * DP] = p24, o[6 * DP] = p34, o[7 * DP] = k4;
            if (DELTA) o[8 * DP] = G4;
        }
        kq_spread_sum<16, 32>(dot, lane); // lane holds sum lane / 2
        float *sc = rec + REC - N_SCALAR;
        const int i = lane / 2, bi = i - 6, row = bi < 1 ? 0 : bi < 3 ? 1 : bi < 6 ? 2 : 3;
        if ((lane & 1) == 0) sc[i < 6 ? 4 + i : 12 + 4 * row + bi - row * (row + 1) / 2] = dot[0];
        else if (i < 6) sc[12 + (i < 3 ? 1 + i : i < 5 ? 3 + i : 11)] = 0.f; // above B's diagonal
        if (DELTA && lane < BT)
            sc[lane] = t0 + lane < p.T ? kq_sigmoid(p.in.b[(seq * p.T + t0 + lane) * p.in.ld + h]) : 0.f;
    }
}

// ---- the walk over the blocks -----------------------------------------------------------------------------
constexpr int TB = 4, STAGES = 3; // blocks per tile, tiles in the ring
constexpr int MAX_WARPS = 8;
constexpr uint64_t LIMIT = 5 * KQ_WAIT_LIMIT_NS;
struct ScanParams {
    KqMatState m;
    KqStateIn in;
    const float *rec, *val;
    int32_t T, pos0, blocks;
    const int32_t *pos0_dev;
    int64_t ldo;
    float *o;
};
__host__ __device__ constexpr int scan_tile_floats(int dp, bool delta, int cols) { return TB * (rec_floats(dp, delta) + cols * BT); }

__device__ __forceinline__ uint64_t pack2(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ float add2(uint64_t a) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
    return x + y;
}

// grid (blocks of columns, heads, sequences).  LPC lanes share NC columns, each with R groups of four key dimensions, so that under
// the delta rule the 8 NC sums of a block are one per lane.  The last warp brings the records.
template <int LPC, int R, bool DELTA>
__global__ void __launch_bounds__((MAX_WARPS + 1) * 32) state_scan_kernel(const __grid_constant__ ScanParams p) {
    constexpr int DP = LPC * R * 4, REC = rec_floats(DP, DELTA), GW = 32 / LPC, NC = LPC / (2 * BT), WC = GW * NC, NV = (DELTA ? 2 : 1) * NC * BT;
    extern __shared__ __align__(128) float sm[];
    __shared__ uint64_t full[STAGES], empty[STAGES];
    __shared__ __align__(16) float s_o[MAX_WARPS][TB * BT][WC];
    __shared__ int s_abort;
    KQ_PDL_ENTER();
    const KqMatState &m = p.m;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = lane % LPC, grp = lane / LPC, warps = (int)(blockDim.x / 32) - 1;
    const int cols = warps * WC; // of the CTA
    const int h = blockIdx.y, e0 = blockIdx.x * cols, ne = min(cols, m.vdim - e0);
    const int64_t seq = blockIdx.z;
    const int pos0 = p.pos0_dev ? *p.pos0_dev : p.pos0;
    if (m.taps)
        kq_move_ring(m, p.in, gridDim.z, p.T, pos0, ((seq * gridDim.y + h) * gridDim.x + blockIdx.x) * blockDim.x + tid,
                  (int64_t)gridDim.x * gridDim.y * gridDim.z * blockDim.x);
    const int tile_floats = scan_tile_floats(DP, DELTA, cols), tiles = (p.blocks + TB - 1) / TB;
    if (tid == 0) {
        for (int i = 0; i < STAGES; i++) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(smem_u32(&full[i])));
            asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(&empty[i])), "r"(warps));
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        s_abort = 0;
    }
    __syncthreads();
    if (warp == warps) {
        for (int tile = 0; tile < tiles; tile++) {
            const int st = tile % STAGES, round = tile / STAGES;
            if (round > 0 && !__all_sync(0xffffffffu, tc_wait(smem_u32(&empty[st]), (uint32_t)((round - 1) & 1), &s_abort, &g_state_error, 1, LIMIT))) break;
            float *dst = sm + st * tile_floats;
            const int b0 = tile * TB, n = min(TB, p.blocks - b0);
            const uint32_t bar = smem_u32(&full[st]);
            if (lane == 0) asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(n * (REC + ne * BT) * 4) : "memory");
            __syncwarp();
            if (lane < 2 * n) { // a lane per copy: the records, and the values of this CTA's columns
                const int i = lane / 2;
                const int64_t at = (seq * p.blocks + b0 + i) * m.heads + h;
                const float *src = lane & 1 ? p.val + (at * m.vdim + e0) * BT : p.rec + at * REC;
                asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                                 smem_u32(dst + (lane & 1 ? TB * REC + i * cols * BT : i * REC))),
                             "l"(src), "r"((lane & 1 ? ne * BT : REC) * 4), "r"(bar)
                             : "memory");
            }
            __syncwarp();
        }
    } else {
        const int c0 = warp * WC + grp * NC; // this lane group's columns inside the CTA
        uint64_t s[NC][R][2];
        const int64_t ld = kq_state_ld(m.dim);
        float *sp = m.s + ((seq * m.heads + h) * m.vdim + e0 + c0) * ld + 4 * part;
#pragma unroll
        for (int c = 0; c < NC; c++)
#pragma unroll
            for (int i = 0; i < R; i++) {
                const ulonglong2 v = pos0 > 0 && c0 + c < ne ? *reinterpret_cast<const ulonglong2 *>(sp + c * ld + 4 * LPC * i) : make_ulonglong2(0, 0);
                s[c][i][0] = v.x, s[c][i][1] = v.y;
            }
        float d_full = 1.f, d_last = 1.f; // fixed decay over a block; the last one may hold fewer tokens
        if (!DELTA)
            for (int j = 0; j < BT; j++) {
                d_full *= m.decay[h];
                if ((p.blocks - 1) * BT + j < p.T) d_last *= m.decay[h];
            }
        float *out = p.o + seq * p.T * p.ldo + (int64_t)h * m.vdim + e0 + warp * WC;
        const int wn = min(WC, ne - warp * WC); // columns of this warp
        const bool vec = WC == 4 && wn == 4 && (p.ldo & 3) == 0 && ((uintptr_t)out & 15) == 0;
        bool ok = true;
        for (int tile = 0; tile < tiles; tile++) {
            const int st = tile % STAGES;
            ok = __all_sync(0xffffffffu, tc_wait(smem_u32(&full[st]), (uint32_t)((tile / STAGES) & 1), &s_abort, &g_state_error, 2, LIMIT));
            if (!ok) break;
            const float *src = sm + st * tile_floats;
            const int nb = min(TB, p.blocks - tile * TB);
            constexpr int KH = DELTA ? 8 : 4; // first of the vectors that are written
            const ulonglong2 *vec2 = reinterpret_cast<const ulonglong2 *>(src) + part; // vector v, group i: vec2[v * DP / 4 + LPC * i]
            constexpr bool AHEAD = R == 1; // vectors wait in registers, where there are few
            ulonglong2 x[KH][R];
            auto load_x = [&](int v) {
#pragma unroll
                for (int i = 0; i < R; i++) x[v][i] = vec2[v * DP / 4 + LPC * i];
            };
            if (AHEAD) {
#pragma unroll
                for (int v = 0; v < KH; v++) load_x(v);
            }
            for (int b = 0; b < nb; b++) {
                const float *sc = src + b * REC + REC - N_SCALAR, *vals = src + TB * REC + (b * cols + c0) * BT;
                float val[NV];
#pragma unroll
                for (int v = 0; v < KH; v++) { // products with the state: [decayed k,] decayed q of the four tokens
                    uint64_t acc[NC];
                    if (!AHEAD) load_x(v);
#pragma unroll
                    for (int i = 0; i < R; i++)
#pragma unroll
                        for (int c = 0; c < NC; c++) acc[c] = fma2(s[c][i][1], x[v][i].y, i == 0 ? mul2(s[c][i][0], x[v][i].x) : fma2(s[c][i][0], x[v][i].x, acc[c]));
#pragma unroll
                    for (int c = 0; c < NC; c++) val[v / BT * NC * BT + c * BT + v % BT] = add2(acc[c]);
                }
                // requested ahead of the reduction: what the rest of the block reads
                ulonglong2 kk[BT][R], gg[R];
                auto load_k = [&]() {
#pragma unroll
                    for (int i = 0; i < R; i++) {
#pragma unroll
                        for (int j = 0; j < BT; j++) kk[j][i] = vec2[(KH + j) * DP / 4 + LPC * i];
                        if (DELTA) gg[i] = vec2[(KH + BT) * DP / 4 + LPC * i];
                    }
                };
                if (AHEAD) load_k();
                // the sum that ends in this lane: column c, token j, of k (lower half of the lanes) or q
                const int idx = part / (LPC / NV), c = idx / BT % NC, j = idx % BT;
                const float4 vt = *reinterpret_cast<const float4 *>(vals + c * BT), B = *reinterpret_cast<const float4 *>(sc + 12 + 4 * j);
                float4 u = vt, be, A0, A1;
                if (DELTA) be = *reinterpret_cast<const float4 *>(sc), A0 = *reinterpret_cast<const float4 *>(sc + 4), A1 = *reinterpret_cast<const float4 *>(sc + 8);
                kq_spread_sum<NV, LPC>(val, lane);
                if (DELTA) { // every lane solves for its column
                    float dk[BT];
#pragma unroll
                    for (int i = 0; i < BT; i++) dk[i] = __shfl_sync(0xffffffffu, val[0], c * BT + i, LPC);
                    u.x = be.x * (vt.x - dk[0]);
                    u.y = be.y * (vt.y - dk[1] - A0.x * u.x);
                    u.z = be.z * (vt.z - dk[2] - A0.y * u.x - A0.z * u.y);
                    u.w = be.w * (vt.w - dk[3] - A0.w * u.x - A1.x * u.y - A1.y * u.z);
                }
                if (DELTA ? part >= LPC / 2 : part % 2 == 0)
                    s_o[warp][b * BT + j][grp * NC + c] = fmaf(B.w, u.w, fmaf(B.z, u.z, fmaf(B.y, u.y, fmaf(B.x, u.x, val[0]))));
                float4 w[NC];
                if (NC == 1) {
                    w[0] = u;
                } else if (DELTA) { // the other column's, from the lane that solves for it
                    const float4 o = make_float4(__shfl_xor_sync(0xffffffffu, u.x, BT), __shfl_xor_sync(0xffffffffu, u.y, BT),
                                                 __shfl_xor_sync(0xffffffffu, u.z, BT), __shfl_xor_sync(0xffffffffu, u.w, BT));
                    w[0] = c ? o : u, w[NC - 1] = c ? u : o;
                } else {
#pragma unroll
                    for (int e = 0; e < NC; e++) w[e] = *reinterpret_cast<const float4 *>(vals + e * BT);
                }
                if (!AHEAD) load_k();
                vec2 += REC / 4;
                if (AHEAD && b + 1 < nb) { // the next block's first vectors
#pragma unroll
                    for (int v = 0; v < KH; v++) load_x(v);
                }
#pragma unroll
                for (int i = 0; i < R; i++) {
                    if (!DELTA) gg[i].x = gg[i].y = tile * TB + b == p.blocks - 1 ? pack2(d_last, d_last) : pack2(d_full, d_full);
#pragma unroll
                    for (int e = 0; e < NC; e++) s[e][i][0] = mul2(s[e][i][0], gg[i].x), s[e][i][1] = mul2(s[e][i][1], gg[i].y);
                }
#pragma unroll
                for (int t = 0; t < BT; t++)
#pragma unroll
                    for (int e = 0; e < NC; e++) {
                        const float f = t == 0 ? w[e].x : t == 1 ? w[e].y : t == 2 ? w[e].z : w[e].w;
                        const uint64_t ff = pack2(f, f);
#pragma unroll
                        for (int i = 0; i < R; i++) s[e][i][0] = fma2(kk[t][i].x, ff, s[e][i][0]), s[e][i][1] = fma2(kk[t][i].y, ff, s[e][i][1]);
                    }
            }
            __syncwarp(); // this warp is done with the tile, its outputs are complete
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&empty[st])) : "memory");
            const int t0 = tile * TB * BT, n = min(TB * BT, p.T - t0);
            if (vec) {
                if (lane < n) *reinterpret_cast<float4 *>(out + (int64_t)(t0 + lane) * p.ldo) = *reinterpret_cast<const float4 *>(s_o[warp][lane]);
            } else {
                for (int i = lane; i < n * WC; i += 32)
                    if (i % WC < wn) out[(int64_t)(t0 + i / WC) * p.ldo + i % WC] = s_o[warp][i / WC][i % WC];
            }
            __syncwarp();
        }
        if (ok) {
#pragma unroll
            for (int c = 0; c < NC; c++)
#pragma unroll
                for (int i = 0; i < R; i++)
                    if (c0 + c < ne) *reinterpret_cast<ulonglong2 *>(sp + c * ld + 4 * LPC * i) = make_ulonglong2(s[c][i][0], s[c][i][1]);
        }
    }
    __syncthreads();
    if (s_abort && tid == 0) // copies in flight must land before the CTA goes away
        for (int i = 0; i < STAGES; i++) {
            kq_mbar_wait(smem_u32(&full[i]), 0u, KQ_WAIT_LIMIT_NS);
            kq_mbar_wait(smem_u32(&full[i]), 1u, KQ_WAIT_LIMIT_NS);
        }
}

// ---- output of a prompt --------------------------------------------------------------------------------
// a warp per row and head; VEC: four elements per access
template <bool VEC>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float *o, int64_t ldo, const float *gate, int64_t ldg, const float *w, float eps, int64_t rows,
                                                             int heads, int vdim, float *out32, int64_t ld32, uint16_t *out16, int64_t ld16) {
    KQ_PDL_ENTER();
    const int64_t id = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5), r = id / heads;
    const int h = (int)(id % heads), lane = threadIdx.x & 31;
    if (r >= rows) return;
    const float *x = o + r * ldo + (int64_t)h * vdim, *gt = gate + r * ldg + (int64_t)h * vdim;
    float ss = 0.f;
    if (VEC) {
        constexpr int KEEP = 2;
        float4 v[KEEP], g[KEEP];
        const int n = vdim / 4;
#pragma unroll
        for (int i = 0; i < KEEP; i++) {
            v[i] = g[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (lane + 32 * i < n) v[i] = reinterpret_cast<const float4 *>(x)[lane + 32 * i], g[i] = reinterpret_cast<const float4 *>(gt)[lane + 32 * i];
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
        for (int d = lane + 32 * KEEP; d < n; d += 32) {
            const float4 a = reinterpret_cast<const float4 *>(x)[d];
            ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
        }
        const float sc = 1.0f / sqrtf(kq_warp_sum(ss) / (float)vdim + eps);
        auto emit = [&](int d, float4 a, const float4 &b) {
            const float4 wv = reinterpret_cast<const float4 *>(w)[d];
            a.x *= sc * wv.x * kq_sigmoid(b.x), a.y *= sc * wv.y * kq_sigmoid(b.y), a.z *= sc * wv.z * kq_sigmoid(b.z), a.w *= sc * wv.w * kq_sigmoid(b.w);
            if (out32) *reinterpret_cast<float4 *>(out32 + r * ld32 + (int64_t)h * vdim + 4 * d) = a;
            if (out16)
                *reinterpret_cast<uint2 *>(out16 + r * ld16 + (int64_t)h * vdim + 4 * d) =
                    make_uint2((uint32_t)kq_f2bf(a.x) | ((uint32_t)kq_f2bf(a.y) << 16), (uint32_t)kq_f2bf(a.z) | ((uint32_t)kq_f2bf(a.w) << 16));
        };
#pragma unroll
        for (int i = 0; i < KEEP; i++)
            if (lane + 32 * i < n) emit(lane + 32 * i, v[i], g[i]);
        for (int d = lane + 32 * KEEP; d < n; d += 32) emit(d, reinterpret_cast<const float4 *>(x)[d], reinterpret_cast<const float4 *>(gt)[d]);
    } else {
        for (int d = lane; d < vdim; d += 32) ss += x[d] * x[d];
        const float sc = 1.0f / sqrtf(kq_warp_sum(ss) / (float)vdim + eps);
        for (int d = lane; d < vdim; d += 32) {
            const float a = x[d] * sc * w[d] * kq_sigmoid(gt[d]);
            if (out32) out32[r * ld32 + (int64_t)h * vdim + d] = a;
            if (out16) out16[r * ld16 + (int64_t)h * vdim + d] = kq_f2bf(a);
        }
    }
    if (out16 && h == heads - 1)
        for (int64_t d = (int64_t)heads * vdim + lane; d < ld16; d += 32) out16[r * ld16 + d] = 0;
}

// ---- one token -----------------------------------------------------------------------------------------
constexpr int STEP_NT = 512, STEP_NW = STEP_NT / 32;
struct StepParams {
    KqMatState m;
    KqStateIn in;
    KqStateStep x;
    const int32_t *pos_dev;
    int32_t pos;
    float *z;
    int64_t ldz;
};

// y[i] = W[i] . x for n rows of bf16 weights (16-byte chunks of padded rows), x in shared memory; groups of lanes share rows.  The
// first chunk of the first rows is requested ahead.
struct SmallMatvec {
    static constexpr int PRE = 4;
    const uint16_t *W;
    int64_t ldw;
    int n, nck, w, l, r0, step;
    uint4 q[PRE];
    __device__ __forceinline__ SmallMatvec(const uint16_t *W_, int64_t ldw_, int n_, int K, int warp, int lane) : W(W_), ldw(ldw_), n(n_), nck((K + 7) / 8) {
        w = 1; // lanes per row
        while (w < nck && w < 32) w *= 2;
        l = lane % w, r0 = warp * (32 / w) + lane / w, step = STEP_NW * (32 / w);
#pragma unroll
        for (int u = 0; u < PRE; u++) q[u] = r0 + u * step < n && l < nck ? kq_ld_stream(W + (int64_t)(r0 + u * step) * ldw + 8 * l) : make_uint4(0, 0, 0, 0);
    }
    __device__ __forceinline__ float dot(const uint4 &v, const float *x, int c, float s) const {
        return kq_dot8(v, *reinterpret_cast<const float4 *>(x + 8 * c), *reinterpret_cast<const float4 *>(x + 8 * c + 4), s);
    }
    __device__ __forceinline__ void row(int r, float s, int c0, const float *x, float *y) const {
        if (r < n)
            for (int c = c0; c < nck; c += w) s = dot(kq_ld_stream(W + (int64_t)r * ldw + 8 * c), x, c, s);
        for (int o = w / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        if (r < n && l == 0) y[r] = s;
    }
    __device__ __forceinline__ void run(const float *x, float *y) const {
#pragma unroll
        for (int u = 0; u < PRE; u++) row(r0 + u * step, l < nck ? dot(q[u], x, l, 0.f) : 0.f, l + w, x, y);
        for (int t = PRE * step; t < n; t += step) row(r0 + t, 0.f, l, x, y); // whole warps: n is the same for all
    }
};
// SiLU of the convolution of one head's channels; the CTA that owns them (`owns`) also stores the new input.  The slot of the
// current position is read by nobody in this launch.
__device__ __forceinline__ void conv_step(const KqMatState &m, const float *x, const float *w, float *ring, int64_t channels, int n, int pos, bool owns, float *out) {
    for (int d = threadIdx.x; d < n; d += STEP_NT) {
        float s = x[d];
        if (m.taps) {
            s = 0.f;
            const KqConvIn ci = {x + d, 0, ring + d, channels, m.taps, pos};
            for (int k = 0; k < m.taps; k++) s = fmaf(w[(int64_t)d * m.taps + k], ci.at(k - (m.taps - 1)), s);
            if (owns) ring[(int64_t)(pos % m.taps) * channels + d] = x[d];
        }
        out[d] = kq_silu(s);
    }
}

// grid (heads, sequences)
template <int DP, bool DELTA>
__global__ void __launch_bounds__(STEP_NT) state_step_kernel(const __grid_constant__ StepParams p) {
    constexpr int R4 = DP / 32, PC = STEP_NT / 8, KEEP = 2; // PC: columns of a pass
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_red[4];
    KQ_PDL_TRIGGER();
    const KqMatState &m = p.m;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, part = tid & 7, col = tid >> 3;
    const int h = blockIdx.x, rep = m.heads / m.kv_heads, kh = h / rep;
    const int64_t seq = blockIdx.y;
    const int ra = (p.x.a_rank + 7) / 8 * 8, rg = (p.x.g_rank + 7) / 8 * 8, vp = (m.vdim + 3) / 4 * 4;
    float *sq = sm, *sk = sq + DP, *sg = sk + DP, *sv = sg + DP, *sgate = sv + vp, *so = sgate + vp, *sa = so + vp, *sg1 = sa + ra;
    const int64_t lda = kq_bf16_ld(p.x.a_rank), ldg = kq_bf16_ld(p.x.g_rank);
    const SmallMatvec wa(p.x.a2 + (int64_t)h * m.dim * lda, lda, DELTA ? m.dim : 0, p.x.a_rank, warp, lane);
    const SmallMatvec wg(p.x.g2 + (int64_t)h * m.vdim * ldg, ldg, DELTA ? m.vdim : 0, p.x.g_rank, warp, lane);
    float *base = m.s + (seq * m.heads + h) * (int64_t)m.vdim * DP;
    for (int i = tid * 32; i < m.vdim * DP; i += STEP_NT * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(base + i));
    KQ_PDL_WAIT();
    const int pos = p.pos_dev ? *p.pos_dev : p.pos;
    const int64_t channels = kq_state_channels(m), nq = (int64_t)m.kv_heads * m.dim, cq = (int64_t)kh * m.dim, cv = (int64_t)h * m.vdim;
    float *ring = m.taps ? m.conv + seq * m.taps * channels : nullptr;
    const bool owns = h % rep == 0;
    // the first columns of the state come while the vectors are made
    float4 first[KEEP][R4];
    auto load = [&](int e, float4 (&s)[R4]) {
#pragma unroll
        for (int i = 0; i < R4; i++)
            s[i] = pos > 0 && e < m.vdim ? *reinterpret_cast<const float4 *>(base + (int64_t)e * DP + 4 * (part + 8 * i)) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
#pragma unroll
    for (int u = 0; u < KEEP; u++) load(u * PC + col, first[u]);
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
        wa.run(sa, sg);
        wg.run(sg1, sgate);
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
    auto column = [&](int e, float4 (&s)[R4]) {
        const bool live = e < m.vdim;
        float *sp = base + (int64_t)(live ? e : 0) * DP;
        const float vt = live ? sv[e] : 0.f;
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
    };
#pragma unroll
    for (int u = 0; u < KEEP; u++)
        if (u * PC < m.vdim) column(u * PC + col, first[u]);
    for (int e0 = KEEP * PC; e0 < m.vdim; e0 += PC) {
        float4 s[R4];
        load(e0 + col, s);
        column(e0 + col, s);
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

template <int LPC, int R, bool DELTA>
b200_status launch_scan(const ScanParams &p, int n_seq, cudaStream_t st) {
    constexpr int DP = LPC * R * 4, per_warp = 32 / LPC * (LPC / (2 * BT));
    // warps per CTA: as few as possible on the busiest SM, then as many as possible in a CTA, which share a record
    int warps = 1;
    int64_t best = INT64_MAX;
    const int most = std::min<int>(MAX_WARPS, (int)((200 * 1024 / 4 / STAGES / TB - rec_floats(DP, DELTA)) / (per_warp * BT)));
    for (int w = 1; w <= most; w++) {
        const int64_t ctas = kq_div_up(p.m.vdim, w * per_warp) * p.m.heads * n_seq, load = kq_div_up(ctas, kq_sm_count()) * w;
        if (load <= best && (w == 1 || (w - 1) * per_warp < p.m.vdim)) best = load, warps = w;
    }
    const int cols = warps * per_warp;
    const size_t smem = (size_t)STAGES * scan_tile_floats(DP, DELTA, cols) * 4;
    static size_t attr[16];
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 16 || attr[dev] < smem) {
        KQ_CUDA(cudaFuncSetAttribute(state_scan_kernel<LPC, R, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        if (dev >= 0 && dev < 16) attr[dev] = smem;
    }
    kq_launch(state_scan_kernel<LPC, R, DELTA>, dim3((unsigned)kq_div_up(p.m.vdim, cols), (unsigned)p.m.heads, (unsigned)n_seq), (warps + 1) * 32, smem, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
template <int C, bool DELTA>
b200_status launch_tokens(const TokParams &p, int n_seq, cudaStream_t st) {
    const dim3 grid((unsigned)(p.head_ctas + kq_div_up((int64_t)p.m.heads * p.m.vdim, 32 * TOK_NW)), (unsigned)kq_div_up(p.blocks, RUN), (unsigned)n_seq);
    kq_launch(state_tokens_kernel<C, DELTA>, grid, TOK_NT, 0, st, p);
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
#define BY_DIM(FN, ARGS32, ARGS64, ARGS128, ARGS256, ...)                                                          \
    switch (kq_state_ld(m.dim)) {                                                                                  \
    case 32: return m.delta ? FN<ARGS32, true>(__VA_ARGS__) : FN<ARGS32, false>(__VA_ARGS__);                      \
    case 64: return m.delta ? FN<ARGS64, true>(__VA_ARGS__) : FN<ARGS64, false>(__VA_ARGS__);                      \
    case 128: return m.delta ? FN<ARGS128, true>(__VA_ARGS__) : FN<ARGS128, false>(__VA_ARGS__);                   \
    default: return m.delta ? FN<ARGS256, true>(__VA_ARGS__) : FN<ARGS256, false>(__VA_ARGS__);                    \
    }
#define TWO(a, b) a, b

} // namespace

int kq_state_error_fetch() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_state_error, sizeof(int)) != cudaSuccess) return -1;
    if (v) cudaMemcpyToSymbol(g_state_error, &zero, sizeof(int));
    return v;
}

int64_t kq_state_rec_floats(const KqMatState &m) {
    return (int64_t)m.heads * std::max<int64_t>(16 / BT * rec_floats(kq_state_ld(m.dim), m.delta != 0), kq_state_chunk_rec_floats(m));
}
int64_t kq_state_val_floats(const KqMatState &m) { return (int64_t)m.heads * m.vdim * 32; }

b200_status kq_state_tokens(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                            cudaStream_t st) {
    KQ_TRY(kq_check_state(m, n_seq, T));
    KQ_REQUIRE((((uintptr_t)t.rec | (uintptr_t)t.val) & 15) == 0, "matrix state: records");
    TokParams p;
    p.m = m, p.in = in, p.rec = t.rec, p.val = t.val, p.T = T, p.pos0 = pos0, p.pos0_dev = pos0_dev;
    p.blocks = (int)kq_div_up(T, BT), p.head_ctas = (int)kq_div_up(m.heads, TOK_NW);
    BY_DIM(launch_tokens, 1, 2, 4, 8, p, n_seq, st)
}

b200_status kq_state_scan(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                          float *o, int64_t ldo, cudaStream_t st) {
    KQ_TRY(kq_check_state(m, n_seq, T));
    ScanParams p;
    p.m = m, p.in = in, p.rec = t.rec, p.val = t.val, p.T = T, p.pos0 = pos0, p.pos0_dev = pos0_dev, p.blocks = (int)kq_div_up(T, BT), p.o = o, p.ldo = ldo;
    BY_DIM(launch_scan, TWO(8, 1), TWO(16, 1), TWO(16, 2), TWO(16, 4), p, n_seq, st)
}

b200_status kq_head_norm_gate(const float *o, int64_t ldo, const float *gate, int64_t ldg, const float *norm_w, float eps, int64_t rows, int heads,
                              int vdim, float *out32, int64_t ld32, uint16_t *out16, int64_t ld16, cudaStream_t st) {
    KQ_REQUIRE(o && gate && norm_w && rows >= 1 && heads >= 1 && vdim >= 1, "head_norm_gate: bad call");
    const uintptr_t al = (uintptr_t)o | (uintptr_t)gate | (uintptr_t)norm_w | (uintptr_t)out32 | (uintptr_t)out16;
    const bool vec = vdim % 4 == 0 && ((ldo | ldg | ld32 | ld16) & 3) == 0 && (al & 15) == 0;
    kq_launch(vec ? head_norm_gate_kernel<true> : head_norm_gate_kernel<false>, (unsigned)kq_div_up(rows * heads, 8), 256, 0, st, o, ldo, gate, ldg, norm_w, eps,
              rows, heads, vdim, out32, ld32, out16, ld16);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

b200_status kq_state_step(const KqMatState &m, const KqStateIn &in, const KqStateStep &x, int n_seq, const int32_t *pos_dev, int pos, float *z,
                          int64_t ldz, cudaStream_t st) {
    KQ_TRY(kq_check_state(m, n_seq, 1));
    StepParams p;
    p.m = m, p.in = in, p.x = x, p.pos_dev = pos_dev, p.pos = pos, p.z = z, p.ldz = ldz;
    const size_t smem = (size_t)(3 * kq_state_ld(m.dim) + 3 * kq_pad(m.vdim, 4) + kq_pad(x.a_rank, 8) + kq_pad(x.g_rank, 8)) * 4;
    KQ_REQUIRE(smem <= 200 * 1024, "matrix state: %d value dimensions", m.vdim);
    BY_DIM(launch_step, 32, 64, 128, 256, p, n_seq, smem, st)
}

b200_status kq_rank_operands(const float *a, int n, uint16_t *a16, const float *g, int m, uint16_t *g16, int64_t ld, int64_t rows, cudaStream_t st) {
    kq_launch(rank_operands_kernel, (unsigned)rows, 256, 0, st, a, n, a16, g, m, g16, ld, rows);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}
