// Recurrences whose state is a matrix per head, for prompts, in chunks of 16 tokens with the products with the state on tensor
// cores.  With S the state in front of a chunk, G_j the product of the chunk's decays up to token j, P_ij that of the
// decays behind token i up to token j, and
//   A_ji = k_j . (P_ij k_i) (i < j),   B_ji = q_j . (P_ij k_i) (i <= j),
// the delta rule's write vectors solve u_j = beta_j (v_j - S^T G_j k_j - sum_(i<j) A_ji u_i).  The solution is linear in S:
//   u_j = U_j - S^T W_j,        W, U: the same recurrence over G_j k_j and over v_j
//   o_j = O_j + S^T Q_j,        O_j = sum_i B_ji U_i,   Q_j = G_j q_j - sum_i B_ji W_i
//   S  <- G_16 S + sum_i (P_i16 k_i) u_i^T
// All but S is known without the chunks before, so one launch makes W, Q, U, O and P k of every chunk in parallel (a CTA per
// chunk and head, a thread per column), and the walk over the chunks is left with three matrix products per chunk.  Four warps
// of the walk hold the state of 16 value dimensions, each a quarter of the key dimensions, as accumulator fragments of
// mma.m16n8k8; a fragment is also the first operand of the next product (the order of the summed dimension is free), so
// only the quarters' sums are exchanged, once per chunk.  The tensor cores see each f32 operand as two parts of 11 bits,
// three products of the parts are summed in f32.
// Decays occur in products only, never in quotients.  The fixed decay has W = 0 and u = v.
#include "kq_state.cuh"

#include <algorithm>

namespace {

constexpr int CT = 16; // tokens per chunk
__device__ int g_chunk_error;

// floats of a record: [W,] Q and P k in fragment order, decay of the chunk per key dimension (delta rule)
__host__ __device__ constexpr int rec_floats(int dp, bool delta) { return (delta ? 49 : 32) * dp; }

struct ChunkParams {
    KqMatState m;
    KqStateIn in;
    float *rec, *val; // [seq][chunk][head][record], [seq][chunk][head][vdim][2 CT]: U, O
    int32_t T, pos0, chunks;
    const int32_t *pos0_dev;
};

// place of row j (of 8 NT rows), key dimension d, as the second operand of a product over d: two neighbouring dimensions and two
// neighbouring 8-row tiles are next to one another, a lane reads four floats
template <int NT>
__device__ __forceinline__ int frag_x(int j, int d) {
    const int kt = d / 8, t = d % 8 / 2, nt = j / 8, g = j % 8;
    return ((kt * (NT / 2) + nt / 2) * 32 + g * 4 + t) * 4 + nt % 2 * 2 + d % 2;
}
// the same of token j, dimension d, for a product over the tokens
__device__ __forceinline__ int frag_k(int j, int d) { return (d / 8 * 32 + d % 8 * 4 + j % 8 / 2) * 4 + j / 8 * 2 + j % 2; }

// the record's fragments in shared memory: 16-byte words exchanged inside groups of eight, so that the columns of a warp, which lie
// whole multiples of 32 words apart, go to different banks
__device__ __forceinline__ int swz(int i) {
    const int w = i / 4;
    return (w ^ (w / 32 & 7)) * 4 + i % 4;
}

// SiLU of the convolution of one channel at N positions from t0 on; zero past the call's rows
template <int N>
__device__ __forceinline__ void conv_column(const ChunkParams &p, const float *x, const float *w, int64_t channel, int64_t seq, int t0, int pos0, float (&out)[N]) {
    const int taps = p.m.taps;
    const int64_t channels = kq_state_channels(p.m);
    const KqConvIn ci = {x + seq * p.T * p.in.ld, p.in.ld, taps ? p.m.conv + seq * taps * channels + channel : nullptr, channels, taps, pos0};
    if (taps == 0) {
#pragma unroll
        for (int j = 0; j < N; j++) out[j] = t0 + j < p.T ? ci.x[(int64_t)(t0 + j) * ci.ld] : 0.f;
    } else if (taps == 4) {
        float in[N + 3];
        if (t0 >= 3 && t0 + N <= p.T) {
#pragma unroll
            for (int k = 0; k < N + 3; k++) in[k] = ci.x[(int64_t)(t0 - 3 + k) * ci.ld];
        } else {
#pragma unroll
            for (int k = 0; k < N + 3; k++) in[k] = t0 - 3 + k < p.T ? ci.at(t0 - 3 + k) : 0.f;
        }
        const float4 cw = *reinterpret_cast<const float4 *>(w);
#pragma unroll
        for (int j = 0; j < N; j++) out[j] = fmaf(cw.w, in[j + 3], fmaf(cw.z, in[j + 2], fmaf(cw.y, in[j + 1], cw.x * in[j])));
    } else {
#pragma unroll 1
        for (int j = 0; j < N; j++) {
            float s = 0.f;
            if (t0 + j < p.T)
                for (int k = 0; k < taps; k++) s = fmaf(w[k], ci.at(t0 + j - (taps - 1) + k), s);
#pragma unroll
            for (int u = 0; u < N; u++)
                if (u == j) out[u] = s;
        }
    }
#pragma unroll
    for (int j = 0; j < N; j++) out[j] = t0 + j < p.T ? kq_silu(out[j]) : 0.f;
}

template <int V>
__device__ __forceinline__ void ld_vec(const float *p, float (&v)[V]) {
    if (V == 4) {
        const float4 x = *reinterpret_cast<const float4 *>(p);
        v[0] = x.x, v[V > 1 ? 1 : 0] = x.y, v[V > 2 ? 2 : 0] = x.z, v[V > 3 ? 3 : 0] = x.w;
    } else if (V == 2) {
        const float2 x = *reinterpret_cast<const float2 *>(p);
        v[0] = x.x, v[V > 1 ? 1 : 0] = x.y;
    } else {
        v[0] = p[0];
    }
}

// grid (chunks, heads, sequences), 2 DP threads
template <int DP, bool DELTA>
__global__ void __launch_bounds__(2 * DP) state_chunks_kernel(const __grid_constant__ ChunkParams p) {
    constexpr int NT = 2 * DP, NW = NT / 32, HT = CT / 2, V = DP / 32, NR = DELTA ? 4 : 2, REC = rec_floats(DP, DELTA), WH = DP / 32;
    extern __shared__ __align__(16) float sm[];
    __shared__ __align__(16) float sA[CT][CT], sB[CT][CT];
    __shared__ float s_sum[2][2 * HT][WH], s_scale[2][2 * HT], s_beta[CT];
    KQ_PDL_ENTER();
    const KqMatState &m = p.m;
    float *sk = sm, *sq = sk + CT * DP, *sg = sq + CT * DP, *rec = sg + CT * DP; // [token][dimension]; the record
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d = tid % DP, half = tid / DP;
    const int h = blockIdx.y, kh = h / (m.heads / m.kv_heads), t0 = blockIdx.x * CT;
    const int64_t seq = blockIdx.z, nq = (int64_t)m.kv_heads * m.dim, cq = (int64_t)kh * m.dim + d, cg = (int64_t)h * m.dim + d;
    const int pos0 = p.pos0_dev ? *p.pos0_dev : p.pos0;
    // ---- q, k and decays of half of the tokens, one key dimension per thread
    {
        float q[HT] = {}, k[HT] = {}, z[HT];
        const int th = t0 + half * HT;
        if (d < m.dim) {
            if (DELTA) {
#pragma unroll
                for (int j = 0; j < HT; j++) z[j] = th + j < p.T ? p.in.z[(seq * p.T + th + j) * p.in.ldz + cg] : 0.f;
            }
            conv_column<HT>(p, p.in.q + cq, m.conv_q + cq * m.taps, cq, seq, th, pos0, q);
            conv_column<HT>(p, p.in.k + cq, m.conv_k + cq * m.taps, nq + cq, seq, th, pos0, k);
        }
        if (DELTA) {
            float ss[2 * HT];
#pragma unroll
            for (int j = 0; j < HT; j++) ss[j] = q[j] * q[j], ss[HT + j] = k[j] * k[j];
            kq_spread_sum<2 * HT, 32>(ss, lane); // lane holds sum lane / 2 of its warp
            if ((lane & 1) == 0) s_sum[half][lane / 2][warp % WH] = ss[0];
            if (tid < CT) s_beta[tid] = t0 + tid < p.T ? kq_sigmoid(p.in.b[(seq * p.T + t0 + tid) * p.in.ld + h]) : 0.f;
            __syncthreads();
            if (tid < 4 * HT) {
                float x = 0.f;
#pragma unroll
                for (int w = 0; w < WH; w++) x += s_sum[tid / (2 * HT)][tid % (2 * HT)][w];
                x = 1.0f / sqrtf(x + 1e-6f);
                s_scale[tid / (2 * HT)][tid % (2 * HT)] = tid % (2 * HT) < HT ? x / sqrtf((float)m.dim) : x;
            }
            __syncthreads();
            const float a = expf(m.a_log[h]), bias = d < m.dim ? m.dt_bias[cg] : 0.f;
#pragma unroll
            for (int j = 0; j < HT; j++) {
                q[j] *= s_scale[half][j];
                k[j] *= s_scale[half][HT + j];
                sg[(half * HT + j) * DP + d] = d < m.dim && th + j < p.T ? expf(-a * kq_softplus(z[j] + bias)) : 1.f;
            }
        } else {
            const float decay = m.decay[h];
#pragma unroll
            for (int j = 0; j < HT; j++) sg[(half * HT + j) * DP + d] = th + j < p.T ? decay : 1.f;
        }
#pragma unroll
        for (int j = 0; j < HT; j++) sq[(half * HT + j) * DP + d] = q[j], sk[(half * HT + j) * DP + d] = k[j];
    }
    __syncthreads();
    // ---- A and B, column i by a warp; what is left of k_i at the end of the chunk
    float *rgc = rec + (NR * 8 + CT) * DP;
    for (int i = warp; i < CT; i += NW) {
        constexpr int NV = DELTA ? 2 * CT : CT, B0 = NV - CT;
        float pk[V], val[NV];
        ld_vec<V>(sk + i * DP + lane * V, pk);
#pragma unroll
        for (int j = 0; j < CT; j++) {
            val[j] = val[B0 + j] = 0.f;
            if (j < i) continue;
            float kj[V], qj[V], gj[V];
            ld_vec<V>(sq + j * DP + lane * V, qj);
            if (j > i) {
                ld_vec<V>(sg + j * DP + lane * V, gj);
                if (DELTA) ld_vec<V>(sk + j * DP + lane * V, kj);
            }
#pragma unroll
            for (int c = 0; c < V; c++) {
                if (j > i) {
                    pk[c] *= gj[c];
                    if (DELTA) val[j] = fmaf(kj[c], pk[c], val[j]);
                }
                val[B0 + j] = fmaf(qj[c], pk[c], val[B0 + j]);
            }
        }
#pragma unroll
        for (int c = 0; c < V; c++) rec[swz(NR * 8 * DP + frag_k(i, lane * V + c))] = pk[c];
        kq_spread_sum<NV, 32>(val, lane);
        if (DELTA) (lane < CT ? sA : sB)[lane % CT][i] = val[0];
        else if ((lane & 1) == 0) sB[lane / 2][i] = val[0];
    }
    __syncthreads();
    // ---- columns: W and Q of a key dimension, U and O of a value dimension
    auto solve = [&](const float (&x)[CT], float (&w)[CT], float (&b)[CT]) { // w: x or the recurrence over it; b = B w
#pragma unroll
        for (int j = 0; j < CT; j++) {
            float s = x[j], t = 0.f;
#pragma unroll
            for (int i = 0; i < CT; i += 4) {
                if (i > j) continue;
                const float4 a4 = *reinterpret_cast<const float4 *>(&sA[j][i]), b4 = *reinterpret_cast<const float4 *>(&sB[j][i]);
                const float av[4] = {a4.x, a4.y, a4.z, a4.w}, bv[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
                for (int e = 0; e < 4; e++)
                    if (i + e < j) {
                        if (DELTA) s = fmaf(-av[e], w[i + e], s);
                        t = fmaf(bv[e], w[i + e], t);
                    }
            }
            w[j] = DELTA ? s_beta[j] * s : s;
            b[j] = fmaf(sB[j][j], w[j], t);
        }
    };
    if (half == 0) {
        float G = 1.f, x[CT], y[CT];
#pragma unroll
        for (int j = 0; j < CT; j++) {
            G *= sg[j * DP + d];
            x[j] = G * sk[j * DP + d], y[j] = G * sq[j * DP + d];
        }
        if (DELTA) {
            float w[CT], b[CT];
            solve(x, w, b);
#pragma unroll
            for (int j = 0; j < CT; j++) rec[swz(frag_x<NR>(j, d))] = w[j], rec[swz(frag_x<NR>(CT + j, d))] = y[j] - b[j];
            rgc[d] = G;
        } else {
#pragma unroll
            for (int j = 0; j < CT; j++) rec[swz(frag_x<NR>(j, d))] = y[j];
        }
    } else {
        float *val = p.val + ((seq * p.chunks + blockIdx.x) * m.heads + h) * (int64_t)m.vdim * 2 * CT;
        for (int e = d; e < m.vdim; e += DP) {
            float x[CT], w[CT], b[CT];
            const int64_t c = (int64_t)h * m.vdim + e;
            conv_column<CT>(p, p.in.v + c, m.conv_v + c * m.taps, 2 * nq + c, seq, t0, pos0, x);
            solve(x, w, b);
#pragma unroll
            for (int j = 0; j < CT; j += 4) {
                *reinterpret_cast<float4 *>(val + (int64_t)e * 2 * CT + j) = make_float4(w[j], w[j + 1], w[j + 2], w[j + 3]);
                *reinterpret_cast<float4 *>(val + (int64_t)e * 2 * CT + CT + j) = make_float4(b[j], b[j + 1], b[j + 2], b[j + 3]);
            }
        }
    }
    __syncthreads();
    float4 *dst = reinterpret_cast<float4 *>(p.rec + ((seq * p.chunks + blockIdx.x) * m.heads + h) * (int64_t)REC);
    constexpr int FRAGS = (NR * 8 + CT) * DP; // the fragments lie swizzled in shared memory
    for (int i = tid; i < REC / 4; i += NT) dst[i] = reinterpret_cast<const float4 *>(rec)[i < FRAGS / 4 ? swz(4 * i) / 4 : i];
}

// ---- the walk ------------------------------------------------------------------------------------------
constexpr int WCOLS = 16, SPLIT = 4, MAX_GROUPS = 2, STAGES = 3; // columns of a group of SPLIT warps
constexpr uint64_t LIMIT = 5 * KQ_WAIT_LIMIT_NS;
struct WalkParams {
    KqMatState m;
    KqStateIn in;
    const float *rec, *val;
    int32_t T, pos0, chunks;
    const int32_t *pos0_dev;
    int64_t ldo;
    float *o;
};
__host__ __device__ constexpr int stage_floats(int dp, bool delta, int cols) { return rec_floats(dp, delta) + cols * 2 * CT; }

// d += a b: 16 x 8 x 8, the operands' upper 19 bits
__device__ __forceinline__ void mma8(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// v = hi + lo, hi the part the tensor cores see
__device__ __forceinline__ void split2(float v, uint32_t &hi, uint32_t &lo) {
    hi = __float_as_uint(v) & 0xffffe000u;
    lo = __float_as_uint(v - __uint_as_float(hi));
}

// grid (blocks of columns, heads, sequences); the last warp brings the records
template <int DP, bool DELTA>
__global__ void __launch_bounds__((MAX_GROUPS * SPLIT + 1) * 32) state_chunk_walk_kernel(const __grid_constant__ WalkParams p) {
    constexpr int REC = rec_floats(DP, DELTA), NR = DELTA ? 4 : 2, TILES = DP / 8 / SPLIT, Q0 = DELTA ? 2 : 0; // 8-row tiles, the first of Q
    extern __shared__ __align__(128) float sm[];
    __shared__ uint64_t full[STAGES], empty[STAGES];
    __shared__ __align__(16) float s_part[MAX_GROUPS][2][SPLIT][NR][32][4];
    __shared__ int s_abort;
    KQ_PDL_ENTER();
    const KqMatState &m = p.m;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane / 4, t = lane % 4, warps = (int)(blockDim.x / 32) - 1;
    const int group = warp / SPLIT, quarter = warp % SPLIT, cols = warps / SPLIT * WCOLS, h = blockIdx.y, e0 = blockIdx.x * cols, ne = min(cols, m.vdim - e0);
    const int64_t seq = blockIdx.z;
    const int pos0 = p.pos0_dev ? *p.pos0_dev : p.pos0;
    if (m.taps)
        kq_move_ring(m, p.in, gridDim.z, p.T, pos0, ((seq * gridDim.y + h) * gridDim.x + blockIdx.x) * blockDim.x + tid,
                     (int64_t)gridDim.x * gridDim.y * gridDim.z * blockDim.x);
    const int floats = stage_floats(DP, DELTA, cols);
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
        for (int c = 0; c < p.chunks; c++) {
            const int st = c % STAGES, round = c / STAGES;
            if (round > 0 && !__all_sync(0xffffffffu, tc_wait(smem_u32(&empty[st]), (uint32_t)((round - 1) & 1), &s_abort, &g_chunk_error, 1, LIMIT))) break;
            float *dst = sm + st * floats;
            const uint32_t bar = smem_u32(&full[st]);
            if (lane == 0) asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"((REC + ne * 2 * CT) * 4) : "memory");
            __syncwarp();
            if (lane < 2) {
                const int64_t at = (seq * p.chunks + c) * m.heads + h;
                const float *src = lane ? p.val + (at * m.vdim + e0) * 2 * CT : p.rec + at * REC;
                asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                                 smem_u32(dst + (lane ? REC : 0))),
                             "l"(src), "r"((lane ? ne * 2 * CT : REC) * 4), "r"(bar)
                             : "memory");
            }
            __syncwarp();
        }
    } else {
        float s[TILES][4]; // S^T: value dimensions g and g + 8, key dimensions 8 i + 2 t and the next, from this warp's quarter on
        const int c0 = group * WCOLS, i0 = quarter * TILES;
        const bool lo_ok = c0 + g < ne, hi_ok = c0 + g + 8 < ne;
        const int64_t ld = kq_state_ld(m.dim);
        float *sp = m.s + ((seq * m.heads + h) * m.vdim + e0 + c0 + g) * ld + 8 * i0 + 2 * t;
#pragma unroll
        for (int i = 0; i < TILES; i++) {
            const float2 a = pos0 > 0 && lo_ok ? *reinterpret_cast<const float2 *>(sp + 8 * i) : make_float2(0.f, 0.f);
            const float2 b = pos0 > 0 && hi_ok ? *reinterpret_cast<const float2 *>(sp + 8 * ld + 8 * i) : make_float2(0.f, 0.f);
            s[i][0] = a.x, s[i][1] = a.y, s[i][2] = b.x, s[i][3] = b.y;
        }
        float d_full = 1.f, d_last = 1.f; // fixed decay over a chunk; the last one may hold fewer tokens
        if (!DELTA)
            for (int j = 0; j < CT; j++) {
                d_full *= m.decay[h];
                if ((p.chunks - 1) * CT + j < p.T) d_last *= m.decay[h];
            }
        float *out = p.o + seq * p.T * p.ldo + (int64_t)h * m.vdim + e0 + c0;
        const int wn = min(WCOLS, ne - c0);
        bool ok = true;
        for (int c = 0; c < p.chunks; c++) {
            const int st = c % STAGES;
            // a warp that gave up runs on (over anything), so that the others of its group do not wait for it at the barrier below
            ok = __all_sync(0xffffffffu, tc_wait(smem_u32(&full[st]), (uint32_t)((c / STAGES) & 1), &s_abort, &g_chunk_error, 2, LIMIT)) && ok;
            const float *src = sm + st * floats;
            const float4 *fx = reinterpret_cast<const float4 *>(src) + i0 * (NR / 2) * 32 + lane,
                         *fk = reinterpret_cast<const float4 *>(src + NR * 8 * DP) + i0 * 32 + lane;
            const float *gc = src + NR * 8 * DP + CT * DP + 8 * i0, *val = src + REC + (c0 + g) * 2 * CT + 2 * t;
            // ---- products with the state: [W,] Q; one sum per pair of parts, so that three chains run side by side
            float acc[NR][3][4];
#pragma unroll
            for (int n = 0; n < NR; n++)
#pragma unroll
                for (int q = 0; q < 3; q++)
#pragma unroll
                    for (int e = 0; e < 4; e++) acc[n][q][e] = 0.f;
#pragma unroll
            for (int i = 0; i < TILES; i++) {
                uint32_t ah[4], al[4]; // rows g, g + 8 at 2 t, then at 2 t + 1
                split2(s[i][0], ah[0], al[0]), split2(s[i][2], ah[1], al[1]), split2(s[i][1], ah[2], al[2]), split2(s[i][3], ah[3], al[3]);
#pragma unroll
                for (int n = 0; n < NR; n += 2) {
                    const float4 x = fx[(i * (NR / 2) + n / 2) * 32];
                    uint32_t h0, h1, l0, l1;
                    split2(x.x, h0, l0), split2(x.y, h1, l1);
                    mma8(acc[n][0], ah, h0, h1), mma8(acc[n][1], ah, l0, l1), mma8(acc[n][2], al, h0, h1);
                    split2(x.z, h0, l0), split2(x.w, h1, l1);
                    mma8(acc[n + 1][0], ah, h0, h1), mma8(acc[n + 1][1], ah, l0, l1), mma8(acc[n + 1][2], al, h0, h1);
                }
            }
            float(*part)[NR][32][4] = s_part[group][c & 1];
#pragma unroll
            for (int n = 0; n < NR; n++)
                *reinterpret_cast<float4 *>(part[quarter][n][lane]) =
                    make_float4(acc[n][0][0] + (acc[n][1][0] + acc[n][2][0]), acc[n][0][1] + (acc[n][1][1] + acc[n][2][1]),
                                acc[n][0][2] + (acc[n][1][2] + acc[n][2][2]), acc[n][0][3] + (acc[n][1][3] + acc[n][2][3]));
            float2 uv[2][2];
#pragma unroll
            for (int n = 0; n < 2; n++) uv[n][0] = *reinterpret_cast<const float2 *>(val + 8 * n), uv[n][1] = *reinterpret_cast<const float2 *>(val + 8 * 2 * CT + 8 * n);
            // what does not wait for the other quarters: G S, and the parts of P k
            const float dc = c == p.chunks - 1 ? d_last : d_full;
            uint32_t kh[TILES][4], kl[TILES][4];
#pragma unroll
            for (int i = 0; i < TILES; i++) {
                const float2 gg = DELTA ? *reinterpret_cast<const float2 *>(gc + 8 * i + 2 * t) : make_float2(dc, dc);
                const float4 x = fk[i * 32];
                s[i][0] *= gg.x, s[i][1] *= gg.y, s[i][2] *= gg.x, s[i][3] *= gg.y;
                split2(x.x, kh[i][0], kl[i][0]), split2(x.y, kh[i][1], kl[i][1]), split2(x.z, kh[i][2], kl[i][2]), split2(x.w, kh[i][3], kl[i][3]);
            }
            asm volatile("bar.sync %0, %1;" ::"r"(1 + group), "n"(SPLIT * 32) : "memory");
            // ---- u = U - S^T W of tokens 8 n + 2 t and the next, as the first operand of the product over the tokens
            uint32_t uh[2][4], ul[2][4];
#pragma unroll
            for (int n = 0; n < 2; n++) {
                float u[4] = {uv[n][0].x, uv[n][0].y, uv[n][1].x, uv[n][1].y};
                if (DELTA) {
#pragma unroll
                    for (int q = 0; q < SPLIT; q++) {
                        const float4 x = *reinterpret_cast<const float4 *>(part[q][n][lane]);
                        u[0] -= x.x, u[1] -= x.y, u[2] -= x.z, u[3] -= x.w;
                    }
                }
                // columns past the call's share hold anything: they stay apart and are not written
                split2(u[0], uh[n][0], ul[n][0]), split2(u[2], uh[n][1], ul[n][1]), split2(u[1], uh[n][2], ul[n][2]), split2(u[3], uh[n][3], ul[n][3]);
            }
            // ---- S <- G S + (P k) u^T, tiles side by side
#pragma unroll
            for (int n = 0; n < 2; n++) {
#pragma unroll
                for (int i = 0; i < TILES; i++) mma8(s[i], uh[n], kl[i][2 * n], kl[i][2 * n + 1]);
#pragma unroll
                for (int i = 0; i < TILES; i++) mma8(s[i], ul[n], kh[i][2 * n], kh[i][2 * n + 1]);
#pragma unroll
                for (int i = 0; i < TILES; i++) mma8(s[i], uh[n], kh[i][2 * n], kh[i][2 * n + 1]);
            }
            { // outputs: a warp takes tile quarter / 2, and of it the lower or upper eight columns
                const int n = quarter / 2, up = quarter % 2, t0 = c * CT + 8 * n + 2 * t;
                float2 o = *reinterpret_cast<const float2 *>(val + up * 8 * 2 * CT + CT + 8 * n);
#pragma unroll
                for (int q = 0; q < SPLIT; q++) {
                    const float2 x = *reinterpret_cast<const float2 *>(&part[q][Q0 + n][lane][2 * up]);
                    o.x += x.x, o.y += x.y;
                }
                if (g + 8 * up < wn) {
                    float *d = out + (int64_t)t0 * p.ldo + g + 8 * up;
                    if (t0 < p.T) d[0] = o.x;
                    if (t0 + 1 < p.T) d[p.ldo] = o.y;
                }
            }
            __syncwarp(); // this warp is done with the stage
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&empty[st])) : "memory");
        }
        if (ok) {
#pragma unroll
            for (int i = 0; i < TILES; i++) {
                if (lo_ok) *reinterpret_cast<float2 *>(sp + 8 * i) = make_float2(s[i][0], s[i][1]);
                if (hi_ok) *reinterpret_cast<float2 *>(sp + 8 * ld + 8 * i) = make_float2(s[i][2], s[i][3]);
            }
        }
    }
    __syncthreads();
    if (s_abort && tid == 0) // copies in flight must land before the CTA goes away
        for (int i = 0; i < STAGES; i++) {
            kq_mbar_wait(smem_u32(&full[i]), 0u, KQ_WAIT_LIMIT_NS);
            kq_mbar_wait(smem_u32(&full[i]), 1u, KQ_WAIT_LIMIT_NS);
        }
}

template <typename K>
b200_status allow(K kern, size_t smem, size_t (&have)[16]) {
    int dev = 0;
    KQ_CUDA(cudaGetDevice(&dev));
    if ((dev < 0 || dev >= 16 || have[dev] < smem)) {
        KQ_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        if (dev >= 0 && dev < 16) have[dev] = smem;
    }
    return B200_OK;
}

template <int DP, bool DELTA>
b200_status launch_chunks(const ChunkParams &p, int n_seq, cudaStream_t st) {
    const size_t smem = (size_t)(3 * CT * DP + rec_floats(DP, DELTA)) * 4;
    static size_t have[16];
    KQ_TRY(allow(state_chunks_kernel<DP, DELTA>, smem, have));
    kq_launch(state_chunks_kernel<DP, DELTA>, dim3((unsigned)p.chunks, (unsigned)p.m.heads, (unsigned)n_seq), 2 * DP, smem, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

template <int DP, bool DELTA>
b200_status launch_walk(const WalkParams &p, int n_seq, cudaStream_t st) {
    // column groups per CTA: as few as possible on the busiest SM, then as many as possible in a CTA, which share a record
    int groups = 1;
    int64_t best = INT64_MAX;
    for (int w = 1; w <= MAX_GROUPS; w++) {
        const int64_t ctas = kq_div_up(p.m.vdim, w * WCOLS) * p.m.heads * n_seq, load = kq_div_up(ctas, kq_sm_count()) * w;
        if (load <= best && (w == 1 || (w - 1) * WCOLS < p.m.vdim)) best = load, groups = w;
    }
    const int cols = groups * WCOLS;
    const size_t smem = (size_t)STAGES * stage_floats(DP, DELTA, cols) * 4;
    static size_t have[16];
    KQ_TRY(allow(state_chunk_walk_kernel<DP, DELTA>, smem, have));
    kq_launch(state_chunk_walk_kernel<DP, DELTA>, dim3((unsigned)kq_div_up(p.m.vdim, cols), (unsigned)p.m.heads, (unsigned)n_seq), (groups * SPLIT + 1) * 32, smem, st, p);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    return B200_OK;
}

#define BY_DIM(FN, ...)                                                                              \
    switch (kq_state_ld(m.dim)) {                                                                    \
    case 32: return m.delta ? FN<32, true>(__VA_ARGS__) : FN<32, false>(__VA_ARGS__);                \
    case 64: return m.delta ? FN<64, true>(__VA_ARGS__) : FN<64, false>(__VA_ARGS__);                \
    default: return m.delta ? FN<128, true>(__VA_ARGS__) : FN<128, false>(__VA_ARGS__);              \
    }

} // namespace

int kq_state_chunk_error_fetch() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_chunk_error, sizeof(int)) != cudaSuccess) return -1;
    if (v) cudaMemcpyToSymbol(g_chunk_error, &zero, sizeof(int));
    return v;
}

bool kq_state_chunks_fit(const KqMatState &m) { return m.dim <= 128; }
int64_t kq_state_chunk_rec_floats(const KqMatState &m) { return kq_state_chunks_fit(m) ? rec_floats(kq_state_ld(m.dim), m.delta != 0) : 0; }

b200_status kq_state_chunks(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                            cudaStream_t st) {
    KQ_TRY(kq_check_state(m, n_seq, T));
    KQ_REQUIRE(kq_state_chunks_fit(m) && (((uintptr_t)t.rec | (uintptr_t)t.val) & 15) == 0, "matrix state: records");
    ChunkParams p;
    p.m = m, p.in = in, p.rec = t.rec, p.val = t.val, p.T = T, p.pos0 = pos0, p.pos0_dev = pos0_dev, p.chunks = (int)kq_div_up(T, CT);
    BY_DIM(launch_chunks, p, n_seq, st)
}

b200_status kq_state_chunk_walk(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                                float *o, int64_t ldo, cudaStream_t st) {
    KQ_TRY(kq_check_state(m, n_seq, T));
    KQ_REQUIRE(kq_state_chunks_fit(m), "matrix state: %d key dimensions", m.dim);
    WalkParams p;
    p.m = m, p.in = in, p.rec = t.rec, p.val = t.val, p.T = T, p.pos0 = pos0, p.pos0_dev = pos0_dev, p.chunks = (int)kq_div_up(T, CT), p.o = o, p.ldo = ldo;
    BY_DIM(launch_walk, p, n_seq, st)
}
