// 16-bit dense weights: launchers of the matrix-vector and matrix-matrix kernels and of the ops of layers that
// are described one by one (latent attention, gated linear recurrence, clamped GLU, sandwich norms).
//
// Weight rows are bfloat16, padded with zeros to a multiple of 64 elements (128 bytes), so that a 64-element
// K slice is one row of a 128-byte-swizzled TMA box and every 16-byte chunk of a row is aligned.  Activations
// between kernels are f32; the tensor-core GEMM reads a 16-bit staging copy with the same row padding.
#pragma once
#include "kq_common.cuh"

#include <cuda_bf16.h>

enum { KQ_ACT_NONE = 0, KQ_ACT_GELU_TANH = 1 };
enum { KQ_OUT_F32 = 0, KQ_OUT_BF16 = 1, KQ_OUT_F16 = 2 };
enum { KQ_PREC_BF16 = 0, KQ_PREC_F32 = 1 };

static inline __host__ __device__ int64_t kq_pad(int64_t n, int64_t to) { return (n + to - 1) / to * to; }
static inline __host__ __device__ int64_t kq_bf16_ld(int64_t k) { return kq_pad(k, 64); } // elements per weight / staging row
static inline __host__ __device__ int64_t kq_f32_ld(int64_t k) { return kq_pad(k, 8); }   // elements per f32 activation row

// One weight matrix of a projection: y[m][col(n)] = act(W[n] . x[m] + bias[n]).  col(n) = n, or with head_in set
// (n / head_in) * head_out + n % head_in: a row that is a sequence of heads goes to a layout with padded heads.
struct KqDenseSeg {
    const uint16_t *W; // bf16 [rows][ldw]
    int32_t n_rows;    // rows of one group
    void *y;
    int64_t ldy;
    const float *bias;
    int32_t act, out; // KQ_ACT_*, KQ_OUT_*
    int32_t head_in, head_out;
    int32_t pad_cols; // 16-bit outputs: columns n_rows .. pad_cols-1 are written as zeros (row padding of a staging copy)
};

struct KqDense {
    KqDenseSeg seg[3];
    int32_t nseg = 0;
    int32_t M = 0, K = 0;
    int64_t ldw = 0;
    // groups > 1: a block-diagonal product, group g reads columns g * xg .. g * xg + K - 1 of x with rows
    // g * n_rows .. of every segment and writes column range g * n_rows (through col())
    int32_t groups = 1;
    int64_t xg = 0;
    // glu: segment 0 is the gate, segment 1 the up matrix: y = g sigmoid(alpha g) (u + 1) with g = min(gate, limit),
    // u = clamp(up, -limit, limit); written through segment 0
    int32_t glu = 0;
    float glu_limit = 0.f, glu_alpha = 0.f;
    // head_gate: y *= sigmoid(head_gate[m * ld_gate + group])
    const float *head_gate = nullptr;
    int64_t ld_gate = 0;
};

// Prologue of a projection: x' = x + norm(sub; sub_w) (sub null: x' = x; sub_w null: plain sum), then
// h = norm(x'; norm_w) (norm_w null: h = x').  norm(v; w) = v / rms(v) * (w_off + w).
struct KqNormPrep {
    const float *x = nullptr;
    int64_t ldx = 0;
    const float *sub = nullptr;
    int64_t ld_sub = 0;
    const float *sub_w = nullptr, *norm_w = nullptr;
    float eps = 0.f, w_off = 0.f;
    float *x_out = nullptr; // where x' goes (null: nowhere); must not be x when several CTAs read it
    int64_t ld_out = 0;
};

#ifdef __CUDACC__
__device__ __forceinline__ float kq_gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
__device__ __forceinline__ float kq_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float kq_clamped_glu(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * kq_sigmoid(alpha * g) * (u + 1.0f);
}
__device__ __forceinline__ uint16_t kq_f2bf(float v) { return __bfloat16_as_ushort(__float2bfloat16_rn(v)); }
__device__ __forceinline__ float kq_bf2f(uint16_t v) { return __uint_as_float((uint32_t)v << 16); }
__device__ __forceinline__ uint16_t kq_f2h_sat(float v) {
    return __half_as_ushort(__float2half_rn(fminf(fmaxf(v, -65504.f), 65504.f)));
}
// Segment i of a call that is a kernel parameter.  The selects keep the parameters in the constant bank: indexed by a
// variable they are read through generic loads, hundreds of cycles each.
__device__ __forceinline__ KqDenseSeg kq_dense_seg(const KqDense &c, int i) {
    KqDenseSeg s = c.seg[0];
    if (i == 1) s = c.seg[1];
    if (i == 2) s = c.seg[2];
    return s;
}
__device__ __forceinline__ int kq_dense_rows(const KqDense &c, int i) { return i == 0 ? c.seg[0].n_rows : i == 1 ? c.seg[1].n_rows : c.seg[2].n_rows; }
__device__ __forceinline__ const uint16_t *kq_dense_w(const KqDense &c, int i) { return i == 0 ? c.seg[0].W : i == 1 ? c.seg[1].W : c.seg[2].W; }
__device__ __forceinline__ int64_t kq_dense_col(const KqDenseSeg &s, int64_t n) {
    return s.head_in ? n / s.head_in * s.head_out + n % s.head_in : n;
}
__device__ __forceinline__ void kq_dense_put(const KqDenseSeg &s, int64_t m, int64_t n, float v) {
    const int64_t i = m * s.ldy + kq_dense_col(s, n);
    if (s.out == KQ_OUT_F32) ((float *)s.y)[i] = v;
    else ((uint16_t *)s.y)[i] = s.out == KQ_OUT_BF16 ? kq_f2bf(v) : kq_f2h_sat(v);
}
// v is the bare product of row n (over all groups) of a segment
__device__ __forceinline__ void kq_dense_store(const KqDense &c, const KqDenseSeg &s, int64_t m, int64_t n, int g, float v) {
    if (s.bias) v += s.bias[n];
    if (s.act == KQ_ACT_GELU_TANH) v = kq_gelu_tanh(v);
    if (c.head_gate) v *= kq_sigmoid(c.head_gate[m * c.ld_gate + g]);
    kq_dense_put(s, m, n, v);
}
#endif

// ---- kq_gemv_bf16.cu: 1..8 rows, f32 activations, exact products of f32 activations and bf16 weights
b200_status kq_gemv_bf16(const KqDense &c, const KqNormPrep &p, cudaStream_t st);
b200_status kq_gemv_grouped_bf16(const KqDense &c, const float *x, int64_t ldx, cudaStream_t st);
// ---- kq_gemm_bf16.cu
// tensor cores: a is a bf16 staging copy [parts][M][lda] (parts > 1: an f32 operand as a sum of bf16 parts)
b200_status kq_gemm_bf16(const KqDense &c, const uint16_t *a, int64_t lda, int parts, cudaStream_t st);
// CUDA cores in f32
b200_status kq_gemm_f32(const KqDense &c, const float *x, int64_t ldx, cudaStream_t st);

// ---- kq_layer_ops.cu
// embedding rows of a bf16 table times `scale`
b200_status kq_embed_bf16(const uint16_t *W, int64_t ldw, const int32_t *ids, int64_t rows, int K, float scale, float *y,
                          int64_t ldy, cudaStream_t st);
// the prologue above as a kernel of its own; h as f32 (h32) and / or as a bf16 staging copy (h16), either may be null
b200_status kq_norm_prep(const KqNormPrep &p, int64_t rows, int K, float *h32, int64_t ld32, uint16_t *h16, int64_t ld16,
                         cudaStream_t st);

// Recurrent state of one layer run: conv ring [seq][taps][width] (the input of position p in slot p % taps) and
// the state of the recurrence [seq][width], both f32.  Position 0 starts from zero whatever they hold.
struct KqRecState {
    float *conv, *s;
};
struct KqRecW {
    const float *conv_w, *conv_b; // [width][taps], [width]
    const uint16_t *ra, *ri;      // [blocks][m][ldw]
    const float *ra_b, *ri_b, *lam;
    float decay; // log a = -decay * r * softplus(lam)
    int32_t width, blocks, taps;
};
// u[row][c] = sum_k taps of x; optional bf16 parts of u per block for the tensor cores: u16 [3][rows][blocks * kq_bf16_ld(m)]
b200_status kq_causal_conv(const KqRecW &w, const KqRecState &s, const float *x, int64_t ldx, int n_seq, int T,
                           const int32_t *pos0_dev, int pos0, float *u, int64_t ldu, uint16_t *u16, cudaStream_t st);
// z[row][c] = S_t * y; r and i hold the gates before the sigmoid (biases included) and are overwritten; also moves the
// conv ring forward (x: the convolution's input).  Output f32 (z32) or bf16 (z16, zero-padded rows of ld16).
b200_status kq_linear_recurrence(const KqRecW &w, const KqRecState &s, float *r, float *i, int64_t ldr, const float *u,
                                 int64_t ldu, const float *x, int64_t ldx, const float *y, int64_t ldy, int n_seq, int T,
                                 const int32_t *pos0_dev, int pos0, float *z32, int64_t ld32, uint16_t *z16, int64_t ld16,
                                 float *scratch, size_t scratch_bytes, cudaStream_t st);
size_t kq_recurrence_scratch_bytes(int width, int rows, int n_seq); // calls of up to `rows` rows
// one token per sequence: convolution, gates, recurrence and the product with y in one launch
b200_status kq_recurrence_step(const KqRecW &w, const KqRecState &s, const float *x, int64_t ldx, const float *y,
                               int64_t ldy, int n_seq, const int32_t *pos_dev, int pos, float *z, int64_t ldz, cudaStream_t st);

// ---- kq_latent_attn.cu
// Latent cache of one layer run: rows [seq][cap][ld], position p in row p % cap; a row holds the normed latent
// (kv_rank values from 0), then the rotated key part (rot_dim values from rot_at).  bf16 or f32.
struct KqLatent {
    int32_t n_head, qk_dim, rot_dim, rot_dims, v_dim, kv_rank, window;
    float scale;
    const double *freq;   // device, rot_dims / 2 frequencies in radians per position
    int32_t cap, f32;     // rows of the ring, cache precision
    int32_t rot_at, ld;   // offset of the rotated part and row length, in elements (multiples of 8)
    void *cache;          // first sequence of the call
    int64_t seq_stride;   // elements between sequences
};
static inline int kq_latent_rot_at(int kv_rank) { return (int)kq_pad(kv_rank, 8); }
static inline int kq_latent_ld(int kv_rank, int rot_dim) { return (int)(kq_pad(kv_rank, 8) + kq_pad(rot_dim, 8)); }
// norm of the latent, rotation of the shared key part and of q's rotated part (in place), cache store
b200_status kq_latent_store(const KqLatent &l, const float *norm_w, float eps, float *q, int64_t ldq, const float *kv,
                            int64_t ldkv, int n_seq, int T, const int32_t *pos0_dev, int pos0, float *q_lat, int64_t ldql,
                            cudaStream_t st);
// Few rows: the store, and in the same launch the absorbed queries q_lat[row][h] = [W_uk[h]^T q_unrot | q_rot]
// (rows laid out like a cache row; `absorb` is that block-diagonal product)
constexpr int KQ_LATENT_ROWS = 8;
b200_status kq_latent_query(const KqLatent &l, const float *norm_w, float eps, float *q, int64_t ldq, const float *kv, int64_t ldkv, int n_seq,
                            int T, const int32_t *pos0_dev, int pos0, float *q_lat, int64_t ldql, const KqDense &absorb, cudaStream_t st);
// Attention over the latent rows.  o_lat given: o_lat [rows][n_head][kq_f32_ld(kv_rank)].  Otherwise (up to KQ_LATENT_ROWS
// rows) partial results of key ranges in scratch, for kq_latent_output: out[row][h * v_dim ..] = sigmoid(gate[row][h]) W_uv[h] o.
// max_keys: the most keys a row can see.
size_t kq_latent_scratch_bytes(const KqLatent &l, int max_keys);
b200_status kq_latent_attention(const KqLatent &l, const float *q_lat, int n_seq, int T, const int32_t *pos0_dev, int pos0, int max_keys,
                                float *o_lat, float *scratch, size_t scratch_bytes, cudaStream_t st);
b200_status kq_latent_output(const KqLatent &l, const float *scratch, int n_seq, int T, const int32_t *pos0_dev, int pos0, int max_keys,
                             const uint16_t *uv, const float *gate, int64_t ldg, float *out, int64_t ldo, cudaStream_t st);

// ---- kq_latent_prefill.cu: the expanded form for prompts of one sequence, bf16 cache
struct KqLatentPrefill {
    const uint16_t *uk, *uv; // bf16 [n_head * dim][kq_bf16_ld(kv_rank)]
    void *work;              // kq_latent_prefill_bytes, zeroed once
    size_t work_bytes;
};
size_t kq_latent_prefill_bytes(const KqLatent &l, int max_rows, int max_keys);
// q [T][n_head * (qk_dim + rot_dim)] f32, rotated; out bf16 [T][ldo]: head h's output times sigmoid(gate[t][h]).  The new
// rows are in the cache already.  B200_ERR_UNSUPPORTED: shapes the kernel is not built for.
b200_status kq_latent_prefill(const KqLatent &l, const KqLatentPrefill &w, const float *q, int64_t ldq, const float *gate, int64_t ldg,
                              int T, int pos0, uint16_t *out, int64_t ldo, cudaStream_t st);
