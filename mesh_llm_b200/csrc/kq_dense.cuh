// 16-bit dense weights: launchers of the matrix-vector and matrix-matrix kernels and of the ops of layers that
// are described one by one (latent and grouped-query attention, linear recurrences with a diagonal or a matrix state,
// GLU feed-forwards, experts, norms around the sub-layers).
//
// Weight rows are bfloat16, padded with zeros to a multiple of 64 elements (128 bytes), so that a 64-element
// K slice is one row of a 128-byte-swizzled TMA box and every 16-byte chunk of a row is aligned.  Activations
// between kernels are f32; the tensor-core GEMM reads a 16-bit staging copy with the same row padding.
#pragma once
#include "kq_common.cuh"

#include <cuda_bf16.h>

enum { KQ_ACT_NONE = 0, KQ_ACT_GELU_TANH = 1, KQ_ACT_SOFT_CAP = 2 }; // SOFT_CAP: cap tanh(y / cap)
enum { KQ_GLU_NONE = 0, KQ_GLU_CLAMPED = 1, KQ_GLU_SILU = 2 };
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
    int32_t pad_cols; // 16-bit outputs of one group: columns n_rows .. pad_cols-1 are written as zeros (row padding of a staging copy)
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
    // glu: segment 0 is the gate, segment 1 the up matrix; written through segment 0.  KQ_GLU_CLAMPED: y = g sigmoid(alpha g)
    // (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit); KQ_GLU_SILU: y = g sigmoid(g) u
    int32_t glu = 0;
    float glu_limit = 0.f, glu_alpha = 0.f;
    // head_gate: y *= sigmoid(head_gate[m * ld_gate + group])
    const float *head_gate = nullptr;
    int64_t ld_gate = 0;
    float cap = 0.f; // KQ_ACT_SOFT_CAP
    // row_mul: y *= row_mul[m * ld_mul + n] (bf16), after the activation
    const uint16_t *row_mul = nullptr;
    int64_t ld_mul = 0;
    // experts > 0 (matrix products): every segment holds `experts` matrices of n_rows rows one after the other; the rows of
    // x come in tiles of KQ_TILE_M, tile i belongs to expert tile_expert[i], *n_tiles of them (device) hold anything
    int32_t experts = 0;
    const int32_t *tile_expert = nullptr, *n_tiles = nullptr;
};
constexpr int KQ_TILE_M = 128;

// Prologue of a projection: x' = x + norm(sub; sub_w) (sub null: x' = x; sub_w null: plain sum), then
// h = norm(x'; norm_w) (norm_w null: h = x') times sigmoid(gate) where a gate is given.
// norm(v; w) = v / rms(v) * (w_off + w).
struct KqNormPrep {
    const float *x = nullptr;
    int64_t ldx = 0;
    const float *sub = nullptr;
    int64_t ld_sub = 0;
    const float *sub_w = nullptr, *norm_w = nullptr;
    float eps = 0.f, w_off = 0.f;
    float *x_out = nullptr; // where x' goes (null: nowhere); must not be x when several CTAs read it
    int64_t ld_out = 0;
    const float *gate = nullptr; // [rows][ld_gate]
    int64_t ld_gate = 0;
};

#ifdef __CUDACC__
__device__ __forceinline__ float kq_sigmoid(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }
// 0.5 z (1 + tanh(u)) = z sigmoid(2 u)
__device__ __forceinline__ float kq_gelu_tanh(float z) { return z * kq_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z)); }
__device__ __forceinline__ float kq_clamped_glu(float g, float u, float limit, float alpha) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * kq_sigmoid(alpha * g) * (u + 1.0f);
}
__device__ __forceinline__ float kq_silu(float z) { return z * kq_sigmoid(z); }
__device__ __forceinline__ float kq_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float kq_glu(const KqDense &c, float g, float u) {
    return c.glu == KQ_GLU_SILU ? kq_silu(g) * u : kq_clamped_glu(g, u, c.glu_limit, c.glu_alpha);
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
    if (s.act == KQ_ACT_SOFT_CAP) v = c.cap * tanhf(v / c.cap);
    if (c.head_gate) v *= kq_sigmoid(c.head_gate[m * c.ld_gate + g]);
    if (c.row_mul) v *= kq_bf2f(c.row_mul[m * c.ld_mul + n]);
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
// rows `ids` of a bf16 table as they are
b200_status kq_gather_bf16(const uint16_t *W, const int32_t *ids, int64_t rows, uint16_t *y, int64_t ld, cudaStream_t st);
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

// ---- kq_prompt_attn.cu
// first position that a query at `pos` sees: the start of its window (window > 0), of its chunk (chunk > 0), or 0
static inline __host__ __device__ int kq_first_key(int pos, int window, int chunk) {
    return window > 0 ? (pos >= window ? pos - window + 1 : 0) : chunk > 0 ? pos / chunk * chunk : 0;
}
// Tensor-core attention of T new positions of one sequence over f16 keys and values.  B200_ERR_UNSUPPORTED: sizes the
// kernel is not built for (kq_prompt_attention_fits says so ahead).
struct KqPromptAttn {
    const float *q = nullptr; // [T][n_head * (dim + rot)], final
    int64_t ldq = 0;
    const uint16_t *k = nullptr, *kr = nullptr, *v = nullptr; // f16 [rows][kv_heads][dims padded to 64]; kr [rows][padded rot]: shared by all heads
    int64_t rows = 0;
    int32_t n_head = 0, kv_heads = 0, dim = 0, rot = 0, vdim = 0, T = 0, pos0 = 0;
    int32_t lo = 0, ring = 0; // position of row 0; ring > 0: position p lies in row p % ring (a multiple of 128)
    int32_t window = 0, chunk = 0;
    float scale = 1.f;
    const float *gate = nullptr; // [T][ldg]: head h's output times sigmoid(gate[t][h])
    int64_t ldg = 0;
    uint16_t *out = nullptr; // bf16 [T][ldo]
    int64_t ldo = 0;
};
bool kq_prompt_attention_fits(int dim, int rot, int vdim);
b200_status kq_prompt_attention(const KqPromptAttn &a, cudaStream_t st);

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

// ---- kq_gqa_attn.cu: grouped-query attention over a ring of keys and values
// Cache of one layer run: rows of [kv_heads][dims padded to 64], position p in row p % cap (cap a multiple of 128), keys
// after their norm; f16 (saturating) or f32.
struct KqGqa {
    int32_t n_head, kv_heads, dim, vdim, window, chunk;
    float scale, eps;
    const float *q_norm, *k_norm; // [dim], plain weights
    int32_t cap, f32;
    void *k, *v;                  // first sequence of the call
    bool own_kv;                  // false: the rows are another layer's, nothing is stored
};
static inline int64_t kq_gqa_ld(int dim) { return kq_pad(dim, 64); }
constexpr int KQ_GQA_MAX_DIM = 512;
// New keys and values into the cache (own_kv), q normed in place.  q, k, v: the columns of projection rows of ldp floats.
b200_status kq_gqa_store(const KqGqa &a, float *q, const float *k, const float *v, int64_t ldp, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                         cudaStream_t st);
// Attention of every row, split over key ranges that the last CTA of a row merges.  fused: T = 1, norms and the store
// happen in here (q, k, v as above; otherwise q is normed and k, v are not read).  Output f32 or bf16 (either may be null).
// scratch: kq_gqa_scratch_bytes; counters: kq_gqa_counters words, zero between launches.  max_keys: the most keys a row can see.
int64_t kq_gqa_counters(const KqGqa &a);
size_t kq_gqa_scratch_bytes(const KqGqa &a, int max_rows, int max_keys);
b200_status kq_gqa_attention(const KqGqa &a, bool fused, const float *q, const float *k, const float *v, int64_t ldp, int n_seq, int T,
                             const int32_t *pos0_dev, int pos0, int max_keys, float *out, int64_t ldo, uint16_t *out16, int64_t ldo16,
                             float *scratch, size_t scratch_bytes, unsigned *counters, cudaStream_t st);

// ---- kq_state_ops.cu: recurrences whose state is a matrix per head
// S <- decay S + k v^T, o = S^T q, or under the delta rule S <- g S (a decay per key channel), u = beta (v - S^T k),
// S <- S + k u^T, o = S^T q.  Query / key head floor(h / (heads / kv_heads)) serves head h.
// State of one layer run: S transposed [seq][heads][vdim][kq_state_ld(dim)] f32, and with taps > 0 a ring of the short
// convolution's last inputs [seq][taps][channels] (the input of position p in slot p % taps; channels: all of q, then k, then
// v).  Position 0 starts from zero whatever they hold.
struct KqMatState {
    int32_t heads, kv_heads, dim, vdim, taps; // taps 0: no convolution
    int32_t delta;                            // delta rule; else a fixed decay per head
    const float *decay;                       // [heads]
    const float *conv_q, *conv_k, *conv_v;    // [channels][taps]
    const float *a_log, *dt_bias;             // delta: g = exp(-exp(a_log[h]) softplus(z + dt_bias)), z the low-rank projection
    float *s, *conv;                          // first sequence of the call
};
constexpr int KQ_STATE_MAX_DIM = 256;
static inline __host__ __device__ int kq_state_ld(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
static inline __host__ __device__ int64_t kq_state_channels(const KqMatState &m) { return 2 * (int64_t)m.kv_heads * m.dim + (int64_t)m.heads * m.vdim; }
// Columns of the fused projection's rows
struct KqStateIn {
    const float *q, *k, *v, *b, *z; // z: decay projection [rows][ldz], bias not added yet; b: write strengths before the sigmoid
    int64_t ld, ldz;
};
// Records of blocks of tokens: for every sequence kq_state_groups(T) times kq_state_rec_floats and kq_state_val_floats floats,
// 16-byte aligned; a launch of kq_state_tokens or kq_state_chunks writes them, the walk that goes with it reads them
struct KqStateTok {
    float *rec, *val;
};
static inline int64_t kq_state_groups(int64_t T) { return (T + 15) / 16; }
int64_t kq_state_rec_floats(const KqMatState &m);
int64_t kq_state_val_floats(const KqMatState &m);
b200_status kq_state_tokens(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                            cudaStream_t st);
// the walk over T positions: o [rows][ldo] f32; also moves the convolution's ring forward (in: its inputs)
b200_status kq_state_scan(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                          float *o, int64_t ldo, cudaStream_t st);
// ---- kq_state_chunk.cu: the same in chunks of 16 tokens, the products with the state on tensor cores (f32 operands in two parts),
// for heads of up to 128 key dimensions
bool kq_state_chunks_fit(const KqMatState &m);
int64_t kq_state_chunk_rec_floats(const KqMatState &m); // per head and chunk
b200_status kq_state_chunks(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                            cudaStream_t st);
b200_status kq_state_chunk_walk(const KqMatState &m, const KqStateIn &in, const KqStateTok &t, int n_seq, int T, const int32_t *pos0_dev, int pos0,
                                float *o, int64_t ldo, cudaStream_t st);
// ---- kq_state_ops.cu
// every head's o over its rms times norm_w [vdim] times sigmoid(gate); f32 or bf16 rows (padded with zeros)
b200_status kq_head_norm_gate(const float *o, int64_t ldo, const float *gate, int64_t ldg, const float *norm_w, float eps, int64_t rows, int heads,
                              int vdim, float *out32, int64_t ld32, uint16_t *out16, int64_t ld16, cudaStream_t st);
// One token per sequence, everything between the projections in one launch.  With delta: z and the gate come out of the low-rank
// products of a1, g1 (columns of the projection's rows) and w_a2, w_g2, and norm_w / eps give the finished rows.
struct KqStateStep {
    const float *a1 = nullptr, *g1 = nullptr;
    const uint16_t *a2 = nullptr, *g2 = nullptr; // bf16 [heads dim or heads vdim][kq_bf16_ld(rank)]
    int32_t a_rank = 0, g_rank = 0;
    const float *norm_w = nullptr;
    float eps = 0.f;
};
b200_status kq_state_step(const KqMatState &m, const KqStateIn &in, const KqStateStep &x, int n_seq, const int32_t *pos_dev, int pos, float *z,
                          int64_t ldz, cudaStream_t st);
// f32 columns into bf16 GEMM operands: a [rows][n] as three parts that add up, g [rows][m] rounded
b200_status kq_rank_operands(const float *a, int n, uint16_t *a16, const float *g, int m, uint16_t *g16, int64_t ld, int64_t rows, cudaStream_t st);

// ---- kq_moe_bf16.cu: SiLU-GLU experts with bf16 weights
// Router logits z [rows][ldz] f32 (bias included); the `top` largest are chosen (ties: the lower expert), weighted by a softmax
// over them.  A shared expert's gate and up products (before the GLU) may lie in the same rows.
struct KqMoe {
    int32_t experts, top, h, ff, ff_shared; // ff_shared 0: none
    const float *z, *sh_gate, *sh_up;       // columns of rows of ldz floats
    int64_t ldz;
};
constexpr int KQ_MOE_MAX_EXPERTS = 2048, KQ_MOE_MAX_TOP = 64;
// Up to a few rows, two launches: act[row * top + s] = GLU of the s-th chosen expert (its choice goes to ids / wts), then
// out = sum_s wts W_down act + shared.  Weights bf16 [experts][rows][kq_bf16_ld(K)].
b200_status kq_moe_few_gate_up(const KqMoe &m, const float *x, int64_t ldx, int rows, const uint16_t *gate, const uint16_t *up, float *act,
                               int64_t ld_act, int32_t *ids, float *wts, cudaStream_t st);
b200_status kq_moe_few_down(const KqMoe &m, const float *act, int64_t ld_act, const int32_t *ids, const float *wts, int rows, const uint16_t *down,
                            const uint16_t *sh_down, float *out, int64_t ldo, cudaStream_t st);
// Many rows: choice, shared GLU (f32 or bf16 rows), order by expert in tiles of KQ_TILE_M rows, gather; after the products with
// experts the weighted sum is added to `out` (which holds the shared expert's output, or is written when first is set).
struct KqMoeOrder {
    int32_t *ids, *pos;           // [rows * top]: chosen expert, place in the tiles
    float *wts;                   // [rows * top]
    int32_t *tile_expert, *n_tiles;
};
int64_t kq_moe_max_tiles(int64_t pairs, int experts);
b200_status kq_moe_route(const KqMoe &m, int rows, const KqMoeOrder &o, float *sh32, int64_t ld32, uint16_t *sh16, int64_t ld16, cudaStream_t st);
b200_status kq_moe_order(const KqMoe &m, int rows, const KqMoeOrder &o, cudaStream_t st);
// rows of elem_bytes-wide elements (ld of them) to their places
b200_status kq_moe_gather(const KqMoe &m, int rows, const KqMoeOrder &o, const void *x, void *y, int64_t ld, int elem_bytes, cudaStream_t st);
b200_status kq_moe_combine(const KqMoe &m, int rows, const KqMoeOrder &o, const float *y, int64_t ldy, float *out, int64_t ldo, bool first, cudaStream_t st);
