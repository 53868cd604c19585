// Stages whose layers are described one by one (b200_stage_create_layers): tensor table, caches and states, and the
// forward pass, on top of the stage object of kq_stage.cuh (loading, decode graphs, logits, counters are shared
// with the K-quant decoder).
//
// The residual stream x is f32.  A sub-layer leaves its output un-normed in `sub`; the next projection's prologue
// forms x + norm_b(sub) and the norm in front of itself, so that no launch of its own does either in a decode step.
// Up to 8 rows (decode) run on the matrix-vector kernels with f32 activations; more rows on the tensor-core GEMM with
// a bf16 copy of each projection's input, or on the f32 GEMM in the 32-bit mode.
//
// State of one layer run and sequence slot: attention keeps a ring of cap rows (window or chunk + micro-batch, so that a
// micro-batch's first row still finds all it sees), a recurrence its state and the convolution's last inputs.
// Weights that are applied to the same input lie one after the other (packs), so that one product makes all of them.
// A slot that starts at position 0 reads none of what it held, so nothing has to be cleared between sequences.
#include "kq_dense.cuh"
#include "kq_stage.cuh"

#include <math.h>
#include <stdlib.h>

#include <algorithm>

struct LayerDesc {
    b200_layer_config c;
    const float *pre1 = nullptr, *post1 = nullptr, *pre2 = nullptr, *post2 = nullptr; // norms in front of (null: none) and behind the sub-layers
    // recurrence
    const uint16_t *wy = nullptr, *wx = nullptr, *wo = nullptr;
    const float *by = nullptr, *bx = nullptr;
    KqRecW rec = {};
    // latent attention
    const uint16_t *wq = nullptr, *dkv = nullptr, *uk = nullptr, *uv = nullptr, *wg = nullptr;
    uint16_t *uk_t = nullptr; // [n_head * kv_rank][kq_bf16_ld(qk_dim)], derived
    const float *kv_norm = nullptr;
    double *freq = nullptr;
    // grouped-query attention, matrix states: all projections of the mixer's input as one matrix, and where each one's rows start
    const uint16_t *win = nullptr;
    int in_pack = -1;
    int64_t in_rows = 0, at_q = 0, at_k = 0, at_v = 0, at_b = 0, at_a = 0, at_g = 0;
    const float *q_norm = nullptr, *k_norm = nullptr, *o_norm = nullptr, *decay = nullptr, *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr,
                *a_log = nullptr, *dt_bias = nullptr;
    const uint16_t *a2 = nullptr, *g2 = nullptr;
    // feed-forward
    const uint16_t *gate = nullptr, *up = nullptr, *down = nullptr;
    // experts: the router and the shared expert's gate and up rows as one matrix (with the router's bias, zero for the rest)
    const uint16_t *wr = nullptr, *sh_down = nullptr;
    float *r_bias = nullptr; // derived
    int r_pack = -1, gate_pack = -1, up_pack = -1, down_pack = -1;
    int64_t r_rows = 0, at_shg = 0, at_shu = 0;
    // per-layer token input
    const uint16_t *side_gate = nullptr, *side_proj = nullptr;
    const float *side_norm = nullptr;
};

// Matrices of equal row length that lie one after the other on the device, each from a row that is a multiple of `align`
struct Pack {
    std::vector<std::string> names;
    int64_t align = 1, rows = 0;
    std::vector<int64_t> at;
    void *dev = nullptr;
};

struct RunState { // one pass over a layer
    int layer;
    float *conv = nullptr, *s = nullptr;
    void *cache = nullptr;              // latents, or keys
    void *vcache = nullptr;             // values
    int cap = 0;
};

struct KqLayers {
    b200_stack_config s;
    std::vector<LayerDesc> layers; // [layer_begin, layer_end)
    std::vector<RunState> runs;
    std::vector<int> seq_pos;
    float *trace = nullptr;
    size_t state_bytes = 0;
    const uint16_t *embed = nullptr;
    const float *final_norm = nullptr;
    // activations, sized for the widest layer
    int64_t ldx = 0;
    float *x[2] = {}, *sub = nullptr, *h32 = nullptr;
    uint16_t *h16 = nullptr;
    float *f[9] = {}; // projections of a mixer
    std::vector<Pack> packs;
    const uint16_t *side_embed = nullptr;
    uint16_t *side_rows = nullptr; // the rows of a call's tokens, all layers
    KqStateTok state_tok = {};
    // experts: activations of few rows; tiles of rows by expert
    float *moe_act = nullptr, *moe_y = nullptr;
    void *moe_x = nullptr, *moe_h = nullptr; // bf16, or f32 in the 32-bit mode
    KqMoeOrder moe = {};
    uint16_t *u16 = nullptr, *z16 = nullptr, *act16 = nullptr;
    float *act32 = nullptr, *att_scratch = nullptr, *rec_scratch = nullptr;
    unsigned *gqa_counters = nullptr;
    size_t att_scratch_bytes = 0, rec_scratch_bytes = 0;
    void *prefill_work = nullptr;
    size_t prefill_bytes = 0;
};

void KqLayersDelete::operator()(KqLayers *p) const { delete p; }

namespace {

constexpr int SMALL_ROWS = KQ_LATENT_ROWS;

// uk [H * dim][ld_in] -> uk_t [H * R][ld_out]
__global__ void transpose_heads_kernel(const uint16_t *in, int64_t ld_in, int H, int dim, int R, uint16_t *out, int64_t ld_out) {
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (int64_t)H * R * ld_out) return;
    const int64_t row = i / ld_out;
    const int d = (int)(i % ld_out), h = (int)(row / R), r = (int)(row % R);
    out[i] = d < dim ? in[((int64_t)h * dim + d) * ld_in + r] : 0;
}

b200_status check_layer(const b200_layer_config &l, int i) {
    if (l.mixer == B200_MIXER_LATENT_ATTN) {
        KQ_REQUIRE(l.n_head >= 1 && l.qk_dim >= 1 && l.rot_dim >= 0 && l.v_dim >= 1 && l.kv_rank >= 1 && l.window >= 0,
                   "layer %d: sizes of the latent attention", i);
        KQ_REQUIRE(l.rot_dims >= 0 && l.rot_dims % 2 == 0 && l.rot_dims <= l.rot_dim && (l.rot_dims == 0 || l.rope_base > 0.f),
                   "layer %d: rotary dimensions %d of %d", i, l.rot_dims, l.rot_dim);
        if (l.kv_rank > 1024) {
            kq_set_error("layer %d: latents of up to 1024 values", i);
            return B200_ERR_UNSUPPORTED;
        }
    } else if (l.mixer == B200_MIXER_LINEAR_REC) {
        KQ_REQUIRE(l.rec_width >= 1 && l.rec_blocks >= 1 && l.rec_width % l.rec_blocks == 0 && l.conv_taps >= 1,
                   "layer %d: sizes of the recurrence", i);
    } else if (l.mixer == B200_MIXER_GQA) {
        KQ_REQUIRE(l.n_head >= 1 && l.n_head_kv >= 1 && l.n_head % l.n_head_kv == 0 && l.qk_dim >= 1 && l.v_dim >= 1 && l.window >= 0 && l.chunk >= 0 &&
                       !(l.window && l.chunk),
                   "layer %d: sizes of the attention", i);
        if (l.qk_dim > KQ_GQA_MAX_DIM || l.v_dim > KQ_GQA_MAX_DIM) {
            kq_set_error("layer %d: heads of up to %d values", i, KQ_GQA_MAX_DIM);
            return B200_ERR_UNSUPPORTED;
        }
    } else if (l.mixer == B200_MIXER_DECAY_STATE || l.mixer == B200_MIXER_DELTA_STATE) {
        const bool delta = l.mixer == B200_MIXER_DELTA_STATE;
        KQ_REQUIRE(l.n_head >= 1 && l.qk_dim >= 1 && l.v_dim >= 1 &&
                       (!delta || (l.n_head_kv >= 1 && l.n_head % l.n_head_kv == 0 && l.conv_taps >= 1 && l.decay_rank >= 1 && l.gate_rank >= 1)),
                   "layer %d: sizes of the linear attention", i);
        if (l.qk_dim > KQ_STATE_MAX_DIM) {
            kq_set_error("layer %d: states of up to %d key dimensions", i, KQ_STATE_MAX_DIM);
            return B200_ERR_UNSUPPORTED;
        }
    } else {
        kq_set_error("layer %d: unknown mixer %d", i, l.mixer);
        return B200_ERR_UNSUPPORTED;
    }
    if (l.ffn == B200_FFN_MOE) {
        KQ_REQUIRE(l.n_expert >= 1 && l.n_expert_used >= 1 && l.n_expert_used <= l.n_expert && l.n_ff_exp >= 1 && l.n_ff_shared >= 0,
                   "layer %d: %d of %d experts", i, l.n_expert_used, l.n_expert);
        if (l.n_expert > KQ_MOE_MAX_EXPERTS || l.n_expert_used > KQ_MOE_MAX_TOP) {
            kq_set_error("layer %d: up to %d of %d experts", i, KQ_MOE_MAX_TOP, KQ_MOE_MAX_EXPERTS);
            return B200_ERR_UNSUPPORTED;
        }
        return B200_OK;
    }
    KQ_REQUIRE(l.ffn == B200_FFN_NONE || (l.ffn == B200_FFN_CLAMPED_GLU && l.n_ff >= 1), "layer %d: feed-forward", i);
    return B200_OK;
}

// a layer that reads another's keys and values: that one comes earlier, has its own, of the same sizes, on the same stage
b200_status check_shared(const b200_layer_config *layers, int i, int begin) {
    const b200_layer_config &l = layers[i];
    if (l.mixer != B200_MIXER_GQA || !l.kv_shared) return B200_OK;
    KQ_REQUIRE(l.kv_layer >= 0 && l.kv_layer < i, "layer %d: keys and values of layer %d", i, l.kv_layer);
    const b200_layer_config &o = layers[l.kv_layer];
    KQ_REQUIRE(o.mixer == B200_MIXER_GQA && !o.kv_shared && o.n_head_kv == l.n_head_kv && o.qk_dim == l.qk_dim && o.v_dim == l.v_dim,
               "layer %d: layer %d has no keys and values of its sizes", i, l.kv_layer);
    KQ_REQUIRE(i < begin || l.kv_layer >= begin, "layer %d and layer %d, whose keys and values it reads, cannot be split between stages", i, l.kv_layer);
    return B200_OK;
}

std::string lname(int i, const char *what) { return "l" + std::to_string(i) + "." + what; }

int64_t max_keys(const b200_stage_config &c, const b200_layer_config &l) {
    return l.window > 0 ? std::min<int64_t>(l.window, c.n_ctx) : l.chunk > 0 ? std::min<int64_t>(l.chunk, c.n_ctx) : c.n_ctx;
}

KqGqa gqa_of(const b200_stage *st, const LayerDesc &L, const RunState &r, int seq0) {
    const b200_layer_config &c = L.c;
    KqGqa a = {};
    a.n_head = c.n_head, a.kv_heads = c.n_head_kv, a.dim = c.qk_dim, a.vdim = c.v_dim, a.window = c.window, a.chunk = c.chunk;
    a.scale = c.attn_scale, a.eps = st->c.rms_eps;
    a.q_norm = L.q_norm, a.k_norm = L.k_norm;
    a.f32 = st->layers_desc->s.precision == B200_PRECISION_F32;
    a.cap = r.cap;
    const int64_t es = a.f32 ? 4 : 2, row = (int64_t)r.cap * c.n_head_kv;
    a.k = (uint8_t *)r.cache + seq0 * row * kq_gqa_ld(c.qk_dim) * es;
    a.v = (uint8_t *)r.vcache + seq0 * row * kq_gqa_ld(c.v_dim) * es;
    a.own_kv = !c.kv_shared;
    return a;
}

KqMatState mat_state_of(const LayerDesc &L, const RunState &r, int seq0) {
    const b200_layer_config &c = L.c;
    KqMatState m = {};
    m.delta = c.mixer == B200_MIXER_DELTA_STATE;
    m.heads = c.n_head, m.kv_heads = m.delta ? c.n_head_kv : c.n_head, m.dim = c.qk_dim, m.vdim = c.v_dim, m.taps = m.delta ? c.conv_taps : 0;
    m.decay = L.decay, m.conv_q = L.conv_q, m.conv_k = L.conv_k, m.conv_v = L.conv_v, m.a_log = L.a_log, m.dt_bias = L.dt_bias;
    m.s = r.s + seq0 * (int64_t)m.heads * m.vdim * kq_state_ld(m.dim);
    m.conv = m.taps ? r.conv + seq0 * m.taps * kq_state_channels(m) : nullptr;
    return m;
}

KqMoe moe_of(const b200_stage *st, const LayerDesc &L, const float *z, int64_t ldz) {
    KqMoe m = {};
    m.experts = L.c.n_expert, m.top = L.c.n_expert_used, m.h = st->c.n_embd, m.ff = L.c.n_ff_exp, m.ff_shared = L.c.n_ff_shared;
    m.z = z, m.sh_gate = z + L.at_shg, m.sh_up = z + L.at_shu, m.ldz = ldz;
    return m;
}

KqLatent latent_of(const b200_stage *st, const LayerDesc &L, const RunState &r, int seq0) {
    const b200_layer_config &c = L.c;
    KqLatent l = {};
    l.n_head = c.n_head, l.qk_dim = c.qk_dim, l.rot_dim = c.rot_dim, l.rot_dims = c.rot_dims, l.v_dim = c.v_dim, l.kv_rank = c.kv_rank;
    l.window = c.window;
    l.scale = c.attn_scale;
    l.freq = L.freq;
    l.cap = r.cap;
    l.f32 = st->layers_desc->s.precision == B200_PRECISION_F32;
    l.rot_at = kq_latent_rot_at(c.kv_rank);
    l.ld = kq_latent_ld(c.kv_rank, c.rot_dim);
    l.seq_stride = (int64_t)r.cap * l.ld;
    l.cache = (uint8_t *)r.cache + seq0 * l.seq_stride * (l.f32 ? 4 : 2);
    return l;
}

// The residual stream of a forward pass: x, plus norm_b(sub) still to be added when sub_w is set.
struct Stream {
    const float *x;
    int64_t ldx;
    const float *sub_w; // null: nothing pending
    int next;           // which of the two x buffers is free
};

struct Pass {
    b200_stage *st;
    KqLayers *k;
    int seq0, n_seq, T, pos0, rows;
    const int32_t *pos_dev;
    bool small, f32;
    unsigned classes;
    cudaStream_t s;
    Stream x;

#define GEMV_(expr) do { if (classes & CLS_GEMV) KQ_TRY(expr); } while (0)
#define ATTN_(expr) do { if (classes & CLS_ATTN) KQ_TRY(expr); } while (0)
#define OTHER_(expr) do { if (classes & CLS_OTHER) KQ_TRY(expr); } while (0)

    KqNormPrep prep(const float *norm_w, bool keep) {
        KqNormPrep p;
        p.x = x.x, p.ldx = x.ldx;
        p.norm_w = norm_w;
        p.eps = st->c.rms_eps;
        p.w_off = k->s.norm_offset;
        if (x.sub_w) {
            p.sub = k->sub, p.ld_sub = k->ldx, p.sub_w = x.sub_w;
            if (keep) p.x_out = k->x[x.next], p.ld_out = k->ldx;
        }
        return p;
    }
    void taken() { // the pending sub-layer output is now part of x
        if (!x.sub_w) return;
        x.x = k->x[x.next], x.ldx = k->ldx, x.sub_w = nullptr;
        x.next ^= 1;
    }
    static KqDenseSeg seg(const uint16_t *W, int64_t n, void *y, int64_t ldy, const float *bias = nullptr, int act = KQ_ACT_NONE,
                          int out = KQ_OUT_F32) {
        KqDenseSeg g = {};
        g.W = W, g.n_rows = (int32_t)n, g.y = y, g.ldy = ldy, g.bias = bias, g.act = act, g.out = out;
        return g;
    }
    KqDense call(int64_t K) {
        KqDense c;
        c.M = rows, c.K = (int)K, c.ldw = kq_bf16_ld(K);
        return c;
    }
    // projection of norm(x): the residual is brought up to date on the way
    b200_status project(const KqDense &c, const float *norm_w) {
        const KqNormPrep p = prep(norm_w, true);
        const int h = st->c.n_embd;
        if (small) {
            GEMV_(kq_gemv_bf16(c, p, s));
        } else if (f32) {
            OTHER_(kq_norm_prep(p, rows, h, k->h32, k->ldx, nullptr, 0, s));
            GEMV_(kq_gemm_f32(c, k->h32, k->ldx, s));
        } else {
            OTHER_(kq_norm_prep(p, rows, h, nullptr, 0, k->h16, kq_bf16_ld(h), s));
            GEMV_(kq_gemm_bf16(c, k->h16, kq_bf16_ld(h), 1, s));
        }
        taken();
        return B200_OK;
    }
    // output projection of a sub-layer: sub = W a, a in f32 (few rows, 32-bit mode) or bf16
    b200_status close(const uint16_t *W, int64_t K, const float *a32, int64_t ld32, const uint16_t *a16, const float *norm_b) {
        KqDense c = call(K);
        c.nseg = 1;
        c.seg[0] = seg(W, st->c.n_embd, k->sub, k->ldx);
        if (small) {
            KqNormPrep p;
            p.x = a32, p.ldx = ld32;
            GEMV_(kq_gemv_bf16(c, p, s));
        } else if (f32) {
            GEMV_(kq_gemm_f32(c, a32, ld32, s));
        } else {
            GEMV_(kq_gemm_bf16(c, a16, kq_bf16_ld(K), 1, s));
        }
        x.sub_w = norm_b;
        return B200_OK;
    }

    // the same of norm(o) times sigmoid(gate), o and the gate in f32
    b200_status close_normed(const uint16_t *W, int64_t K, const float *o, int64_t ldo, const float *norm_w, const float *gate, int64_t ldg, const float *norm_b) {
        KqDense c = call(K);
        c.nseg = 1;
        c.seg[0] = seg(W, st->c.n_embd, k->sub, k->ldx);
        KqNormPrep p;
        p.x = o, p.ldx = ldo, p.norm_w = norm_w, p.eps = st->c.rms_eps, p.gate = gate, p.ld_gate = ldg;
        if (small) {
            GEMV_(kq_gemv_bf16(c, p, s));
        } else if (f32) {
            OTHER_(kq_norm_prep(p, rows, (int)K, k->f[8], kq_f32_ld(K), nullptr, 0, s));
            GEMV_(kq_gemm_f32(c, k->f[8], kq_f32_ld(K), s));
        } else {
            OTHER_(kq_norm_prep(p, rows, (int)K, nullptr, 0, k->z16, kq_bf16_ld(K), s));
            GEMV_(kq_gemm_bf16(c, k->z16, kq_bf16_ld(K), 1, s));
        }
        x.sub_w = norm_b;
        return B200_OK;
    }

    b200_status recurrence(const LayerDesc &L, const RunState &r) {
        const int W = L.c.rec_width, B = L.c.rec_blocks, m = W / B;
        const int64_t ld = kq_f32_ld(W);
        float *y = k->f[0], *xi = k->f[1], *u = k->f[2], *gr = k->f[3], *gi = k->f[4], *z = k->f[5];
        KqDense c = call(st->c.n_embd);
        c.nseg = 2;
        c.seg[0] = seg(L.wy, W, y, ld, L.by, KQ_ACT_GELU_TANH);
        c.seg[1] = seg(L.wx, W, xi, ld, L.bx);
        KQ_TRY(project(c, L.pre1));
        KqRecState rs;
        rs.conv = r.conv + (int64_t)seq0 * L.c.conv_taps * W;
        rs.s = r.s + (int64_t)seq0 * W;
        if (T == 1 && small) {
            OTHER_(kq_recurrence_step(L.rec, rs, xi, ld, y, ld, n_seq, pos_dev, pos0, z, ld, s));
            return close(L.wo, W, z, ld, nullptr, L.post1);
        }
        const bool tc = !small && !f32;
        const int64_t ldu = (int64_t)B * kq_bf16_ld(m);
        OTHER_(kq_causal_conv(L.rec, rs, xi, ld, n_seq, T, pos_dev, pos0, u, ld, tc ? k->u16 : nullptr, s));
        KqDense g = call(m);
        g.nseg = 2;
        g.groups = B;
        g.seg[0] = seg(L.rec.ra, m, gr, ld, L.rec.ra_b);
        g.seg[1] = seg(L.rec.ri, m, gi, ld, L.rec.ri_b);
        g.xg = tc ? kq_bf16_ld(m) : m;
        if (small) OTHER_(kq_gemv_grouped_bf16(g, u, ld, s));
        else if (f32) OTHER_(kq_gemm_f32(g, u, ld, s));
        else OTHER_(kq_gemm_bf16(g, k->u16, ldu, 3, s)); // the gates see u in full f32
        OTHER_(kq_linear_recurrence(L.rec, rs, gr, gi, ld, u, ld, xi, ld, y, ld, n_seq, T, pos_dev, pos0, tc ? nullptr : z, ld,
                                    tc ? k->z16 : nullptr, kq_bf16_ld(W), k->rec_scratch, k->rec_scratch_bytes, s));
        return close(L.wo, W, z, ld, k->z16, L.post1);
    }

    b200_status latent(const LayerDesc &L, const RunState &r) {
        const b200_layer_config &c = L.c;
        const int H = c.n_head, hd = c.qk_dim + c.rot_dim;
        const int64_t ldq = kq_f32_ld((int64_t)H * hd), ldkv = kq_f32_ld(c.kv_rank + c.rot_dim), ldg = kq_f32_ld(H), rp = kq_f32_ld(c.kv_rank);
        const int64_t lda = kq_f32_ld((int64_t)H * c.v_dim);
        float *q = k->f[0], *kv = k->f[1], *g = k->f[2], *q_lat = k->f[3], *o_lat = k->f[4], *att = k->f[5];
        KqDense p = call(st->c.n_embd);
        p.nseg = 3;
        p.seg[0] = seg(L.wq, (int64_t)H * hd, q, ldq);
        p.seg[1] = seg(L.dkv, c.kv_rank + c.rot_dim, kv, ldkv);
        p.seg[2] = seg(L.wg, H, g, ldg);
        KQ_TRY(project(p, L.pre1));
        const KqLatent l = latent_of(st, L, r, seq0);
        const bool tc = !small && !f32;
        // prompts on tensor cores: keys and values of the visible rows are worked out per head
        if (tc && T > SMALL_ROWS && !pos_dev && k->prefill_work) {
            OTHER_(kq_latent_store(l, L.kv_norm, st->c.rms_eps, q, ldq, kv, ldkv, n_seq, T, pos_dev, pos0, nullptr, 0, s));
            const KqLatentPrefill w = {L.uk, L.uv, k->prefill_work, k->prefill_bytes};
            b200_status rc = B200_OK;
            for (int i = 0; i < n_seq && rc == B200_OK; i++) {
                KqLatent li = l;
                li.cache = (uint8_t *)l.cache + i * l.seq_stride * 2;
                if (classes & CLS_ATTN)
                    rc = kq_latent_prefill(li, w, q + (int64_t)i * T * ldq, ldq, g + (int64_t)i * T * ldg, ldg, T, pos0,
                                           k->z16 + (int64_t)i * T * kq_bf16_ld((int64_t)H * c.v_dim), kq_bf16_ld((int64_t)H * c.v_dim), s);
            }
            if (rc == B200_OK) return close(L.wo, (int64_t)H * c.v_dim, nullptr, 0, k->z16, L.post1);
            if (rc != B200_ERR_UNSUPPORTED) return rc;
            // q is rotated already: only its copy into the latent layout is missing
            KQ_TRY(copy_rotated(L, l, q, ldq, hd, q_lat));
        } else if (small) {
            const int keys = (int)max_keys(st->c, c);
            ATTN_(kq_latent_query(l, L.kv_norm, st->c.rms_eps, q, ldq, kv, ldkv, n_seq, T, pos_dev, pos0, q_lat, (int64_t)H * l.ld,
                                  absorb(L, l, hd, q_lat), s));
            ATTN_(kq_latent_attention(l, q_lat, n_seq, T, pos_dev, pos0, keys, nullptr, k->att_scratch, k->att_scratch_bytes, s));
            ATTN_(kq_latent_output(l, k->att_scratch, n_seq, T, pos_dev, pos0, keys, L.uv, g, ldg, att, lda, s));
            return close(L.wo, (int64_t)H * c.v_dim, att, lda, nullptr, L.post1);
        } else {
            OTHER_(kq_latent_store(l, L.kv_norm, st->c.rms_eps, q, ldq, kv, ldkv, n_seq, T, pos_dev, pos0, q_lat, (int64_t)H * l.ld, s));
        }
        ATTN_(kq_gemm_f32(absorb(L, l, hd, q_lat), q, ldq, s));
        ATTN_(kq_latent_attention(l, q_lat, n_seq, T, pos_dev, pos0, (int)max_keys(st->c, c), o_lat, nullptr, 0, s));
        KqDense v = call(c.kv_rank);
        v.nseg = 1;
        v.groups = H;
        v.xg = rp;
        v.head_gate = g;
        v.ld_gate = ldg;
        v.seg[0] = tc ? seg(L.uv, c.v_dim, k->z16, kq_bf16_ld((int64_t)H * c.v_dim), nullptr, KQ_ACT_NONE, KQ_OUT_BF16)
                      : seg(L.uv, c.v_dim, att, lda);
        ATTN_(kq_gemm_f32(v, o_lat, H * rp, s));
        return close(L.wo, (int64_t)H * c.v_dim, att, lda, k->z16, L.post1);
    }
    // q_lat[h] = W_uk[h]^T q_unrot, into rows laid out like a cache row
    KqDense absorb(const LayerDesc &L, const KqLatent &l, int hd, float *q_lat) {
        KqDense a = call(L.c.qk_dim);
        a.nseg = 1;
        a.groups = L.c.n_head;
        a.xg = hd;
        a.seg[0] = seg(L.uk_t, L.c.kv_rank, q_lat, (int64_t)L.c.n_head * l.ld);
        a.seg[0].head_in = L.c.kv_rank;
        a.seg[0].head_out = l.ld;
        return a;
    }
    b200_status copy_rotated(const LayerDesc &L, const KqLatent &l, const float *q, int64_t ldq, int hd, float *q_lat) {
        KQ_CUDA(cudaMemsetAsync(q_lat, 0, (size_t)rows * L.c.n_head * l.ld * 4, s));
        for (int i = 0; i < rows && L.c.rot_dim; i++)
            KQ_CUDA(cudaMemcpy2DAsync(q_lat + (int64_t)i * L.c.n_head * l.ld + l.rot_at, (size_t)l.ld * 4, q + i * ldq + L.c.qk_dim, (size_t)hd * 4,
                                      (size_t)L.c.rot_dim * 4, (size_t)L.c.n_head, cudaMemcpyDeviceToDevice, s));
        return B200_OK;
    }

    // all projections of a mixer's input, side by side in f[0]
    b200_status project_in(const LayerDesc &L, int64_t &ldp) {
        ldp = kq_f32_ld(L.in_rows);
        KqDense p = call(st->c.n_embd);
        p.nseg = 1;
        p.seg[0] = seg(L.win, L.in_rows, k->f[0], ldp);
        return project(p, L.pre1);
    }

    b200_status gqa(const LayerDesc &L, const RunState &r) {
        const b200_layer_config &c = L.c;
        const int64_t K = (int64_t)c.n_head * c.v_dim, lda = kq_f32_ld(K), ld16 = kq_bf16_ld(K);
        int64_t ldp;
        KQ_TRY(project_in(L, ldp));
        float *q = k->f[0] + L.at_q, *att = k->f[6];
        const float *kk = k->f[0] + L.at_k, *v = k->f[0] + L.at_v;
        const KqGqa a = gqa_of(st, L, r, seq0);
        const bool tc = !small && !f32, fused = T == 1;
        const int keys = (int)max_keys(st->c, c);
        if (!fused) OTHER_(kq_gqa_store(a, q, kk, v, ldp, n_seq, T, pos_dev, pos0, s));
        if (tc && T > SMALL_ROWS && !pos_dev && kq_prompt_attention_fits(c.qk_dim, 0, c.v_dim)) {
            KqPromptAttn w;
            w.ldq = ldp, w.rows = w.ring = r.cap, w.n_head = c.n_head, w.kv_heads = c.n_head_kv, w.dim = c.qk_dim, w.vdim = c.v_dim;
            w.T = T, w.pos0 = pos0, w.window = c.window, w.chunk = c.chunk, w.scale = c.attn_scale, w.ldo = ld16;
            for (int i = 0; i < n_seq; i++) {
                const int64_t row = (int64_t)i * r.cap * c.n_head_kv;
                w.q = q + (int64_t)i * T * ldp;
                w.k = (const uint16_t *)a.k + row * kq_gqa_ld(c.qk_dim), w.v = (const uint16_t *)a.v + row * kq_gqa_ld(c.v_dim);
                w.out = k->z16 + (int64_t)i * T * ld16;
                ATTN_(kq_prompt_attention(w, s));
            }
        } else {
            ATTN_(kq_gqa_attention(a, fused, q, kk, v, ldp, n_seq, T, pos_dev, pos0, keys, tc ? nullptr : att, lda, tc ? k->z16 : nullptr, ld16,
                                   k->att_scratch, k->att_scratch_bytes, k->gqa_counters, s));
        }
        return close(L.wo, K, att, lda, k->z16, L.post1);
    }

    // linear attention with a matrix state per head, under fixed decays or the delta rule
    b200_status mat_state(const LayerDesc &L, const RunState &r) {
        const b200_layer_config &c = L.c;
        const KqMatState m = mat_state_of(L, r, seq0);
        const int64_t K = (int64_t)m.heads * m.vdim, ldv = kq_f32_ld(K), ld16 = kq_bf16_ld(K), ldg = kq_f32_ld((int64_t)m.heads * m.dim);
        int64_t ldp;
        KQ_TRY(project_in(L, ldp));
        const float *in = k->f[0], *gate = in + L.at_g; // under the delta rule at_g is the gate's low-rank input
        const KqStateIn si = {in + L.at_q, in + L.at_k, in + L.at_v, in + L.at_b, k->f[4], ldp, ldg};
        float *z = k->f[8], *o = k->f[6];
        if (T == 1 && small) {
            KqStateStep x;
            if (m.delta) {
                x.a1 = in + L.at_a, x.g1 = gate, x.a2 = L.a2, x.g2 = L.g2, x.a_rank = c.decay_rank, x.g_rank = c.gate_rank;
                x.norm_w = L.o_norm, x.eps = st->c.rms_eps;
            }
            OTHER_(kq_state_step(m, si, x, n_seq, pos_dev, pos0, z, ldv, s));
            return m.delta ? close(L.wo, K, z, ldv, nullptr, L.post1) : close_normed(L.wo, K, z, ldv, L.o_norm, gate, ldp, L.post1);
        }
        const bool tc = !small && !f32;
        if (m.delta) { // second halves of the low-rank projections; the decays' with the first half's result in full f32
            KqDense d = call(c.decay_rank), g = call(c.gate_rank);
            d.nseg = g.nseg = 1;
            d.seg[0] = seg(L.a2, (int64_t)m.heads * m.dim, k->f[4], ldg);
            g.seg[0] = seg(L.g2, K, k->f[5], ldv);
            if (small) {
                KqNormPrep pd, pg;
                pd.x = in + L.at_a, pg.x = gate, pd.ldx = pg.ldx = ldp;
                OTHER_(kq_gemv_bf16(d, pd, s));
                OTHER_(kq_gemv_bf16(g, pg, s));
            } else if (f32) {
                OTHER_(kq_gemm_f32(d, in + L.at_a, ldp, s));
                OTHER_(kq_gemm_f32(g, gate, ldp, s));
            } else {
                const int64_t lda = kq_bf16_ld(c.decay_rank);
                uint16_t *g16 = k->u16 + 3 * rows * lda;
                OTHER_(kq_rank_operands(in + L.at_a, c.decay_rank, k->u16, gate, c.gate_rank, g16, ldp, rows, s));
                OTHER_(kq_gemm_bf16(d, k->u16, lda, 3, s));
                OTHER_(kq_gemm_bf16(g, g16, kq_bf16_ld(c.gate_rank), 1, s));
            }
        }
        if (tc && kq_state_chunks_fit(m)) {
            OTHER_(kq_state_chunks(m, si, k->state_tok, n_seq, T, pos_dev, pos0, s));
            OTHER_(kq_state_chunk_walk(m, si, k->state_tok, n_seq, T, pos_dev, pos0, o, ldv, s));
        } else {
            OTHER_(kq_state_tokens(m, si, k->state_tok, n_seq, T, pos_dev, pos0, s));
            OTHER_(kq_state_scan(m, si, k->state_tok, n_seq, T, pos_dev, pos0, o, ldv, s));
        }
        if (!m.delta) return close_normed(L.wo, K, o, ldv, L.o_norm, gate, ldp, L.post1);
        OTHER_(kq_head_norm_gate(o, ldv, k->f[5], ldv, L.o_norm, st->c.rms_eps, rows, m.heads, m.vdim, tc ? nullptr : z, ldv, tc ? k->z16 : nullptr, ld16, s));
        return close(L.wo, K, z, ldv, k->z16, L.post1);
    }

    b200_status moe(const LayerDesc &L) {
        const b200_layer_config &c = L.c;
        const int h = st->c.n_embd, ff = c.n_ff_exp, ffs = c.n_ff_shared;
        const int64_t ldz = kq_f32_ld(L.r_rows), ldf = kq_f32_ld(ff), ld16 = kq_bf16_ld(h), lds = kq_bf16_ld(std::max(ffs, 1)), lds32 = kq_f32_ld(std::max(ffs, 1));
        float *z = k->f[0];
        KqDense p = call(h);
        p.nseg = 1;
        p.seg[0] = seg(L.wr, L.r_rows, z, ldz, L.r_bias);
        if (small && L.pre2) { // the experts read the normed row: it is made once
            OTHER_(kq_norm_prep(prep(L.pre2, true), rows, h, k->h32, k->ldx, nullptr, 0, s));
            taken();
            KqNormPrep n;
            n.x = k->h32, n.ldx = k->ldx;
            GEMV_(kq_gemv_bf16(p, n, s));
        } else {
            KQ_TRY(project(p, L.pre2));
        }
        const KqMoe m = moe_of(st, L, z, ldz);
        x.sub_w = L.post2;
        if (small) {
            GEMV_(kq_moe_few_gate_up(m, L.pre2 ? k->h32 : x.x, L.pre2 ? k->ldx : x.ldx, rows, L.gate, L.up, k->moe_act, ldf, k->moe.ids, k->moe.wts, s));
            GEMV_(kq_moe_few_down(m, k->moe_act, ldf, k->moe.ids, k->moe.wts, rows, L.down, L.sh_down, k->sub, k->ldx, s));
            return B200_OK;
        }
        OTHER_(kq_moe_route(m, rows, k->moe, f32 ? k->act32 : nullptr, lds32, f32 ? nullptr : k->act16, lds, s));
        OTHER_(kq_moe_order(m, rows, k->moe, s));
        OTHER_(kq_moe_gather(m, rows, k->moe, f32 ? (const void *)k->h32 : k->h16, k->moe_x, f32 ? k->ldx : ld16, f32 ? 4 : 2, s));
        KqDense g = call(h), d = call(ff), sh = call(ffs);
        g.M = d.M = (int)(kq_moe_max_tiles((int64_t)rows * c.n_expert_used, c.n_expert) * KQ_TILE_M);
        g.experts = d.experts = c.n_expert;
        g.tile_expert = d.tile_expert = k->moe.tile_expert, g.n_tiles = d.n_tiles = k->moe.n_tiles;
        g.nseg = 2, g.glu = KQ_GLU_SILU;
        g.seg[0] = f32 ? seg(L.gate, ff, k->moe_h, ldf) : seg(L.gate, ff, k->moe_h, kq_bf16_ld(ff), nullptr, KQ_ACT_NONE, KQ_OUT_BF16);
        if (!f32) g.seg[0].pad_cols = (int32_t)kq_bf16_ld(ff);
        g.seg[1] = seg(L.up, ff, nullptr, 0);
        d.nseg = sh.nseg = 1;
        d.seg[0] = seg(L.down, h, k->moe_y, k->ldx);
        sh.seg[0] = seg(L.sh_down, h, k->sub, k->ldx);
        if (f32) {
            GEMV_(kq_gemm_f32(g, (const float *)k->moe_x, k->ldx, s));
            GEMV_(kq_gemm_f32(d, (const float *)k->moe_h, ldf, s));
            if (ffs) GEMV_(kq_gemm_f32(sh, k->act32, lds32, s));
        } else {
            GEMV_(kq_gemm_bf16(g, (const uint16_t *)k->moe_x, ld16, 1, s));
            GEMV_(kq_gemm_bf16(d, (const uint16_t *)k->moe_h, kq_bf16_ld(ff), 1, s));
            if (ffs) GEMV_(kq_gemm_bf16(sh, k->act16, lds, 1, s));
        }
        OTHER_(kq_moe_combine(m, rows, k->moe, k->moe_y, k->ldx, k->sub, k->ldx, ffs == 0, s));
        return B200_OK;
    }

    // the token's own embedding for this layer, behind a gate made from the residual
    b200_status side(const LayerDesc &L, int layer) {
        const int sd = k->s.side_dim;
        const bool tc = !small && !f32;
        KqDense c = call(st->c.n_embd);
        c.nseg = 1;
        c.seg[0] = tc ? seg(L.side_gate, sd, k->u16, kq_bf16_ld(sd), nullptr, KQ_ACT_GELU_TANH, KQ_OUT_BF16)
                      : seg(L.side_gate, sd, k->f[1], kq_f32_ld(sd), nullptr, KQ_ACT_GELU_TANH);
        if (tc) c.seg[0].pad_cols = (int32_t)kq_bf16_ld(sd);
        c.row_mul = k->side_rows + (int64_t)layer * sd;
        c.ld_mul = kq_bf16_ld((int64_t)st->c.n_layer * sd);
        KQ_TRY(project(c, nullptr));
        return close(L.side_proj, sd, k->f[1], kq_f32_ld(sd), k->u16, L.side_norm);
    }

    b200_status feed_forward(const LayerDesc &L) {
        const int ff = L.c.n_ff;
        const bool tc = !small && !f32;
        KqDense c = call(st->c.n_embd);
        c.nseg = 2;
        c.glu = KQ_GLU_CLAMPED;
        c.glu_limit = L.c.glu_limit;
        c.glu_alpha = L.c.glu_alpha;
        c.seg[0] = tc ? seg(L.gate, ff, k->act16, kq_bf16_ld(ff), nullptr, KQ_ACT_NONE, KQ_OUT_BF16) : seg(L.gate, ff, k->act32, kq_f32_ld(ff));
        if (tc) c.seg[0].pad_cols = (int32_t)kq_bf16_ld(ff);
        c.seg[1] = seg(L.up, ff, nullptr, 0);
        KQ_TRY(project(c, L.pre2));
        return close(L.down, ff, k->act32, kq_f32_ld(ff), k->act16, L.post2);
    }

    b200_status head(float *logits, int all_logits, int32_t *next_tokens) {
        const b200_stage_config &c = st->c;
        const int out_rows = all_logits ? rows : n_seq, h = c.n_embd;
        float *lg = logits ? logits : st->logits_int;
        if (!lg || !(logits || next_tokens)) return B200_OK;
        KQ_REQUIRE(logits || out_rows <= c.n_seq, "stage: internal logits hold one row per sequence");
        KqNormPrep p = prep(k->final_norm, false);
        if (!all_logits) { // last token of each sequence
            p.x += (int64_t)(T - 1) * p.ldx, p.ldx *= T;
            if (p.sub) p.sub += (int64_t)(T - 1) * p.ld_sub, p.ld_sub *= T;
        }
        KqDense d = call(h);
        d.M = out_rows;
        d.nseg = 1;
        d.seg[0] = seg(k->embed, c.n_vocab, lg, c.n_vocab, nullptr, k->s.logit_softcap > 0.f ? KQ_ACT_SOFT_CAP : KQ_ACT_NONE);
        d.cap = k->s.logit_softcap;
        if (out_rows <= SMALL_ROWS) {
            GEMV_(kq_gemv_bf16(d, p, s));
        } else if (f32) {
            OTHER_(kq_norm_prep(p, out_rows, h, k->h32, k->ldx, nullptr, 0, s));
            GEMV_(kq_gemm_f32(d, k->h32, k->ldx, s));
        } else {
            OTHER_(kq_norm_prep(p, out_rows, h, nullptr, 0, k->h16, kq_bf16_ld(h), s));
            GEMV_(kq_gemm_bf16(d, k->h16, kq_bf16_ld(h), 1, s));
        }
        if (next_tokens)
            OTHER_(b200_logit_signals(lg, out_rows, c.n_vocab, nullptr, nullptr, next_tokens, st->scan_scratch, st->scan_scratch_bytes, s));
        return B200_OK;
    }
    // the residual stream as it stands, into a buffer of n_embd-wide rows
    b200_status residual_to(float *out) {
        KqNormPrep p = prep(nullptr, false);
        p.x_out = out;
        p.ld_out = st->c.n_embd;
        OTHER_(kq_norm_prep(p, rows, st->c.n_embd, nullptr, 0, nullptr, 0, s));
        return B200_OK;
    }
};

} // namespace

b200_status kq_layers_forward(b200_stage *st, const int32_t *tokens, const float *hidden_in, int seq0, int n_seq, int T, int pos0,
                              bool pos_from_dev, float *hidden_out, float *logits, int all_logits, int32_t *next_tokens, cudaStream_t s,
                              unsigned classes) {
    KqLayers *k = st->layers_desc.get();
    const b200_stage_config &c = st->c;
    Pass P;
    P.st = st, P.k = k, P.seq0 = seq0, P.n_seq = n_seq, P.T = T, P.pos0 = pos0, P.rows = n_seq * T;
    P.pos_dev = pos_from_dev ? st->pos0_dev : nullptr;
    P.small = P.rows <= SMALL_ROWS;
    P.f32 = k->s.precision == B200_PRECISION_F32;
    P.classes = classes;
    P.s = s;
    P.x = {hidden_in, c.n_embd, nullptr, 0};
    if (c.has_embd) {
        if (classes & CLS_OTHER) KQ_TRY(kq_embed_bf16(k->embed, kq_bf16_ld(c.n_embd), tokens, P.rows, c.n_embd, k->s.embd_scale, k->x[0], k->ldx, s));
        P.x = {k->x[0], k->ldx, nullptr, 1};
    }
    if (k->s.side_dim && (classes & CLS_OTHER))
        KQ_TRY(kq_gather_bf16(k->side_embed, tokens, P.rows, k->side_rows, kq_bf16_ld((int64_t)c.n_layer * k->s.side_dim), s));
    int run = 0;
    for (const RunState &r : k->runs) {
        const LayerDesc &L = k->layers[r.layer - c.layer_begin];
        switch (L.c.mixer) {
        case B200_MIXER_LATENT_ATTN: KQ_TRY(P.latent(L, r)); break;
        case B200_MIXER_LINEAR_REC: KQ_TRY(P.recurrence(L, r)); break;
        case B200_MIXER_GQA: KQ_TRY(P.gqa(L, r)); break;
        default: KQ_TRY(P.mat_state(L, r)); break;
        }
        if (L.c.ffn != B200_FFN_NONE) KQ_TRY(L.c.ffn == B200_FFN_MOE ? P.moe(L) : P.feed_forward(L));
        if (k->s.side_dim) KQ_TRY(P.side(L, r.layer));
        if (k->trace) KQ_TRY(P.residual_to(k->trace + (int64_t)run * P.rows * c.n_embd));
        run++;
    }
    if (hidden_out) KQ_TRY(P.residual_to(hidden_out));
    if (c.has_output) KQ_TRY(P.head(logits, all_logits, next_tokens));
    return B200_OK;
}

b200_status kq_layers_resolve(b200_stage *st) {
    KqLayers *k = st->layers_desc.get();
    const b200_stage_config &c = st->c;
    auto f32 = [&](const std::string &n) { return (const float *)kq_stage_find(st, n)->dev; };
    auto b16 = [&](const std::string &n) { return (const uint16_t *)kq_stage_find(st, n)->dev; };
    for (int i = c.layer_begin; i < c.layer_end; i++) {
        LayerDesc &L = k->layers[i - c.layer_begin];
        const bool sandwich = k->s.norm_place == B200_NORM_SANDWICH;
        if (sandwich) L.pre1 = f32(lname(i, "norm1"));
        L.post1 = f32(lname(i, sandwich ? "norm1b" : "norm1"));
        L.wo = b16(lname(i, "mix.o"));
        if (L.in_pack >= 0) {
            const Pack &in = k->packs[L.in_pack];
            L.win = (const uint16_t *)in.dev;
            L.in_rows = in.rows;
            auto at = [&](const char *leaf) {
                for (size_t j = 0; j < in.names.size(); j++)
                    if (in.names[j] == lname(i, leaf)) return in.at[j];
                return (int64_t)0;
            };
            L.at_q = at("mix.q"), L.at_k = at("mix.k"), L.at_v = at("mix.v"), L.at_b = at("mix.b"), L.at_a = at("mix.a1");
            L.at_g = at(L.c.mixer == B200_MIXER_DELTA_STATE ? "mix.g1" : "mix.g");
        }
        if (L.c.mixer == B200_MIXER_GQA) {
            L.q_norm = f32(lname(i, "mix.q.norm"));
            if (!L.c.kv_shared) L.k_norm = f32(lname(i, "mix.k.norm"));
        } else if (L.c.mixer == B200_MIXER_DECAY_STATE) {
            L.o_norm = f32(lname(i, "mix.norm")), L.decay = f32(lname(i, "mix.decay"));
        } else if (L.c.mixer == B200_MIXER_DELTA_STATE) {
            L.o_norm = f32(lname(i, "mix.norm")), L.a_log = f32(lname(i, "mix.A_log")), L.dt_bias = f32(lname(i, "mix.dt_bias"));
            L.conv_q = f32(lname(i, "mix.q.conv")), L.conv_k = f32(lname(i, "mix.k.conv")), L.conv_v = f32(lname(i, "mix.v.conv"));
            L.a2 = b16(lname(i, "mix.a2")), L.g2 = b16(lname(i, "mix.g2"));
        } else if (L.c.mixer == B200_MIXER_LINEAR_REC) {
            L.wy = b16(lname(i, "mix.y")), L.by = f32(lname(i, "mix.y.b"));
            L.wx = b16(lname(i, "mix.x")), L.bx = f32(lname(i, "mix.x.b"));
            L.rec.conv_w = f32(lname(i, "mix.conv")), L.rec.conv_b = f32(lname(i, "mix.conv.b"));
            L.rec.ra = b16(lname(i, "mix.ra")), L.rec.ra_b = f32(lname(i, "mix.ra.b"));
            L.rec.ri = b16(lname(i, "mix.ri")), L.rec.ri_b = f32(lname(i, "mix.ri.b"));
            L.rec.lam = f32(lname(i, "mix.lam"));
            L.rec.decay = L.c.rec_decay;
            L.rec.width = L.c.rec_width, L.rec.blocks = L.c.rec_blocks, L.rec.taps = L.c.conv_taps;
        } else {
            L.wq = b16(lname(i, "mix.q")), L.dkv = b16(lname(i, "mix.dkv")), L.kv_norm = f32(lname(i, "mix.dkv.norm"));
            L.uk = b16(lname(i, "mix.uk")), L.uv = b16(lname(i, "mix.uv")), L.wg = b16(lname(i, "mix.g"));
            const int64_t ld = kq_bf16_ld(L.c.qk_dim), n = (int64_t)L.c.n_head * L.c.kv_rank * ld;
            transpose_heads_kernel<<<(unsigned)kq_div_up(n, 256), 256>>>(L.uk, kq_bf16_ld(L.c.kv_rank), L.c.n_head, L.c.qk_dim, L.c.kv_rank, L.uk_t, ld);
            KQ_LAUNCH_CHECK();
        }
        if (L.c.ffn != B200_FFN_NONE) {
            if (sandwich) L.pre2 = f32(lname(i, "norm2"));
            L.post2 = f32(lname(i, sandwich ? "norm2b" : "norm2"));
        }
        if (k->s.side_dim) L.side_gate = b16(lname(i, "side.gate")), L.side_proj = b16(lname(i, "side.proj")), L.side_norm = f32(lname(i, "side.norm"));
        if (L.c.ffn == B200_FFN_MOE) {
            const Pack &rp = k->packs[L.r_pack];
            L.wr = (const uint16_t *)rp.dev, L.r_rows = rp.rows;
            if (L.c.n_ff_shared) L.at_shg = rp.at[1], L.at_shu = rp.at[2], L.sh_down = b16(lname(i, "mlp.shared.down"));
            L.gate = (const uint16_t *)k->packs[L.gate_pack].dev, L.up = (const uint16_t *)k->packs[L.up_pack].dev;
            L.down = (const uint16_t *)k->packs[L.down_pack].dev;
            KQ_CUDA(cudaMemcpy(L.r_bias, f32(lname(i, "mlp.router.b")), (size_t)L.c.n_expert * 4, cudaMemcpyDeviceToDevice));
        } else if (L.c.ffn != B200_FFN_NONE) {
            L.gate = b16(lname(i, "mlp.gate")), L.up = b16(lname(i, "mlp.up")), L.down = b16(lname(i, "mlp.down"));
        }
    }
    if (c.has_embd || c.has_output) k->embed = b16("embed");
    if (k->s.side_dim) k->side_embed = b16("side.embed");
    if (c.has_output) k->final_norm = f32("final.norm");
    KQ_CUDA(cudaDeviceSynchronize());
    return B200_OK;
}

b200_status kq_layers_check_pos(b200_stage *st, int seq0, int n_seq, int T, int pos0) {
    const KqLayers *k = st->layers_desc.get();
    (void)T;
    for (int i = seq0; i < seq0 + n_seq; i++)
        if (pos0 != 0 && pos0 != k->seq_pos[i]) {
            kq_set_error("stage_forward: sequence %d stands at position %d, the call starts at %d", i, k->seq_pos[i], pos0);
            return B200_ERR_STATE;
        }
    return B200_OK;
}

void kq_layers_advance(b200_stage *st, int seq0, int n_seq, int pos) {
    if (!st->layers_desc) return;
    for (int i = seq0; i < seq0 + n_seq; i++) st->layers_desc->seq_pos[i] = pos;
}

bool kq_layers_read_tokens(const b200_stage *st) { return st->layers_desc && st->layers_desc->s.side_dim > 0; }

bool kq_layers_plain_norm(const b200_stage *st, const std::string &name) {
    const bool vector_norm = name.find("norm") != std::string::npos;
    // inside a mixer and of the token input norms are plain; the others are relative to the model's offset
    const bool inner = name.find(".mix.") != std::string::npos || name.find(".side.") != std::string::npos;
    return vector_norm && (inner || st->layers_desc->s.norm_offset == 0.f);
}

bool kq_layers_tracing(const b200_stage *st) { return st->layers_desc && st->layers_desc->trace; }

b200_status kq_layers_peek(b200_stage *st, const char *which, float *host_out, size_t n_floats) {
    KqLayers *k = st->layers_desc.get();
    KQ_REQUIRE(std::string(which) == "sub", "stage_peek: no buffer named %s (sub: the last sub-layer's output)", which);
    KQ_REQUIRE(n_floats <= (size_t)st->rows_max * k->ldx, "stage_peek: %s holds %zu floats", which, (size_t)st->rows_max * k->ldx);
    KqDevGuard dev_guard(st->c.device);
    KQ_CUDA(cudaDeviceSynchronize());
    KQ_CUDA(cudaMemcpy(host_out, k->sub, n_floats * 4, cudaMemcpyDeviceToHost));
    return B200_OK;
}

extern "C" {

b200_status b200_stage_create_layers(const b200_stage_config *cfg, const b200_stack_config *stack, const b200_layer_config *layers,
                                     b200_stage **out) {
    KQ_REQUIRE(cfg && stack && layers && out, "stage_create_layers: null argument");
    b200_stage_config c = *cfg;
    KQ_REQUIRE(c.n_embd > 0 && c.n_layer > 0 && c.layer_begin >= 0 && c.layer_begin <= c.layer_end && c.layer_end <= c.n_layer,
               "stage: bad layer range [%d,%d) of %d", c.layer_begin, c.layer_end, c.n_layer);
    KQ_REQUIRE(c.n_ctx > 0 && c.n_seq > 0 && c.n_ubatch > 0, "stage: n_ctx, n_seq, n_ubatch");
    KQ_REQUIRE(!(c.has_embd || c.has_output) || c.n_vocab > 0, "stage: n_vocab");
    KQ_REQUIRE(stack->precision == B200_PRECISION_BF16 || stack->precision == B200_PRECISION_F32, "stage: precision %d", stack->precision);
    const bool loop = stack->loop_times > 1 && stack->loop_stop > stack->loop_start;
    if (loop) {
        KQ_REQUIRE(stack->loop_start >= 0 && stack->loop_stop <= c.n_layer, "stage: looped layers [%d,%d) of %d", stack->loop_start,
                   stack->loop_stop, c.n_layer);
        const bool outside = c.layer_end <= stack->loop_start || c.layer_begin >= stack->loop_stop;
        const bool inside = c.layer_begin <= stack->loop_start && c.layer_end >= stack->loop_stop;
        KQ_REQUIRE(outside || inside, "stage: the looped layers [%d,%d) cannot be split between stages", stack->loop_start, stack->loop_stop);
    }
    KQ_REQUIRE(stack->norm_place == B200_NORM_SANDWICH || stack->norm_place == B200_NORM_OUTPUT, "stage: norm place %d", stack->norm_place);
    KQ_REQUIRE(stack->side_dim >= 0 && (!stack->side_dim || c.n_vocab > 0), "stage: token input of %d values", stack->side_dim);
    for (int i = 0; i < c.n_layer; i++) KQ_TRY(check_layer(layers[i], i));
    for (int i = 0; i < c.layer_end; i++) KQ_TRY(check_shared(layers, i, c.layer_begin));
    KqDevGuard dev_guard(c.device);
    b200_stage *st = new b200_stage();
    c.n_head = c.n_head_kv = c.head_dim = c.n_ff = c.n_expert = 0;
    st->c = c;
    st->layers_desc.reset(new KqLayers());
    KqLayers *k = st->layers_desc.get();
    k->s = *stack;
    k->seq_pos.assign(c.n_seq, -1);
    for (int i = c.layer_begin; i < c.layer_end; i++) {
        LayerDesc L;
        L.c = layers[i];
        k->layers.push_back(L);
        const int times = loop && i == stack->loop_start ? stack->loop_times : 1;
        const int last = loop && i == stack->loop_start ? stack->loop_stop : i + 1;
        for (int t = 0; t < times; t++)
            for (int j = i; j < last; j++)
                if (times > 1 || !loop || j < stack->loop_start || j >= stack->loop_stop) {
                    RunState r;
                    r.layer = j;
                    k->runs.push_back(r);
                }
    }
    const int64_t h = c.n_embd, R = c.n_ubatch;
    if (c.has_embd || c.has_output) kq_stage_add_tensor(st, "embed", B200_TYPE_BF16, h, c.n_vocab, 1);
    if (stack->side_dim) kq_stage_add_tensor(st, "side.embed", B200_TYPE_BF16, (int64_t)c.n_layer * stack->side_dim, c.n_vocab, 1);
    int64_t fmax[9] = {}, wmax16 = 0, u16max = 0, ffmax = 0, scratch = 0, rec_scratch = 0, prefill = 0;
    int64_t gqa_counters = 0, state_rec = 0, state_val = 0, few_act = 0, moe_rows = 0, moe_ff = 0, moe_pairs = 0, moe_tiles = 0;
    const bool f32 = stack->precision == B200_PRECISION_F32;
    auto grow = [](int64_t &a, int64_t b) { a = std::max(a, b); };
    for (int i = c.layer_begin; i < c.layer_end; i++) {
        const b200_layer_config &l = layers[i];
        auto mat = [&](const char *w, int64_t in, int64_t rows, int64_t n = 1) { kq_stage_add_tensor(st, lname(i, w), B200_TYPE_BF16, in, rows, n); };
        auto vec = [&](const char *w, int64_t a, int64_t b = 1) { kq_stage_add_tensor(st, lname(i, w), B200_TYPE_F32, a, b, 1); };
        const bool sandwich = stack->norm_place == B200_NORM_SANDWICH;
        LayerDesc &L = k->layers[i - c.layer_begin];
        auto pack = [&](std::vector<std::string> names, int64_t align) { // of matrices that are tensors already
            Pack p;
            p.names = std::move(names), p.align = align;
            k->packs.push_back(p);
            return (int)k->packs.size() - 1;
        };
        vec("norm1", h);
        if (sandwich) vec("norm1b", h);
        if (l.mixer == B200_MIXER_GQA) {
            const int64_t H = l.n_head, G = l.n_head_kv, K = H * l.v_dim;
            std::vector<std::string> in = {lname(i, "mix.q")};
            mat("mix.q", h, H * l.qk_dim);
            vec("mix.q.norm", l.qk_dim);
            if (!l.kv_shared) {
                mat("mix.k", h, G * l.qk_dim);
                vec("mix.k.norm", l.qk_dim);
                mat("mix.v", h, G * l.v_dim);
                in.push_back(lname(i, "mix.k")), in.push_back(lname(i, "mix.v"));
            }
            mat("mix.o", K, h);
            L.in_pack = pack(in, 8);
            grow(fmax[6], kq_f32_ld(K));
            grow(wmax16, kq_bf16_ld(K));
            KqGqa a = {};
            a.n_head = l.n_head, a.kv_heads = l.n_head_kv, a.dim = l.qk_dim, a.vdim = l.v_dim;
            grow(gqa_counters, kq_gqa_counters(a));
            grow(scratch, (int64_t)kq_gqa_scratch_bytes(a, (int)std::max<int64_t>(R, c.n_seq), (int)max_keys(c, l)));
        } else if (l.mixer == B200_MIXER_DECAY_STATE || l.mixer == B200_MIXER_DELTA_STATE) {
            const bool delta = l.mixer == B200_MIXER_DELTA_STATE;
            const int64_t H = l.n_head, G = delta ? l.n_head_kv : l.n_head, K = H * l.v_dim;
            std::vector<std::string> in = {lname(i, "mix.q"), lname(i, "mix.k"), lname(i, "mix.v")};
            mat("mix.q", h, G * l.qk_dim);
            mat("mix.k", h, G * l.qk_dim);
            mat("mix.v", h, K);
            if (delta) {
                vec("mix.q.conv", l.conv_taps, G * l.qk_dim);
                vec("mix.k.conv", l.conv_taps, G * l.qk_dim);
                vec("mix.v.conv", l.conv_taps, K);
                mat("mix.b", h, H);
                vec("mix.A_log", H);
                mat("mix.a1", h, l.decay_rank);
                mat("mix.a2", l.decay_rank, H * l.qk_dim);
                vec("mix.dt_bias", H * l.qk_dim);
                mat("mix.g1", h, l.gate_rank);
                mat("mix.g2", l.gate_rank, K);
                vec("mix.norm", l.v_dim);
                in.push_back(lname(i, "mix.b")), in.push_back(lname(i, "mix.a1")), in.push_back(lname(i, "mix.g1"));
                grow(u16max, 3 * kq_bf16_ld(l.decay_rank) + kq_bf16_ld(l.gate_rank));
            } else {
                vec("mix.decay", H);
                mat("mix.g", h, K);
                vec("mix.norm", K);
                in.push_back(lname(i, "mix.g"));
            }
            mat("mix.o", K, h);
            L.in_pack = pack(in, 8);
            if (delta) grow(fmax[4], kq_f32_ld(H * l.qk_dim));
            for (int f : {5, 6, 8}) grow(fmax[f], kq_f32_ld(K));
            KqMatState m = {};
            m.heads = l.n_head, m.dim = l.qk_dim, m.vdim = l.v_dim, m.delta = delta;
            grow(state_rec, kq_state_rec_floats(m));
            grow(state_val, kq_state_val_floats(m));
            grow(wmax16, kq_bf16_ld(K));
        } else if (l.mixer == B200_MIXER_LINEAR_REC) {
            const int64_t W = l.rec_width, m = W / l.rec_blocks;
            mat("mix.y", h, W);
            vec("mix.y.b", W);
            mat("mix.x", h, W);
            vec("mix.x.b", W);
            vec("mix.conv", l.conv_taps, W);
            vec("mix.conv.b", W);
            mat("mix.ra", m, m, l.rec_blocks);
            vec("mix.ra.b", m, l.rec_blocks);
            mat("mix.ri", m, m, l.rec_blocks);
            vec("mix.ri.b", m, l.rec_blocks);
            vec("mix.lam", W);
            mat("mix.o", W, h);
            for (int f = 0; f < 6; f++) grow(fmax[f], kq_f32_ld(W));
            grow(wmax16, kq_bf16_ld(W));
            grow(rec_scratch, (int64_t)kq_recurrence_scratch_bytes(l.rec_width, (int)R, c.n_seq));
            grow(u16max, 3 * l.rec_blocks * kq_bf16_ld(m));
        } else {
            const int64_t H = l.n_head, hd = l.qk_dim + l.rot_dim;
            mat("mix.q", h, H * hd);
            mat("mix.dkv", h, l.kv_rank + l.rot_dim);
            vec("mix.dkv.norm", l.kv_rank);
            mat("mix.uk", l.kv_rank, H * l.qk_dim);
            mat("mix.uv", l.kv_rank, H * l.v_dim);
            mat("mix.g", h, H);
            mat("mix.o", H * l.v_dim, h);
            grow(fmax[0], kq_f32_ld(H * hd));
            grow(fmax[1], kq_f32_ld(l.kv_rank + l.rot_dim));
            grow(fmax[2], kq_f32_ld(H));
            grow(fmax[3], H * kq_latent_ld(l.kv_rank, l.rot_dim));
            grow(fmax[4], H * kq_f32_ld(l.kv_rank));
            grow(fmax[5], kq_f32_ld(H * l.v_dim));
            grow(wmax16, kq_bf16_ld(H * l.v_dim));
            KqLatent q = {};
            q.n_head = l.n_head, q.qk_dim = l.qk_dim, q.rot_dim = l.rot_dim, q.v_dim = l.v_dim, q.kv_rank = l.kv_rank, q.window = l.window;
            q.f32 = f32, q.ld = kq_latent_ld(l.kv_rank, l.rot_dim);
            grow(scratch, (int64_t)kq_latent_scratch_bytes(q, (int)max_keys(c, l)));
            if (!f32) grow(prefill, (int64_t)kq_latent_prefill_bytes(q, (int)R, (int)std::min<int64_t>(c.n_ctx, max_keys(c, l) - 1 + R)));
        }
        if (L.in_pack >= 0) {
            int64_t n = 0;
            for (const std::string &s : k->packs[L.in_pack].names) n += kq_pad(kq_stage_find(st, s)->ne[1], 8);
            grow(fmax[0], n);
        }
        if (l.ffn != B200_FFN_NONE) {
            vec("norm2", h);
            if (sandwich) vec("norm2b", h);
        }
        if (stack->side_dim) {
            mat("side.gate", h, stack->side_dim);
            mat("side.proj", stack->side_dim, h);
            vec("side.norm", h);
            grow(fmax[1], kq_f32_ld(stack->side_dim));
            grow(u16max, kq_bf16_ld(stack->side_dim));
        }
        if (l.ffn == B200_FFN_MOE) {
            auto expert = [&](const std::string &e, int64_t ff, std::vector<std::string> *to) { // gate, up, down
                const std::string n = "mlp." + e;
                mat((n + ".gate").c_str(), h, ff);
                mat((n + ".up").c_str(), h, ff);
                mat((n + ".down").c_str(), ff, h);
                if (!to) return;
                to[0].push_back(lname(i, (n + ".gate").c_str()));
                to[1].push_back(lname(i, (n + ".up").c_str()));
                to[2].push_back(lname(i, (n + ".down").c_str()));
            };
            std::vector<std::string> parts[3];
            for (int e = 0; e < l.n_expert; e++) expert("e" + std::to_string(e), l.n_ff_exp, parts);
            mat("mlp.router", h, l.n_expert);
            vec("mlp.router.b", l.n_expert);
            std::vector<std::string> in = {lname(i, "mlp.router")};
            if (l.n_ff_shared) {
                expert("shared", l.n_ff_shared, nullptr);
                in.push_back(lname(i, "mlp.shared.gate")), in.push_back(lname(i, "mlp.shared.up"));
            }
            L.gate_pack = pack(parts[0], 1), L.up_pack = pack(parts[1], 1), L.down_pack = pack(parts[2], 1);
            L.r_pack = pack(in, 8);
            grow(fmax[0], kq_pad(l.n_expert, 8) + 2 * kq_pad(l.n_ff_shared, 8));
            grow(ffmax, std::max(l.n_ff_shared, 1));
            grow(few_act, std::min<int64_t>(R, SMALL_ROWS) * l.n_expert_used * kq_f32_ld(l.n_ff_exp));
            grow(moe_pairs, R * l.n_expert_used);
            grow(moe_tiles, kq_moe_max_tiles(R * l.n_expert_used, l.n_expert));
            grow(moe_rows, kq_moe_max_tiles(R * l.n_expert_used, l.n_expert) * KQ_TILE_M);
            grow(moe_ff, l.n_ff_exp);
        } else if (l.ffn != B200_FFN_NONE) {
            mat("mlp.gate", h, l.n_ff);
            mat("mlp.up", h, l.n_ff);
            mat("mlp.down", l.n_ff, h);
            grow(ffmax, l.n_ff);
        }
    }
    if (c.has_output) kq_stage_add_tensor(st, "final.norm", B200_TYPE_F32, h, 1, 1);
    b200_status rc = B200_OK;
    auto A = [&](void *p, size_t bytes) { // zeroed: padding is read (times zero weights), so it must not hold NaNs
        void **pp = (void **)p;
        if (rc == B200_OK) rc = kq_stage_alloc(st, pp, bytes);
        if (rc == B200_OK && bytes && cudaMemset(*pp, 0, bytes) != cudaSuccess) rc = B200_ERR_CUDA;
    };
    for (Pack &p : k->packs) {
        const int64_t ld = kq_bf16_ld(kq_stage_find(st, p.names[0])->ne[0]);
        for (const std::string &n : p.names) {
            p.at.push_back(p.rows);
            p.rows += kq_pad(kq_stage_find(st, n)->ne[1], p.align);
        }
        A(&p.dev, (size_t)(p.rows * ld * 2) + 16);
        for (size_t j = 0; j < p.names.size() && rc == B200_OK; j++) kq_stage_find(st, p.names[j])->dev = (uint16_t *)p.dev + p.at[j] * ld;
    }
    for (auto &t : st->tensors)
        if (!t.dev) A(&t.dev, t.dev_bytes + 16);
    for (LayerDesc &L : k->layers)
        if (L.r_pack >= 0) A(&L.r_bias, (size_t)k->packs[L.r_pack].rows * 4);
    for (size_t i = 0; i < k->layers.size(); i++) {
        LayerDesc &L = k->layers[i];
        if (L.c.mixer != B200_MIXER_LATENT_ATTN) continue;
        A(&L.uk_t, (size_t)L.c.n_head * L.c.kv_rank * kq_bf16_ld(L.c.qk_dim) * 2);
        std::vector<double> fr(L.c.rot_dims / 2 + 1, 0.0);
        for (int j = 0; j < L.c.rot_dims / 2; j++) fr[j] = pow((double)L.c.rope_base, -2.0 * j / L.c.rot_dims);
        A(&L.freq, fr.size() * 8);
        if (rc == B200_OK && cudaMemcpy(L.freq, fr.data(), fr.size() * 8, cudaMemcpyHostToDevice) != cudaSuccess) rc = B200_ERR_CUDA;
    }
    auto ring_rows = [&](const b200_layer_config &l) { return std::min<int64_t>(c.n_ctx, max_keys(c, l) - 1 + R); };
    for (RunState &r : k->runs) {
        const b200_layer_config &l = k->layers[r.layer - c.layer_begin].c;
        size_t b;
        if (l.mixer == B200_MIXER_GQA) {
            if (l.kv_shared) { // the latest pass over that layer
                for (RunState *o = &r - 1; o >= &k->runs[0]; o--)
                    if (o->layer == l.kv_layer) {
                        r.cache = o->cache, r.vcache = o->vcache, r.cap = o->cap;
                        break;
                    }
                continue;
            }
            int64_t cap = ring_rows(l);
            for (const LayerDesc &o : k->layers) // whoever reads these rows may look further back
                if (o.c.mixer == B200_MIXER_GQA && o.c.kv_shared && o.c.kv_layer == r.layer) cap = std::max(cap, ring_rows(o.c));
            r.cap = (int)kq_pad(cap, 128); // whole key tiles of the tensor-core kernel
            const size_t rows = (size_t)c.n_seq * r.cap * l.n_head_kv * (f32 ? 4 : 2);
            A(&r.cache, b = rows * kq_gqa_ld(l.qk_dim));
            k->state_bytes += b;
            A(&r.vcache, b = rows * kq_gqa_ld(l.v_dim));
        } else if (l.mixer == B200_MIXER_DECAY_STATE || l.mixer == B200_MIXER_DELTA_STATE) {
            if (l.mixer == B200_MIXER_DELTA_STATE) {
                A(&r.conv, b = (size_t)c.n_seq * l.conv_taps * (2 * (size_t)l.n_head_kv * l.qk_dim + (size_t)l.n_head * l.v_dim) * 4);
                k->state_bytes += b;
            }
            A(&r.s, b = (size_t)c.n_seq * l.n_head * l.v_dim * kq_state_ld(l.qk_dim) * 4);
        } else if (l.mixer == B200_MIXER_LINEAR_REC) {
            A(&r.conv, b = (size_t)c.n_seq * l.conv_taps * l.rec_width * 4);
            k->state_bytes += b;
            A(&r.s, b = (size_t)c.n_seq * l.rec_width * 4);
        } else {
            r.cap = (int)ring_rows(l);
            A(&r.cache, b = (size_t)c.n_seq * r.cap * kq_latent_ld(l.kv_rank, l.rot_dim) * (f32 ? 4 : 2));
        }
        k->state_bytes += b;
    }
    st->rows_max = (int)R;
    k->ldx = kq_f32_ld(h);
    for (int i = 0; i < 2; i++) A(&k->x[i], (size_t)(R * k->ldx * 4));
    A(&k->sub, (size_t)(R * k->ldx * 4));
    const bool wide = R > SMALL_ROWS || c.n_seq > SMALL_ROWS;
    if (wide || moe_pairs) A(&k->h32, (size_t)(R * k->ldx * 4));
    if (wide) A(&k->h16, (size_t)(R * kq_bf16_ld(h) * 2));
    for (int f = 0; f < 9; f++)
        if (fmax[f]) A(&k->f[f], (size_t)(R * fmax[f] * 4));
    if (wide) A(&k->z16, (size_t)(R * wmax16 * 2));
    if (wide) A(&k->u16, (size_t)(R * u16max * 2));
    if (ffmax) A(&k->act32, (size_t)((f32 ? R : std::min<int64_t>(R, SMALL_ROWS)) * kq_f32_ld(ffmax) * 4));
    if (ffmax && wide) A(&k->act16, (size_t)(R * kq_bf16_ld(ffmax) * 2));
    if (state_rec) {
        const int64_t blocks = R / 16 + std::min<int64_t>(R, c.n_seq) + 1; // groups of 16 positions of all sequences of a call
        A(&k->state_tok.rec, (size_t)(blocks * state_rec * 4));
        A(&k->state_tok.val, (size_t)(blocks * state_val * 4));
    }
    if (gqa_counters) A(&k->gqa_counters, (size_t)gqa_counters * 4);
    if (moe_pairs) {
        A(&k->moe_act, (size_t)few_act * 4);
        A(&k->moe.ids, (size_t)moe_pairs * 4);
        A(&k->moe.wts, (size_t)moe_pairs * 4);
    }
    if (moe_pairs && wide) {
        A(&k->moe.pos, (size_t)moe_pairs * 4);
        A(&k->moe.tile_expert, (size_t)moe_tiles * 4);
        A(&k->moe.n_tiles, 16);
        A(&k->moe_x, (size_t)(moe_rows * (f32 ? k->ldx * 4 : kq_bf16_ld(h) * 2)));
        A(&k->moe_h, (size_t)(moe_rows * (f32 ? kq_f32_ld(moe_ff) * 4 : kq_bf16_ld(moe_ff) * 2)));
        A(&k->moe_y, (size_t)(moe_rows * k->ldx * 4));
    }
    if (stack->side_dim) A(&k->side_rows, (size_t)(R * kq_bf16_ld((int64_t)c.n_layer * stack->side_dim) * 2));
    k->rec_scratch_bytes = (size_t)rec_scratch;
    A(&k->rec_scratch, (size_t)rec_scratch);
    k->att_scratch_bytes = (size_t)scratch;
    A(&k->att_scratch, (size_t)scratch);
    k->prefill_bytes = wide ? (size_t)prefill : 0;
    if (k->prefill_bytes) A(&k->prefill_work, k->prefill_bytes);
    A(&st->pos0_dev, 256);
    A(&st->rid_scratch, 1024);
    A(&st->xn, (size_t)(c.n_seq * h * 4));
    A(&st->att, (size_t)(c.n_seq * h * 4));
    if (c.has_output) {
        A(&st->logits_int, (size_t)c.n_seq * c.n_vocab * 4);
        st->scan_scratch_bytes = b200_logit_signals_scratch_bytes(std::max<int64_t>(R, c.n_seq));
        A(&st->scan_scratch, st->scan_scratch_bytes);
    }
    if (rc == B200_OK && cudaStreamCreateWithFlags(&st->cap_stream, cudaStreamNonBlocking) != cudaSuccess) {
        kq_set_error("stage: cudaStreamCreate failed");
        rc = B200_ERR_CUDA;
    }
    if (rc == B200_OK && cudaDeviceSynchronize() != cudaSuccess) rc = B200_ERR_CUDA;
    if (rc != B200_OK) {
        b200_stage_free(st);
        return rc;
    }
    const char *ng = getenv("B200_NO_GRAPH");
    st->use_graph = !(ng && ng[0] == '1');
    *out = st;
    return B200_OK;
}

b200_status b200_stage_trace_residual(b200_stage *st, float *buf) {
    KQ_REQUIRE(st && st->layers_desc, "stage_trace_residual: a stage with described layers");
    st->layers_desc->trace = buf;
    return B200_OK;
}

int32_t b200_stage_layer_runs(b200_stage *st) {
    if (!st) return -1;
    return st->layers_desc ? (int32_t)st->layers_desc->runs.size() : st->c.layer_end - st->c.layer_begin;
}

int32_t b200_stage_seq_pos(b200_stage *st, int32_t seq) {
    if (!st || !st->layers_desc || seq < 0 || seq >= st->c.n_seq) return -1;
    return st->layers_desc->seq_pos[seq];
}

size_t b200_stage_state_bytes(b200_stage *st) {
    if (!st) return 0;
    if (st->layers_desc) return st->layers_desc->state_bytes / (size_t)st->c.n_seq;
    return (size_t)(st->c.layer_end - st->c.layer_begin) * st->c.n_ctx * st->c.n_head_kv * (st->k_row + st->v_row);
}

} // extern "C"
