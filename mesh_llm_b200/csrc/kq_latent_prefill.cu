// Latent attention for prompts in the expanded form: the latents of the rows that the prompt's queries can see are gathered
// out of the ring, one GEMM turns them into per-head keys and values (f16), and the tensor-core attention of
// kq_prompt_attn.cu runs over them, with the rotated key part that all heads share as the second part of a key.
#include "kq_dense.cuh"

#include <algorithm>

namespace {

// rows lo .. lo + n - 1 of the ring in order: latents to a GEMM operand, the shared key part to f16
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint16_t *cache, int ld, int cap, int rank, int rot_at, int rot, int lo, uint16_t *c,
                                                            int64_t ldc, uint16_t *kr, int64_t ldr) {
    KQ_PDL_ENTER();
    const int64_t r = blockIdx.x;
    const uint16_t *src = cache + (int64_t)((lo + (int)r) % cap) * ld;
    const int r8 = rank / 8 * 8;
    for (int i = threadIdx.x * 8; i < r8; i += 128 * 8) *reinterpret_cast<uint4 *>(c + r * ldc + i) = *reinterpret_cast<const uint4 *>(src + i);
    for (int i = r8 + threadIdx.x; i < ldc; i += 128) c[r * ldc + i] = i < rank ? src[i] : 0;
    for (int i = threadIdx.x; i < ldr; i += 128) kr[r * ldr + i] = i < rot ? kq_f2h_sat(kq_bf2f(src[rot_at + i])) : 0;
}

struct Work {
    int64_t ldc, ldr, ldk, ldv; // elements per row
    size_t at_r, at_k, at_v, total;
};
Work layout(const KqLatent &l, int64_t keys) {
    Work w;
    auto up = [](size_t v) { return (v + 255) / 256 * 256; };
    w.ldc = kq_bf16_ld(l.kv_rank);
    w.ldr = kq_pad(l.rot_dim, 64);
    w.ldk = l.n_head * kq_pad(l.qk_dim, 64);
    w.ldv = l.n_head * kq_pad(l.v_dim, 64);
    w.at_r = up((size_t)(keys * w.ldc * 2));
    w.at_k = w.at_r + up((size_t)(keys * w.ldr * 2));
    w.at_v = w.at_k + up((size_t)(keys * w.ldk * 2));
    w.total = w.at_v + up((size_t)(keys * w.ldv * 2));
    return w;
}
bool supported(const KqLatent &l) { return kq_prompt_attention_fits(l.qk_dim, l.rot_dim, l.v_dim); }

} // namespace

size_t kq_latent_prefill_bytes(const KqLatent &l, int max_rows, int max_keys) {
    (void)max_rows;
    return supported(l) ? layout(l, max_keys).total : 0;
}

b200_status kq_latent_prefill(const KqLatent &l, const KqLatentPrefill &w, const float *q, int64_t ldq, const float *gate, int64_t ldg,
                              int T, int pos0, uint16_t *out, int64_t ldo, cudaStream_t st) {
    if (!supported(l) || l.f32) return B200_ERR_UNSUPPORTED;
    const int lo = l.window > 0 ? std::max(0, pos0 - l.window + 1) : 0, keys = pos0 + T - lo;
    const Work k = layout(l, keys);
    KQ_REQUIRE(keys <= l.cap && k.total <= w.work_bytes, "latent_prefill: %d visible rows, the cache holds %d", keys, l.cap);
    uint16_t *c = (uint16_t *)w.work, *kr = (uint16_t *)((uint8_t *)w.work + k.at_r), *ku = (uint16_t *)((uint8_t *)w.work + k.at_k),
             *v = (uint16_t *)((uint8_t *)w.work + k.at_v);
    kq_launch(latent_gather_kernel, (unsigned)keys, 128, 0, st, (const uint16_t *)l.cache, l.ld, l.cap, l.kv_rank, l.rot_at, l.rot_dim, lo, c, k.ldc, kr,
              k.ldr);
    KQ_COUNT_LAUNCH();
    KQ_LAUNCH_CHECK();
    KqDense d;
    d.M = keys, d.K = l.kv_rank, d.ldw = kq_bf16_ld(l.kv_rank), d.nseg = 2;
    d.seg[0] = {};
    d.seg[0].W = w.uk, d.seg[0].n_rows = l.n_head * l.qk_dim, d.seg[0].y = ku, d.seg[0].ldy = k.ldk, d.seg[0].out = KQ_OUT_F16;
    d.seg[0].head_in = l.qk_dim, d.seg[0].head_out = (int32_t)kq_pad(l.qk_dim, 64);
    d.seg[1] = {};
    d.seg[1].W = w.uv, d.seg[1].n_rows = l.n_head * l.v_dim, d.seg[1].y = v, d.seg[1].ldy = k.ldv, d.seg[1].out = KQ_OUT_F16;
    d.seg[1].head_in = l.v_dim, d.seg[1].head_out = (int32_t)kq_pad(l.v_dim, 64);
    b200_status rc = kq_gemm_bf16(d, c, k.ldc, 1, st);
    if (rc != B200_OK) return rc;
    KqPromptAttn a;
    a.q = q, a.ldq = ldq, a.k = ku, a.kr = kr, a.v = v, a.rows = keys, a.lo = lo;
    a.n_head = a.kv_heads = l.n_head, a.dim = l.qk_dim, a.rot = l.rot_dim, a.vdim = l.v_dim;
    a.T = T, a.pos0 = pos0, a.window = l.window, a.scale = l.scale;
    a.gate = gate, a.ldg = ldg, a.out = out, a.ldo = ldo;
    return kq_prompt_attention(a, st);
}
