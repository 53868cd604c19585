#include "kq_dense.cuh"
struct KqLatentPrefill { const uint16_t *uk, *uv; void *work; size_t work_bytes; };
int kq_latent_tc_error_fetch() { return 0; }
size_t kq_latent_prefill_bytes(const KqLatent &l, int max_rows, int max_keys) { return 0; }
b200_status kq_latent_prefill(const KqLatent &l, const KqLatentPrefill &w, const float *q, int64_t ldq, const float *gate, int64_t ldg,
                              int T, int pos0, uint16_t *out, int64_t ldo, cudaStream_t st) { return B200_ERR_UNSUPPORTED; }
