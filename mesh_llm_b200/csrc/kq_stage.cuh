// The stage object, shared by the forward pass of the K-quant decoder (kq_stage.cu) and that of stages whose
// layers are described one by one (kq_layers.cu): both use its tensor table, loading, graphs, logits and counters.
#pragma once
#include "kq_common.cuh"
#include "kq_kvq.cuh"

#include <string.h>

#include <map>
#include <memory>
#include <string>
#include <vector>

struct StTensor {
    std::string name;
    uint32_t type = 0;
    int64_t ne[3] = {0, 0, 0};
    void *dev = nullptr;
    size_t dev_bytes = 0;
    bool loaded = false;
};

struct LayerW {
    const float *attn_norm = nullptr, *ffn_norm = nullptr, *bq = nullptr, *bk = nullptr, *bv = nullptr,
                *q_norm = nullptr, *k_norm = nullptr, *router = nullptr;
    StTensor *wq = nullptr, *wk = nullptr, *wv = nullptr, *wo = nullptr, *gate = nullptr, *up = nullptr,
             *down = nullptr, *gate_e = nullptr, *up_e = nullptr, *down_e = nullptr;
};

struct GraphKey {
    int n_seq, n_split, seq0, pad_;
    const void *tokens, *hidden_in, *hidden_out, *logits, *next;
    bool operator<(const GraphKey &o) const {
        return memcmp(this, &o, sizeof(GraphKey)) < 0;
    }
};

struct GraphEntry {
    int n_split = 0; // attention slices the instantiated graph was last captured / updated for
    cudaGraphExec_t exec = nullptr;
    long long launches = 0;
};

struct KqLayers; // kq_layers.cu
struct KqLayersDelete {
    void operator()(KqLayers *p) const;
};

struct b200_stage {
    b200_stage_config c;
    std::vector<StTensor> tensors;
    std::map<std::string, int> index;
    std::vector<LayerW> layers;
    StTensor *tok_embd = nullptr, *out_w = nullptr;
    const float *out_norm = nullptr;
    bool resolved = false;
    // KV cache [layer_local][seq][ctx][n_kv][hd] f16
    uint16_t *kc = nullptr, *vc = nullptr;
    KqKvTypes kvt;
    int k_row = 0, v_row = 0; // bytes of one (position, kv head) row of each cache
    // activations
    int rows_max = 0;
    float *x = nullptr, *xn = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *att = nullptr, *g = nullptr,
          *u = nullptr, *last = nullptr, *logits_int = nullptr, *att_scratch = nullptr, *rl = nullptr,
          *rw = nullptr, *hp = nullptr, *hp2 = nullptr, *yp = nullptr;
    int32_t *moe_sorted = nullptr; // expert-major order of the routed pairs of a batch
    size_t moe_sorted_bytes = 0;
    uint8_t *expert_mask = nullptr; // one byte per expert, 1 = allowed (all ones when no mask is set)
    int32_t *rid = nullptr, *pos0_dev = nullptr, *rid_scratch = nullptr, *attn_counters = nullptr;
    unsigned int *moe_counters = nullptr; // one word per token row, zero between launches (moe_router_fused_kernel)
    int32_t *emit_counters = nullptr;     // one word per 256 rows of the feed-forward width, zero between launches (KqEmitQ8)
    size_t att_scratch_bytes = 0;
    void *scan_scratch = nullptr; // slices and counters of the vocabulary scan
    size_t scan_scratch_bytes = 0;
    int8_t *aq = nullptr;
    float *ad = nullptr;
    int16_t *abs16 = nullptr;
    int64_t kmax = 0;
    std::map<GraphKey, GraphEntry> graphs;
    cudaStream_t cap_stream = nullptr;
    long long launches = 0;
    bool use_graph = true;
    std::vector<void *> allocs;
    std::unique_ptr<KqLayers, KqLayersDelete> layers_desc; // set: the stage's layers are described one by one (kq_layers.cu)
};

// kernel classes of a decode step, selectable for timing (b200_stage_profile_decode)
enum { CLS_GEMV = 1, CLS_ATTN = 2, CLS_OTHER = 4, CLS_ALL = 7 };

b200_status kq_stage_alloc(b200_stage *st, void **p, size_t bytes);
void kq_stage_add_tensor(b200_stage *st, const std::string &name, uint32_t type, int64_t ne0, int64_t ne1, int64_t ne2);
StTensor *kq_stage_find(b200_stage *st, const std::string &name);

// ---- stages whose layers are described one by one
b200_status kq_layers_resolve(b200_stage *st);
b200_status kq_layers_forward(b200_stage *st, const int32_t *tokens, const float *hidden_in, int seq0, int n_seq, int T, int pos0,
                              bool pos_from_dev, float *hidden_out, float *logits, int all_logits, int32_t *next_tokens, cudaStream_t s,
                              unsigned classes);
// positions a call may run at: a sequence starts at 0 and continues where it stopped
b200_status kq_layers_check_pos(b200_stage *st, int seq0, int n_seq, int T, int pos0);
void kq_layers_advance(b200_stage *st, int seq0, int n_seq, int pos); // pos < 0: the state is no longer usable
bool kq_layers_tracing(const b200_stage *st);
bool kq_layers_read_tokens(const b200_stage *st); // every stage of such a model takes the token ids, next to hidden_in
bool kq_layers_plain_norm(const b200_stage *st, const std::string &name); // a norm weight around one, not around zero
b200_status kq_layers_peek(b200_stage *st, const char *which, float *host_out, size_t n_floats);
