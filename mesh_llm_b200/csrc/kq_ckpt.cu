// Checkpoint folders (config.json + model.safetensors): a small JSON reader, the safetensors index, the table of
// architectures that turns a config into layer descriptions, and the selective load of a stage's own tensors
// (host code only).
#include "kq_common.cuh"

#include <errno.h>
#include <fcntl.h>
#include <math.h>
#include <stdlib.h>
#include <string.h>
#include <sys/stat.h>
#include <unistd.h>

#include <algorithm>
#include <cmath>
#include <map>
#include <string>
#include <utility>
#include <vector>

namespace {

constexpr uint64_t MAX_CONFIG_BYTES = 64u << 20, MAX_HEADER_BYTES = 256u << 20;
constexpr int MAX_DEPTH = 64;

// ---- JSON ----------------------------------------------------------------------------------------
struct Json {
    enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ } kind = NUL;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<Json> arr;
    std::vector<std::pair<std::string, Json>> obj;
    const Json *get(const char *key) const {
        if (kind == OBJ)
            for (const auto &kv : obj)
                if (kv.first == key) return &kv.second;
        return nullptr;
    }
};

struct JsonReader {
    const char *p, *end;
    const char *err = nullptr;
    bool fail(const char *what) {
        if (!err) err = what;
        return false;
    }
    void ws() {
        while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) p++;
    }
    bool lit(const char *s) {
        const size_t n = strlen(s);
        if ((size_t)(end - p) < n || memcmp(p, s, n)) return fail("unexpected token");
        p += n;
        return true;
    }
    bool hex4(uint32_t &v) {
        if (end - p < 4) return fail("short escape");
        v = 0;
        for (int i = 0; i < 4; i++, p++) {
            const char c = *p;
            const int d = c >= '0' && c <= '9' ? c - '0' : c >= 'a' && c <= 'f' ? c - 'a' + 10 : c >= 'A' && c <= 'F' ? c - 'A' + 10 : -1;
            if (d < 0) return fail("bad escape");
            v = v * 16 + (uint32_t)d;
        }
        return true;
    }
    bool string(std::string &s) {
        if (p >= end || *p != '"') return fail("expected a string");
        for (p++; p < end && *p != '"';) {
            if ((unsigned char)*p < 0x20) return fail("control character in a string");
            if (*p != '\\') {
                s += *p++;
                continue;
            }
            if (++p >= end) break;
            const char c = *p++;
            static const char from[] = "\"\\/bfnrt", to[] = "\"\\/\b\f\n\r\t";
            if (c == 'u') {
                uint32_t u = 0, lo = 0;
                if (!hex4(u)) return false;
                if (u >= 0xD800 && u < 0xDC00) { // a surrogate pair
                    if (end - p < 2 || p[0] != '\\' || p[1] != 'u') return fail("lone surrogate");
                    p += 2;
                    if (!hex4(lo)) return false;
                    if (lo < 0xDC00 || lo > 0xDFFF) return fail("lone surrogate");
                    u = 0x10000 + ((u - 0xD800) << 10) + (lo - 0xDC00);
                }
                if (u < 0x80) s += (char)u;
                else if (u < 0x800) s += (char)(0xC0 | u >> 6), s += (char)(0x80 | (u & 63));
                else if (u < 0x10000) s += (char)(0xE0 | u >> 12), s += (char)(0x80 | (u >> 6 & 63)), s += (char)(0x80 | (u & 63));
                else s += (char)(0xF0 | u >> 18), s += (char)(0x80 | (u >> 12 & 63)), s += (char)(0x80 | (u >> 6 & 63)), s += (char)(0x80 | (u & 63));
            } else {
                const char *q = strchr(from, c);
                if (!q || !c) return fail("bad escape");
                s += to[q - from];
            }
        }
        if (p >= end) return fail("unterminated string");
        p++;
        return true;
    }
    bool value(Json &v, int depth = 0) {
        if (depth > MAX_DEPTH) return fail("nested too deeply");
        ws();
        if (p >= end) return fail("unexpected end");
        switch (*p) {
        case '{':
            v.kind = Json::OBJ;
            p++;
            ws();
            if (p < end && *p == '}') return p++, true;
            for (;;) {
                ws();
                std::string k;
                if (!string(k)) return false;
                ws();
                if (p >= end || *p++ != ':') return fail("expected ':'");
                v.obj.emplace_back(std::move(k), Json());
                if (!value(v.obj.back().second, depth + 1)) return false;
                ws();
                if (p >= end) return fail("unexpected end");
                if (*p == ',') { p++; continue; }
                if (*p == '}') return p++, true;
                return fail("expected ',' or '}'");
            }
        case '[':
            v.kind = Json::ARR;
            p++;
            ws();
            if (p < end && *p == ']') return p++, true;
            for (;;) {
                v.arr.emplace_back();
                if (!value(v.arr.back(), depth + 1)) return false;
                ws();
                if (p >= end) return fail("unexpected end");
                if (*p == ',') { p++; continue; }
                if (*p == ']') return p++, true;
                return fail("expected ',' or ']'");
            }
        case '"': v.kind = Json::STR; return string(v.str);
        case 't': v.kind = Json::BOOL; v.b = true; return lit("true");
        case 'f': v.kind = Json::BOOL; return lit("false");
        case 'n': return lit("null");
        default: {
            const std::string s(p, (size_t)std::min<ptrdiff_t>(end - p, 64));
            char *e = nullptr;
            if (*p != '-' && (*p < '0' || *p > '9')) return fail("unexpected token");
            v.kind = Json::NUM;
            v.num = strtod(s.c_str(), &e);
            if (e == s.c_str() || !std::isfinite(v.num)) return fail("bad number");
            p += e - s.c_str();
            return true;
        }
        }
    }
    bool document(Json &v) {
        if (!value(v)) return false;
        ws();
        return p == end || fail("trailing characters");
    }
};

bool read_all(int fd, uint64_t pos, void *dst, uint64_t n) {
    for (uint64_t done = 0; done < n;) {
        const ssize_t r = pread(fd, (char *)dst + done, (size_t)std::min<uint64_t>(n - done, 1u << 30), (off_t)(pos + done));
        if (r <= 0) return false;
        done += (uint64_t)r;
    }
    return true;
}

// ---- config access: a missing or ill-typed key is an error that names it ---------------------------
struct Cfg {
    b200_status rc = B200_OK;
    void bad(const std::string &where, const char *key, const char *what) {
        if (rc == B200_OK) kq_set_error("config.json: %s%s%s %s", where.c_str(), where.empty() ? "" : ".", key, what);
        rc = B200_ERR_INVALID;
    }
    const Json *need(const Json *o, const std::string &where, const char *key) {
        const Json *v = o ? o->get(key) : nullptr;
        if (!v) bad(where, key, "is missing");
        return v;
    }
    int32_t integer(const Json *o, const std::string &where, const char *key, int64_t lo, int64_t hi) {
        const Json *v = need(o, where, key);
        if (!v) return 0;
        if (v->kind != Json::NUM || v->num != floor(v->num) || v->num < (double)lo || v->num > (double)hi) {
            bad(where, key, "is not an integer in range");
            return 0;
        }
        return (int32_t)v->num;
    }
    float number(const Json *o, const std::string &where, const char *key) {
        const Json *v = need(o, where, key);
        if (!v) return 0.f;
        if (v->kind != Json::NUM) bad(where, key, "is not a number");
        return (float)v->num;
    }
};
constexpr int64_t BIG = 1 << 28;

} // namespace

struct b200_ckpt {
    Json cfg;
    std::string arch;
    int fd = -1;
    uint64_t data_at = 0;
    std::vector<b200_gguf_tensor> tensors;
    std::map<std::string, int> index;
    // what the architecture's reader made of the config
    int32_t n_embd = 0, n_vocab = 0;
    float eps = 0.f;
    b200_stack_config stack = {};
    std::vector<b200_layer_config> layers;
    std::map<std::string, std::vector<float>> constants; // vectors that the config holds and a stage takes as tensors
    ~b200_ckpt() {
        if (fd >= 0) close(fd);
    }
};

namespace {

// Gonetar: recurrent blocks and windowed latent attention in any order, norms around every sub-layer, one range of
// layers possibly run several times, clamped GLU feed-forwards, tied output head.
b200_status read_gonetar(b200_ckpt &ck) {
    Cfg r;
    const Json *c = &ck.cfg;
    ck.n_embd = r.integer(c, "", "width", 1, BIG);
    ck.n_vocab = r.integer(c, "", "vocab", 1, BIG);
    ck.eps = r.number(r.need(c, "", "norm"), "norm", "eps");
    ck.stack.embd_scale = r.number(r.need(c, "", "embedding"), "embedding", "scale");
    ck.stack.norm_offset = 1.0f;
    const Json *layers = r.need(c, "", "layers");
    if (layers && layers->kind != Json::ARR) r.bad("", "layers", "is not a list");
    if (r.rc != B200_OK) return r.rc;
    for (size_t i = 0; i < layers->arr.size(); i++) {
        const Json *l = &layers->arr[i];
        const std::string at = "layers[" + std::to_string(i) + "]";
        const Json *type = r.need(l, at, "type"), *m = r.need(l, at, "mixer");
        if (r.rc != B200_OK) return r.rc;
        b200_layer_config d = {};
        const std::string in = at + ".mixer";
        if (type->str == "latent_attention") {
            d.mixer = B200_MIXER_LATENT_ATTN;
            d.n_head = r.integer(m, in, "heads", 1, 65536);
            d.qk_dim = r.integer(m, in, "dim", 1, 65536);
            d.rot_dim = r.integer(m, in, "rot_dim", 0, 65536);
            d.v_dim = r.integer(m, in, "vdim", 1, 65536);
            d.kv_rank = r.integer(m, in, "kv_rank", 1, 65536);
            d.attn_scale = r.number(m, in, "scale");
            const Json *mask = r.need(m, in, "mask"), *rot = r.need(m, in, "rot");
            d.window = r.integer(mask, in + ".mask", "size", 1, BIG);
            d.rope_base = r.number(rot, in + ".rot", "base");
            d.rot_dims = r.integer(rot, in + ".rot", "dims", 0, d.rot_dim);
        } else if (type->str == "rglru") {
            d.mixer = B200_MIXER_LINEAR_REC;
            d.rec_width = r.integer(m, in, "width", 1, BIG);
            d.rec_blocks = r.integer(m, in, "blocks", 1, BIG);
            d.conv_taps = r.integer(m, in, "conv", 1, 4096);
            d.rec_decay = 8.0f;
        } else {
            kq_set_error("config.json: %s.type \"%s\" is not a mixer of this architecture", at.c_str(), type->str.c_str());
            return B200_ERR_UNSUPPORTED;
        }
        const Json *mlp = l->get("mlp");
        if (mlp && mlp->kind != Json::NUL) {
            const std::string im = at + ".mlp";
            const Json *kind = r.need(mlp, im, "kind");
            if (kind && kind->str != "dense") {
                kq_set_error("config.json: %s.kind \"%s\" is not a feed-forward of this architecture", im.c_str(), kind->str.c_str());
                return B200_ERR_UNSUPPORTED;
            }
            d.ffn = B200_FFN_CLAMPED_GLU;
            d.n_ff = r.integer(mlp, im, "ff", 1, BIG);
            d.glu_limit = r.number(mlp, im, "limit");
            d.glu_alpha = 1.702f;
        }
        if (r.rc != B200_OK) return r.rc;
        ck.layers.push_back(d);
    }
    const Json *loop = c->get("loop");
    if (loop && loop->kind != Json::NUL) {
        const int64_t n = (int64_t)ck.layers.size();
        ck.stack.loop_start = r.integer(loop, "loop", "start", 0, n);
        ck.stack.loop_stop = r.integer(loop, "loop", "stop", 0, n);
        ck.stack.loop_times = r.integer(loop, "loop", "times", 1, 4096);
    }
    return r.rc;
}

// Lomodra: linear attention with fixed decays, chunked attention and gated delta rules in any order, norms behind the
// sub-layers, experts with a shared one, a per-layer token input, tied output head with a soft cap.
b200_status read_lomodra(b200_ckpt &ck) {
    Cfg r;
    const Json *c = &ck.cfg;
    ck.n_embd = r.integer(c, "", "width", 1, BIG);
    ck.n_vocab = r.integer(c, "", "vocab", 1, BIG);
    ck.eps = r.number(r.need(c, "", "norm"), "norm", "eps");
    ck.stack.embd_scale = 1.0f;
    ck.stack.norm_place = B200_NORM_OUTPUT;
    auto given = [](const Json *o, const char *key) { // absent and null are the same
        const Json *v = o ? o->get(key) : nullptr;
        return v && v->kind != Json::NUL ? v : nullptr;
    };
    if (const Json *side = given(c, "token_side")) ck.stack.side_dim = r.integer(side, "token_side", "dim", 1, BIG);
    if (given(c, "logit_softcap")) {
        ck.stack.logit_softcap = r.number(c, "", "logit_softcap");
        if (!(ck.stack.logit_softcap > 0.f)) r.bad("", "logit_softcap", "is not positive");
    }
    const Json *layers = r.need(c, "", "layers");
    if (layers && layers->kind != Json::ARR) r.bad("", "layers", "is not a list");
    if (r.rc != B200_OK) return r.rc;
    for (size_t i = 0; i < layers->arr.size(); i++) {
        const Json *l = &layers->arr[i];
        const std::string at = "layers[" + std::to_string(i) + "]", in = at + ".mixer", mix = "l" + std::to_string(i) + ".mix.";
        const Json *type = r.need(l, at, "type"), *m = r.need(l, at, "mixer");
        if (r.rc != B200_OK) return r.rc;
        b200_layer_config d = {};
        d.n_head = r.integer(m, in, "heads", 1, 65536);
        d.qk_dim = r.integer(m, in, "dim", 1, 65536);
        d.v_dim = r.integer(m, in, "vdim", 1, 65536);
        if (type->str == "attention") {
            d.mixer = B200_MIXER_GQA;
            d.n_head_kv = r.integer(m, in, "kv_heads", 1, 65536);
            d.attn_scale = r.number(m, in, "scale");
            d.chunk = r.integer(r.need(m, in, "mask"), in + ".mask", "size", 1, BIG);
            if (given(m, "kv_from")) {
                d.kv_shared = 1;
                d.kv_layer = r.integer(m, in, "kv_from", 0, (int64_t)i - 1);
            }
        } else if (type->str == "lightning") {
            d.mixer = B200_MIXER_DECAY_STATE;
            const Json *decay = r.need(m, in, "decay");
            if (decay && (decay->kind != Json::ARR || (int64_t)decay->arr.size() != d.n_head)) r.bad(in, "decay", "is not a list of one number per head");
            if (r.rc != B200_OK) return r.rc;
            std::vector<float> &v = ck.constants[mix + "decay"];
            for (const Json &x : decay->arr) {
                if (x.kind != Json::NUM) r.bad(in, "decay", "is not a list of one number per head");
                v.push_back((float)x.num);
            }
        } else if (type->str == "channel_delta") {
            d.mixer = B200_MIXER_DELTA_STATE;
            d.n_head_kv = r.integer(m, in, "kv_heads", 1, 65536);
            d.conv_taps = r.integer(m, in, "conv", 1, 4096);
            auto rank = [&](const char *leaf) { // the inner size of a low-rank projection: the rows of its first matrix
                const auto it = ck.index.find(mix + leaf);
                if (it != ck.index.end()) return (int32_t)ck.tensors[(size_t)it->second].ne[1];
                kq_set_error("model.safetensors: no tensor %s%s", mix.c_str(), leaf);
                r.rc = B200_ERR_INVALID;
                return 0;
            };
            d.decay_rank = rank("a1");
            d.gate_rank = rank("g1");
        } else {
            kq_set_error("config.json: %s.type \"%s\" is not a mixer of this architecture", at.c_str(), type->str.c_str());
            return B200_ERR_UNSUPPORTED;
        }
        if (const Json *mlp = given(l, "mlp")) {
            const std::string im = at + ".mlp";
            const Json *kind = r.need(mlp, im, "kind");
            if (kind && kind->str != "moe") {
                kq_set_error("config.json: %s.kind \"%s\" is not a feed-forward of this architecture", im.c_str(), kind->str.c_str());
                return B200_ERR_UNSUPPORTED;
            }
            d.ffn = B200_FFN_MOE;
            const Json *router = r.need(mlp, im, "router");
            d.n_expert = r.integer(router, im + ".router", "experts", 1, 65536);
            d.n_expert_used = r.integer(router, im + ".router", "top", 1, d.n_expert);
            d.n_ff_exp = r.integer(r.need(mlp, im, "expert"), im + ".expert", "ff", 1, BIG);
            if (const Json *sh = given(mlp, "shared")) d.n_ff_shared = r.integer(sh, im + ".shared", "ff", 1, BIG);
        }
        if (r.rc != B200_OK) return r.rc;
        ck.layers.push_back(d);
    }
    return r.rc;
}

struct Architecture {
    const char *name;
    b200_status (*read)(b200_ckpt &);
};
const Architecture ARCHITECTURES[] = {
    {"Gonetar", read_gonetar},
    {"Lomodra", read_lomodra},
};

b200_status index_safetensors(b200_ckpt &ck, const std::string &path) {
    ck.fd = open(path.c_str(), O_RDONLY | O_CLOEXEC);
    struct stat sb;
    if (ck.fd < 0 || fstat(ck.fd, &sb) != 0) {
        kq_set_error("%s: %s", path.c_str(), strerror(errno));
        return B200_ERR_INVALID;
    }
    const uint64_t size = (uint64_t)sb.st_size;
    uint64_t n = 0;
    KQ_REQUIRE(size >= 8 && read_all(ck.fd, 0, &n, 8) && n <= size - 8 && n <= MAX_HEADER_BYTES, "%s: bad header length", path.c_str());
    std::string text((size_t)n, '\0');
    KQ_REQUIRE(read_all(ck.fd, 8, &text[0], n), "%s: short header", path.c_str());
    Json h;
    JsonReader rd{text.data(), text.data() + text.size()};
    KQ_REQUIRE(rd.document(h) && h.kind == Json::OBJ, "%s: header: %s", path.c_str(), rd.err ? rd.err : "not an object");
    ck.data_at = 8 + n;
    for (const auto &kv : h.obj) {
        if (kv.first == "__metadata__") continue;
        const Json *ty = kv.second.get("dtype"), *sh = kv.second.get("shape"), *of = kv.second.get("data_offsets");
        const char *name = kv.first.c_str();
        KQ_REQUIRE(ty && ty->kind == Json::STR && sh && sh->kind == Json::ARR && of && of->kind == Json::ARR && of->arr.size() == 2,
                   "%s: entry of %s", path.c_str(), name);
        b200_gguf_tensor t;
        memset(&t, 0, sizeof(t));
        KQ_REQUIRE(kv.first.size() < sizeof(t.name), "%s: name %s is too long", path.c_str(), name);
        snprintf(t.name, sizeof(t.name), "%s", name);
        uint64_t es = 0;
        if (ty->str == "BF16") t.type = B200_TYPE_BF16, es = 2;
        else if (ty->str == "F16") t.type = B200_TYPE_F16, es = 2;
        else if (ty->str == "F32") t.type = B200_TYPE_F32, es = 4;
        else if (ty->str == "I32") t.type = B200_TYPE_I32, es = 4;
        KQ_REQUIRE(es, "%s: %s has type %s", path.c_str(), name, ty->str.c_str());
        KQ_REQUIRE(sh->arr.size() <= 4, "%s: %s has %zu dimensions", path.c_str(), name, sh->arr.size());
        t.n_dims = (uint32_t)sh->arr.size();
        double count = 1;
        for (int d = 0; d < 4; d++) t.ne[d] = 1;
        for (size_t d = 0; d < sh->arr.size(); d++) {
            const Json &v = sh->arr[sh->arr.size() - 1 - d];
            KQ_REQUIRE(v.kind == Json::NUM && v.num >= 0 && v.num == floor(v.num) && v.num < 9e15, "%s: shape of %s", path.c_str(), name);
            t.ne[d] = (int64_t)v.num;
            count *= v.num;
        }
        const Json &a = of->arr[0], &b = of->arr[1];
        KQ_REQUIRE(a.kind == Json::NUM && b.kind == Json::NUM && a.num >= 0 && b.num >= a.num && b.num <= (double)(size - ck.data_at) &&
                       b.num - a.num == count * (double)es,
                   "%s: data range of %s", path.c_str(), name);
        t.file_offset = ck.data_at + (uint64_t)a.num;
        t.nbytes = (uint64_t)(b.num - a.num);
        ck.index[kv.first] = (int)ck.tensors.size();
        ck.tensors.push_back(t);
    }
    return B200_OK;
}

b200_status open_into(b200_ckpt &ck, const std::string &dir) {
    const std::string path = dir + "/config.json";
    const int fd = open(path.c_str(), O_RDONLY | O_CLOEXEC);
    struct stat sb;
    if (fd < 0 || fstat(fd, &sb) != 0 || !S_ISREG(sb.st_mode)) {
        kq_set_error("%s: %s", path.c_str(), fd < 0 ? strerror(errno) : "not a file");
        if (fd >= 0) close(fd);
        return B200_ERR_INVALID;
    }
    const uint64_t n = (uint64_t)sb.st_size;
    std::string text;
    const bool ok = n <= MAX_CONFIG_BYTES && (text.resize((size_t)n), n == 0 || read_all(fd, 0, &text[0], n));
    close(fd);
    KQ_REQUIRE(ok, "%s: cannot be read", path.c_str());
    JsonReader rd{text.data(), text.data() + text.size()};
    KQ_REQUIRE(rd.document(ck.cfg) && ck.cfg.kind == Json::OBJ, "%s: %s", path.c_str(), rd.err ? rd.err : "not an object");
    const Json *a = ck.cfg.get("architecture");
    KQ_REQUIRE(a && a->kind == Json::STR, "%s: no architecture", path.c_str());
    ck.arch = a->str;
    for (const Architecture &ar : ARCHITECTURES)
        if (ck.arch == ar.name) {
            const b200_status rc = index_safetensors(ck, dir + "/model.safetensors"); // some sizes are those of the tensors
            return rc == B200_OK ? ar.read(ck) : rc;
        }
    kq_set_error("%s: architecture %s is not one of this library", path.c_str(), ck.arch.c_str());
    return B200_ERR_UNSUPPORTED;
}

} // namespace

extern "C" {

b200_status b200_ckpt_open(const char *dir, b200_ckpt **out) {
    KQ_REQUIRE(dir && out, "ckpt_open: null argument");
    b200_ckpt *ck = new b200_ckpt();
    const b200_status rc = open_into(*ck, dir);
    if (rc != B200_OK) {
        delete ck;
        return rc;
    }
    *out = ck;
    return B200_OK;
}

void b200_ckpt_close(b200_ckpt *ck) { delete ck; }

const char *b200_ckpt_architecture(const b200_ckpt *ck) { return ck ? ck->arch.c_str() : ""; }
int64_t b200_ckpt_tensor_count(const b200_ckpt *ck) { return ck ? (int64_t)ck->tensors.size() : -1; }
int32_t b200_ckpt_layer_count(const b200_ckpt *ck) { return ck ? (int32_t)ck->layers.size() : -1; }

b200_status b200_ckpt_tensor_info(const b200_ckpt *ck, int64_t i, b200_gguf_tensor *out) {
    KQ_REQUIRE(ck && out && i >= 0 && i < (int64_t)ck->tensors.size(), "ckpt_tensor_info: bad argument");
    *out = ck->tensors[(size_t)i];
    return B200_OK;
}

b200_status b200_ckpt_read_tensor(const b200_ckpt *ck, int64_t i, void *dst, size_t nbytes) {
    KQ_REQUIRE(ck && dst && i >= 0 && i < (int64_t)ck->tensors.size(), "ckpt_read_tensor: bad argument");
    const b200_gguf_tensor &t = ck->tensors[(size_t)i];
    if (nbytes != t.nbytes) {
        kq_set_error("ckpt_read_tensor: %s holds %llu bytes", t.name, (unsigned long long)t.nbytes);
        return B200_ERR_BOUNDS;
    }
    KQ_REQUIRE(read_all(ck->fd, t.file_offset, dst, nbytes), "ckpt_read_tensor: reading %s failed", t.name);
    return B200_OK;
}

b200_status b200_ckpt_stage_config(const b200_ckpt *ck, int32_t layer_begin, int32_t layer_end, int32_t n_ctx,
                                   int32_t n_seq, int32_t n_ubatch, int32_t device, int32_t precision,
                                   b200_stage_config *cfg, b200_stack_config *stack, b200_layer_config *layers) {
    KQ_REQUIRE(ck && cfg && stack && layers, "ckpt_stage_config: null argument");
    memset(cfg, 0, sizeof(*cfg));
    cfg->n_layer = (int32_t)ck->layers.size();
    cfg->layer_begin = layer_begin;
    cfg->layer_end = layer_end < 0 ? cfg->n_layer : layer_end;
    KQ_REQUIRE(cfg->layer_begin >= 0 && cfg->layer_begin <= cfg->layer_end && cfg->layer_end <= cfg->n_layer,
               "ckpt_stage_config: layer range [%d, %d) outside [0, %d)", layer_begin, layer_end, cfg->n_layer);
    cfg->n_embd = ck->n_embd;
    cfg->n_vocab = ck->n_vocab;
    cfg->n_ctx = n_ctx;
    cfg->n_seq = n_seq;
    cfg->n_ubatch = n_ubatch;
    cfg->device = device;
    cfg->rms_eps = ck->eps;
    cfg->has_embd = cfg->layer_begin == 0;
    cfg->has_output = cfg->layer_end == cfg->n_layer;
    *stack = ck->stack;
    stack->precision = precision;
    for (size_t i = 0; i < ck->layers.size(); i++) layers[i] = ck->layers[i];
    return B200_OK;
}

b200_status b200_stage_load_ckpt(b200_stage *st, const b200_ckpt *ck, int64_t *n_loaded, int64_t *bytes_read) {
    KQ_REQUIRE(st && ck, "stage_load_ckpt: null argument");
    int64_t loaded = 0, total = 0;
    std::vector<uint8_t> host;
    const int64_t n = b200_stage_tensor_count(st);
    for (int64_t i = 0; i < n; i++) {
        char name[128];
        uint32_t type = 0;
        int64_t ne[3];
        b200_status rc = b200_stage_tensor_info(st, i, name, sizeof(name), &type, ne);
        if (rc != B200_OK) return rc;
        const auto it = ck->index.find(name);
        const auto given = ck->constants.find(name);
        if (given != ck->constants.end()) {
            rc = b200_stage_set_tensor(st, name, B200_TYPE_F32, given->second.data(), given->second.size() * 4);
            if (rc != B200_OK) return rc;
            continue;
        }
        if (it == ck->index.end()) {
            kq_set_error("stage_load_ckpt: the file has no tensor %s", name);
            return B200_ERR_STATE;
        }
        const b200_gguf_tensor &t = ck->tensors[(size_t)it->second];
        if (t.type != B200_TYPE_BF16 && !(t.type == B200_TYPE_F32 && type == B200_TYPE_F32)) {
            kq_set_error("stage_load_ckpt: %s is stored as type %u", name, t.type);
            return B200_ERR_UNSUPPORTED;
        }
        // leading dimensions may be folded (a vector per block is one row per block)
        const int64_t have = t.ne[0] * t.ne[1] * t.ne[2] * t.ne[3];
        KQ_REQUIRE(t.ne[0] == ne[0] && have == ne[0] * ne[1] * ne[2], "stage_load_ckpt: %s is [%lld x %lld] in the file, the stage expects [%lld x %lld]",
                   name, (long long)t.ne[0], (long long)(t.ne[0] ? have / t.ne[0] : 0), (long long)ne[0], (long long)(ne[1] * ne[2]));
        host.resize((size_t)t.nbytes);
        rc = b200_ckpt_read_tensor(ck, it->second, host.data(), host.size());
        if (rc == B200_OK) rc = b200_stage_set_tensor(st, name, t.type, host.data(), host.size());
        if (rc != B200_OK) return rc;
        loaded++;
        total += (int64_t)t.nbytes;
    }
    if (n_loaded) *n_loaded = loaded;
    if (bytes_read) *bytes_read = total;
    return B200_OK;
}

} // extern "C"
