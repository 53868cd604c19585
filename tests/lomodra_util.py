"""Small random Lomodra models, and the helpers of the tests that run them."""
import numpy as np

from hybrid_util import bf16


def experts(n, top, ff, shared=None):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def light(heads, dim, vdim, decay=None, mlp=None):
    decay = decay or [float(d) for d in np.linspace(0.55, 0.995, heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def attn(heads, kv_heads, dim, vdim, chunk, scale=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "scale": scale or dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv=4, ranks=(12, 20), mlp=None):
    """ranks: inner sizes of the decay's and the gate's projections (they show in the tensors' shapes only)"""
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp,
            "_ranks": ranks}


def config(layers, width, vocab, side=None, cap=None, eps=1e-6):
    c = {"architecture": "Lomodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side:
        c["token_side"] = {"dim": side}
    if cap:
        c["logit_softcap"] = cap
    return c


def shapes(cfg):
    """name -> shape of every tensor of the model"""
    h, n = cfg["width"], len(cfg["layers"])
    out = {"embed": (cfg["vocab"], h)}
    side = cfg.get("token_side", {}).get("dim")
    if side:
        out["side.embed"] = (cfg["vocab"], n * side)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, d, e = m["heads"], m["dim"], m["vdim"]
        out[p + "norm1"] = (h,)
        x = p + "mix."
        if l["type"] == "lightning":
            out.update({x + "q": (H * d, h), x + "k": (H * d, h), x + "v": (H * e, h), x + "g": (H * e, h), x + "norm": (H * e,)})
        elif l["type"] == "attention":
            G = m["kv_heads"]
            out.update({x + "q": (H * d, h), x + "q.norm": (d,)})
            if m.get("kv_from") is None:
                out.update({x + "k": (G * d, h), x + "k.norm": (d,), x + "v": (G * e, h)})
        else:
            G, t, (ra, rg) = m["kv_heads"], m["conv"], l["_ranks"]
            for name, c in (("q", G * d), ("k", G * d), ("v", H * e)):
                out.update({x + name: (c, h), x + name + ".conv": (c, t)})
            out.update({x + "b": (H, h), x + "A_log": (H,), x + "dt_bias": (H * d,), x + "norm": (e,), x + "a1": (ra, h), x + "a2": (H * d, ra),
                        x + "g1": (rg, h), x + "g2": (H * e, rg)})
        out[x + "o"] = (h, H * e)
        if l["mlp"]:
            f = p + "mlp."
            out[p + "norm2"] = (h,)
            parts = [(f"e{j}", l["mlp"]["expert"]["ff"]) for j in range(l["mlp"]["router"]["experts"])]
            if l["mlp"]["shared"]:
                parts.append(("shared", l["mlp"]["shared"]["ff"]))
            for name, ff in parts:
                out.update({f + name + ".gate": (ff, h), f + name + ".up": (ff, h), f + name + ".down": (h, ff)})
            out.update({f + "router": (l["mlp"]["router"]["experts"], h), f + "router.b": (l["mlp"]["router"]["experts"],)})
        if side:
            out.update({p + "side.gate": (side, h), p + "side.proj": (h, side), p + "side.norm": (h,)})
    out["final.norm"] = (h,)
    return out


def weights(cfg, seed):
    """bf16 values as float32; sized so that gates, decays, unit norms and attention scores all vary.  The first dimensions of the
    residual carry a code of the token that no sub-layer touches and that the routers read, one per expert: choices
    differ from token to token and none of them is close."""
    rng = np.random.default_rng(seed)
    code = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l["mlp"]] + [0])
    assert code < cfg["width"]
    levels = np.linspace(-2, 2, code) if code > 1 else np.zeros(code)
    out = {}
    for name, s in shapes(cfg).items():
        w = rng.standard_normal(s)
        leaf = name.split(".", 1)[1] if name[0] == "l" and "." in name else name
        if leaf in ("norm1", "norm2", "side.norm"):
            w = 0.5 + 0.2 * w
            w[:code] = 0
        elif leaf.endswith("norm"):
            w = 1 + 0.2 * w
        elif leaf == "embed":
            if code:
                w[:, :code] = rng.permuted(np.tile(levels, (s[0], 1)), axis=1)
        elif leaf == "mlp.router":
            w = 0.02 * w / np.sqrt(s[-1])
            w[:, :s[0]] += 0.75 * max(1, s[0] - 1) * np.eye(s[0])
        elif leaf == "mlp.router.b":
            w = 0.1 * w
        elif leaf == "mix.A_log":
            w = rng.uniform(-3.0, 0.5, s)
        elif leaf == "mix.dt_bias":
            w = rng.uniform(-4.0, 0.5, s)
        elif leaf.endswith(".conv"):
            w = w / np.sqrt(s[-1])
        elif leaf != "side.embed":
            w = w / np.sqrt(s[-1])
        out[name] = bf16(w)
    return out


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


def engine(path, precision, n_ctx=512, n_seq=1, n_ubatch=256):
    from mesh_llm_b200.engine import Engine, open_stage

    return Engine(open_stage(path, precision, n_ctx=n_ctx, n_seq=n_seq, n_ubatch=n_ubatch))


def run(eng, toks, portions, rid="r"):
    """feeds the tokens in portions (the last one repeats) and returns all logits"""
    out, at = [], 0
    for i in range(len(toks)):
        n = portions[min(i, len(portions) - 1)]
        part = toks[at:at + n]
        if not len(part):
            break
        out.append(eng.feed(rid, part, range(len(part))))
        at += len(part)
    eng.check()
    eng.end(rid)
    return np.concatenate(out)
