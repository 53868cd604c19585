"""Small random models for the tests of stages whose layers are described one by one."""
import json
import os
import struct

import numpy as np


def bf16(a):
    """round to bfloat16 (nearest, ties to even), as float32"""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.view(np.float32)


def rec(width, blocks, conv, ff=None, limit=1.5):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def attn(heads, dim, rot_dim, vdim, kv_rank, window, base=10000.0, scale=None, ff=None, limit=1.5):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
                      "scale": scale or (dim + rot_dim) ** -0.5},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def config(layers, width, vocab, loop=None, scale=1.0, eps=1e-6):
    c = {"architecture": "Gonetar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
         "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def shapes(cfg):
    """name -> shape of every tensor of the model"""
    h, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"] = out[p + "norm1b"] = (h,)
        if l["type"] == "rglru":
            W, B, n = m["width"], m["blocks"], m["width"] // m["blocks"]
            out.update({p + "mix.y": (W, h), p + "mix.y.b": (W,), p + "mix.x": (W, h), p + "mix.x.b": (W,),
                        p + "mix.conv": (W, m["conv"]), p + "mix.conv.b": (W,), p + "mix.ra": (B, n, n), p + "mix.ra.b": (B, n),
                        p + "mix.ri": (B, n, n), p + "mix.ri.b": (B, n), p + "mix.lam": (W,), p + "mix.o": (h, W)})
        else:
            H, d, r, v, R = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            out.update({p + "mix.q": (H * (d + r), h), p + "mix.dkv": (R + r, h), p + "mix.dkv.norm": (R,),
                        p + "mix.uk": (H * d, R), p + "mix.uv": (H * v, R), p + "mix.g": (H, h), p + "mix.o": (h, H * v)})
        if l["mlp"]:
            f = l["mlp"]["ff"]
            out[p + "norm2"] = out[p + "norm2b"] = (h,)
            out.update({p + "mlp.gate": (f, h), p + "mlp.up": (f, h), p + "mlp.down": (h, f)})
    out["final.norm"] = (h,)
    return out


def weights(cfg, seed):
    """bf16 values as float32; sized so that gates, clamps, decays and attention scores all vary"""
    rng = np.random.default_rng(seed)
    out = {}
    for name, s in shapes(cfg).items():
        w = rng.standard_normal(s)
        leaf = name.split(".", 1)[1] if name[0] == "l" and "." in name else name
        if leaf == "mix.dkv.norm":
            w = 1 + 0.2 * w
        elif leaf.startswith("norm") or leaf == "final.norm":
            w = 0.3 * w
        elif leaf == "mix.lam":
            w = rng.uniform(-5.0, -0.5, s)
        elif leaf.endswith(".b"):
            w = 0.3 * w
        elif leaf == "mix.conv":
            w = w / np.sqrt(s[-1])
        elif leaf == "mix.q":
            w = 2.5 * w / np.sqrt(s[-1])
        elif leaf != "embed":
            w = w / np.sqrt(s[-1])
        out[name] = bf16(w)
    return out


def write_checkpoint(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, data = {}, []
    at = 0
    for name, a in w.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        data.append(raw)
        at += len(raw)
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(data))
    return str(path)


def rel(got, ref):
    """rms error of every row over the rms of all of ref"""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())
