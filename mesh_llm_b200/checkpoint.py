"""Host-side view of the library's checkpoint reader: a folder with config.json and model.safetensors.

The counterpart of gguf.py for models whose layers are described one by one.  All parsing happens in
libb200kq.so, which also holds the table of architectures.
"""
from __future__ import annotations

import ctypes as C

import numpy as np

from .capi import GgufTensor, LayerConfig, StackConfig, StageConfig, check, lib


class Checkpoint:
    def __init__(self, path):
        h = C.c_void_p()
        check(lib().b200_ckpt_open(str(path).encode(), C.byref(h)))
        self.h = h
        self.path = str(path)

    def close(self):
        if getattr(self, "h", None):
            lib().b200_ckpt_close(self.h)
            self.h = None

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    @property
    def architecture(self):
        return lib().b200_ckpt_architecture(self.h).decode()

    def tensors(self):
        """-> {name: (index, ggml type id, shape with the contiguous dimension last)}"""
        out = {}
        for i in range(lib().b200_ckpt_tensor_count(self.h)):
            t = GgufTensor()
            check(lib().b200_ckpt_tensor_info(self.h, i, C.byref(t)))
            out[t.name.decode()] = (i, t.type, [int(t.ne[d]) for d in range(t.n_dims)][::-1])
        return out

    def read(self, name):
        """raw bytes of a tensor"""
        i = self.tensors()[name][0]
        t = GgufTensor()
        check(lib().b200_ckpt_tensor_info(self.h, i, C.byref(t)))
        out = np.empty(t.nbytes, np.uint8)
        check(lib().b200_ckpt_read_tensor(self.h, i, out.ctypes.data, out.size))
        return out

    def stage_config(self, layer_begin=0, layer_end=-1, n_ctx=4096, n_seq=1, n_ubatch=512, device=0, precision=0):
        """-> (StageConfig, StackConfig, [LayerConfig])"""
        cfg, stack = StageConfig(), StackConfig()
        n = lib().b200_ckpt_layer_count(self.h)
        layers = (LayerConfig * max(n, 1))()
        check(lib().b200_ckpt_stage_config(self.h, layer_begin, layer_end, n_ctx, n_seq, n_ubatch, device, precision,
                                           C.byref(cfg), C.byref(stack), layers))
        return cfg, stack, list(layers)[:n]
