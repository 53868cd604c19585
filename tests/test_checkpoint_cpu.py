"""No GPU: the checkpoint reader (config.json + model.safetensors), its table of architectures, and the layouts of the
structs it fills."""
import ctypes as C
import json
import os
import struct

import numpy as np
import pytest

from hybrid_util import attn, config, rec, shapes, weights, write_checkpoint
from test_abi_layout_cpu import compiler_layout, header_struct_fields


def small():
    return config([rec(24, 3, 5, ff=20), attn(2, 6, 4, 5, 9, window=7, base=123.5, scale=0.25, ff=12, limit=2.5), rec(8, 2, 1)],
                  width=12, vocab=19, loop=(1, 3, 4), scale=3.5, eps=2e-4)


def opened(path):
    from mesh_llm_b200.checkpoint import Checkpoint

    return Checkpoint(path)


def test_config_becomes_layer_descriptions(tmp_path):
    from mesh_llm_b200 import capi

    cfg = small()
    with opened(write_checkpoint(tmp_path, cfg, weights(cfg, 1))) as ck:
        assert ck.architecture == "Gonetar"
        c, s, layers = ck.stage_config(n_ctx=50, n_seq=3, n_ubatch=16, precision=capi.PRECISION_F32)
        assert (c.n_layer, c.layer_begin, c.layer_end, c.n_embd, c.n_vocab) == (3, 0, 3, 12, 19)
        assert (c.n_ctx, c.n_seq, c.n_ubatch, c.has_embd, c.has_output) == (50, 3, 16, 1, 1)
        assert c.rms_eps == np.float32(2e-4) and s.embd_scale == 3.5 and s.norm_offset == 1.0
        assert (s.loop_start, s.loop_stop, s.loop_times, s.precision) == (1, 3, 4, 1)
        a, b, d = layers
        assert (a.mixer, a.rec_width, a.rec_blocks, a.conv_taps, a.rec_decay) == (capi.MIXER_LINEAR_REC, 24, 3, 5, 8.0)
        assert (a.ffn, a.n_ff, a.glu_limit) == (capi.FFN_CLAMPED_GLU, 20, 1.5) and a.glu_alpha == np.float32(1.702)
        assert (b.mixer, b.n_head, b.qk_dim, b.rot_dim, b.rot_dims, b.v_dim, b.kv_rank, b.window) == (capi.MIXER_LATENT_ATTN, 2, 6, 4, 4, 5, 9, 7)
        assert (b.rope_base, b.attn_scale, b.n_ff, b.glu_limit) == (123.5, 0.25, 12, 2.5)
        assert (d.ffn, d.conv_taps) == (capi.FFN_NONE, 1)
        c, _, _ = ck.stage_config(1, 3)
        assert (c.has_embd, c.has_output) == (0, 1)


def test_no_loop_and_null_loop(tmp_path):
    cfg = small()
    for k, loop in enumerate((None, "drop")):
        c = json.loads(json.dumps(cfg))
        c["loop"] = None
        if loop == "drop":
            del c["loop"]
        with opened(write_checkpoint(tmp_path / str(k), c, weights(cfg, 1))) as ck:
            assert ck.stage_config()[1].loop_times <= 1


def test_tensor_index_and_bytes(tmp_path):
    cfg = small()
    w = weights(cfg, 2)
    with opened(write_checkpoint(tmp_path, cfg, w)) as ck:
        t = ck.tensors()
        assert {n: tuple(s) for n, (_, _, s) in t.items()} == {n: tuple(s) for n, s in shapes(cfg).items()}
        for n in ("embed", "l0.mix.ra", "l1.mix.dkv.norm"):
            got = ck.read(n).view("<u2").astype(np.uint32) << 16
            assert np.array_equal(got.view(np.float32).reshape(w[n].shape), w[n])


def test_unicode_and_numbers_in_json(tmp_path):
    cfg = small()
    path = write_checkpoint(tmp_path, cfg, weights(cfg, 1))
    text = json.dumps(dict(cfg, note='é中\U0001F600 "\\ \n', unknown=[1e3, -2.5E-7, [], {}, True, False, None]), indent=3)
    (tmp_path / "config.json").write_text(text)
    with opened(path) as ck:
        assert ck.stage_config()[0].n_embd == 12


@pytest.mark.parametrize("edit,what", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "layers[0].mixer.conv"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][1]["mixer"].update(heads=2.5), "heads"),
    (lambda c: c["layers"][1]["mixer"].update(scale="x"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), "dims"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][2].update(type="mamba"), "mamba"),
    (lambda c: c["layers"][0]["mlp"].update(kind="experts"), "experts"),
    (lambda c: c.update(architecture="Other"), "Other"),
    (lambda c: c.update(loop={"start": 0, "stop": 9, "times": 2}), "stop"),
])
def test_bad_configs_are_refused_by_name(tmp_path, edit, what):
    from mesh_llm_b200.capi import B200Error

    cfg = small()
    path = write_checkpoint(tmp_path, cfg, weights(cfg, 1))
    edit(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(B200Error) as e:
        opened(path)
    assert what in str(e.value)


@pytest.mark.parametrize("text", ["", "{", "[1]", '{"a" 1}', '{"architecture": "Gonetar",}', '{"a": 01x}', '{"a": "\\ud800"}',
                                  '{"a": "x', "{}{}", '{"a": nul}', "[" * 200 + "]" * 200])
def test_malformed_json_is_refused(tmp_path, text):
    from mesh_llm_b200.capi import B200Error

    cfg = small()
    path = write_checkpoint(tmp_path, cfg, weights(cfg, 1))
    (tmp_path / "config.json").write_text(text)
    with pytest.raises(B200Error):
        opened(path)


def test_malformed_safetensors_are_refused(tmp_path):
    from mesh_llm_b200.capi import B200Error

    cfg = small()
    path = write_checkpoint(tmp_path, cfg, weights(cfg, 1))
    file = tmp_path / "model.safetensors"
    good = file.read_bytes()
    n = struct.unpack("<Q", good[:8])[0]
    head = json.loads(good[8:8 + n])

    def with_head(h):
        t = json.dumps(h).encode()
        return struct.pack("<Q", len(t)) + t + good[8 + n:]

    bad = [b"", good[:5], good[:8 + n // 2], struct.pack("<Q", 1 << 60) + good[8:], good[:-1]]
    for change in ({"dtype": "F8"}, {"shape": [3, -1]}, {"shape": [1] * 9}, {"data_offsets": [0, 1 << 50]}, {"data_offsets": [4, 2]},
                   {"data_offsets": [0]}):
        h = json.loads(json.dumps(head))
        h["embed"].update(change)
        bad.append(with_head(h))
    for b in bad:
        file.write_bytes(b)
        with pytest.raises(B200Error):
            opened(path)
    os.unlink(file)
    with pytest.raises(B200Error):
        opened(path)
    with pytest.raises(B200Error):
        opened(tmp_path / "nowhere")


def test_struct_layouts_agree_between_header_and_ctypes(tmp_path):
    from mesh_llm_b200 import capi

    for name, cls in (("b200_layer_config", capi.LayerConfig), ("b200_stack_config", capi.StackConfig)):
        fields = header_struct_fields(name)
        size, offs = compiler_layout(name, fields, tmp_path)
        assert C.sizeof(cls) == size
        assert [f for f, _, _ in fields] == [f for f, _ in cls._fields_]
        for f, _, _ in fields:
            assert getattr(cls, f).offset == offs[f], f
