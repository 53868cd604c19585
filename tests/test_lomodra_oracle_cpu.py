"""No GPU: the plain restatement the GPU tests compare with, checked against direct formulas and its own invariances; the
checkpoint reader's view of the architecture."""
import json

import numpy as np
import pytest

import lomodra_oracle as orc
from hybrid_util import write_checkpoint
from lomodra_util import attn, config, delta, experts, light, shapes, tokens, weights

rng = np.random.default_rng(0)


def test_decayed_outer_products_are_a_weighted_sum_over_the_past():
    q, k, v, d = rng.standard_normal((7, 2, 3)), rng.standard_normal((7, 2, 3)), rng.standard_normal((7, 2, 4)), np.array([0.5, 0.9])
    o = orc.decayed_outer_products(q, k, v, d)
    for t in range(7):
        for h in range(2):
            want = sum(d[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert np.allclose(o[t, h], want)


def test_delta_rule_recalls_what_it_wrote_last():
    """unit keys, full write strength, no decay: reading with the key just written gives its value"""
    T, H, d, e = 6, 2, 5, 3
    k, v = orc.unit(rng.standard_normal((T, H, d))), rng.standard_normal((T, H, e))
    one = np.ones((T, H, d))
    assert np.allclose(orc.delta_rule(k, k, v, one, np.ones((T, H))), v, atol=1e-4)
    # orthogonal keys, half strength: a plain sum of halves, decayed by the products of what came after
    k = np.repeat(np.eye(d)[None, :, None].transpose(1, 2, 0, 3).reshape(d, 1, d), H, 1)
    v, g = rng.standard_normal((d, H, e)), rng.uniform(0.3, 1, (d, H, d))
    q = rng.standard_normal((d, H, d))
    o = orc.delta_rule(q, k, v, g, np.full((d, H), 0.5))
    for t in range(d):
        want = sum(0.5 * q[t, :, s, None] * np.prod(g[s + 1:t + 1, :, s], axis=0)[:, None] * v[s] for s in range(t + 1))
        assert np.allclose(o[t], want)


@pytest.mark.parametrize("chunk", [1, 4, 100])
def test_chunked_attention_by_loops(chunk):
    q, k, v = rng.standard_normal((11, 4, 3)), rng.standard_normal((11, 2, 3)), rng.standard_normal((11, 2, 5))
    o = orc.chunked_attention(q, k, v, 0.7, chunk)
    for t in range(11):
        lo = t - t % chunk
        for h in range(4):
            w = np.exp(0.7 * k[lo:t + 1, h // 2] @ q[t, h])
            assert np.allclose(o[t, h], (w / w.sum()) @ v[lo:t + 1, h // 2])


def test_convolution_by_loops():
    x, taps = rng.standard_normal((7, 3)), rng.standard_normal((3, 4))
    y = orc.causal_conv(x, taps)
    for t in range(7):
        assert np.allclose(y[t], sum(taps[:, 3 - j] * x[t - j] for j in range(4) if t - j >= 0))
    assert np.allclose(orc.causal_conv(x, taps[:, -1:]), x * taps[:, -1])


def test_routes_weigh_the_chosen_logits_only():
    z = np.array([[1.0, 3.0, 2.0, -5.0], [400.0, -400.0, 0.0, 399.0]])
    r = orc.route(z, 2)
    assert np.allclose(r[0], [0, 1 / (1 + np.exp(-1)), 1 / (1 + np.exp(1)), 0])
    assert np.allclose(r[1, [0, 3]].sum(), 1) and (r[1, 1:3] == 0).all()
    assert np.allclose(orc.route(z[:1], 4), np.exp(z[:1]) / np.exp(z[:1]).sum())
    assert (orc.route(z, 1) == np.array([[0, 1, 0, 0], [1, 0, 0, 0]])).all()


def test_token_input_takes_the_layers_own_slice():
    cfg = config([light(1, 4, 4), light(1, 4, 4)], 8, 10, side=3)
    w = weights(cfg, 1)
    x, t = rng.standard_normal((2, 8)), np.array([3, 9])
    a = orc.token_input(x, w, 1, t, 3, 0.0)
    y = (orc.gelu_tanh(x @ w["l1.side.gate"].T) * w["side.embed"][t, 3:6]) @ w["l1.side.proj"].T
    assert np.allclose(a, y / np.sqrt((y * y).mean(-1, keepdims=True)) * w["l1.side.norm"])


def test_causal_and_every_mechanism_reaches_the_logits():
    cfg = config([delta(2, 1, 6, 5, mlp=experts(5, 2, 6, 7)), light(2, 4, 6, mlp=experts(4, 4, 5)), attn(4, 2, 6, 5, 8), attn(4, 2, 6, 5, 8, kv_from=2)],
                 24, 30, side=4, cap=3.0)
    w = weights(cfg, 3)
    toks = tokens(cfg, 20)
    full, _ = orc.forward(cfg, w, toks)
    assert np.abs(full).max() < 3.0
    assert np.allclose(orc.forward(cfg, w, toks[:13])[0], full[:13])
    for name in w:  # no tensor is without effect
        if ".mlp.e" in name:  # an expert may not be chosen
            continue
        changed = dict(w, **{name: w[name] * rng.uniform(0.5, 1.5, w[name].shape)})
        assert np.abs(orc.forward(cfg, changed, toks)[0] - full).max() > 1e-6, name


def test_chunks_do_not_see_one_another():
    cfg = config([attn(2, 1, 6, 5, 7)], 16, 30)
    w = weights(cfg, 4)
    toks = tokens(cfg, 20)
    other = toks.copy()
    other[6] = (other[6] + 1) % 30
    d = np.abs(orc.forward(cfg, w, other)[0] - orc.forward(cfg, w, toks)[0]).max(-1)
    assert d[6] > 1e-6 and d[:6].max() == 0 and d[7:].max() == 0


# ---- the checkpoint reader -----------------------------------------------------------------------------
def small():
    return config([delta(6, 2, 8, 10, conv=3, ranks=(5, 7), mlp=experts(5, 2, 6, 7)), light(2, 4, 6, [0.25, 0.75], mlp=experts(4, 4, 5)),
                   attn(4, 2, 6, 5, 9, scale=0.3), attn(8, 2, 6, 5, 17, kv_from=2)], 24, 19, side=4, cap=3.0, eps=2e-4)



def test_config_becomes_layer_descriptions(tmp_path):
    from mesh_llm_b200 import capi
    from mesh_llm_b200.checkpoint import Checkpoint

    cfg = small()
    with Checkpoint(write_checkpoint(tmp_path, cfg, weights(cfg, 1))) as ck:
        assert ck.architecture == "Lomodra"
        assert {n: tuple(s) for n, (_, _, s) in ck.tensors().items()} == {n: tuple(s) for n, s in shapes(cfg).items()}
        c, s, layers = ck.stage_config(n_ctx=50, n_seq=3, n_ubatch=16)
        assert (c.n_layer, c.n_embd, c.n_vocab) == (4, 24, 19) and c.rms_eps == np.float32(2e-4)
        assert (s.embd_scale, s.norm_offset, s.norm_place, s.side_dim, s.logit_softcap, s.loop_times) == (1.0, 0.0, capi.NORM_OUTPUT, 4, 3.0, 0)
        a, b, d, e = layers
        assert (a.mixer, a.n_head, a.n_head_kv, a.qk_dim, a.v_dim, a.conv_taps) == (capi.MIXER_DELTA_STATE, 6, 2, 8, 10, 3)
        assert (a.decay_rank, a.gate_rank) == (5, 7)
        assert (a.ffn, a.n_expert, a.n_expert_used, a.n_ff_exp, a.n_ff_shared) == (capi.FFN_MOE, 5, 2, 6, 7)
        assert (b.mixer, b.n_head, b.qk_dim, b.v_dim, b.n_ff_shared) == (capi.MIXER_DECAY_STATE, 2, 4, 6, 0)
        assert (d.mixer, d.n_head, d.n_head_kv, d.chunk, d.window, d.kv_shared, d.ffn) == (capi.MIXER_GQA, 4, 2, 9, 0, 0, capi.FFN_NONE)
        assert d.attn_scale == np.float32(0.3)
        assert (e.kv_shared, e.kv_layer, e.chunk, e.n_head) == (1, 2, 17, 8)


def test_optional_parts_may_be_absent_or_null(tmp_path):
    from mesh_llm_b200.checkpoint import Checkpoint

    cfg = config([light(1, 4, 4)], 8, 10)
    for k, extra in enumerate(({}, {"token_side": None, "logit_softcap": None})):
        c = dict(cfg, **extra)
        w = weights(cfg, 1)
        with Checkpoint(write_checkpoint(tmp_path / str(k), c, w)) as ck:
            _, s, layers = ck.stage_config()
            assert (s.side_dim, s.logit_softcap, layers[0].ffn) == (0, 0.0, 0)


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "layers[0].mixer.conv"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_heads"), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, "x"]), "decay"),
    (lambda c: c["layers"][2]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "dense"),
    (lambda c: c["layers"][1].update(type="mamba"), "mamba"),
    (lambda c: c["token_side"].pop("dim"), "token_side.dim"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
])
def test_bad_configs_are_refused_by_name(tmp_path, edit, what):
    from mesh_llm_b200.capi import B200Error
    from mesh_llm_b200.checkpoint import Checkpoint

    cfg = small()
    path = write_checkpoint(tmp_path, cfg, weights(cfg, 1))
    edit(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(B200Error) as e:
        Checkpoint(path)
    assert what in str(e.value)
