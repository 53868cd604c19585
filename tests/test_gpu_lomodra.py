"""Lomodra on the GPU (matrix-state linear attention under fixed decays and the delta rule, chunked attention with shared
keys and values, experts, per-layer token input) against the plain numpy restatement in lomodra_oracle.py, on small
random models, in bf16 and in 32-bit."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import lomodra_oracle as orc
from hybrid_util import bf16, rel, write_checkpoint
from lomodra_util import attn, config, delta, engine, experts, light, run, tokens, weights

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

CONFIGS = {
    # every mixer alone, with sizes that no vector access divides, heads shared and not, one tap and many
    "light": config([light(3, 20, 36), light(5, 9, 7), light(1, 96, 40)], 88, 101),
    "delta": config([delta(4, 4, 24, 40), delta(6, 2, 13, 11, conv=3, ranks=(9, 5)), delta(3, 1, 40, 17, conv=1, ranks=(30, 70))], 72, 97),
    "attn": config([attn(6, 2, 24, 40, 33), attn(3, 3, 17, 9, 64), attn(5, 1, 72, 70, 21)], 104, 131),
    # queries on another layer's keys and values, behind smaller and larger chunks and with other head counts
    "shared": config([attn(4, 2, 32, 48, 30), attn(4, 2, 32, 48, 75, kv_from=0), attn(8, 2, 32, 48, 11, kv_from=0), light(2, 16, 16),
                      attn(2, 1, 16, 24, 50), attn(2, 1, 16, 24, 50, kv_from=4)], 80, 90),
    # feed-forwards: few and all experts, without a shared one, odd sizes
    "experts": config([light(2, 16, 24, mlp=experts(11, 3, 37, 53)), light(2, 16, 24, mlp=experts(7, 7, 24)), light(2, 16, 24, mlp=experts(5, 1, 40, 24)),
                       light(1, 16, 24), light(2, 16, 24, mlp=experts(1, 1, 16, 8))], 60, 83),
    "side": config([light(2, 16, 16), attn(2, 1, 16, 16, 40), delta(2, 2, 16, 16)], 64, 77, side=21, cap=20.0),
    # everything together
    "mixed": config([delta(4, 2, 32, 48, mlp=experts(8, 2, 48, 72)), attn(4, 2, 40, 32, 45, mlp=experts(6, 3, 32, 40)), light(3, 32, 64, mlp=experts(8, 4, 40)),
                     attn(6, 2, 40, 32, 45, scale=0.25, kv_from=1, mlp=experts(8, 2, 32, 64)), light(2, 48, 16), delta(2, 2, 64, 32, conv=2, mlp=experts(4, 2, 24, 16))],
                    128, 160, side=24, cap=30.0, eps=1e-5),
    # head sizes of large models, more than one key tile per chunk, heads in several groups
    "wide": config([delta(6, 3, 128, 96, ranks=(40, 64), mlp=experts(40, 6, 96, 160)), attn(16, 2, 128, 128, 200, mlp=experts(16, 4, 128, 128)), light(2, 256, 128),
                    attn(4, 4, 192, 256, 150), delta(2, 2, 160, 64), attn(2, 1, 64, 300, 70)], 192, 211, side=64, cap=25.0),
    # values that sizes can happen to share or that are one
    "ones": config([delta(1, 1, 8, 8, conv=1, ranks=(1, 1), mlp=experts(1, 1, 8, 8)), attn(1, 1, 8, 8, 1), light(1, 8, 8, [1.0]), attn(8, 8, 8, 8, 8),
                    light(8, 1, 8)], 48, 64, side=1, cap=50.0),
}
LIMIT = {"float32": 2e-5, "bfloat16": 3e-2}
SMALL = {"ones": 4}  # heads of 8 values or of one do not average their roundings out
SEEDS = {"ones": 1}
PRECISIONS = ("float32", "bfloat16")


def limit(name, precision):
    return LIMIT[precision] * SMALL.get(name, 1)


def worst(err, name, precision):
    """of all rows; where heads are that small, the norms behind them magnify a near-zero output's roundings without bound in
    16 bits: there all but a tenth of the rows"""
    return np.quantile(err, 0.9) if name in SMALL and precision == "bfloat16" else err.max()


_models = {}


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    """name -> (config, weights, checkpoint folder), made once"""
    def get(name):
        if name not in _models:
            cfg = CONFIGS[name]
            w = weights(cfg, SEEDS.get(name, 7))
            _models[name] = (cfg, w, write_checkpoint(tmp_path_factory.mktemp(name), cfg, w))
        return _models[name]
    return get


# ---- every layer, whole prompts ------------------------------------------------------------------------
@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_after_every_layer(model, name, precision):
    import torch

    from mesh_llm_b200.engine import open_stage

    cfg, w, path = model(name)
    toks = tokens(cfg, 170)
    ref, res = orc.forward(cfg, w, toks)
    st = open_stage(path, precision, n_ctx=256, n_seq=1, n_ubatch=256)
    assert st.layer_runs() == len(res)
    for T in (170, 5, 1):  # matrix products, matrix-vector products with several rows and with one
        buf = torch.zeros((len(res), T, cfg["width"]), device="cuda")
        st.trace_residual(buf)
        _, lg, _ = st.forward(tokens=torch.from_numpy(toks[:T]).cuda(), all_logits=True)
        st.trace_residual(None)
        st.synchronize()
        got = buf.cpu().numpy()
        for i in range(len(res)):
            err = rel(got[i], res[i][:T])
            assert worst(err, name, precision) < limit(name, precision), (T, i, int(err.argmax()), err.max())
        assert worst(rel(lg.cpu().numpy(), ref[:T]), name, precision) < limit(name, precision)
    st.close()


# ---- portions, decoding, ring wrap ------------------------------------------------------------------------
@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding(model, name, precision):
    cfg, w, path = model(name)
    toks = tokens(cfg, 330, 1)
    ref, _ = orc.forward(cfg, w, toks)
    # micro-batches of 64: the rings of chunks smaller than the sequence wrap many times
    for n_ubatch, portions in ((256, [330]), (64, [330]), (64, [2, 3, 64, 9, 1, 40, 8, 2, 10, 33, 64, 5]), (64, [200, 1]), (16, [17]), (64, [2])):
        eng = engine(path, precision, n_ctx=330, n_ubatch=n_ubatch)
        err = rel(run(eng, toks, portions), ref)
        assert worst(err, name, precision) < limit(name, precision), (n_ubatch, portions, int(err.argmax()), err.max())
        eng.stage.close()


@pytest.mark.parametrize("precision", PRECISIONS)
def test_long_decoding_token_by_token(model, precision):
    cfg, w, path = model("mixed")
    toks = tokens(cfg, 700, 2)
    ref, _ = orc.forward(cfg, w, toks)
    eng = engine(path, precision, n_ctx=700, n_ubatch=8)
    err = rel(run(eng, toks, [1]), ref)
    assert err.max() < LIMIT[precision], (int(err.argmax()), err.max())


# ---- keys far away and at the chunks' edges --------------------------------------------------------------------
def needle_model(chunk, shared_chunk=None, dim=24, vdim=16):
    """Attention that looks for one token: its key direction is what every query asks for, with a score far above the
    others', and its value is unlike theirs.  Whether it is visible decides the logits.  With shared_chunk a second layer
    looks for it among the first one's keys, and the first one's own queries do not."""
    layers = [attn(2, 1, dim, vdim, chunk)]
    if shared_chunk:
        layers.append(attn(2, 1, dim, vdim, shared_chunk, kv_from=0))
    cfg = config(layers, 48, 64)
    w = weights(cfg, 11)
    e = w["embed"].copy()
    e[:, 40:] = 0
    e[:, 40] = 3.0           # every token: what queries are made from
    e[5] = 0
    e[5, 41] = 6.0           # the needle
    w["embed"] = bf16(e)
    for i in range(len(layers)):
        w[f"l{i}.norm1"][40:] = 0
        q = 0.05 * w[f"l{i}.mix.q"]
        if i == len(layers) - 1:
            q.reshape(2, dim, 48)[:, 0, 40] = 12.0
        w[f"l{i}.mix.q"] = bf16(q)
        w[f"l{i}.mix.q.norm"][:] = w[f"l{i}.mix.q.norm"][:] * 0 + 4
    k, v = 0.4 * w["l0.mix.k"], 0.3 * w["l0.mix.v"]
    k[:, 41] = 0
    k[0, 41] = 8.0
    v[:, 41] = bf16(np.linspace(-2, 2, vdim))
    w["l0.mix.k"], w["l0.mix.v"] = bf16(k), bf16(v)
    w["l0.mix.k.norm"][:] = 4
    return cfg, w


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("chunk", [2, 31, 32, 33, 64, 127, 128, 129, 200])
def test_chunk_edges(tmp_path, chunk, precision):
    cfg, w = needle_model(chunk)
    path = write_checkpoint(tmp_path, cfg, w)
    n = 420
    toks = np.random.default_rng(chunk).integers(6, 64, n).astype(np.int32)
    start = (100 // chunk + 1) * chunk  # a chunk's first position
    last = start + chunk - 1            # and its last
    for needle in (start, start - 1):
        t = toks.copy()
        t[needle] = 5
        ref, _ = orc.forward(cfg, w, t)
        without, _ = orc.forward(cfg, w, toks)
        # the test is sharp: the needle moves the last row of its own chunk and no row of the next
        inside = last if needle == start else start - 1
        if inside != needle:
            assert rel(ref[inside:inside + 1], without[inside:inside + 1]).max() > 0.2
        assert rel(ref[inside + 1:inside + 2], without[inside + 1:inside + 2]).max() < 1e-9
        for portions in ([n], [start, 1], [start - 1, 2], [start + 1, 2], [last, 1, 1], [last + 1, 2], [1], [128, 100, 1], [130, 3]):
            eng = engine(path, precision, n_ctx=n, n_ubatch=128)
            err = rel(run(eng, t, portions), ref)
            assert err.max() < LIMIT[precision], (needle, portions, int(err.argmax()), err.max())
            eng.stage.close()


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("own,other", [(20, 300), (300, 20), (64, 128), (1, 150)])
def test_shared_keys_behind_another_chunk(tmp_path, own, other, precision):
    cfg, w = needle_model(own, other)
    path = write_checkpoint(tmp_path, cfg, w)
    toks = np.random.default_rng(own).integers(6, 64, 400).astype(np.int32)
    needle = other + 2 if other < 100 else 3
    t = toks.copy()
    t[needle] = 5
    ref, _ = orc.forward(cfg, w, t)
    last = needle // other * other + other - 1
    assert rel(ref[last:last + 1], orc.forward(cfg, w, toks)[0][last:last + 1]).max() > 0.2
    for portions in ([400], [last, 1, 1], [64], [needle + 1, 9, 1]):
        eng = engine(path, precision, n_ctx=400, n_ubatch=64)
        err = rel(run(eng, t, portions), ref)
        assert err.max() < LIMIT[precision], (portions, int(err.argmax()), err.max())
        eng.stage.close()


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("dim,vdim", [(24, 16), (128, 128), (256, 320)])
def test_far_key_among_many_in_prompt_and_decoding(tmp_path, dim, vdim, precision):
    cfg, w = needle_model(600, dim=dim, vdim=vdim)
    path = write_checkpoint(tmp_path, cfg, w)
    toks = np.random.default_rng(3).integers(6, 64, 520).astype(np.int32)
    toks[3] = 5
    ref, _ = orc.forward(cfg, w, toks)
    for portions in ([520], [500, 1], [257, 256, 2], [7, 64]):
        eng = engine(path, precision, n_ctx=520, n_ubatch=256)
        err = rel(run(eng, toks, portions), ref)
        assert err.max() < LIMIT[precision], (portions, int(err.argmax()), err.max())
        eng.stage.close()


# ---- states ------------------------------------------------------------------------------------------------------
def slow_model():
    """what the first tokens leave in the states is still there hundreds of tokens later"""
    cfg = config([delta(2, 1, 24, 20, mlp=experts(4, 2, 16)), light(2, 24, 20, [0.9999, 1.0])], 40, 50)
    w = weights(cfg, 5)
    w["l0.mix.A_log"][:] = -9.0
    w["l0.mix.b"][:] = bf16(-0.2 * np.abs(w["l0.mix.b"]))
    return cfg, w


@pytest.mark.parametrize("precision", PRECISIONS)
def test_first_tokens_and_lost_state_show(tmp_path, precision):
    cfg, w = slow_model()
    path = write_checkpoint(tmp_path, cfg, w)
    toks = tokens(cfg, 260, 9)
    ref, _ = orc.forward(cfg, w, toks)
    other = toks.copy()
    other[0] = (other[0] + 1) % cfg["vocab"]
    assert rel(orc.forward(cfg, w, other)[0][-1:], ref[-1:]).max() > 20 * LIMIT["float32"]
    for portions in ([260], [1], [2], [3, 1, 1, 200, 1], [100, 7, 64]):
        eng = engine(path, precision, n_ctx=260, n_ubatch=100)
        err = rel(run(eng, toks, portions), ref)
        assert err.max() < LIMIT[precision], (portions, int(err.argmax()), err.max())
        eng.stage.close()


@pytest.mark.parametrize("precision", PRECISIONS)
def test_decays_that_forget_at_once(tmp_path, precision):
    cfg = config([delta(2, 2, 16, 16), light(2, 16, 16, [1e-3, 0.1])], 40, 50)
    w = weights(cfg, 6)
    w["l0.mix.A_log"][:] = 4.0
    w["l0.mix.dt_bias"][::2] = 3.0  # half of the channels: exp(-55 softplus) is zero in 32-bit
    path = write_checkpoint(tmp_path, cfg, w)
    toks = tokens(cfg, 150, 9)
    ref, _ = orc.forward(cfg, w, toks)
    for portions in ([150], [40, 1], [3, 30]):
        eng = engine(path, precision, n_ctx=150, n_ubatch=64)
        assert rel(run(eng, toks, portions), ref).max() < LIMIT[precision]
        eng.stage.close()


@pytest.mark.parametrize("taps", [2, 4, 7])
def test_convolution_reaches_back_across_portions(tmp_path, taps):
    """the oldest tap alone: a token's q, k and v come from `taps - 1` tokens before it"""
    cfg = config([delta(2, 1, 16, 16, conv=taps)], 40, 50)
    w = weights(cfg, 8)
    for n in ("q", "k", "v"):
        w[f"l0.mix.{n}.conv"][:, 1:] = 0
        w[f"l0.mix.{n}.conv"][:, 0] = 1
    path = write_checkpoint(tmp_path, cfg, w)
    toks = tokens(cfg, 60, 3)
    ref, _ = orc.forward(cfg, w, toks)
    for portions in ([60], [1], [2], [3, 2, 1, 1, 9, 1, 30], [20, 1]):
        eng = engine(path, "float32", n_ctx=60, n_ubatch=32)
        err = rel(run(eng, toks, portions), ref)
        assert err.max() < LIMIT["float32"], (portions, int(err.argmax()), err.max())
        eng.stage.close()


# ---- experts -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("precision", PRECISIONS)
def test_bias_decides_and_weights_are_over_the_chosen(tmp_path, precision):
    """logits far apart: a softmax over all experts would underflow for those that are chosen second and third"""
    cfg = config([light(1, 8, 8, mlp=experts(9, 3, 24, 16)), light(1, 8, 8, mlp=experts(300, 40, 8))], 320, 50)
    w = weights(cfg, 6)
    w["l0.mlp.router"][:] = 0
    w["l0.mlp.router.b"] = bf16(np.array([-150, 300, 5, 299, -2, 0, 298.0, 3, 1]))
    w["l1.mlp.router"][:] = 0
    w["l1.mlp.router.b"] = bf16(np.random.default_rng(0).permutation(300) / 64.0)
    path = write_checkpoint(tmp_path, cfg, w)
    toks = tokens(cfg, 150, 9)
    ref, _ = orc.forward(cfg, w, toks)
    for portions in ([150], [40, 1], [3, 30]):  # every token goes to the same experts: more than one tile each
        eng = engine(path, precision, n_ctx=150, n_ubatch=150)
        assert rel(run(eng, toks, portions), ref).max() < LIMIT[precision]
        eng.stage.close()


# ---- slots ------------------------------------------------------------------------------------------------------------
def test_positions_cannot_be_skipped_or_rewound(model):
    import torch

    from mesh_llm_b200.capi import B200Error
    from mesh_llm_b200.engine import open_stage

    cfg, _, path = model("mixed")
    st = open_stage(path, n_ctx=64, n_seq=2, n_ubatch=32)
    t = torch.from_numpy(tokens(cfg, 12)).cuda()
    st.forward(tokens=t, pos0=0)
    for p in (3, 11, 13):
        with pytest.raises(B200Error):
            st.forward(tokens=t, pos0=p)
    st.forward(tokens=t, pos0=12)
    assert st.seq_pos(0) == 24 and st.seq_pos(1) == -1
    st.close()


@pytest.mark.parametrize("precision", PRECISIONS)
def test_slots_are_reused_and_sequences_do_not_mix(model, precision):
    cfg, w, path = model("mixed")
    eng = engine(path, precision, n_ctx=256, n_seq=3, n_ubatch=64)
    seqs = {i: tokens(cfg, n, 20 + i) for i, n in enumerate((150, 3, 97, 41, 200, 66))}
    alone = {i: run(eng, t, [64], rid=i) for i, t in seqs.items()}
    for i, t in seqs.items():
        assert rel(alone[i], orc.forward(cfg, w, t)[0]).max() < LIMIT[precision]
    # interleaved in three slots; a finished sequence's slot goes to the next one
    got = {i: [] for i in seqs}
    at = dict.fromkeys(seqs, 0)
    waiting, live = list(seqs), []
    rng = np.random.default_rng(4)
    while waiting or live:
        while waiting and len(live) < 3:
            live.append(waiting.pop(0))
        i = live[rng.integers(len(live))]
        n = int(rng.choice([1, 1, 2, 5, 9, 30, 64]))
        part = seqs[i][at[i]:at[i] + n]
        got[i].append(eng.feed(i, part, range(len(part))))
        at[i] += len(part)
        if at[i] == len(seqs[i]):
            eng.end(i)
            live.remove(i)
    for i in seqs:
        assert rel(np.concatenate(got[i]), alone[i]).max() < LIMIT[precision]
    # the same sequence in the same slot after others: bit for bit what it was
    assert np.array_equal(run(eng, seqs[2], [64], rid="again"), alone[2])


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("name", ["mixed", "wide", "delta", "shared"])
def test_batches_of_sequences_equal_each_alone(model, name, precision):
    import torch

    from mesh_llm_b200.engine import open_stage

    cfg, w, path = model(name)
    seqs = np.stack([tokens(cfg, 60, 30 + i) for i in range(12)])
    ref = np.stack([orc.forward(cfg, w, s)[0] for s in seqs])
    st = open_stage(path, precision, n_ctx=64, n_seq=12, n_ubatch=12 * 40)
    for n_seq in (1, 3, 12):
        t = torch.from_numpy(seqs[:n_seq]).cuda()
        _, lg, _ = st.forward(tokens=t[:, :40].contiguous(), n_seq=n_seq, T=40, pos0=0)
        assert rel(lg.cpu().numpy(), ref[:n_seq, 39]).max() < LIMIT[precision]
        _, lg, _ = st.forward(tokens=t[:, 40:42].contiguous(), n_seq=n_seq, T=2, pos0=40)
        assert rel(lg.cpu().numpy(), ref[:n_seq, 41]).max() < LIMIT[precision]
        for p in range(42, 60):
            _, lg, nxt = st.forward(tokens=t[:, p].contiguous(), n_seq=n_seq, T=1, pos0=p)
            err = rel(lg.cpu().numpy(), ref[:n_seq, p])
            assert err.max() < LIMIT[precision], (n_seq, p, err)
            assert np.array_equal(nxt.cpu().numpy(), lg.cpu().numpy().argmax(-1))
    st.synchronize()
    st.close()


# ---- stages -------------------------------------------------------------------------------------------------------------
def test_two_stages_equal_one(model):
    import torch

    from mesh_llm_b200.capi import B200Error
    from mesh_llm_b200.checkpoint import Checkpoint
    from mesh_llm_b200.stage import Stage

    cfg, w, path = model("mixed")
    toks = tokens(cfg, 50, 8)
    ref, _ = orc.forward(cfg, w, toks)
    with Checkpoint(path) as ck:
        a, _, _ = Stage.from_checkpoint(ck, 0, 4, n_ctx=64, n_ubatch=64, precision=1)
        b, _, _ = Stage.from_checkpoint(ck, 4, -1, n_ctx=64, n_ubatch=64, precision=1)
        assert (a.cfg.has_embd, a.cfg.has_output, b.cfg.has_embd, b.cfg.has_output) == (1, 0, 0, 1)
        with pytest.raises(B200Error):  # a layer that reads another's keys stays with it
            Stage.from_checkpoint(ck, 2, -1, n_ctx=64)
    t = torch.from_numpy(toks).cuda()
    for lo, hi in ((0, 40), (40, 41), (41, 50)):
        part = t[lo:hi].contiguous()
        hid, _, _ = a.forward(tokens=part, pos0=lo)
        with pytest.raises(B200Error):  # the token input of the later layers needs the ids
            b.forward(hidden_in=hid, pos0=lo)
        _, lg, _ = b.forward(tokens=part, hidden_in=hid, pos0=lo, all_logits=True)
        assert rel(lg.cpu().numpy(), ref[lo:hi]).max() < LIMIT["float32"]


# ---- generation and commands ---------------------------------------------------------------------------------------------
def continuation(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(orc.forward(cfg, w, seq)[0][-1].argmax()))
    return seq[len(prompt):]


def test_greedy_generation(model):
    for name in ("mixed", "delta"):
        cfg, w, path = model(name)
        prompts = [tokens(cfg, n, 50 + n).tolist() for n in (1, 7, 40, 7, 7)]
        want = [continuation(cfg, w, p, 12) for p in prompts]
        for n_seq in (1, 2, 5):  # one after the other, slots that come free, all at once
            eng = engine(path, "float32", n_ctx=64, n_seq=n_seq, n_ubatch=32)
            assert eng.generate(prompts, 12) == want
            assert eng.free == list(range(n_seq)) and not eng.live


def test_generate_command(model):
    cfg, w, path = model("side")
    p = tokens(cfg, 9, 1).tolist()
    out = subprocess.run([sys.executable, "-m", "mesh_llm_b200.generate", "--model", path, "--dtype", "float32", "-n", "6",
                          "--tokens", ",".join(map(str, p)), "--tokens", str(p[0])], capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert out.returncode == 0, out.stderr[-2000:]
    assert out.stdout.split() == [",".join(map(str, continuation(cfg, w, q, 6))) for q in (p, p[:1])]


@pytest.mark.parametrize("precision", PRECISIONS)
def test_trace_command(model, tmp_path, precision):
    cfg, w, path = model("mixed")
    a, b = tokens(cfg, 70, 1), tokens(cfg, 33, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50].tolist(), "want": [0, 49, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:69].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[69:].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b.tolist(), "want": [32]}], "end": ["b"]}]
    out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", precision, "--out", str(tmp_path),
                          "--max-tokens", "80"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                         cwd=ROOT, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    assert [l for l in out.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb = orc.forward(cfg, w, a)[0], orc.forward(cfg, w, b)[0]
    assert not (tmp_path / "1.f32").exists()
    for n, ref in ((0, ra[[0, 49, 7]]), (2, ra[[69]]), (3, rb[[32]])):
        got = np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(len(ref), cfg["vocab"])
        assert rel(got, ref).max() < LIMIT[precision], n
