"""Gonetar on the GPU (gated linear recurrence, windowed latent attention, sandwich norms, looped layers) against the
plain numpy restatement in hybrid_oracle.py, on small random models, in bf16 and in 32-bit."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import hybrid_oracle as orc
from hybrid_util import attn, bf16, config, rec, rel, weights, write_checkpoint

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

CONFIGS = {
    # recurrence alone: block sizes and widths that are no multiple of anything, one tap, one block
    "rec": config([rec(120, 3, 4), rec(72, 1, 1, ff=88), rec(56, 7, 6, ff=40)], width=88, vocab=101, scale=3.0),
    # latent attention alone
    "attn": config([attn(3, 24, 8, 40, 48, window=17, ff=72), attn(5, 40, 16, 16, 72, window=33)], width=104, vocab=131, scale=2.0),
    # both, looped, a feed-forward missing, layers behind the loop
    "mixed": config([rec(96, 2, 3, ff=64), attn(2, 32, 32, 48, 56, window=25, base=500.0, ff=80), rec(128, 8, 4), rec(64, 4, 2, ff=96)],
                    width=96, vocab=160, loop=(0, 3, 3), scale=5.0, eps=1e-5),
    # sizes no vector access divides
    "odd": config([rec(51, 3, 4, ff=37), attn(3, 13, 6, 11, 29, window=9, ff=53), rec(26, 2, 2)], width=45, vocab=77, loop=(1, 2, 2)),
    # values that sizes can happen to share or that are one
    "ones": config([attn(1, 8, 2, 1, 8, window=1, ff=8), rec(8, 8, 1, ff=8), attn(1, 16, 16, 16, 16, window=64)], width=16, vocab=32),
    # head sizes of large models: several 64-wide boxes per operand, more than one key tile per window
    "wide": config([attn(2, 128, 64, 128, 256, window=150, ff=160), rec(256, 1, 4, ff=128), attn(20, 64, 32, 80, 320, window=300)],
                   width=160, vocab=211, scale=4.0),
    "unrotated": config([attn(4, 32, 0, 32, 64, window=40, ff=64)], width=64, vocab=97),
}
LIMIT = {"float32": 2e-5, "bfloat16": 3e-2}
SMALL = {"ones": 3}  # a row of 16 values does not average its bf16 roundings out
PRECISIONS = ("float32", "bfloat16")


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


_stage_dirs = {}


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    """name -> (config, weights, checkpoint folder), made once"""
    def get(name):
        if name not in _stage_dirs:
            cfg = CONFIGS[name]
            w = weights(cfg, 7)
            _stage_dirs[name] = (cfg, w, write_checkpoint(tmp_path_factory.mktemp(name), cfg, w))
        return _stage_dirs[name]
    return get


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


# ---- projections -----------------------------------------------------------------------------------
@pytest.mark.parametrize("N,K", [(1, 8), (37, 45), (300, 192), (129, 1000), (768, 2560), (65, 12296)])
def test_bf16_mul_mat(N, K):
    import torch

    from mesh_llm_b200 import ops

    rng = np.random.default_rng(N + K)
    w = torch.from_numpy(bf16(rng.standard_normal((N, K)))).cuda()
    W = ops.upload_bf16(w)
    for M in (1, 2, 3, 5, 8, 9, 64, 130):
        x = torch.from_numpy(rng.standard_normal((M, K)).astype(np.float32)).cuda()
        got = ops.mul_mat_bf16(W, x, N, K).double()
        ref = (x if M <= 8 else x.bfloat16().float()).double() @ w.double().T
        err = ((got - ref).abs().max() / ref.abs().max()).item()
        # the operands are exact, what is left is the f32 sum: rounded per step on CUDA cores, truncated on tensor cores
        assert err < (3e-6 if M <= 8 else 3e-6 + 2e-9 * K), (M, err)


# ---- every layer run, whole prompts ------------------------------------------------------------------
@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_residual_after_every_layer_run(model, name, precision):
    import torch

    from mesh_llm_b200.engine import open_stage

    cfg, w, path = model(name)
    toks = tokens(cfg, 90)
    ref, res = orc.forward(cfg, w, toks)
    st = open_stage(path, precision, n_ctx=128, n_seq=1, n_ubatch=128)
    assert st.layer_runs() == len(res)
    for T in (90, 5):  # tensor-core / f32 GEMM path, matrix-vector path
        buf = torch.zeros((len(res), T, cfg["width"]), device="cuda")
        st.trace_residual(buf)
        _, lg, _ = st.forward(tokens=torch.from_numpy(toks[:T]).cuda(), all_logits=True)
        st.trace_residual(None)
        st.synchronize()
        got = buf.cpu().numpy()
        for i in range(len(res)):
            assert rel(got[i], res[i][:T]).max() < LIMIT[precision], (T, i, rel(got[i], res[i][:T]).max())
        assert rel(lg.cpu().numpy(), ref[:T]).max() < LIMIT[precision]
    st.close()


# ---- portions, decoding, ring wrap --------------------------------------------------------------------
@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding(model, name, precision):
    cfg, w, path = model(name)
    toks = tokens(cfg, 330, 1)
    ref, _ = orc.forward(cfg, w, toks)
    # micro-batches of 64: the ring of a window smaller than the sequence wraps many times
    for n_ubatch, portions in ((256, [330]), (64, [330]), (64, [2, 3, 64, 9, 1, 40, 8, 2, 10, 33, 64, 5]), (64, [200, 1]), (16, [17])):
        eng = engine(path, precision, n_ctx=330, n_ubatch=n_ubatch)
        err = rel(run(eng, toks, portions), ref)
        assert err.max() < LIMIT[precision] * SMALL.get(name, 1), (n_ubatch, portions, int(err.argmax()), err.max())
        eng.stage.close()


@pytest.mark.parametrize("precision", PRECISIONS)
def test_long_decoding_token_by_token(model, precision):
    cfg, w, path = model("mixed")
    toks = tokens(cfg, 700, 2)
    ref, _ = orc.forward(cfg, w, toks)
    eng = engine(path, precision, n_ctx=700, n_ubatch=8)
    err = rel(run(eng, toks, [1]), ref)
    assert err.max() < LIMIT[precision], (int(err.argmax()), err.max())


# ---- keys at the window's edges -------------------------------------------------------------------------
def needle_model(window, vdim=16):
    """One attention layer that looks for one token: its key direction is what every query asks for, with a score far
    above the others', and its value is unlike theirs.  Whether it is inside the window decides the logits."""
    cfg = config([attn(2, 16, 8, vdim, 32, window=window)], width=48, vocab=64, scale=1.0)
    w = weights(cfg, 11)
    e = w["embed"].copy()
    e[:, 40:] = 0
    e[:, 40] = 1.0          # every token: what queries are made from
    e[5] = 0
    e[5, 41] = 6.0          # the needle
    w["embed"] = bf16(e)
    w["l0.norm1"][40:] = 0
    q = 0.05 * w["l0.mix.q"]
    q.reshape(2, 24, 48)[:, 0, 40] = 12.0
    w["l0.mix.q"] = bf16(q)
    dkv = 0.3 * w["l0.mix.dkv"]
    dkv[0] = 0
    dkv[0, 41] = 8.0        # latent value 0: the needle's
    w["l0.mix.dkv"] = bf16(dkv)
    uk = 0.1 * w["l0.mix.uk"]
    uk.reshape(2, 16, 32)[:, 0, 0] = 4.0
    w["l0.mix.uk"] = bf16(uk)
    return cfg, w


@pytest.mark.parametrize("precision", PRECISIONS)
@pytest.mark.parametrize("window", [2, 31, 32, 33, 64, 127, 128, 129, 200])
def test_window_edges(tmp_path, window, precision):
    cfg, w = needle_model(window)
    path = write_checkpoint(tmp_path, cfg, w)
    n = 300
    rng = np.random.default_rng(window)
    toks = rng.integers(6, 64, n).astype(np.int32)
    needle = 64
    toks[needle] = 5
    ref, _ = orc.forward(cfg, w, toks)
    inside, outside = needle + window - 1, needle + window
    without, _ = orc.forward(cfg, w, np.where(toks == 5, 6, toks))
    # the test is sharp: the needle moves the last row that sees it, and no later one
    assert rel(ref[inside:inside + 1], without[inside:inside + 1]).max() > 0.2
    assert rel(ref[outside:outside + 1], without[outside:outside + 1]).max() < 1e-9
    for portions in ([n], [inside, 1], [outside, 1], [needle, 2], [needle + 1, window - 1, 2, 9], [1], [128, 100, 1]):
        eng = engine(path, precision, n_ctx=n, n_ubatch=128)
        err = rel(run(eng, toks, portions), ref)
        assert err.max() < LIMIT[precision], (portions, int(err.argmax()), err.max())
        eng.stage.close()


@pytest.mark.parametrize("precision", PRECISIONS)
def test_far_key_among_many_in_prompt_and_decoding(tmp_path, precision):
    cfg, w = needle_model(600)
    path = write_checkpoint(tmp_path, cfg, w)
    toks = np.random.default_rng(3).integers(6, 64, 520).astype(np.int32)
    toks[3] = 5
    ref, _ = orc.forward(cfg, w, toks)
    for portions in ([520], [500, 1], [257, 256, 2], [7, 64]):
        eng = engine(path, precision, n_ctx=520, n_ubatch=256)
        err = rel(run(eng, toks, portions), ref)
        assert err.max() < LIMIT[precision], (portions, int(err.argmax()), err.max())
        eng.stage.close()


# ---- the state at the start of a sequence ----------------------------------------------------------------
@pytest.mark.parametrize("precision", PRECISIONS)
def test_first_tokens_and_lost_state_show(tmp_path, precision):
    """slow decays: what the first token leaves in the state is still there hundreds of tokens later"""
    cfg = config([rec(64, 4, 4), rec(48, 2, 3, ff=40)], width=40, vocab=50, scale=2.0)
    w = weights(cfg, 5)
    for i in (0, 1):
        w[f"l{i}.mix.lam"] = bf16(np.full_like(w[f"l{i}.mix.lam"], -9.0))
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


def test_positions_cannot_be_skipped_or_rewound(model):
    import torch

    from mesh_llm_b200.capi import B200Error
    from mesh_llm_b200.engine import open_stage

    cfg, _, path = model("mixed")
    st = open_stage(path, n_ctx=64, n_seq=2, n_ubatch=32)
    t = torch.from_numpy(tokens(cfg, 12)).cuda()
    with pytest.raises(B200Error):
        st.forward(tokens=t, pos0=3)
    st.forward(tokens=t, pos0=0)
    assert st.seq_pos(0) == 12 and st.seq_pos(1) == -1
    for p in (11, 13, 1):
        with pytest.raises(B200Error):
            st.forward(tokens=t, pos0=p)
    st.forward(tokens=t, pos0=12)
    st.forward(tokens=t, pos0=0)  # a new sequence
    assert st.seq_pos(0) == 12
    st.close()


# ---- slots ------------------------------------------------------------------------------------------------
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
    again = run(eng, seqs[2], [64], rid="again")
    assert np.array_equal(again, alone[2])


@pytest.mark.parametrize("precision", PRECISIONS)
def test_batches_of_sequences_equal_each_alone(model, precision):
    import torch

    from mesh_llm_b200.engine import open_stage

    for name in ("mixed", "wide", "odd"):
        cfg, w, path = model(name)
        seqs = np.stack([tokens(cfg, 60, 30 + i) for i in range(12)])
        ref = np.stack([orc.forward(cfg, w, s)[0] for s in seqs])
        st = open_stage(path, precision, n_ctx=64, n_seq=12, n_ubatch=12 * 40)
        for n_seq in (1, 3, 12):
            t = torch.from_numpy(seqs[:n_seq]).cuda()
            _, lg, _ = st.forward(tokens=t[:, :40].contiguous(), n_seq=n_seq, T=40, pos0=0)
            assert rel(lg.cpu().numpy(), ref[:n_seq, 39]).max() < LIMIT[precision]
            for p in range(40, 60):
                _, lg, nxt = st.forward(tokens=t[:, p].contiguous(), n_seq=n_seq, T=1, pos0=p)
                assert rel(lg.cpu().numpy(), ref[:n_seq, p]).max() < LIMIT[precision], (name, n_seq, p)
                assert np.array_equal(nxt.cpu().numpy(), lg.cpu().numpy().argmax(-1))
        st.synchronize()
        st.close()


# ---- stages -------------------------------------------------------------------------------------------------
def test_two_stages_equal_one(model):
    import torch

    from mesh_llm_b200.capi import B200Error
    from mesh_llm_b200.checkpoint import Checkpoint
    from mesh_llm_b200.stage import Stage

    cfg, w, path = model("mixed")
    toks = tokens(cfg, 50, 8)
    ref, _ = orc.forward(cfg, w, toks)
    with Checkpoint(path) as ck:
        a, _, _ = Stage.from_checkpoint(ck, 0, 3, n_ctx=64, n_ubatch=64, precision=1)
        b, _, _ = Stage.from_checkpoint(ck, 3, -1, n_ctx=64, n_ubatch=64, precision=1)
        assert (a.cfg.has_embd, a.cfg.has_output, b.cfg.has_embd, b.cfg.has_output) == (1, 0, 0, 1)
        with pytest.raises(B200Error):  # the loop's layers stay together
            Stage.from_checkpoint(ck, 0, 2, n_ctx=64)
    t = torch.from_numpy(toks).cuda()
    for lo, hi in ((0, 40), (40, 41), (41, 50)):
        hid, _, _ = a.forward(tokens=t[lo:hi].contiguous(), pos0=lo)
        _, lg, _ = b.forward(hidden_in=hid, pos0=lo, all_logits=True)
        assert rel(lg.cpu().numpy(), ref[lo:hi]).max() < LIMIT["float32"]


# ---- generation and commands --------------------------------------------------------------------------------
def test_greedy_generation(model):
    for name in ("mixed", "attn"):
        cfg, w, path = model(name)
        prompts = [tokens(cfg, n, 50 + n).tolist() for n in (1, 7, 40, 7, 7)]
        want = []
        for p in prompts:
            seq = list(p)
            for _ in range(12):
                seq.append(int(orc.forward(cfg, w, seq)[0][-1].argmax()))
            want.append(seq[len(p):])
        for n_seq in (1, 2, 5):  # one after the other, slots that come free, all at once
            eng = engine(path, "float32", n_ctx=64, n_seq=n_seq, n_ubatch=32)
            assert eng.generate(prompts, 12) == want
            assert eng.free == list(range(n_seq)) and not eng.live
        stop = want[2][4]
        assert eng.generate([prompts[2]], 12, stop=[stop])[0] == want[2][:want[2].index(stop) + 1]


def test_generate_command(model):
    cfg, w, path = model("rec")
    p = tokens(cfg, 9, 1).tolist()
    out = subprocess.run([sys.executable, "-m", "mesh_llm_b200.generate", "--model", path, "--dtype", "float32", "-n", "6",
                          "--tokens", ",".join(map(str, p)), "--tokens", str(p[0])], capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert out.returncode == 0, out.stderr[-2000:]
    want = []
    for q in (p, p[:1]):
        seq = list(q)
        for _ in range(6):
            seq.append(int(orc.forward(cfg, w, seq)[0][-1].argmax()))
        want.append(",".join(map(str, seq[len(q):])))
    assert out.stdout.split() == want


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
