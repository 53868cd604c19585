"""No GPU: the engine's slots, micro-batches and decode batches, with a stage that only records what it is asked to run."""
import types

import numpy as np
import pytest
import torch

from mesh_llm_b200.engine import Engine, PrecisionError, open_stage


class FakeStage:
    """next token of a sequence = (sum of its tokens so far + number of them) mod vocab; logits are one-hot of it"""

    def __init__(self, n_ctx=64, n_seq=3, n_ubatch=8, vocab=50):
        self.cfg = types.SimpleNamespace(has_embd=1, has_output=1, n_ctx=n_ctx, n_seq=n_seq, n_ubatch=n_ubatch, n_vocab=vocab)
        self.device = torch.device("cpu")
        self.seqs = [[] for _ in range(n_seq)]
        self.calls = []

    def forward(self, tokens, n_seq, T, pos0, logits, next_tokens, all_logits=False, seq0=0):
        assert tokens.numel() == n_seq * T <= self.cfg.n_ubatch and pos0 + T <= self.cfg.n_ctx
        self.calls.append((seq0, n_seq, T, pos0, bool(all_logits)))
        for s in range(n_seq):
            q = self.seqs[seq0 + s]
            if pos0 == 0:
                q.clear()
            assert len(q) == pos0
            for t in range(T):
                q.append(int(tokens.reshape(n_seq, T)[s, t]))
                row = s * T + t if all_logits else s
                if all_logits or t == T - 1:
                    nxt = expected(q, self.cfg.n_vocab)
                    logits[row] = 0
                    logits[row, nxt] = 1
                    next_tokens[row] = nxt

    def synchronize(self):
        pass


def expected(q, vocab=50):
    return (sum(q) + len(q)) % vocab


def continuation(prompt, n, vocab=50):
    q = list(prompt)
    for _ in range(n):
        q.append(expected(q, vocab))
    return q[len(prompt):]


def test_feed_cuts_micro_batches_and_returns_wanted_places():
    st = FakeStage()
    eng = Engine(st)
    toks = list(range(1, 21))
    out = eng.feed("a", toks, [0, 7, 8, 19])
    assert [c[2:] for c in st.calls] == [(8, 0, True), (8, 8, True), (4, 16, False)]
    assert [int(r.argmax()) for r in out] == [expected(toks[:i + 1]) for i in (0, 7, 8, 19)]
    out = eng.feed("a", [3], [0])
    assert st.calls[-1][2:] == (1, 20, False) and int(out[0].argmax()) == expected(toks + [3])
    assert eng.feed("a", [4, 5]).shape == (0, 50) and eng.live["a"].pos == 23


def test_slots_come_and_go():
    eng = Engine(FakeStage(n_seq=2))
    eng.feed("a", [1])
    eng.feed("b", [2])
    with pytest.raises(RuntimeError):
        eng.feed("c", [3])
    slot = eng.live["a"].slot
    eng.end("a")
    eng.feed("c", [3, 4])
    assert eng.live["c"].slot == slot and eng.stage.seqs[slot] == [3, 4]
    with pytest.raises(ValueError):
        eng.start("c")
    with pytest.raises(KeyError):
        eng.end("a")


def test_bad_input_is_refused_before_it_runs():
    st = FakeStage()
    eng = Engine(st)
    for toks, want in (([50], []), ([-1], []), ([1], [1]), ([1], [-1]), (list(range(40)) * 2, [])):
        with pytest.raises(ValueError):
            eng.feed("a", toks, want)
    assert not st.calls


@pytest.mark.parametrize("n_seq", [1, 2, 3, 5])
def test_generation_equals_each_alone(n_seq):
    prompts = [[5], [1, 2, 3], list(range(17)), [7, 7, 7], [9, 1, 4], [2, 2]]
    st = FakeStage(n_seq=n_seq)
    eng = Engine(st)
    assert eng.generate(prompts, 9) == [continuation(p, 9) for p in prompts]
    assert not eng.live and eng.free == list(range(n_seq))
    if n_seq >= 3:  # neighbours at one position are one batch
        assert any(c[1] > 1 for c in st.calls)
    assert all(c[1] == 1 or c[2] == 1 for c in st.calls)


def test_generation_stops():
    eng = Engine(FakeStage())
    full = continuation([4, 5], 12)
    stop = full[5]
    assert eng.generate([[4, 5]], 12, stop=[stop]) == [full[:full.index(stop) + 1]]
    assert eng.generate([[4, 5]], 0) == [[]]
    with pytest.raises(ValueError):
        eng.generate([[]], 3)
    with pytest.raises(ValueError):  # more tokens than the cache has room for
        Engine(FakeStage(n_ctx=10)).generate([[1, 2, 3]], 20)


def test_quantised_model_has_no_32_bit_mode(tmp_path):
    f = tmp_path / "m.gguf"
    f.write_bytes(b"")
    with pytest.raises(PrecisionError):
        open_stage(str(f), "float32")


def test_trace_command_refuses_32_bit_of_a_quantised_model(tmp_path):
    from mesh_llm_b200 import trace

    f = tmp_path / "m.gguf"
    f.write_bytes(b"")
    assert trace.main(["--model", str(f), "--dtype", "float32", "--out", str(tmp_path)]) == 3
