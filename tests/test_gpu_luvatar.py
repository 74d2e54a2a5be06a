"""Luvatar on the GPU against the tests' plain model: every mechanism alone and together, in bf16 and f32, in prompts, in
portions, token by token, in batches and slots, through the engine's own entry points."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from tests import luvatar_models as L
from tests import oracle_luvatar as O
from tests.oracle_luvatar import OracleLuvatar

pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ("float32", "bfloat16")


def engine(cfg, w, dtype, **kw):
    from ironmill_b200.engine import CudaConfig, CudaInference
    e = CudaInference(CudaConfig(dtype=dtype, **kw))
    e.load_weights(L.Provider(cfg, w))
    return e


def tokens(n, vocab=203, seed=1):
    return np.random.default_rng(seed).integers(0, vocab, n).astype(np.uint32)


def decoded(e, toks):
    return np.stack([e.decode_step(int(t)) for t in toks])


MIX = L.config([L.gla(), L.attention(), L.gla(heads=2, dim=36, vdim=20, tau=2.0, rank=9, ff=33), L.attention(chunk=50, kv_from=1, ff=0),
                L.attention(heads=4, kv_heads=4, dim=40, vdim=12, rot_dims=40, chunk=0, factor=None)])

# each mechanism by itself, at sizes that divide nothing, and at sizes that take the wide kernels
ALONE = {
    "attention": L.config([L.attention(ff=0)]),
    "attention_all_positions": L.config([L.attention(ff=0, chunk=0)]),
    "attention_plain_rotation": L.config([L.attention(ff=0, factor=None, base=500.0, rot_dims=24)]),
    "attention_chunks_of_one": L.config([L.attention(ff=0, chunk=1)]),
    "attention_chunks_of_64": L.config([L.attention(ff=0, chunk=64)]),
    "attention_small_chunks": L.config([L.attention(ff=0, chunk=5)]),
    "attention_one_head": L.config([L.attention(heads=1, kv_heads=1, dim=9, vdim=7, rot_dims=2, ff=0)], width=50, vocab=61),
    "attention_all_heads_alone": L.config([L.attention(heads=5, kv_heads=5, dim=16, vdim=33, rot_dims=16, ff=0)]),
    "attention_twelve_heads_a_key": L.config([L.attention(heads=24, kv_heads=2, dim=16, vdim=24, rot_dims=10, chunk=90, ff=0)]),
    "attention_twenty_heads_a_key": L.config([L.attention(heads=20, kv_heads=1, dim=32, vdim=16, rot_dims=32, chunk=0, ff=0)]),
    "attention_wide": L.config([L.attention(heads=8, kv_heads=2, dim=128, vdim=128, rot_dims=64, chunk=100, ff=0)], width=136, vocab=90),
    "attention_widest": L.config([L.attention(heads=18, kv_heads=1, dim=256, vdim=256, rot_dims=128, chunk=70, ff=0)], width=64, vocab=90),
    "attention_large_keys": L.config([L.attention(heads=2, kv_heads=1, dim=520, vdim=40, rot_dims=100, chunk=70, ff=0)], width=64, vocab=90),
    "attention_large_values": L.config([L.attention(heads=2, kv_heads=2, dim=40, vdim=264, rot_dims=40, chunk=70, ff=0)], width=64, vocab=90),
    "attention_feedforward": L.config([L.attention()]),
    "shared_keys": L.config([L.attention(ff=0, chunk=20), L.attention(ff=0, chunk=45, kv_from=0, scale=0.4), L.attention(ff=0), L.attention(ff=0, chunk=0, kv_from=0)]),
    "gla": L.config([L.gla()]),
    "gla_long_memory": L.config([L.gla(tau=32.0, bias=(2.0, 8.0))]),
    "gla_short_memory": L.config([L.gla(tau=0.5, bias=(-9.0, 2.0))]),
    "gla_tau_one": L.config([L.gla(tau=1.0)]),
    "gla_one_head": L.config([L.gla(heads=1, dim=5, vdim=3, rank=1)], width=50, vocab=61),
    "gla_wide": L.config([L.gla(heads=2, dim=128, vdim=128, rank=16)], width=96, vocab=90),
    "gla_widest": L.config([L.gla(heads=1, dim=256, vdim=256, rank=24)], width=64, vocab=90),
    "gla_large_gate": L.config([L.gla(heads=2, dim=72, vdim=40, rank=131)], width=96, vocab=90),
    "gla_large_keys": L.config([L.gla(heads=1, dim=300, vdim=24)], width=96, vocab=90),
    "gla_large_values": L.config([L.gla(heads=2, dim=24, vdim=530)], width=64, vocab=90),
    "gla_feedforward": L.config([L.gla(ff=129)]),
    "small_embedding": L.config([L.attention(), L.gla()], scale=0.02),
    "large_embedding": L.config([L.attention(), L.gla()], scale=11.0),
    "large_eps": L.config([L.attention(), L.gla(ff=24)], eps=0.5),
    "odd_width": L.config([L.attention(ff=31), L.gla(heads=1, dim=7, vdim=11, ff=3)], width=37, vocab=45),
    "mix": MIX,
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism(name, dtype):
    """A prompt of 150 tokens (the prompt kernels), of 40 and of 13 (the short-portion ones), then decoding."""
    cfg = ALONE[name]
    w = L.weights(cfg, 11)
    toks = tokens(162, cfg["vocab"])
    want = OracleLuvatar(cfg, w).forward(toks)
    e = engine(cfg, w, dtype, max_seq_len=200)
    for n in (150, 40, 13):
        e.reset()
        got = e.prefill_all_logits(toks[:n])
        for rows, ref in ((got, want[:n]), (decoded(e, toks[n:n + 12]), want[n:n + 12])):
            assert L.close(rows, ref, dtype) if name == "mix" else L.error(rows, ref) < L.TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_every_size(dtype):
    w = L.weights(MIX, 12)
    toks = tokens(300)
    want = OracleLuvatar(MIX, w).forward(toks)
    e = engine(MIX, w, dtype, max_seq_len=320, max_batch=2)
    for sizes in ([300], [2] * 20 + [3] * 20 + [200], [1] * 30 + [15, 16, 17, 63, 64, 65, 30], [128, 129, 43], [7, 256, 2, 2, 33], [9, 10, 11, 12, 13, 14, 31, 37, 50, 113]):
        sid = e.open_sequence()
        at, rows = 0, []
        for n in sizes:
            rows.append(e.extend_sequence(sid, toks[at:at + n], range(n)))
            at += n
        assert e.sequence_position(sid) == 300
        assert L.close(np.concatenate(rows), want, dtype)
        e.remove_sequence(sid)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_in_internal_chunks(dtype):
    """The engine's own portion size must not show; only some places are asked for."""
    w = L.weights(MIX, 13)
    toks = tokens(700)
    want = OracleLuvatar(MIX, w).forward(toks)
    places = [0, 1, 63, 64, 65, 127, 128, 299, 300, 301, 511, 512, 699]
    for portion in (None, 300, 70, 5):
        e = engine(MIX, w, dtype, max_seq_len=700, prefill_chunk_size=portion)
        sid = e.open_sequence()
        assert L.close(e.extend_sequence(sid, toks, places), want[places], dtype)
        e.reset()
        assert L.close(e.prefill(toks)[None], want[-1:], dtype)
        e.close()


def content_scores(cfg, w, h):
    """Scores of head 0 of layer 0 between every two tokens of the vocabulary, rotation left out."""
    mx = cfg["layers"][0]["mixer"]
    d = mx["dim"]
    q = O.rms(h @ w["l0.mix.q"][:d].T.astype(np.float64), w["l0.mix.q.norm"], 3e-6)
    k = O.rms(h @ w["l0.mix.k"][:d].T.astype(np.float64), w["l0.mix.k.norm"], 3e-6)
    return q @ k.T * mx["scale"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("wide", [False, True])
def test_a_far_key_and_the_edges_of_a_chunk(monkeypatch, dtype, wide):
    """One key fits the last query far better than all others.  Just inside the query's chunk and at the borders of tiles and
    shares it must show, just outside it must not; in a prompt, after a portion and in decoding."""
    chunk = 700 if wide else 96
    layer = L.attention(heads=2, kv_heads=1, dim=128, vdim=96, rot_dims=4, chunk=chunk, ff=0) if wide else \
        L.attention(heads=2, kv_heads=2, dim=40, vdim=16, rot_dims=4, chunk=chunk, ff=0)
    cfg = L.config([layer], width=120, vocab=256)
    w = L.weights(cfg, 14, sharp=2.5)
    score = content_scores(cfg, w, w["embed"].astype(np.float64) * 0.4)
    asks, needle = np.unravel_index(np.argmax(score), score.shape)
    dull = np.argsort(score[asks])[:40]
    e = engine(cfg, w, dtype, max_seq_len=1500, max_batch=2)
    rng = np.random.default_rng(15)
    begin = 2 * chunk
    seen = hidden = 0
    for n in (begin + 90, begin + 65, begin + 1, begin + 2):
        for at in {begin - 1, begin, begin + 1, begin + 15, begin + 16, begin + 31, begin + 32, begin + 63, begin + 64, n - 2}:
            if not 0 <= at < n - 1:
                continue
            toks = rng.choice(dull, n).astype(np.uint32)
            toks[-1] = asks
            without = OracleLuvatar(cfg, w).forward(toks)[-1:]
            toks[at] = needle
            want = OracleLuvatar(cfg, w).forward(toks)[-1:]
            if at >= begin:
                assert L.error(without, want) > 4 * L.TOL[dtype]
                seen += 1
            else:
                monkeypatch.setattr(O, "chunk_start", lambda p, s: max(0, p // s * s - 1))
                assert L.error(OracleLuvatar(cfg, w).forward(toks)[-1:], want) > 4 * L.TOL[dtype]
                monkeypatch.undo()
                hidden += 1
            e.reset()
            assert L.error(e.prefill(toks)[None], want) < L.TOL[dtype]
            e.reset()
            e.prefill(toks[:-1])
            assert L.error(e.decode_step(int(toks[-1]))[None], want) < L.TOL[dtype]
            e.reset()
            sid = e.open_sequence()
            cut = min(begin - 1, n - 2)
            e.extend_sequence(sid, toks[:cut], [])
            assert L.error(e.extend_sequence(sid, toks[cut:], [n - cut - 1]), want) < L.TOL[dtype]
    assert seen > 12 and hidden >= 4


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_in_the_chunk_of_the_sharing_layer_only(dtype):
    """Layer 1 reads layer 0's keys through a longer chunk of its own."""
    cfg = L.config([L.attention(heads=2, kv_heads=1, dim=40, vdim=16, rot_dims=4, chunk=30, ff=0),
                    L.attention(heads=2, kv_heads=1, dim=40, vdim=16, rot_dims=4, chunk=150, kv_from=0, ff=0)], width=120)
    w = L.weights(cfg, 16, sharp=2.0)
    toks = tokens(290, seed=3)
    want = OracleLuvatar(cfg, w).forward(toks)
    narrow = json.loads(json.dumps(cfg))
    narrow["layers"][1]["mixer"]["mask"]["size"] = 30
    assert L.error(OracleLuvatar(narrow, w).forward(toks), want) > 4 * L.TOL[dtype]
    e = engine(cfg, w, dtype, max_seq_len=300)
    assert L.error(e.prefill_all_logits(toks[:200]), want[:200]) < L.TOL[dtype]
    assert L.error(decoded(e, toks[200:]), want[200:]) < L.TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_state_that_lasts(dtype):
    """Decays close to one: what the first tokens left is in the output 900 tokens on, whatever the cut."""
    cfg = L.config([L.gla(heads=2, dim=36, vdim=40, tau=64.0, bias=(5.0, 9.0)), L.gla(heads=1, dim=72, vdim=20, tau=64.0, bias=(3.0, 9.0), ff=24)])
    w = L.weights(cfg, 30)
    toks = tokens(920)
    want = OracleLuvatar(cfg, w).forward(toks)
    other = toks.copy()
    other[:40] = (other[:40] + 50) % 203
    assert L.error(OracleLuvatar(cfg, w).forward(other)[900:], want[900:]) > 4 * L.TOL[dtype]
    e = engine(cfg, w, dtype, max_seq_len=920)
    for first in (0, 2, 37, 300):
        e.reset()
        if first:
            e.prefill(toks[:first])
        assert L.error(e.prefill(toks[first:900])[None], want[899:900]) < L.TOL[dtype]
        assert L.error(decoded(e, toks[900:]), want[900:]) < L.TOL[dtype]


def test_prompt_chunks_keep_32_bit():
    """bf16: the state after a prompt in chunks against the state after the same tokens one by one.  What the two round
    differently is only the recurrence, so the next logits agree far better than either agrees with the plain model."""
    cfg = L.config([L.gla(heads=2, dim=64, vdim=64, tau=16.0, bias=(0.0, 6.0))], width=128)
    w = L.weights(cfg, 31)
    toks = tokens(400)
    e = engine(cfg, w, "bfloat16", max_seq_len=512)
    a = e.prefill_all_logits(toks)[-100:]
    e.reset()
    b = np.concatenate([e.prefill_all_logits(toks[i:i + 12]) for i in range(0, 400, 12)])[-100:]
    assert L.error(a, b.astype(np.float64)) < 4e-3


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(dtype):
    """Sequences of one token and a few, in one portion and one by one."""
    w = L.weights(MIX, 16)
    toks = tokens(6)
    want = OracleLuvatar(MIX, w).forward(toks)
    e = engine(MIX, w, dtype, max_seq_len=64)
    for n in range(1, 7):
        e.reset()
        assert L.close(e.prefill(toks[:n])[None], want[n - 1:n], dtype)
    e.reset()
    assert L.close(decoded(e, toks), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nseq", [3, 11, 18])
def test_unequal_requests_in_a_batch(dtype, nseq):
    """Sequences of different lengths decode together (matvec and GEMM batch sizes), some leave, others take their slots."""
    w = L.weights(MIX, 17)
    rng = np.random.default_rng(18)
    lens = [int(n) for n in rng.integers(1, 90, nseq)]
    toks = [tokens(n + 8, seed=100 + i) for i, n in enumerate(lens)]
    want = [OracleLuvatar(MIX, w).forward(t) for t in toks]
    e = engine(MIX, w, dtype, max_seq_len=128, max_batch=nseq)
    ids = [e.add_sequence(t[:n]) for t, n in zip(toks, lens)]
    for k in range(4):
        for sid, lg in e.batch_decode_step({s: int(t[n + k]) for s, t, n in zip(ids, toks, lens)}):
            i = ids.index(sid)
            assert L.close(lg[None], want[i][lens[i] + k:lens[i] + k + 1], dtype)
    # one leaves, its slot goes to a new sequence; the rest decode on, in another order
    fresh = tokens(37, seed=999)
    fresh_want = OracleLuvatar(MIX, w).forward(fresh)
    e.remove_sequence(ids[0])
    sid = e.open_sequence()
    assert sid == ids[0]
    assert L.close(e.extend_sequence(sid, fresh[:30], [29]), fresh_want[29:30], dtype)
    for k in range(4):
        feed = {sid: int(fresh[30 + k])}
        feed.update({ids[i]: int(toks[i][lens[i] + 4 + k]) for i in range(nseq - 1, 0, -1)})
        for s, lg in e.batch_decode_step(feed):
            ref = fresh_want[30 + k] if s == sid else want[ids.index(s)][lens[ids.index(s)] + 4 + k]
            assert L.close(lg[None], ref[None], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_slot_used_again_remembers_nothing(dtype):
    w = L.weights(MIX, 19)
    a, b = tokens(120, seed=1), tokens(50, seed=2)
    want = OracleLuvatar(MIX, w).forward(b)
    e = engine(MIX, w, dtype, max_seq_len=128)
    for _ in range(2):
        sid = e.add_sequence(a)
        e.batch_decode_step({sid: 5})
        e.remove_sequence(sid)
        sid = e.open_sequence()
        rows = [e.extend_sequence(sid, [int(t)], [0]) for t in b[:3]] + [e.extend_sequence(sid, b[3:], range(47))]
        assert L.close(np.concatenate(rows), want, dtype)
        e.remove_sequence(sid)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    w = L.weights(MIX, 20)
    toks = tokens(420)
    want = OracleLuvatar(MIX, w).forward(toks)
    e = engine(MIX, w, dtype, max_seq_len=420)
    e.prefill(toks[:5])
    assert L.close(decoded(e, toks[5:]), want[5:], dtype)


@pytest.mark.parametrize("kv_heads", [1, 4])
def test_many_shares_of_a_long_context(kv_heads):
    """bf16 decoding far into a sequence: the positions are shared out over many CTAs; one and several sequences."""
    cfg = L.config([L.attention(heads=4, kv_heads=kv_heads, dim=64, vdim=64, rot_dims=64, base=2e5, chunk=2500, ff=0)], width=64, vocab=90)
    w = L.weights(cfg, 33)
    toks = tokens(2110, 90)
    want = OracleLuvatar(cfg, w).forward(toks)
    e = engine(cfg, w, "bfloat16", max_seq_len=2600, max_batch=3)
    ids = [e.add_sequence(toks[:2100]), e.add_sequence(toks[:70]), e.add_sequence(toks[:1])]
    at = [2100, 70, 1]
    for _ in range(8):
        for s, lg in e.batch_decode_step({i: int(toks[a]) for i, a in zip(ids, at)}):
            assert L.error(lg[None], want[at[ids.index(s)]][None]) < L.TOL["bfloat16"]
        at = [a + 1 for a in at]
    assert L.error(e.extend_sequence(ids[0], toks[2108:2110], [0, 1]), want[2108:2110]) < L.TOL["bfloat16"]


def test_greedy_generation():
    """Tokens picked on the device, step after step, are the plain model's; sequences of a batch and of the scheduler agree."""
    w = L.weights(MIX, 21)
    prompt = tokens(40)
    m = OracleLuvatar(MIX, w)
    picks, lg = [], m.forward(prompt)[-1]
    for _ in range(30):
        two = np.sort(lg)[-2:]
        assert two[1] - two[0] > 1e-3, "the test's tokens must not be ties"
        picks.append(int(np.argmax(lg)))
        lg = m.forward([picks[-1]])[-1]
    e = engine(MIX, w, "float32", max_seq_len=128, max_batch=3)
    first = int(np.argmax(e.prefill(prompt)))
    got, ms = e.decode_greedy([first], 29)
    assert [first] + got[:, 0].tolist() == picks and ms > 0
    e.reset()
    ids = [e.add_sequence(prompt), e.add_sequence(prompt[:20]), e.add_sequence(prompt)]
    seen = {i: [e._next[i]] for i in ids}
    for _ in range(10):
        for sid, logits in e.batch_decode_step():
            seen[sid].append(int(np.argmax(logits)))
    assert seen[ids[0]] == seen[ids[2]] == picks[:11]
    e.reset()
    rows = e.generate([prompt, prompt[:20]], 12)
    assert rows[0] == picks[:12] and rows[1][:11] == seen[ids[1]]


def test_command_line_generation(tmp_path):
    """The same continuation from a checkpoint folder and from a bundle written from it."""
    from ironmill_b200.bundle import write_gpu_bundle
    w = L.weights(MIX, 21)
    prompt = tokens(40)
    e = engine(MIX, w, "float32", max_seq_len=128)
    want = e.generate([prompt], 8)[0]
    L.write_checkpoint(tmp_path / "model", MIX, w)
    p = L.Provider(MIX, w)
    write_gpu_bundle(str(tmp_path / "bundle"), p.config(), {n: p.tensor(n) for n in p.tensor_names()})
    for folder in ("model", "bundle"):
        r = subprocess.run([sys.executable, "-m", "ironmill_b200", "generate", "--model", str(tmp_path / folder), "--dtype", "float32", "--max-new-tokens", "8",
                            "--tokens", ",".join(map(str, prompt))], capture_output=True, text=True, timeout=200, cwd=ROOT)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [int(t) for t in r.stdout.split(",")] == want


def test_repeated_steps_are_bit_identical():
    w = L.weights(MIX, 22)
    toks = tokens(90)
    e = engine(MIX, w, "bfloat16", max_seq_len=128)
    runs = []
    for _ in range(2):
        e.reset()
        runs.append(np.concatenate([e.prefill_all_logits(toks[:70]), decoded(e, toks[70:])]))
    assert (runs[0] == runs[1]).all()


def test_profiling_and_hidden_state_leave_the_sequence_alone():
    w = L.weights(MIX, 23)
    toks = tokens(30)
    want = OracleLuvatar(MIX, w).forward(toks)
    e = engine(MIX, w, "float32", max_seq_len=64)
    e.prefill(toks[:20])
    assert L.close((e.last_hidden_state() @ w["embed"].T.astype(np.float64))[None], want[19:20], "float32")
    assert e.profile_step()["attention"] > 0
    lg = decoded(e, toks[20:])
    assert L.close(lg, want[20:], "float32")
    assert L.close((e.last_hidden_state() @ w["embed"].T.astype(np.float64))[None], want[-1:], "float32")
    assert e.step_launches() > 0 and e.step_bytes(30) > 0


def test_positions_and_going_back():
    from ironmill_b200.engine import InferenceError
    w = L.weights(MIX, 24)
    e = engine(MIX, w, "bfloat16", max_seq_len=32, max_batch=2)
    e.prefill(tokens(20))
    with pytest.raises(InferenceError, match="recurrent state"):
        e.truncate_to(10)
    with pytest.raises(InferenceError, match="max_seq_len"):
        e.prefill(tokens(13))
    # only attention layers: an earlier position is still there
    cfg = L.config([L.attention(), L.attention(kv_from=0, chunk=0)])
    w = L.weights(cfg, 25)
    toks = tokens(40)
    want = OracleLuvatar(cfg, w).forward(toks)
    e = engine(cfg, w, "float32", max_seq_len=64)
    e.prefill(np.concatenate([toks[:30], tokens(9, seed=7)]))
    e.truncate_to(30)
    assert L.close(decoded(e, toks[30:]), want[30:], "float32")


def test_loading_is_checked():
    from ironmill_b200.engine import InferenceError
    cfg = L.config([L.attention(), L.gla()])
    w = L.weights(cfg, 26)
    with pytest.raises(InferenceError, match="gate of rank"):
        engine(cfg, {k: v for k, v in w.items() if k != "l1.mix.a1"}, "bfloat16", max_seq_len=16)
    for name in ("l1.mix.norm", "l1.mix.a2", "l0.mix.k.norm", "l0.norm2", "final.norm"):
        with pytest.raises(InferenceError, match=name):
            engine(cfg, {k: v for k, v in w.items() if k != name}, "bfloat16", max_seq_len=16)
    for name in ("l0.mix.k", "l0.mix.q.norm", "l1.mix.a2", "l1.mix.a2.b"):
        with pytest.raises(InferenceError, match=name.replace(".", r"\.") + ": expected shape"):
            engine(cfg, dict(w, **{name: w[name][:-1]}), "bfloat16", max_seq_len=16)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(tmp_path, dtype):
    """bin/trace_run on a checkpoint folder: requests in portions, several alive at once, slots given back."""
    w = L.weights(MIX, 27)
    L.write_checkpoint(tmp_path / "model", MIX, w)
    (tmp_path / "out").mkdir()
    reqs = {k: tokens(n, seed=50 + i) for i, (k, n) in enumerate((("a", 100), ("b", 45), ("c", 70), ("d", 3)))}
    plan = [[("a", 60)], [("b", 2), ("a", 2)], [("a", 1)], [("b", 43)], [("c", 70)], [("a", 37), ("d", 3)]]
    at, lines, rows = dict.fromkeys(reqs, 0), [], []
    for n, step in enumerate(plan):
        entries, end, r = [], [], []
        for k, c in step:
            want = sorted({0, c - 1}) if n != 1 else []
            entries.append({"id": k, "tokens": reqs[k][at[k]:at[k] + c].tolist(), "want": want})
            r += [(k, at[k] + p) for p in want]
            at[k] += c
            if at[k] == len(reqs[k]):
                end.append(k)
        lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
        rows.append(r)
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(tmp_path / "out"),
                        "--max-tokens", "200", "--max-requests", "2"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=200)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {n}" for n in range(len(plan))]
    want = {k: OracleLuvatar(MIX, w).forward(t) for k, t in reqs.items()}
    for n, r in enumerate(rows):
        f = tmp_path / "out" / f"{n}.f32"
        assert f.exists() == bool(r)
        if r:
            got = np.fromfile(f, dtype="<f4").reshape(len(r), -1)
            assert L.close(got, np.stack([want[k][p] for k, p in r]), dtype)
