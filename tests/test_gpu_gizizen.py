"""Gizizen on the GPU against the tests' plain model: every mechanism alone and together, in bf16 and f32, in prompts, in
portions, token by token, in batches and slots, through the engine's own entry points."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from tests import gizizen_models as G
from tests.oracle_gizizen import OracleGizizen

pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ("float32", "bfloat16")


def engine(cfg, w, dtype, **kw):
    from ironmill_b200.engine import CudaConfig, CudaInference
    e = CudaInference(CudaConfig(dtype=dtype, **kw))
    e.load_weights(G.Provider(cfg, w))
    return e


def tokens(n, vocab, seed=1):
    return np.random.default_rng(seed).integers(0, vocab, n).astype(np.uint32)


def decoded(e, toks):
    return np.stack([e.decode_step(int(t)) for t in toks])


MIX = G.config([G.latent(), G.lightning(), G.latent(heads=2, dim=16, rot_dim=8, vdim=36, kv_rank=33, ff=0), G.lightning(heads=2, dim=36, vdim=20, ff=0)],
               loop=(0, 2, 2))

# each mechanism by itself, at sizes that divide nothing, and at sizes that take the wide kernels
ALONE = {
    "latent": G.config([G.latent(ff=0)]),
    "latent_plain_rotation": G.config([G.latent(ff=0, scaling=None, base=500.0)]),
    "latent_one_head": G.config([G.latent(heads=1, dim=8, rot_dim=2, vdim=9, kv_rank=7, ff=0)], width=50, vocab=61),
    "latent_wide": G.config([G.latent(heads=5, dim=128, rot_dim=64, vdim=128, kv_rank=512, ff=0)], width=136, vocab=90),
    "latent_many_heads": G.config([G.latent(heads=36, dim=32, rot_dim=16, vdim=40, kv_rank=200, ff=0)], width=96, vocab=90),
    "latent_large_values": G.config([G.latent(heads=2, dim=40, rot_dim=20, vdim=264, kv_rank=600, ff=0)], width=64, vocab=90),
    "latent_feedforward": G.config([G.latent()]),
    "linear": G.config([G.lightning(ff=0)]),
    "linear_edge_decays": G.config([G.lightning(decay=(0.0, 1.0, 0.05), ff=0)]),
    "linear_wide": G.config([G.lightning(heads=2, dim=128, vdim=160, decay=(0.9, 0.9995), ff=0)], width=96, vocab=90),
    "linear_large_keys": G.config([G.lightning(heads=1, dim=300, vdim=24, decay=(0.97,), ff=0)], width=96, vocab=90),
    "linear_keys_200": G.config([G.lightning(heads=3, dim=200, vdim=40, ff=0)], width=96, vocab=90),
    "linear_feedforward": G.config([G.lightning(ff=129)]),
    "loop_once": G.config([G.latent(ff=0), G.lightning(ff=0)], loop=(1, 2, 1)),
    "loop_all_layers": G.config([G.latent(), G.lightning()], loop=(0, 2, 3)),
    "no_cap": G.config([G.latent()], cap=None),
    "tight_cap": G.config([G.latent()], cap=0.8),
    "large_eps": G.config([G.latent(), G.lightning()], eps=0.5),
    "odd_width": G.config([G.latent(ff=31), G.lightning(heads=1, dim=5, vdim=11, decay=(0.7,), ff=3)], width=37, vocab=45, loop=(0, 2, 2)),
    "mix": MIX,
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism(name, dtype):
    """A prompt of 150 tokens (the wide kernels) and of 40 (the short-chunk ones), then decoding."""
    cfg = ALONE[name]
    w = G.weights(cfg, 11)
    toks = tokens(162, cfg["vocab"])
    want = OracleGizizen(cfg, w).forward(toks)
    e = engine(cfg, w, dtype, max_seq_len=200)
    for n in (150, 40):
        e.reset()
        got = e.prefill_all_logits(toks[:n])
        assert G.error(got, want[:n]) < G.TOL[dtype]
        assert G.error(decoded(e, toks[n:n + 12]), want[n:n + 12]) < G.TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_every_size(dtype):
    w = G.weights(MIX, 12)
    toks = tokens(300, 203)
    want = OracleGizizen(MIX, w).forward(toks)
    e = engine(MIX, w, dtype, max_seq_len=320, max_batch=2)
    for sizes in ([300], [2] * 20 + [3] * 20 + [200], [1] * 30 + [15, 16, 17, 63, 64, 65, 30], [128, 129, 43], [7, 256, 2, 2, 33]):
        sid = e.open_sequence()
        at, rows = 0, []
        for n in sizes:
            rows.append(e.extend_sequence(sid, toks[at:at + n], range(n)))
            at += n
        assert e.sequence_position(sid) == 300
        assert G.error(np.concatenate(rows), want) < G.TOL[dtype]
        e.remove_sequence(sid)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_in_internal_chunks(dtype):
    """The engine's own chunk size must not show; only some places are asked for."""
    w = G.weights(MIX, 13)
    toks = tokens(700, 203)
    want = OracleGizizen(MIX, w).forward(toks)
    places = [0, 1, 63, 64, 65, 127, 128, 299, 300, 301, 511, 512, 699]
    for chunk in (None, 300, 70, 5):
        e = engine(MIX, w, dtype, max_seq_len=700, prefill_chunk_size=chunk)
        sid = e.open_sequence()
        assert G.error(e.extend_sequence(sid, toks, places), want[places]) < G.TOL[dtype]
        e.reset()
        assert G.error(e.prefill(toks)[None], want[-1:]) < G.TOL[dtype]
        e.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("wide", [False, True])
def test_a_far_key_at_every_border(dtype, wide):
    """One key that fits the last query far better than all others, at tile and split borders: the logits must show it,
    in a prompt and in decoding, with the cache long enough for many splits."""
    layer = G.latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=448, ff=0) if wide else G.latent(heads=2, dim=40, rot_dim=8, vdim=16, kv_rank=48, ff=0)
    cfg = G.config([layer], width=120, vocab=256)
    w = G.weights(cfg, 14, sharp=2.0)
    from tests import oracle_gizizen as O
    mx = layer["mixer"]
    h = O.rms(O.rms(w["embed"].astype(np.float64), w["embed.norm"], 3e-6), w["l0.norm1"], 3e-6)
    d, r = mx["dim"], mx["rot_dim"]
    q = (h @ w["l0.mix.q"].T.astype(np.float64)).reshape(-1, 2, d + r)[:, 0, :d]
    lat = O.rms(h @ w["l0.mix.dkv"][:mx["kv_rank"]].T.astype(np.float64), w["l0.mix.dkv.norm"], 3e-6)
    score = q @ (lat @ w["l0.mix.uk"][:d].T.astype(np.float64)).T * mx["scale"]
    asks, needle = np.unravel_index(np.argmax(score), score.shape)
    dull = np.argsort(score[asks])[:40]
    e = engine(cfg, w, dtype, max_seq_len=4096)  # more splits than one group of threads adds up
    rng = np.random.default_rng(15)
    for n, at in ((200, 0), (200, 63), (200, 64), (200, 65), (200, 127), (200, 128), (200, 198), (517, 0), (517, 191), (517, 511), (517, 512), (70, 3)):
        toks = rng.choice(dull, n).astype(np.uint32)
        toks[-1] = asks
        without = OracleGizizen(cfg, w).forward(toks)[-1:]
        toks[at] = needle
        want = OracleGizizen(cfg, w).forward(toks)[-1:]
        assert G.error(without, want) > 4 * G.TOL[dtype]
        e.reset()
        assert G.error(e.prefill(toks)[None], want) < G.TOL[dtype]
        e.reset()
        e.prefill(toks[:-1])
        assert G.error(e.decode_step(int(toks[-1]))[None], want) < G.TOL[dtype]


def test_prompts_long_enough_for_parallel_segments():
    """bf16: a 900-token prompt's recurrence runs in segments; cut elsewhere it does not; then decoding from the state."""
    cfg = G.config([G.lightning(heads=2, dim=36, vdim=40, decay=(0.995, 0.9999)), G.lightning(heads=1, dim=72, vdim=20, decay=(0.98,), ff=0)])
    w = G.weights(cfg, 30)
    toks = tokens(920, 203)
    want = OracleGizizen(cfg, w).forward(toks)
    e = engine(cfg, w, "bfloat16", max_seq_len=920)
    for first in (0, 37, 300):
        e.reset()
        if first:
            e.prefill(toks[:first])
        assert G.error(e.prefill(toks[first:900])[None], want[899:900]) < G.TOL["bfloat16"]
        assert G.error(decoded(e, toks[900:]), want[900:]) < G.TOL["bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(dtype):
    """Sequences of one token and a few, in one portion and one by one."""
    w = G.weights(MIX, 16)
    toks = tokens(6, 203)
    want = OracleGizizen(MIX, w).forward(toks)
    e = engine(MIX, w, dtype, max_seq_len=64)
    for n in range(1, 7):
        e.reset()
        assert G.error(e.prefill(toks[:n])[None], want[n - 1:n]) < G.TOL[dtype]
    e.reset()
    assert G.error(decoded(e, toks), want) < G.TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nseq", [3, 7, 18])
def test_unequal_requests_in_a_batch(dtype, nseq):
    """Sequences of different lengths decode together (matvec and GEMM batch sizes), some leave, others take their slots."""
    w = G.weights(MIX, 17)
    rng = np.random.default_rng(18)
    lens = [int(n) for n in rng.integers(1, 90, nseq)]
    toks = [tokens(n + 8, 203, 100 + i) for i, n in enumerate(lens)]
    want = [OracleGizizen(MIX, w).forward(t) for t in toks]
    e = engine(MIX, w, dtype, max_seq_len=128, max_batch=nseq)
    ids = [e.add_sequence(t[:n]) for t, n in zip(toks, lens)]
    for k in range(4):
        for sid, lg in e.batch_decode_step({s: int(t[n + k]) for s, t, n in zip(ids, toks, lens)}):
            i = ids.index(sid)
            assert G.error(lg[None], want[i][lens[i] + k:lens[i] + k + 1]) < G.TOL[dtype]
    # every other one leaves, its slot goes to a new sequence; the rest decode on, in another order
    fresh = tokens(37, 203, 999)
    fresh_want = OracleGizizen(MIX, w).forward(fresh)
    e.remove_sequence(ids[0])
    sid = e.open_sequence()
    assert sid == ids[0]
    assert G.error(e.extend_sequence(sid, fresh[:30], [29]), fresh_want[29:30]) < G.TOL[dtype]
    for k in range(4):
        feed = {sid: int(fresh[30 + k])}
        feed.update({ids[i]: int(toks[i][lens[i] + 4 + k]) for i in range(nseq - 1, 0, -1)})
        for s, lg in e.batch_decode_step(feed):
            ref = fresh_want[30 + k] if s == sid else want[ids.index(s)][lens[ids.index(s)] + 4 + k]
            assert G.error(lg[None], ref[None]) < G.TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_slot_used_again_remembers_nothing(dtype):
    w = G.weights(MIX, 19)
    a, b = tokens(120, 203, 1), tokens(50, 203, 2)
    want = OracleGizizen(MIX, w).forward(b)
    e = engine(MIX, w, dtype, max_seq_len=128)
    for _ in range(2):
        sid = e.add_sequence(a)
        e.batch_decode_step({sid: 5})
        e.remove_sequence(sid)
        sid = e.open_sequence()
        rows = [e.extend_sequence(sid, [int(t)], [0]) for t in b[:3]] + [e.extend_sequence(sid, b[3:], range(47))]
        assert G.error(np.concatenate(rows), want) < G.TOL[dtype]
        e.remove_sequence(sid)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    w = G.weights(MIX, 20)
    toks = tokens(420, 203)
    want = OracleGizizen(MIX, w).forward(toks)
    e = engine(MIX, w, dtype, max_seq_len=420)
    e.prefill(toks[:5])
    assert G.error(decoded(e, toks[5:]), want[5:]) < G.TOL[dtype]


def test_greedy_generation():
    """Tokens picked on the device, step after step, are the plain model's; sequences of a batch and of the scheduler agree."""
    w = G.weights(MIX, 21)
    prompt = tokens(40, 203)
    m = OracleGizizen(MIX, w)
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
    assert seen[ids[0]] == seen[ids[2]] == picks[:11] and seen[ids[1]] != picks[:11]
    e.reset()
    rows = e.generate([prompt, prompt[:20]], 12)
    assert rows[0] == picks[:12] and rows[1] == seen[ids[1]] + rows[1][11:]


def test_command_line_generation(tmp_path):
    """The same continuation from a checkpoint folder and from a bundle written from it."""
    from ironmill_b200.bundle import write_gpu_bundle
    w = G.weights(MIX, 21)
    prompt = tokens(40, 203)
    e = engine(MIX, w, "float32", max_seq_len=128)
    want = e.generate([prompt], 8)[0]
    G.write_checkpoint(tmp_path / "model", MIX, w)
    p = G.Provider(MIX, w)
    write_gpu_bundle(str(tmp_path / "bundle"), p.config(), {n: p.tensor(n) for n in p.tensor_names()})
    for folder in ("model", "bundle"):
        r = subprocess.run([sys.executable, "-m", "ironmill_b200", "generate", "--model", str(tmp_path / folder), "--dtype", "float32", "--max-new-tokens", "8",
                            "--tokens", ",".join(map(str, prompt))], capture_output=True, text=True, timeout=200, cwd=ROOT)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [int(t) for t in r.stdout.split(",")] == want


def test_repeated_steps_are_bit_identical():
    w = G.weights(MIX, 22)
    toks = tokens(90, 203)
    e = engine(MIX, w, "bfloat16", max_seq_len=128)
    runs = []
    for _ in range(2):
        e.reset()
        runs.append(np.concatenate([e.prefill_all_logits(toks[:70]), decoded(e, toks[70:])]))
    assert (runs[0] == runs[1]).all()


def test_profiling_and_hidden_state_leave_the_sequence_alone():
    w = G.weights(MIX, 23)
    toks = tokens(30, 203)
    m = OracleGizizen(MIX, w)
    want = m.forward(toks)
    e = engine(MIX, w, "float32", max_seq_len=64)
    e.prefill(toks[:20])
    assert e.profile_step()["attention"] > 0
    lg = np.stack([e.decode_step(int(t)) for t in toks[20:]])
    assert G.error(lg, want[20:]) < G.TOL["float32"]
    z = e.last_hidden_state() @ w["head"].T.astype(np.float64)
    assert G.error(7.0 * np.tanh(z / 7.0)[None], want[-1:]) < G.TOL["float32"]
    assert e.step_launches() > 0 and e.step_bytes(30) > 0


def test_positions_and_bounds():
    from ironmill_b200.engine import InferenceError
    w = G.weights(MIX, 24)
    e = engine(MIX, w, "bfloat16", max_seq_len=32, max_batch=2)
    e.prefill(tokens(20, 203))
    with pytest.raises(InferenceError, match="recurrent state"):
        e.truncate_to(10)
    e.truncate_to(20)
    with pytest.raises(InferenceError, match="max_seq_len"):
        e.prefill(tokens(13, 203))
    e.truncate_to(0)
    assert e.seq_pos() == 0
    e.reset()
    ids = [e.open_sequence(), e.open_sequence()]
    with pytest.raises(InferenceError, match="slots are in use"):
        e.open_sequence()
    with pytest.raises(InferenceError, match="ascend"):
        e.extend_sequence(ids[0], [1, 2, 3], [2, 1])
    with pytest.raises(InferenceError, match="no sequence"):
        e.extend_sequence(5, [1, 2], [])
    # only latent layers: an earlier position is still there
    cfg = G.config([G.latent(), G.latent(heads=2)])
    w = G.weights(cfg, 25)
    toks = tokens(40, 203)
    want = OracleGizizen(cfg, w).forward(toks)
    e = engine(cfg, w, "float32", max_seq_len=64)
    e.prefill(np.concatenate([toks[:30], tokens(9, 203, 7)]))
    e.truncate_to(30)
    assert G.error(decoded(e, toks[30:]), want[30:]) < G.TOL["float32"]


def test_loading_is_checked():
    from ironmill_b200.engine import InferenceError
    cfg = G.config([G.latent(), G.lightning()], loop=(0, 1, 2))
    w = G.weights(cfg, 26)
    short = {k: v for k, v in w.items() if k != "l1.mix.norm"}
    with pytest.raises(InferenceError, match="l1.mix.norm"):
        engine(cfg, short, "bfloat16", max_seq_len=16)
    bad = dict(w)
    bad["l0.mix.uk"] = w["l0.mix.uk"][:-1]
    with pytest.raises(InferenceError, match="l0.mix.uk: expected shape"):
        engine(cfg, bad, "bfloat16", max_seq_len=16)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(tmp_path, dtype):
    """bin/trace_run on a checkpoint folder: requests in portions, several alive at once, slots given back."""
    w = G.weights(MIX, 27)
    G.write_checkpoint(tmp_path / "model", MIX, w)
    (tmp_path / "out").mkdir()
    reqs = {k: tokens(n, 203, 50 + i) for i, (k, n) in enumerate((("a", 100), ("b", 45), ("c", 70), ("d", 3)))}
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
    want = {k: OracleGizizen(MIX, w).forward(t) for k, t in reqs.items()}
    for n, r in enumerate(rows):
        f = tmp_path / "out" / f"{n}.f32"
        assert f.exists() == bool(r)
        if r:
            got = np.fromfile(f, dtype="<f4").reshape(len(r), -1)
            assert G.error(got, np.stack([want[k][p] for k, p in r])) < G.TOL[dtype]
