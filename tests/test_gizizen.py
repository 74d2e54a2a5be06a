"""Gizizen on the CPU: configuration and checkpoint readers, the registry, and the tests' own plain model (that its
mechanisms matter: a mistake planted in it moves the logits by far more than the tolerances of the GPU tests)."""
import json

import numpy as np
import pytest

from ironmill_b200.architectures import LayerStack, QuantizedBlocks, config_from_json, family_of
from ironmill_b200.bundle import CudaBundleProvider, GpuBundleError, ModelConfig, write_gpu_bundle
from ironmill_b200.checkpoint import CheckpointProvider
from ironmill_b200.stack_config import LatentAttention, LinearAttention, StackConfig
from tests import gizizen_models as G
from tests import oracle_gizizen as O

CFG = G.config([G.latent(), G.lightning(), G.latent(heads=2, ff=0)], loop=(0, 2, 2))


def test_config_reader_takes_every_field():
    c = StackConfig.from_json(CFG)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.logit_softcap) == (203, 88, 3e-6, 7.0)
    assert (c.loop_start, c.loop_stop, c.loop_times) == (0, 2, 2)
    a, b, d = c.layers
    assert isinstance(a.mixer, LatentAttention) and isinstance(b.mixer, LinearAttention) and d.ff == 0 and a.ff == 56
    assert (a.mixer.rot.factor, a.mixer.rot.original, a.mixer.rot.fast, a.mixer.rot.slow) == (5.0, 300.0, 20.0, 1.5)
    assert b.mixer.decay == [0.4, 0.93, 0.998]
    shapes = c.tensors()
    assert shapes["l0.mix.q"] == (3 * 36, 88) and shapes["loop.in"] == (88, 176) and "l2.mlp.up" not in shapes
    plain = G.config([G.latent(scaling=None)], loop=None, cap=None)
    p = StackConfig.from_json(plain)
    assert p.loop_times == 0 and p.logit_softcap == 0.0 and p.layers[0].mixer.rot.factor == 0.0 and "loop.in" not in p.tensors()


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="other"), "unknown type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mixer"]["decay"].pop(), "decays"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "feed-forward"),
    (lambda c: c.update(width="88"), "width"),
])
def test_config_reader_refuses(edit, text):
    c = json.loads(json.dumps(CFG))
    edit(c)
    with pytest.raises(GpuBundleError, match=text):
        StackConfig.from_json(c)


def test_registry_picks_the_family():
    assert family_of(config_from_json(CFG)) is LayerStack
    llama = ModelConfig("llama", 256, 512, 2, 2, 2, 128, 300).to_json()
    assert family_of(config_from_json(llama)) is QuantizedBlocks


def test_checkpoint_and_bundle_round_trip(tmp_path):
    w = G.weights(CFG)
    G.write_checkpoint(tmp_path / "m", CFG, w)
    p = CheckpointProvider(str(tmp_path / "m"))
    assert set(p.tensor_names()) == set(p.config().tensors()) == set(w)
    for n in ("l0.mix.dkv", "l1.mix.norm", "head"):
        t = p.tensor(n)
        assert t.dtype == "bfloat16" and t.shape == w[n].shape and (t.data == G.bf16_bits(w[n])).all()
    write_gpu_bundle(str(tmp_path / "b"), p.config(), {n: p.tensor(n) for n in p.tensor_names()})
    b = CudaBundleProvider(str(tmp_path / "b"))
    assert isinstance(b.config(), StackConfig) and b.config().tensors() == p.config().tensors()
    assert (b.tensor("loop.step").data == G.bf16_bits(w["loop.step"])).all()


def test_checkpoint_reader_refuses_broken_files(tmp_path):
    with pytest.raises(GpuBundleError, match="config.json"):
        CheckpointProvider(str(tmp_path))
    G.write_checkpoint(tmp_path / "m", CFG, G.weights(CFG))
    f = tmp_path / "m" / "model.safetensors"
    f.write_bytes(f.read_bytes()[:-10])
    with pytest.raises(GpuBundleError, match="data range"):
        CheckpointProvider(str(tmp_path / "m"))


def test_plain_model_does_not_depend_on_the_cut():
    w = G.weights(CFG, 3)
    toks = np.random.default_rng(4).integers(0, 203, 90)
    whole = O.OracleGizizen(CFG, w).forward(toks)
    for cut in ([2] * 45, [1, 88, 1], [33, 3, 54]):
        m, at, parts = O.OracleGizizen(CFG, w), 0, []
        for n in cut:
            parts.append(m.forward(toks[at:at + n]))
            at += n
        assert np.abs(np.concatenate(parts) - whole).max() < 1e-9


def test_rotation_keeps_the_relative_angle_and_scales_both_halves():
    rot = {"dims": 8, "base": 1e3, "scaling": dict(G.YARN)}
    f, amp = O.rope_freqs(rot)
    plain, one = O.rope_freqs({"dims": 8, "base": 1e3})
    assert one == 1.0 and amp == pytest.approx(1 + 0.1 * np.log(5.0))
    assert f[0] == pytest.approx(plain[0]) and f[-1] == pytest.approx(plain[-1] / 5.0)   # fast pairs kept, slow ones stretched
    x = np.random.default_rng(0).normal(size=(2, 8))
    dots = [float((O.rotate(x[:1], np.array([p]), rot) * O.rotate(x[1:], np.array([p + 7]), rot)).sum()) for p in (0, 11, 500)]
    assert np.ptp(dots) < 1e-9


# A mistake in one mechanism of the plain model: (patch name, replacement maker).  Each must show above the bf16 tolerance.
def _no_sink(s, sink):
    e = np.exp(s - s.max())
    return e / e.sum()


def _half_split(x, pos, rot):
    f, amp = O.rope_freqs(rot)
    a = pos.reshape((-1,) + (1,) * (x.ndim - 1)) * f
    n = len(f)
    u, v, c, s = x[..., :n], x[..., n:], np.cos(a) * amp, np.sin(a) * amp
    return np.concatenate([u * c - v * s, v * c + u * s], axis=-1)


def _unscaled(rot):
    d = rot["dims"]
    return np.array([rot["base"] ** (-2.0 * i / d) for i in range(d // 2)]), 1.0


@pytest.mark.parametrize("attr, wrong", [("sink_softmax", _no_sink), ("rotate", _half_split), ("rope_freqs", _unscaled), ("gelu_tanh", lambda z: z * O.sigmoid(z) * 0.9)])
def test_a_wrong_mechanism_shows(monkeypatch, attr, wrong):
    w = G.weights(CFG, 5)
    toks = np.random.default_rng(6).integers(0, 203, 120)
    right = O.OracleGizizen(CFG, w).forward(toks)
    monkeypatch.setattr(O, attr, wrong)
    assert G.error(O.OracleGizizen(CFG, w).forward(toks), right) > 2 * G.TOL["bfloat16"]


def test_a_lost_state_or_key_shows():
    """Dropping one early token's latent row, or the recurrent state, in the middle of a sequence."""
    w = G.weights(CFG, 7)
    toks = np.random.default_rng(8).integers(0, 203, 100)
    right = O.OracleGizizen(CFG, w).forward(toks)[60:]
    for what in ("S", "lat"):
        m = O.OracleGizizen(CFG, w)
        m.forward(toks[:60])
        for st in m.states.values():
            if what == "S" and "S" in st:
                st["S"] = st["S"] * 0
            if what == "lat" and "lat" in st:
                st["lat"] = [r * (i != 31) for i, r in enumerate(st["lat"])]
        assert G.error(m.forward(toks[60:]), right) > G.TOL["bfloat16"]


def test_trace_replay_drives_the_sequence_interface(tmp_path):
    """Portions, wanted places in any order, slots given back; the engine is a stand-in that records calls."""
    from ironmill_b200.trace import replay

    class Engine:
        def __init__(self):
            self.live, self.calls = set(), []

        def open_sequence(self):
            i = min(set(range(9)) - self.live)
            self.live.add(i)
            return i

        def extend_sequence(self, sid, tokens, want):
            self.calls.append((sid, list(tokens), list(want)))
            return np.array([[sid, tokens[k], 0.5] for k in want], dtype=np.float32).reshape(len(want), 3)

        def remove_sequence(self, sid):
            self.live.remove(sid)

    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [4, 5, 6], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [7], "want": []}, {"id": "a", "tokens": [8], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "c", "tokens": [9, 1], "want": [1]}], "end": ["b", "c"]}]
    e, said = Engine(), []
    replay(e, [json.dumps(s) + "\n" for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not e.live
    assert e.calls == [(0, [4, 5, 6], [0, 2]), (1, [7], []), (0, [8], []), (0, [9, 1], [1])]
    assert np.fromfile(tmp_path / "0.f32", "<f4").reshape(-1, 3)[:, 1].tolist() == [6, 4]
    assert not (tmp_path / "1.f32").exists() and np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [0, 1, 0.5]
