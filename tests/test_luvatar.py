"""Luvatar on the CPU: configuration and checkpoint readers, the registry, and the tests' own plain model (that its
mechanisms matter: a mistake planted in it moves the logits by far more than the tolerances of the GPU tests)."""
import json

import numpy as np
import pytest

from ironmill_b200.architectures import LayerStack, config_from_json, family_of
from ironmill_b200.bundle import CudaBundleProvider, GpuBundleError, write_gpu_bundle
from ironmill_b200.checkpoint import CheckpointProvider
from ironmill_b200.stack_config import GatedLinearAttention, GroupedAttention, StackConfig
from tests import luvatar_models as L
from tests import oracle_luvatar as O

CFG = L.config([L.gla(), L.attention(), L.attention(chunk=50, kv_from=1, ff=0), L.gla(heads=2, ff=40)])


def test_config_reader_takes_every_field():
    c = StackConfig.from_json(CFG)
    assert (c.vocab_size, c.hidden_size, c.norm_eps, c.embed_scale, c.loop_times, c.logit_softcap) == (203, 88, 3e-6, 0.4, 0, 0.0)
    d = c.design
    assert d.post_norm and d.silu and d.scaled_embedding and d.tied_head
    a, b, s, _ = c.layers
    assert isinstance(a.mixer, GatedLinearAttention) and a.mixer.tau == 8.0 and a.ff == 0
    m = b.mixer
    assert isinstance(m, GroupedAttention) and (m.heads, m.kv_heads, m.dim, m.vdim, m.chunk, m.kv_from) == (6, 2, 24, 20, 37, None)
    assert (m.rot.dims, m.rot.base, m.rot.divide) == (16, 3e4, 3.0) and b.ff == 56
    assert s.mixer.kv_from == 1 and s.mixer.chunk == 50 and s.ff == 0
    assert StackConfig.from_json(L.config([L.attention(chunk=0, factor=None)])).layers[0].mixer.chunk == 0
    assert StackConfig.from_json(L.config([L.attention(chunk=0, factor=None)])).layers[0].mixer.rot.divide == 1.0


def test_sizes_that_only_the_tensors_give():
    w = L.weights(CFG)
    p = L.Provider(CFG, w)
    c = p.config()
    family_of(c).complete(c, p)
    shapes = c.tensors()
    assert c.layers[0].mixer.rank == 5 and shapes["l0.mix.a1"] == (5, 88) and shapes["l0.mix.a2"] == (60, 5)
    assert set(shapes) == set(w) and all(w[n].shape == s for n, s in shapes.items())
    assert "head" not in shapes and "embed.norm" not in shapes and "l2.mix.k" not in shapes and "l1.norm2" in shapes and "l0.norm2" not in shapes


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "share"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "rotation"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "rotation"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "keys and values"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "keys and values"),
    (lambda c: c["layers"][2]["mixer"].update(dim=32), "keys and values"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0), "tau"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c.pop("embedding"), "embedding.scale"),
])
def test_config_reader_refuses(edit, text):
    c = json.loads(json.dumps(CFG))
    edit(c)
    with pytest.raises(GpuBundleError, match=text):
        StackConfig.from_json(c)


def test_registry_and_round_trips(tmp_path):
    assert family_of(config_from_json(CFG)) is LayerStack
    w = L.weights(CFG)
    L.write_checkpoint(tmp_path / "m", CFG, w)
    p = CheckpointProvider(str(tmp_path / "m"))
    write_gpu_bundle(str(tmp_path / "b"), p.config(), {n: p.tensor(n) for n in p.tensor_names()})
    for q in (p, CudaBundleProvider(str(tmp_path / "b"))):
        c = q.config()
        family_of(c).complete(c, q)
        assert c.tensors() == {n: t.shape for n, t in w.items()}
        assert (q.tensor("l1.mix.q.norm").data == L.bf16_bits(w["l1.mix.q.norm"])).all()


def test_plain_model_does_not_depend_on_the_cut():
    w = L.weights(CFG, 3)
    toks = np.random.default_rng(4).integers(0, 203, 90)
    whole = O.OracleLuvatar(CFG, w).forward(toks)
    for cut in ([2] * 45, [1, 88, 1], [33, 3, 54]):
        m, at, parts = O.OracleLuvatar(CFG, w), 0, []
        for n in cut:
            parts.append(m.forward(toks[at:at + n]))
            at += n
        assert np.abs(np.concatenate(parts) - whole).max() < 1e-9


def test_rotation_keeps_the_relative_angle():
    rot = {"dims": 8, "base": 1e3, "scaling": {"factor": 5.0}}
    assert np.allclose(O.rope_freqs(rot) * 5.0, O.rope_freqs({"dims": 8, "base": 1e3}))
    x = np.random.default_rng(0).normal(size=(2, 1, 11))
    y = O.rotate(x, np.array([7, 9]), rot)
    assert (y[..., 8:] == x[..., 8:]).all() and np.allclose((y ** 2).sum(-1), (x ** 2).sum(-1))
    dots = [float((O.rotate(x[:1], np.array([p]), rot) * O.rotate(x[1:], np.array([p + 7]), rot)).sum()) for p in (0, 11, 500)]
    assert np.ptp(dots) < 1e-9


# A mistake in one mechanism of the plain model.  Each must show above the bf16 tolerance.
def _no_sink(s, sink):
    e = np.exp(s - s.max())
    return e / e.sum()


def _half_split(x, pos, rot):
    f, n = O.rope_freqs(rot), rot["dims"] // 2
    a = (pos[:, None] * f)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., 2 * n:]], axis=-1)


_decay, _embed = O.decay, O.embed
MISTAKES = {
    "sink": ("sink_softmax", _no_sink),
    "pairs": ("rotate", _half_split),
    "frequencies": ("rope_freqs", lambda rot: np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])),
    "no rotation": ("rotate", lambda x, pos, rot: x),
    "chunk": ("chunk_start", lambda pos, size: 0),
    "sliding window": ("chunk_start", lambda pos, size: max(0, pos - size + 1) if size else 0),
    "gate": ("gate_values", lambda o, z: o),
    "key heads": ("shared_head", lambda h, heads, kv: h % kv),
    "temperature": ("decay", lambda h, W, tau: _decay(h, W, 1.0)),
    "decay without its bias": ("decay", lambda h, W, tau: _decay(h, dict(W, **{"a2.b": 0}), tau)),
    "one decay a head": ("decay", lambda h, W, tau: _decay(h, W, tau).reshape(len(h), -1, 20).mean(-1, keepdims=True).repeat(20, -1).reshape(len(h), -1)),
    "embedding": ("embed", lambda t, k, s: _embed(t, k, 1.0)),
}


@pytest.mark.parametrize("name", sorted(MISTAKES))
def test_a_wrong_mechanism_shows(monkeypatch, name):
    w = L.weights(CFG, 5)
    toks = np.random.default_rng(6).integers(0, 203, 120)
    right = O.OracleLuvatar(CFG, w).forward(toks)
    monkeypatch.setattr(O, *MISTAKES[name])
    assert L.error(O.OracleLuvatar(CFG, w).forward(toks), right) > 2 * L.TOL["bfloat16"]


def test_a_lost_state_or_key_shows():
    w = L.weights(CFG, 7)
    toks = np.random.default_rng(8).integers(0, 203, 70)
    right = O.OracleLuvatar(CFG, w).forward(toks)[60:]
    for what in ("S", "k"):
        m = O.OracleLuvatar(CFG, w)
        m.forward(toks[:60])
        for st in m.states.values():
            if what == "S" and "S" in st:
                st["S"] = st["S"] * 0
            if what == "k" and "k" in st:
                st["k"] = [r * (i != 58) for i, r in enumerate(st["k"])]
        assert L.error(m.forward(toks[60:]), right) > L.TOL["bfloat16"]
