"""Small Luvatar models with random weights for the tests: configurations and weights (bf16-exact).  Provider, checkpoint writer
and error measure are those of gizizen_models."""
import numpy as np

from ironmill_b200.stack_config import StackConfig
from tests.gizizen_models import TOL, Provider, bf16, bf16_bits, error, write_checkpoint  # noqa: F401


def attention(heads=6, kv_heads=2, dim=24, vdim=20, rot_dims=16, base=3e4, factor=3.0, chunk=37, scale=None, kv_from=None, ff=56):
    rot = {"base": base, "dims": rot_dims}
    if factor:
        rot["scaling"] = {"factor": factor}
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": scale if scale is not None else 1.4 / np.sqrt(dim)}
    if chunk:
        mixer["mask"] = {"size": chunk}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


# rank, bias: of the decay's tensors, which config.json does not give (the reader passes over them)
def gla(heads=3, dim=20, vdim=28, tau=8.0, rank=5, bias=(-3.0, 4.0), ff=0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "rank": rank, "bias": list(bias)}


def config(layers, width=88, vocab=203, scale=0.4, eps=3e-6):
    return {"architecture": "Luvatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


def weights(cfg, seed=0, sharp=1.6):
    rng = np.random.default_rng(seed)
    c = StackConfig.from_json(cfg)
    c.complete(lambda name: (cfg["layers"][int(name[1:name.index(".")])]["rank"],))
    out = {}
    for name, shape in c.tensors().items():
        leaf = name.split(".", 1)[-1] if name[0] == "l" and name[1].isdigit() else name
        layer = cfg["layers"][int(name[1:name.index(".")])] if leaf != name else {}
        if leaf in ("mix.q.norm", "mix.k.norm"):
            a = rng.uniform(0.6, 1.6, shape) * (sharp if leaf == "mix.q.norm" else 1.0)
        elif leaf.endswith(("norm", "norm1", "norm2")):
            a = rng.uniform(0.6, 1.6, shape)
        elif leaf == "mix.sink":
            a = rng.normal(1.0, 1.5, shape)
        elif leaf == "mix.a2.b":
            a = rng.uniform(*layer["bias"], shape)
        elif leaf == "embed":
            a = rng.normal(0, 1.0, shape)
        else:
            a = rng.normal(0, 1.0 / np.sqrt(shape[-1]), shape)
        out[name] = bf16(a)
    return out


def close(got, want, dtype):
    """For models of several layers.  Every sublayer's output is normed, so where one happens to be small its rounding is blown up:
    rounding the plain model's activations to bf16 moves single rows of the tests' models by up to 0.11, all rows together by
    less than 0.05.  So: all rows (eight and more) within TOL, and no row beyond three times that."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want)
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    spread = np.sqrt(np.mean((want - want.mean(axis=-1, keepdims=True)) ** 2))
    rows = np.sqrt((d * d).mean(axis=-1)) / spread
    return rows.max() < 3 * TOL[dtype] and (len(rows) < 8 or np.sqrt((rows * rows).mean()) < TOL[dtype])
