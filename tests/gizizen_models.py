"""Small Gizizen models with random weights for the tests: configurations, weights (bf16-exact), a weight provider."""
import numpy as np

from ironmill_b200.bundle import WeightTensor
from ironmill_b200.stack_config import StackConfig


def bf16(a):
    """Nearest bf16 values of an f32 array, as f32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).view(np.float32)


def bf16_bits(a):
    return (bf16(a).view(np.uint32) >> 16).astype(np.uint16)


YARN = {"factor": 5.0, "fast": 20.0, "slow": 1.5, "original": 300}


def latent(heads=3, dim=24, rot_dim=12, vdim=20, kv_rank=40, scale=None, base=2e4, scaling=YARN, ff=56):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
                      "scale": scale if scale is not None else 1.3 / np.sqrt(dim + rot_dim)}}


def lightning(heads=3, dim=20, vdim=28, decay=(0.4, 0.93, 0.998), ff=72):
    return {"type": "lightning", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)[:heads]}}


def config(layers, width=88, vocab=203, loop=None, cap=7.0, eps=3e-6):
    return {"architecture": "Gizizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]} if loop else None, "logit_softcap": cap}


# sharp: gain on queries and keys, so that a row of attention weights has few large entries and every key can be the one
def weights(cfg, seed=0, sharp=1.6):
    rng = np.random.default_rng(seed)
    c = StackConfig.from_json(cfg)
    out = {}
    for name, shape in c.tensors().items():
        leaf = name.split(".", 1)[-1] if name[0] == "l" and name[1].isdigit() else name
        if leaf.endswith("norm") or leaf == "norm1":
            a = rng.uniform(0.6, 1.6, shape)
        elif leaf == "mix.sink":
            a = rng.normal(1.0, 1.5, shape)
        elif leaf == "loop.step":
            a = rng.normal(0, 0.7, shape)
        elif leaf == "embed":
            a = rng.normal(0, 1.0, shape)
        else:
            a = rng.normal(0, 1.0 / np.sqrt(shape[-1]), shape)
            if leaf in ("mix.q", "mix.uk", "mix.dkv"):
                a *= sharp
            if leaf == "mix.o" or leaf == "head":
                a *= 2.0
            if leaf == "mlp.down":
                a *= 1.5
        out[name] = bf16(a)
    return out


class Provider:
    def __init__(self, cfg, tensors):
        self._cfg, self._t = StackConfig.from_json(cfg), tensors

    def config(self):
        return self._cfg

    def tensor_names(self):
        return list(self._t)

    def has_tensor(self, name):
        return name in self._t

    def tensor(self, name):
        a = self._t[name]
        return WeightTensor(bf16_bits(a), a.shape, "bfloat16")


def write_checkpoint(path, cfg, tensors):
    """config.json + model.safetensors of the model, bf16."""
    import json
    import struct
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    header, blob = {}, b""
    for name, a in tensors.items():
        raw = bf16_bits(a).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    h = json.dumps(header).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + blob)


def error(got, want):
    """Largest root-mean-square logit error of a row (its mean taken off), in units of the logits' spread."""
    d = np.asarray(got, dtype=np.float64) - want
    d = d - d.mean(axis=-1, keepdims=True)
    spread = np.sqrt(np.mean((want - want.mean(axis=-1, keepdims=True)) ** 2))
    return float(np.sqrt((d * d).mean(axis=-1)).max() / spread)


TOL = {"float32": 1e-4, "bfloat16": 0.06}
