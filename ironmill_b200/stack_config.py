"""Configuration of models given as a list of layers (the Gizizen and Luvatar designs and relatives): the reader of their
config.json.

Every size and every constant that may differ between models is a field here; a block takes them as arguments
(im_stack_layer in include/ironmill_cuda.h), so a layer kind can be combined with others in another design.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .bundle import GpuBundleError


def _get(obj, path: str, kind=int, default=...):
    cur = obj
    for k in path.split("."):
        if not isinstance(cur, dict) or k not in cur:
            if default is ...:
                raise GpuBundleError(f"missing field: {path}")
            return default
        cur = cur[k]
    if cur is None and default is not ...:
        return default
    if kind is int and (not isinstance(cur, int) or isinstance(cur, bool)):
        raise GpuBundleError(f"{path} must be an integer")
    if kind is float:
        if not isinstance(cur, (int, float)) or isinstance(cur, bool):
            raise GpuBundleError(f"{path} must be a number")
        return float(cur)
    return cur


@dataclass
class Rotation:
    dims: int
    base: float
    factor: float = 0.0      # 0: plain rotation; otherwise the interpolation of long contexts
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0
    divide: float = 1.0      # every frequency is divided by this (linear scaling)


@dataclass
class LatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotation

    @staticmethod
    def read(m: dict, where: str) -> "LatentAttention":
        sc = _get(m, "rot.scaling", dict, None)
        rot = Rotation(_get(m, "rot.dims"), _get(m, "rot.base", float))
        if sc:
            rot.factor, rot.original = _get(sc, "factor", float), _get(sc, "original", float)
            rot.fast, rot.slow = _get(sc, "fast", float), _get(sc, "slow", float)
        a = LatentAttention(_get(m, "heads"), _get(m, "dim"), _get(m, "rot_dim"), _get(m, "vdim"), _get(m, "kv_rank"), _get(m, "scale", float), rot)
        if rot.dims > a.rot_dim:
            raise GpuBundleError(f"{where}: {rot.dims} rotated dimensions in a part of {a.rot_dim}")
        return a

    def tensors(self, width: int) -> dict:
        h, n = self.heads, self.kv_rank
        return {"q": (h * (self.dim + self.rot_dim), width), "dkv": (n + self.rot_dim, width), "dkv.norm": (n,), "uk": (h * self.dim, n),
                "uv": (h * self.vdim, n), "sink": (h,), "o": (width, h * self.vdim)}


@dataclass
class LinearAttention:
    heads: int
    dim: int
    vdim: int
    decay: list

    @staticmethod
    def read(m: dict, where: str) -> "LinearAttention":
        d = _get(m, "decay", list)
        a = LinearAttention(_get(m, "heads"), _get(m, "dim"), _get(m, "vdim"), [float(x) for x in d])
        if len(a.decay) != a.heads:
            raise GpuBundleError(f"{where}: {len(a.decay)} decays for {a.heads} heads")
        return a

    def tensors(self, width: int) -> dict:
        h = self.heads
        return {"q": (h * self.dim, width), "k": (h * self.dim, width), "v": (h * self.vdim, width), "g": (h * self.vdim, width),
                "norm": (h * self.vdim,), "o": (width, h * self.vdim)}


@dataclass
class GroupedAttention:
    """Grouped-query attention: normed and rotated queries and keys, chunks, a sink, an output gate."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation
    chunk: int = 0               # positions of a chunk; 0: all earlier positions are seen
    kv_from: int | None = None   # layer whose keys and values are used

    @staticmethod
    def read(m: dict, where: str) -> "GroupedAttention":
        rot = Rotation(0, 1.0)
        if _get(m, "rot", dict, None):
            rot = Rotation(_get(m, "rot.dims"), _get(m, "rot.base", float))
            if _get(m, "rot.scaling", dict, None):
                rot.divide = _get(m, "rot.scaling.factor", float)
        a = GroupedAttention(_get(m, "heads"), _get(m, "kv_heads"), _get(m, "dim"), _get(m, "vdim"), _get(m, "scale", float), rot,
                             _get(m, "mask.size") if _get(m, "mask", dict, None) else 0, _get(m, "kv_from", int, None))
        if rot.dims > a.dim or rot.dims % 2 or rot.divide <= 0.0:
            raise GpuBundleError(f"{where}: bad rotation")
        if a.kv_heads <= 0 or a.heads % a.kv_heads:
            raise GpuBundleError(f"{where}: {a.heads} query heads do not share {a.kv_heads} key / value heads evenly")
        return a

    def tensors(self, width: int) -> dict:
        h, g = self.heads, self.kv_heads
        out = {"q": (h * self.dim, width), "q.norm": (self.dim,), "sink": (h,), "g": (h * self.vdim, width), "o": (width, h * self.vdim)}
        if self.kv_from is None:
            out.update({"k": (g * self.dim, width), "k.norm": (self.dim,), "v": (g * self.vdim, width)})
        return out


@dataclass
class GatedLinearAttention:
    """Linear attention with a decay per token and key channel, sigmoid(a2 (a1 h) + b)^(1 / tau)."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 0   # rows of a1: the checkpoint's tensor says (complete())

    @staticmethod
    def read(m: dict, where: str) -> "GatedLinearAttention":
        a = GatedLinearAttention(_get(m, "heads"), _get(m, "dim"), _get(m, "vdim"), _get(m, "tau", float))
        if a.tau <= 0.0:
            raise GpuBundleError(f"{where}: tau must be positive")
        return a

    def complete(self, shape_of) -> None:
        s = shape_of("a1")
        if s:
            self.rank = int(s[0])

    def tensors(self, width: int) -> dict:
        h, r = self.heads, self.rank
        return {"q": (h * self.dim, width), "k": (h * self.dim, width), "v": (h * self.vdim, width), "g": (h * self.vdim, width),
                "norm": (self.vdim,), "a1": (r, width), "a2": (h * self.dim, r), "a2.b": (h * self.dim,), "o": (width, h * self.vdim)}


# layer kinds by the name config.json gives them
MIXERS = {"latent_attention": LatentAttention, "lightning": LinearAttention, "attention": GroupedAttention, "gla": GatedLinearAttention}


@dataclass(frozen=True)
class Design:
    """What a design fixes beside its layers."""
    post_norm: bool = False      # x += rms(mixer(x)) g1, x += rms(ffn(x)) g2; otherwise x += mixer(n) + ffn(n), n = rms(x) g1
    silu: bool = False           # activation of the feed-forwards: SiLU, otherwise gelu_tanh
    scaled_embedding: bool = False  # embedding.scale in place of a norm after the embedding
    tied_head: bool = False      # the embedding table is the output head


# designs by their architecture name in lower case
DESIGNS = {"gizizen": Design(), "luvatar": Design(post_norm=True, silu=True, scaled_embedding=True, tied_head=True)}


@dataclass
class StackLayer:
    mixer: object
    ff: int = 0


@dataclass
class StackConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: list = field(default_factory=list)
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0
    logit_softcap: float = 0.0
    embed_scale: float = 0.0     # 0: the embedding is normed
    design: Design = Design()
    raw: dict = field(default_factory=dict)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @staticmethod
    def from_json(obj: dict) -> "StackConfig":
        c = StackConfig(_get(obj, "architecture", str), _get(obj, "vocab"), _get(obj, "width"), _get(obj, "norm.eps", float), raw=obj)
        c.design = DESIGNS.get(c.architecture.lower(), c.design)
        if c.design.scaled_embedding:
            c.embed_scale = _get(obj, "embedding.scale", float)
            if c.embed_scale == 0.0:
                raise GpuBundleError("embedding.scale must not be zero")
        for i, e in enumerate(_get(obj, "layers", list)):
            kind = _get(e, "type", str)
            if kind not in MIXERS:
                raise GpuBundleError(f"layer {i}: unknown type '{kind}'")
            mlp = _get(e, "mlp", dict, None)
            if mlp and _get(mlp, "kind", str) != "dense":
                raise GpuBundleError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
            c.layers.append(StackLayer(MIXERS[kind].read(_get(e, "mixer", dict), f"layer {i}"), _get(mlp, "ff") if mlp else 0))
        for i, L in enumerate(c.layers):
            j = getattr(L.mixer, "kv_from", None)
            if j is None:
                continue
            o = c.layers[j].mixer if 0 <= j < i else None
            if not isinstance(o, GroupedAttention) or o.kv_from is not None or (o.kv_heads, o.dim, o.vdim) != (L.mixer.kv_heads, L.mixer.dim, L.mixer.vdim):
                raise GpuBundleError(f"layer {i}: layer {j} has no keys and values that it could use")
        loop = _get(obj, "loop", dict, None)
        if loop:
            c.loop_start, c.loop_stop, c.loop_times = _get(loop, "start"), _get(loop, "stop"), _get(loop, "times")
        c.logit_softcap = _get(obj, "logit_softcap", float, 0.0)
        return c

    def to_json(self) -> dict:
        return self.raw

    def complete(self, shape_of) -> None:
        """Fills in the sizes that only the checkpoint's tensors give.  shape_of(name): a tensor's shape, None without it."""
        for i, L in enumerate(self.layers):
            if hasattr(L.mixer, "complete"):
                L.mixer.complete(lambda name: shape_of(f"l{i}.mix.{name}"))

    def tensors(self) -> dict:
        """{checkpoint name: shape} of everything the model loads."""
        w = self.hidden_size
        out = {"embed": (self.vocab_size, w)}
        if not self.design.scaled_embedding:
            out["embed.norm"] = (w,)
        if self.loop_times:
            out["loop.in"], out["loop.step"] = (w, 2 * w), (self.loop_times, w)
        for i, L in enumerate(self.layers):
            out[f"l{i}.norm1"] = (w,)
            out.update({f"l{i}.mix.{k}": s for k, s in L.mixer.tensors(w).items()})
            if L.ff:
                out.update({f"l{i}.mlp.gate": (L.ff, w), f"l{i}.mlp.up": (L.ff, w), f"l{i}.mlp.down": (w, L.ff)})
                if self.design.post_norm:
                    out[f"l{i}.norm2"] = (w,)
        out["final.norm"] = (w,)
        if not self.design.tied_head:
            out["head"] = (self.vocab_size, w)
        return out
