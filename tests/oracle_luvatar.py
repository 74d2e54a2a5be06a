"""Plain numpy model of the Luvatar design (tests only): one function per mechanism, token loops where a loop is the
definition, no code shared with the package.  Everything is float64 unless `dtype` says otherwise.

A decoder whose sublayers read the residual as it is and are normed on the way out, x += rms(mixer(x)) g1 and then
x += rms(ffn(x)) g2; the mixer is linear attention with a learned decay per key channel, or grouped-query attention inside
fixed chunks of the sequence with normed and rotated queries and keys, a sink and an output gate, whose keys and values may
be those of an earlier layer.  The embedding table, scaled on the way in, is the output head too.
"""
import math

import numpy as np

from tests.oracle_gizizen import rms, sigmoid, silu, sink_softmax


def embed(table, tokens, scale):
    return table[np.asarray(tokens, dtype=np.int64)] * scale


def rope_freqs(rot):
    d, sc = rot["dims"], rot.get("scaling")
    f = np.array([float(rot["base"]) ** (-2.0 * i / d) for i in range(d // 2)])
    return f / sc["factor"] if sc else f


def rotate(x, pos, rot):
    """x [T, heads, dim]: the first rot.dims of each head turn, neighbours paired; pos [T]."""
    y = x.copy()
    for i, f in enumerate(rope_freqs(rot)):
        c, s = np.cos(pos * f)[:, None], np.sin(pos * f)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i], y[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def chunk_start(pos, size):
    """First position that a query at `pos` may see."""
    return pos // size * size if size else 0


def gate_values(o, z):
    return o * sigmoid(z)


def shared_head(h, heads, kv_heads):
    return h // (heads // kv_heads)


def attention(h, W, mx, eps, state, kv_state=None):
    """h [T, width]; state: dict with 'k' and 'v' (and 'n', the tokens so far) of this layer; kv_state: of the layer whose
    keys and values are used instead (it has run on these tokens already)."""
    H, G, d, vd = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T, p0 = h.shape[0], state.setdefault("n", 0)
    pos = np.arange(p0, p0 + T)
    state["n"] += T
    q = rotate(rms((h @ W["q"].T).reshape(T, H, d), W["q.norm"], eps), pos, mx["rot"])
    if kv_state is None:
        k = rotate(rms((h @ W["k"].T).reshape(T, G, d), W["k.norm"], eps), pos, mx["rot"])
        state.setdefault("k", []).extend(list(k))
        state.setdefault("v", []).extend(list((h @ W["v"].T).reshape(T, G, vd)))
        kv_state = state
    K, V = np.array(kv_state["k"]), np.array(kv_state["v"])
    size = (mx.get("mask") or {}).get("size", 0)
    out = np.zeros((T, H, vd))
    for t in range(T):
        a, b = chunk_start(p0 + t, size), p0 + t + 1
        for hh in range(H):
            g = shared_head(hh, H, G)
            out[t, hh] = sink_softmax(K[a:b, g] @ q[t, hh] * mx["scale"], float(W["sink"][hh])) @ V[a:b, g]
    return gate_values(out.reshape(T, H * vd), h @ W["g"].T) @ W["o"].T


def decay(h, W, tau):
    """Per token and key channel: sigmoid(z)^(1 / tau)."""
    return sigmoid(h @ W["a1"].T @ W["a2"].T + W["a2.b"]) ** (1.0 / tau)


def gla(h, W, mx, eps, state):
    H, d, vd = mx["heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q, k = (h @ W["q"].T).reshape(T, H, d) / math.sqrt(d), (h @ W["k"].T).reshape(T, H, d)
    v, a = (h @ W["v"].T).reshape(T, H, vd), decay(h, W, mx["tau"]).reshape(T, H, d)
    S = state.setdefault("S", np.zeros((H, d, vd)))
    o = np.zeros((T, H, vd))
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    state["S"] = S
    o = rms(o, W["norm"], eps).reshape(T, H * vd) * silu(h @ W["g"].T)
    return o @ W["o"].T


def dense_ffn(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


class OracleLuvatar:
    """cfg: the parsed config.json; tensors: {name: array}.  forward(tokens) continues the sequence."""

    def __init__(self, cfg, tensors, dtype=np.float64):
        self.cfg = cfg
        self.t = {k: np.asarray(v, dtype=dtype) for k, v in tensors.items()}
        self.reset()

    def reset(self):
        self.states = {}

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def forward(self, tokens, layers_out=None):
        t, eps = self.t, self.cfg["norm"]["eps"]
        x = embed(t["embed"], tokens, self.cfg["embedding"]["scale"])
        for i, L in enumerate(self.cfg["layers"]):
            st, mx, W = self.states.setdefault(i, {}), L["mixer"], self._sub(f"l{i}.mix.")
            if L["type"] == "gla":
                y = gla(x, W, mx, eps, st)
            else:
                src = mx.get("kv_from")
                y = attention(x, W, mx, eps, st, None if src is None else self.states[src])
            x = x + rms(y, t[f"l{i}.norm1"], eps)
            if L.get("mlp"):
                x = x + rms(dense_ffn(x, self._sub(f"l{i}.mlp.")), t[f"l{i}.norm2"], eps)
            if layers_out is not None:
                layers_out.append(x)
        return rms(x, t["final.norm"], eps) @ t["embed"].T
