"""Plain numpy model of the Gizizen design (tests only): one function per mechanism, token loops where a loop is the
definition, no code shared with the package.  Everything is float64 unless `dtype` says otherwise.

A decoder of parallel blocks x += mixer(n) + ffn(n), n = rms(x) g, whose mixer is latent attention with a sink and
rotary keys or decayed linear attention; a run of layers is repeated with shared weights, each pass preceded by a linear
map of [x, x0] (x0: the normed embedding) and a learned vector of the pass.
"""
import math

import numpy as np


def rms(x, g, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * g


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rope_freqs(rot):
    """(angular frequencies, amplitude) of the rotary pairs, with the piecewise interpolation of long contexts if any."""
    d, base = rot["dims"], float(rot["base"])
    f = np.array([base ** (-2.0 * i / d) for i in range(d // 2)])
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def turn_dim(turns):
        return d * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turn_dim(sc["fast"])), 0), min(math.ceil(turn_dim(sc["slow"])), d - 1)
    ramp = np.clip((np.arange(d // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """x [T, ..., dims], neighbours paired; pos [T]."""
    f, amp = rope_freqs(rot)
    a = pos[:, None].astype(np.float64) * f[None, :]
    a = a.reshape((len(pos),) + (1,) * (x.ndim - 2) + (len(f),))
    c, s = np.cos(a) * amp, np.sin(a) * amp
    u, v = x[..., 0::2], x[..., 1::2]
    y = np.empty_like(x)
    y[..., 0::2] = u * c - v * s
    y[..., 1::2] = v * c + u * s
    return y


def sink_softmax(s, sink):
    """Rows of scores (-inf = not seen) with one extra keyless logit."""
    m = max(np.max(s), sink)
    e = np.exp(s - m)
    return e / (e.sum() + math.exp(sink - m))


def latent_attention(h, W, mx, eps, state):
    """h [T, width]; state: dict with 'lat' and 'kr' lists of the tokens before these.  Returns [T, width]."""
    H, d, r, vd, kr = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    T, p0 = h.shape[0], len(state.setdefault("lat", []))
    pos = np.arange(p0, p0 + T)
    q = (h @ W["q"].T).reshape(T, H, d + r)
    qr = rotate(q[..., d:], pos, mx["rot"])
    dkv = h @ W["dkv"].T
    state["lat"] += list(rms(dkv[:, :kr], W["dkv.norm"], eps))
    state.setdefault("kr", []).extend(list(rotate(dkv[:, kr:], pos, mx["rot"])))
    lat, krot = np.array(state["lat"]), np.array(state["kr"])
    k = (lat @ W["uk"].T).reshape(-1, H, d)
    v = (lat @ W["uv"].T).reshape(-1, H, vd)
    out = np.zeros((T, H, vd))
    for hh in range(H):
        s = (q[:, hh, :d] @ k[:, hh].T + qr[:, hh] @ krot.T) * mx["scale"]
        for t in range(T):
            n = p0 + t + 1
            out[t, hh] = sink_softmax(s[t, :n], float(W["sink"][hh])) @ v[:n, hh]
    return out.reshape(T, H * vd) @ W["o"].T


def lightning(h, W, mx, eps, state):
    H, d, vd = mx["heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q, k = silu(h @ W["q"].T).reshape(T, H, d), silu(h @ W["k"].T).reshape(T, H, d)
    v = silu(h @ W["v"].T).reshape(T, H, vd)
    S = state.setdefault("S", np.zeros((H, d, vd)))
    dec = np.asarray(mx["decay"], dtype=np.float64)[:, None, None]
    o = np.zeros((T, H, vd))
    for t in range(T):
        S = dec * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    state["S"] = S
    o = rms(o.reshape(T, H * vd), W["norm"], eps) * sigmoid(h @ W["g"].T)
    return o @ W["o"].T


MIXERS = {"latent_attention": latent_attention, "lightning": lightning}


def dense_ffn(h, W):
    return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


class OracleGizizen:
    """cfg: the parsed config.json; tensors: {name: array}.  forward(tokens) continues the sequence."""

    def __init__(self, cfg, tensors, dtype=np.float64):
        self.cfg = cfg
        self.t = {k: np.asarray(v, dtype=dtype) for k, v in tensors.items()}
        self.reset()

    def reset(self):
        self.states = {}

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def schedule(self):
        """[(layer, pass or -1, first layer of its pass)]"""
        lp, n = self.cfg.get("loop"), len(self.cfg["layers"])
        if not lp:
            return [(i, -1, False) for i in range(n)]
        out = [(i, -1, False) for i in range(lp["start"])]
        for p in range(lp["times"]):
            out += [(i, p, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
        return out + [(i, -1, False) for i in range(lp["stop"], n)]

    def forward(self, tokens, layers_out=None):
        t, eps = self.t, self.cfg["norm"]["eps"]
        x = rms(t["embed"][np.asarray(tokens, dtype=np.int64)], t["embed.norm"], eps)
        x0 = x
        for i, p, first in self.schedule():
            if first:
                x = np.concatenate([x, x0], axis=-1) @ t["loop.in"].T + t["loop.step"][p]
            L = self.cfg["layers"][i]
            h = rms(x, t[f"l{i}.norm1"], eps)
            st = self.states.setdefault((i, p), {})
            y = MIXERS[L["type"]](h, self._sub(f"l{i}.mix."), L["mixer"], eps, st)
            if L.get("mlp"):
                y = y + dense_ffn(h, self._sub(f"l{i}.mlp."))
            x = x + y
            if layers_out is not None:
                layers_out.append(x)
        z = rms(x, t["final.norm"], eps) @ t["head"].T
        cap = self.cfg.get("logit_softcap")
        return cap * np.tanh(z / cap) if cap else z
