"""Plain, slow NumPy statement of the Nuzopel design: one function per mechanism, float64, one token at a time where the
mechanism is a recurrence.  It is the yardstick of the GPU tests and shares no code with the product path."""
from __future__ import annotations

import numpy as np

F = np.float64


def rms_unit(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def rotate_half(x, pos, base):
    """x [T, ..., R] rotated in pairs (i, i + R/2) by pos * base^(-2i/R)."""
    r = x.shape[-1]
    half = r // 2
    freq = F(base) ** (-2.0 * np.arange(half, dtype=F) / r)
    ang = np.asarray(pos, F)[:, None] * freq[None, :]
    ang = ang.reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (half,))
    u, v = x[..., :half], x[..., half:]
    return np.concatenate([u * np.cos(ang) - v * np.sin(ang), v * np.cos(ang) + u * np.sin(ang)], axis=-1)


def mlstm_recurrence(q, k, v, ig, fg, state=None):
    """q, k [T, H, D] (q scaled), v [T, H, V], log gates ig, fg [T, H] -> o [T, H, V] and the state (S, n, m)."""
    T, H, D = q.shape
    V = v.shape[-1]
    S, n, m = (np.zeros((H, D, V), F), np.zeros((H, D), F), np.zeros(H, F)) if state is None else [np.array(s, F) for s in state]
    o = np.zeros((T, H, V), F)
    for t in range(T):
        m_new = np.maximum(fg[t] + m, ig[t])
        keep, add = np.exp(fg[t] + m - m_new), np.exp(ig[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        num = np.einsum("hdv,hd->hv", S, q[t])
        den = np.maximum(np.abs(np.sum(n * q[t], axis=-1)), np.exp(-m)) + 1e-6
        o[t] = num / den[:, None]
    return o, (S, n, m)


def exact(a):
    return a


def mlstm_mixer(h, W, c, eps, state=None, r=exact):
    """W: dict of float64 tensors without the layer prefix; c: the layer's sizes; r: applied to what a 16-bit path rounds."""
    T = h.shape[0]
    H, D, V, cap = c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    h = r(h)
    q = r(h @ W["q"].T).reshape(T, H, D) * D ** -0.5
    k = r(h @ W["k"].T).reshape(T, H, D)
    v = r(h @ W["v"].T).reshape(T, H, V)
    ig = cap * np.tanh((h @ W["i"].T + W["i.b"]) / cap)
    fg = log_sigmoid(cap * np.tanh((h @ W["f"].T + W["f.b"]) / cap))
    o, state = mlstm_recurrence(q, k, v, ig, fg, state)
    o = rms_unit(o, eps).reshape(T, H * V) * W["norm"] * sigmoid(r(h @ W["g"].T))
    return r(o) @ W["o"].T, state


def latent_rows(h, W, c, eps, pos, r=exact):
    """The cached rows of a latent-attention layer: normed latent and rotated key part."""
    y = r(h) @ W["dkv"].T
    n = c["kv_rank"]
    return r(rms_norm(y[:, :n], W["dkv.norm"], eps)), r(rotate_half(y[:, n:], pos, c["rot"]["base"]))


def window_softmax(q, k, v, scale, size, pos0):
    """q [T, H, D] at positions pos0 .., k [N, H, D], v [N, H, V] at positions 0 .. N-1; size None = all earlier ones."""
    T, N = q.shape[0], k.shape[0]
    s = np.einsum("thd,nhd->htn", q, k) * scale
    dist = (pos0 + np.arange(T))[:, None] - np.arange(N)[None, :]
    see = (dist >= 0) & ((dist < size) if size else True)
    s = np.where(see[None], s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return np.einsum("htn,nhv->thv", p / p.sum(-1, keepdims=True), v)


def latent_mixer(h, W, c, eps, lat, pos0, r=exact):
    """lat = (latents [N, rank], rotated key parts [N, R]) of positions 0 .. N-1, this call's own included."""
    T = h.shape[0]
    H, D, R, V = c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    pos = pos0 + np.arange(T)
    q = r(r(h) @ W["q"].T).reshape(T, H, D + R)
    q = np.concatenate([q[..., :D], rotate_half(q[..., D:], pos, c["rot"]["base"])], -1)
    lc, lr = lat
    N = lc.shape[0]
    ku = r(lc @ W["uk"].T).reshape(N, H, D)
    vv = r(lc @ W["uv"].T).reshape(N, H, V)
    k = np.concatenate([ku, np.broadcast_to(lr[:, None, :], (N, H, R))], -1)
    o = window_softmax(q, k, vv, c["scale"], c["mask"]["size"], pos0)
    return r(o.reshape(T, H * V)) @ W["o"].T


def dense_ff(h, W, r=exact):
    h = r(h)
    return r(gelu_tanh(r(h @ W["gate"].T)) * r(h @ W["up"].T)) @ W["down"].T


class PlainModel:
    """A whole model; keeps each sequence's states and latents in the object returned by `start`."""

    def __init__(self, config, tensors):
        self.c = config
        self.t = {k: np.asarray(v, F) for k, v in tensors.items()}

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def start(self):
        return dict(pos=0, layers=[None] * len(self.c["layers"]))

    def forward(self, seq, tokens, trace=None, r=exact):
        """Runs `tokens` behind what `seq` has seen; returns logits [T, vocab].  `r` may disturb what a 16-bit path rounds."""
        c, eps, p0 = self.c, self.c["norm"]["eps"], seq["pos"]
        x = self.t["embed"][np.asarray(tokens)] * c["embedding"]["scale"]
        pos = p0 + np.arange(len(tokens))
        for i, layer in enumerate(c["layers"]):
            W, mc = self._sub(f"l{i}.mix."), layer["mixer"]
            if layer["type"] == "mlstm":
                y, seq["layers"][i] = mlstm_mixer(x, W, mc, eps, seq["layers"][i], r)
            else:
                src = mc.get("kv_from")
                if src is None:
                    src = i
                    new = latent_rows(x, W, mc, eps, pos, r)
                    old = seq["layers"][i]
                    seq["layers"][i] = new if old is None else tuple(np.concatenate([a, b]) for a, b in zip(old, new))
                y = latent_mixer(x, W, mc, eps, seq["layers"][src], p0, r)
            x = x + rms_norm(y, self.t[f"l{i}.norm1"], eps)
            if layer["mlp"] is not None:
                x = x + rms_norm(dense_ff(x, self._sub(f"l{i}.mlp."), r), self.t[f"l{i}.norm2"], eps)
            if trace is not None:
                trace.append(x.copy())
        seq["pos"] = p0 + len(tokens)
        return r(rms_norm(x, self.t["final.norm"], eps)) @ self.t["embed"].T * c["logit_scale"]
