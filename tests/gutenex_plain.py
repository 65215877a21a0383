"""Plain, slow NumPy statement of the Gutenex design: one function per mechanism, float64, one token at a time where the
mechanism is a recurrence.  It is the yardstick of the GPU tests and shares no code with the product path."""
from __future__ import annotations

import numpy as np

from nuzopel_plain import exact, rms_norm, rms_unit, sigmoid

F = np.float64


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def unit(x):
    """x over its length along the last axis."""
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def rotate_pairs(x, pos, base, dims):
    """x [T, ..., D]: of the first `dims` values, pairs (2i, 2i + 1) are turned by pos * base^(-2i / dims)."""
    ang = np.asarray(pos, F)[:, None] * F(base) ** (-2.0 * np.arange(dims // 2, dtype=F) / dims)[None, :]
    ang = ang.reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (dims // 2,))
    out = np.array(x, F)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(ang) - v * np.sin(ang)
    out[..., 1:dims:2] = v * np.cos(ang) + u * np.sin(ang)
    return out


# ---- lightning attention: a matrix memory with one constant decay per head -------------------------------------------------
def decay_recurrence(q, k, v, decay, S=None):
    """q, k [T, H, D], v [T, H, V], decay [H] -> o [T, H, V], S [H, D, V]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[-1]), F) if S is None else np.array(S)
    o = np.zeros((T, H, v.shape[-1]), F)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def lightning_mixer(h, W, c, eps, S=None, r=exact):
    T, H, D, V = h.shape[0], c["heads"], c["dim"], c["vdim"]
    h = r(h)
    q = r(silu(h @ W["q"].T)).reshape(T, H, D)
    k = r(silu(h @ W["k"].T)).reshape(T, H, D)
    v = r(silu(h @ W["v"].T)).reshape(T, H, V)
    o, S = decay_recurrence(q, k, v, np.asarray(c["decay"], F), S)
    o = rms_norm(o.reshape(T, H * V), W["norm"], eps) * sigmoid(r(h @ W["g"].T))
    return r(o) @ W["o"].T, S


# ---- gated delta rule with a decay per key channel -----------------------------------------------------------------------------
def short_conv(y, w, hist):
    """y [T, C] behind hist [taps - 1, C]; w [C, taps], the last column is the current token's.  Returns output and new hist."""
    taps = w.shape[1]
    full = np.concatenate([hist, y])
    out = np.zeros_like(y)
    for j in range(taps):
        out += full[j:j + len(y)] * w[:, j]
    return out, full[len(full) - (taps - 1):]


def channel_delta_recurrence(q, k, v, g, beta, S=None):
    """q, k, g [T, H, D] (g: decay factors), v [T, H, V], beta [T, H] -> o [T, H, V], S [H, D, V]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[-1]), F) if S is None else np.array(S)
    o = np.zeros((T, H, v.shape[-1]), F)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def channel_delta_mixer(h, W, c, eps, state=None, r=exact):
    T, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    h = r(h)
    if state is None:
        state = dict(S=None, q=np.zeros((c["conv"] - 1, G * D)), k=np.zeros((c["conv"] - 1, G * D)), v=np.zeros((c["conv"] - 1, H * V)))
    new, y = {}, {}
    for n in "qkv":
        y[n], new[n] = short_conv(r(h @ W[n].T), W[n + ".conv"], state[n])
        y[n] = r(silu(y[n]))
    own = np.arange(H) // (H // G)
    q = (unit(y["q"].reshape(T, G, D)) * F(D) ** -0.5)[:, own]
    k = unit(y["k"].reshape(T, G, D))[:, own]
    v = y["v"].reshape(T, H, V)
    beta = sigmoid(h @ W["b"].T)
    a = r(h @ W["a1"].T) @ W["a2"].T + W["dt_bias"]
    g = np.exp(-np.exp(W["A_log"])[None, :, None] * softplus(a).reshape(T, H, D))
    o, new["S"] = channel_delta_recurrence(q, k, v, g, beta, state["S"])
    gate = sigmoid(r(r(h @ W["g1"].T) @ W["g2"].T)).reshape(T, H, V)
    o = rms_norm(o, W["norm"], eps) * gate
    return r(o.reshape(T, H * V)) @ W["o"].T, new


# ---- differential attention ---------------------------------------------------------------------------------------------------------
def visible(pos_q, pos_k, size, keep_first):
    d = pos_q[:, None] - pos_k[None, :]
    return (d >= 0) & ((d < size) | (pos_k[None, :] < keep_first))


def softmax_attention(q, k, v, scale, see):
    """q [T, H, D], k [N, H, D], v [N, H, V], see [T, N]."""
    s = np.where(see[None], np.einsum("thd,nhd->htn", q, k) * scale, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return np.einsum("htn,nhv->thv", p / p.sum(-1, keepdims=True), v)


def diff_keys(h, W, c, eps, pos, r=exact):
    """The cached keys [T, G, 2, D] and values [T, G, V] of these rows."""
    T, G, D, V = h.shape[0], c["kv_heads"], c["dim"], c["vdim"]
    k = rms_norm((r(h) @ W["k"].T).reshape(T, G, 2, D), W["k.norm"], eps)
    return r(rotate_pairs(k, pos, c["rot"]["base"], c["rot"]["dims"])), r(r(h) @ W["v"].T).reshape(T, G, V)


def diff_lambda(W, c):
    return np.exp(np.sum(W["lq1"] * W["lk1"])) - np.exp(np.sum(W["lq2"] * W["lk2"])) + c["diff"]


def diff_mixer(h, W, c, eps, kv, pos0, r=exact):
    """kv = keys and values of positions 0 .. N-1, this call's own included."""
    T, H, G, D, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    pos = pos0 + np.arange(T)
    q = rms_norm((r(h) @ W["q"].T).reshape(T, H, 2, D), W["q.norm"], eps)
    q = r(rotate_pairs(q, pos, c["rot"]["base"], c["rot"]["dims"]))
    own = np.arange(H) // (H // G)
    k, v = kv[0][:, own], kv[1][:, own]
    see = visible(pos, np.arange(k.shape[0]), c["mask"]["size"], c["mask"]["keep_first"])
    a1, a2 = (softmax_attention(q[:, :, m], k[:, :, m], v, c["scale"], see) for m in (0, 1))
    o = rms_unit(a1 - diff_lambda(W, c) * a2, eps) * (1.0 - c["diff"])
    return r(o.reshape(T, H * V)) @ W["o"].T


def dense_ff(h, W, r=exact):
    h = r(h)
    return r(silu(r(h @ W["gate"].T)) * r(h @ W["up"].T)) @ W["down"].T


def layer_runs(config):
    """(layer, True where the embedding output is added ahead of it) in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


class PlainModel:
    """A whole model; a sequence's states and keys live in the object returned by `start`."""

    def __init__(self, config, tensors):
        self.c = config
        self.t = {k: np.asarray(v, F) for k, v in tensors.items()}

    def _sub(self, prefix):
        return {k[len(prefix):]: v for k, v in self.t.items() if k.startswith(prefix)}

    def start(self):
        return dict(pos=0, runs=[None] * len(layer_runs(self.c)))

    def forward(self, seq, tokens, trace=None, r=exact):
        """Runs `tokens` behind what `seq` has seen; returns logits [T, vocab].  `r` may disturb what a 16-bit path rounds."""
        c, eps, p0 = self.c, self.c["norm"]["eps"], seq["pos"]
        x0 = x = self.t["embed"][np.asarray(tokens)]
        pos = p0 + np.arange(len(tokens))
        for n, (i, again) in enumerate(layer_runs(c)):
            layer, W, mc = c["layers"][i], self._sub(f"l{i}.mix."), c["layers"][i]["mixer"]
            if again:
                x = x + x0
            h = rms_norm(x, self.t[f"l{i}.norm1"], eps)
            if layer["type"] == "lightning":
                y, seq["runs"][n] = lightning_mixer(h, W, mc, eps, seq["runs"][n], r)
            elif layer["type"] == "channel_delta":
                y, seq["runs"][n] = channel_delta_mixer(h, W, mc, eps, seq["runs"][n], r)
            else:
                new, old = diff_keys(h, W, mc, eps, pos, r), seq["runs"][n]
                seq["runs"][n] = new if old is None else tuple(np.concatenate([a, b]) for a, b in zip(old, new))
                y = diff_mixer(h, W, mc, eps, seq["runs"][n], p0, r)
            x = x + y
            if layer["mlp"] is not None:
                x = x + dense_ff(rms_norm(x, self.t[f"l{i}.norm2"], eps), self._sub(f"l{i}.mlp."), r)
            if trace is not None:
                trace.append(x.copy())
        seq["pos"] = p0 + len(tokens)
        logits = r(rms_norm(x, self.t["final.norm"], eps)) @ self.t["head"].T
        cap = c["logit_softcap"]
        return cap * np.tanh(logits / cap)
