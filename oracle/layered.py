"""Plain restatement of the models built from a list of layers (architecture "Tolevik"): one function per mechanism, numpy, one
token after the other wherever the definition is a recurrence.  Test infrastructure only; it shares nothing with the product path.

Notation.  A sequence is a matrix of row vectors x[t].  Every weight is [out, in].  ``st`` arguments carry what a sequence keeps
between calls (GLA: the state matrices; latent attention: the latents and rotated keys), so a prompt may be fed in portions.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def rotate_pairs(x, positions, base, dims):
    """Rotation of neighbouring pairs (2i, 2i+1) of the first ``dims`` entries of the last axis by positions * base^(-2i/dims);
    x is [T, ..., n], positions [T]."""
    i = np.arange(dims // 2)
    ang = np.asarray(positions, np.float64)[:, None] * np.power(float(base), -2.0 * i / dims)
    ang = ang.reshape((ang.shape[0],) + (1,) * (x.ndim - 2) + (dims // 2,))
    c, s = np.cos(ang), np.sin(ang)
    y = np.array(x, copy=True)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y[..., 0:dims:2] = u * c - v * s
    y[..., 1:dims:2] = v * c + u * s
    return y


def gla_decay(h, a1, a2, a2_b, tau):
    """Per key channel: alpha = sigmoid(z)^(1/tau), z = A2 (A1 h) + b."""
    return np.exp(log_sigmoid(h @ a1.T @ a2.T + a2_b) / tau)


def gla_recurrence(q, k, v, alpha, state):
    """q, k, alpha [T, H, D], v [T, H, V], state [H, D, V] (updated in place): S <- diag(alpha) S + k v^T, o = S^T q."""
    out = np.zeros(v.shape, state.dtype)
    for t in range(q.shape[0]):
        for hd in range(q.shape[1]):
            s = state[hd]
            s *= alpha[t, hd][:, None]
            s += np.outer(k[t, hd], v[t, hd])
            out[t, hd] = q[t, hd] @ s
    return out


def gla_mixer(h, p, m, eps, state):
    """p: the mixer's tensors by their short names, m: its sizes; h [T, width] -> [T, width]."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ p["q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ p["k"].T).reshape(T, H, D)
    v = (h @ p["v"].T).reshape(T, H, V)
    alpha = gla_decay(h, p["a1"], p["a2"], p["a2.b"], m["tau"]).reshape(T, H, D)
    o = gla_recurrence(q, k, v, alpha, state)
    o = rms_norm(o, p["norm"], eps).reshape(T, H * V)
    return (o * silu(h @ p["g"].T)) @ p["o"].T


def latents_of(h, p, m, eps, positions):
    """What latent attention keeps of a token: the normed latent and the rotated key part shared by the heads."""
    kv = h @ p["dkv"].T
    r = m["kv_rank"]
    return rms_norm(kv[:, :r], p["dkv.norm"], eps), rotate_pairs(kv[:, r:], positions, m["rot"]["base"], m["rot"]["dims"])


def latent_queries(h, p, m, eps, positions):
    """(unrotated [T, H, dim], rotated [T, H, rot_dim])"""
    q = (rms_norm(h @ p["dq"].T, p["dq.norm"], eps) @ p["uq"].T).reshape(h.shape[0], m["heads"], m["dim"] + m["rot_dim"])
    return q[..., :m["dim"]], rotate_pairs(q[..., m["dim"]:], positions, m["rot"]["base"], m["rot"]["dims"])


def latent_attention_core(qn, qr, c, kr, p, m, first):
    """Causal softmax attention of queries at positions first, first + 1, ... over the keys 0 .. of the latents c and rotated parts kr."""
    H, D, V = m["heads"], m["dim"], m["vdim"]
    kn = (c @ p["uk"].T).reshape(-1, H, D)
    v = (c @ p["uv"].T).reshape(-1, H, V)
    out = np.zeros((qn.shape[0], H, V), c.dtype)
    for t in range(qn.shape[0]):
        n = first + t + 1
        for hd in range(H):
            s = (kn[:n, hd] @ qn[t, hd] + kr[:n] @ qr[t, hd]) * m["scale"]
            w = np.exp(s - s.max())
            out[t, hd] = (w / w.sum()) @ v[:n, hd]
    return out


def latent_attention_mixer(h, p, m, eps, st):
    """st: {"c": [n, kv_rank], "kr": [n, rot_dim]} of the tokens before h (extended in place)."""
    first = st["c"].shape[0]
    pos = first + np.arange(h.shape[0])
    c, kr = latents_of(h, p, m, eps, pos)
    st["c"], st["kr"] = np.concatenate([st["c"], c]), np.concatenate([st["kr"], kr])
    qn, qr = latent_queries(h, p, m, eps, pos)
    o = latent_attention_core(qn, qr, st["c"], st["kr"], p, m, first)
    o = o * sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(h.shape[0], -1) @ p["o"].T


def dense_mlp(h, p):
    return (silu(h @ p["gate"].T + p["gate.b"]) * (h @ p["up"].T + p["up.b"])) @ p["down"].T + p["down.b"]


class LayeredOracle:
    """config: the dictionary of config.json; params: {tensor name: array}.  ``feed`` runs the next tokens of the sequence."""

    def __init__(self, config, params, dtype=np.float64):
        self.c, self.dtype = config, dtype
        self.p = {k: np.asarray(v, dtype) for k, v in params.items()}
        self.reset()

    def reset(self):
        self.states = []
        for la in self.c["layers"]:
            m = la["mixer"]
            if la["type"] == "gla":
                self.states.append(np.zeros((m["heads"], m["dim"], m["vdim"]), self.dtype))
            elif la["type"] == "latent_attention":
                self.states.append({"c": np.zeros((0, m["kv_rank"]), self.dtype), "kr": np.zeros((0, m["rot_dim"]), self.dtype)})
            else:
                raise ValueError(la["type"])

    def _sub(self, prefix):
        n = len(prefix)
        return {k[n:]: v for k, v in self.p.items() if k.startswith(prefix)}

    def feed(self, tokens, taps=None):
        eps = self.c["norm"]["eps"]
        x = self.p["embed"][np.asarray(tokens)]
        for i, la in enumerate(self.c["layers"]):
            mix = gla_mixer if la["type"] == "gla" else latent_attention_mixer
            x = x + rms_norm(mix(x, self._sub(f"l{i}.mix."), la["mixer"], eps, self.states[i]), self.p[f"l{i}.norm1"], eps)
            if la["mlp"] is not None:
                x = x + rms_norm(dense_mlp(x, self._sub(f"l{i}.mlp.")), self.p[f"l{i}.norm2"], eps)
            if taps is not None:
                taps.append(x)
        return rms_norm(x, self.p["final.norm"], eps) @ self.p["head"].T
