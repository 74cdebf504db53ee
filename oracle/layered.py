"""Plain restatement of the models built from a list of layers (architectures "Tolevik" and "Bulidra"): one function per mechanism,
numpy, one token after the other wherever the definition is a recurrence.  Test infrastructure only; it shares nothing with the
product path.

Notation.  A sequence is a matrix of row vectors x[t].  Every weight is [out, in].  ``st`` arguments carry what a sequence keeps
between calls (GLA: the state matrices; latent attention: the latents and rotated keys; attention: keys, values and the last
projected rows before its convolutions), so a prompt may be fed in portions.
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


def relu(z):
    return np.maximum(z, 0.0)


def dense_mlp(h, p, act=silu):
    """down(act(gate h) * (up h)); the biases are left out where there are none."""
    b = lambda name: p.get(name + ".b", 0.0)
    return (act(h @ p["gate"].T + b("gate")) * (h @ p["up"].T + b("up"))) @ p["down"].T + b("down")


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def short_convolution(u, w, tail):
    """u [T, C] projected rows, w [C, K], tail [K - 1, C] the rows before u (zeros in front of a sequence): y[t] = sum_j w[:, j] *
    u[t - (K - 1) + j].  Returns (y, the new tail)."""
    taps = w.shape[1]
    line = np.concatenate([tail, u])
    y = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * line[t + j]
    return y, line[line.shape[0] - (taps - 1):]


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, np.float64) + 1.0) / every) + 1.0)


def distance_slopes(heads):
    return 2.0 ** (-8.0 * (np.arange(heads) + 1.0) / heads)


def window_attention(q, k, v, first, window, scale, slopes):
    """q [T, H, D] at positions first, first + 1, ...; k [n, G, D], v [n, G, V] of positions 0 .. n - 1; head h reads key/value head
    h // (H / G).  Position i sees the last ``window`` positions up to i itself; score = q . k * scale - slope_h * (i - j)."""
    H, G = q.shape[1], k.shape[1]
    out = np.zeros((q.shape[0], H, v.shape[2]), q.dtype)
    for t in range(q.shape[0]):
        i = first + t
        seen = np.arange(max(0, i - window + 1), i + 1)
        for h in range(H):
            g = h // (H // G)
            s = k[seen, g] @ q[t, h] * scale - slopes[h] * (i - seen)
            w = np.exp(s - s.max())
            out[t, h] = (w / w.sum()) @ v[seen, g]
    return out


def attention_mixer(h, p, m, st, source):
    """st: {"n": positions seen, "tails": {"q" | "k" | "v": rows}, "k": [n, G, D], "v": [n, G, V]}; source: the state whose keys and
    values are read (st itself, or that of the layer named by "kv_from", which has run on the same tokens)."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    first = st["n"]

    def projected(name):
        y, st["tails"][name] = short_convolution(h @ p[name].T, p[name + ".conv"], st["tails"][name])
        return y

    q = projected("q").reshape(T, H, D) * query_temperature(first + np.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    if source is st:
        st["k"] = np.concatenate([st["k"], projected("k").reshape(T, G, D)])
        st["v"] = np.concatenate([st["v"], projected("v").reshape(T, G, V)])
    st["n"] = first + T
    o = window_attention(q, source["k"], source["v"], first, m["mask"]["size"], m["scale"], distance_slopes(H))
    return (o.reshape(T, H * V) * sigmoid(h @ p["g"].T)) @ p["o"].T


def token_side(x, e, p, eps):
    """The per-layer token input: e [T, dim] is the layer's part of the tokens' rows in the side table."""
    y = (gelu_tanh(x @ p["gate"].T) * e) @ p["proj"].T
    return x + rms_norm(y, p["norm"], eps)


# How the layers of an architecture join the residual stream: "parallel" or "post" (the norm behind the sublayer), the activation of the
# feed-forward, whether the head is the embedding table, and whether the stream starts scaled and takes per-layer token inputs
DESIGNS = {"Tolevik": dict(block="post", act=silu, tied=False, token_side=False, embedding_scale=False),
           "Bulidra": dict(block="parallel", act=relu, tied=True, token_side=True, embedding_scale=True)}


class LayeredOracle:
    """config: the dictionary of config.json; params: {tensor name: array}.  ``feed`` runs the next tokens of the sequence."""

    def __init__(self, config, params, dtype=np.float64):
        self.c, self.dtype, self.design = config, dtype, DESIGNS[config["architecture"]]
        self.p = {k: np.asarray(v, dtype) for k, v in params.items()}
        self.reset()

    def reset(self):
        self.states = []
        for la in self.c["layers"]:
            m = la["mixer"]
            if la["type"] == "gla":
                self.states.append(np.zeros((m["heads"], m["dim"], m["vdim"]), self.dtype))
            elif la["type"] == "attention":
                G, D, V = m["kv_heads"], m["dim"], m["vdim"]
                self.states.append({"n": 0, "k": np.zeros((0, G, D), self.dtype), "v": np.zeros((0, G, V), self.dtype),
                                    "tails": {n: np.zeros((m["conv"] - 1, c), self.dtype) for n, c in (("q", m["heads"] * D), ("k", G * D), ("v", G * V))}})
            elif la["type"] == "latent_attention":
                self.states.append({"c": np.zeros((0, m["kv_rank"]), self.dtype), "kr": np.zeros((0, m["rot_dim"]), self.dtype)})
            else:
                raise ValueError(la["type"])

    def _sub(self, prefix):
        n = len(prefix)
        return {k[n:]: v for k, v in self.p.items() if k.startswith(prefix)}

    def _mix(self, i, h):
        la, eps = self.c["layers"][i], self.c["norm"]["eps"]
        m, p, st = la["mixer"], self._sub(f"l{i}.mix."), self.states[i]
        if la["type"] == "gla":
            return gla_mixer(h, p, m, eps, st)
        if la["type"] == "latent_attention":
            return latent_attention_mixer(h, p, m, eps, st)
        return attention_mixer(h, p, m, st, self.states[m["kv_from"]] if "kv_from" in m else st)

    def feed(self, tokens, taps=None):
        eps, d, tokens = self.c["norm"]["eps"], self.design, np.asarray(tokens)
        x = self.p["embed"][tokens]
        if d["embedding_scale"]:
            x = x * self.c["embedding"]["scale"]
        for i, la in enumerate(self.c["layers"]):
            mlp = None if la["mlp"] is None else (lambda h: dense_mlp(h, self._sub(f"l{i}.mlp."), d["act"]))
            if d["block"] == "parallel":
                h = rms_norm(x, self.p[f"l{i}.norm1"], eps)
                x = x + self._mix(i, h) + (mlp(h) if mlp else 0.0)
            else:
                x = x + rms_norm(self._mix(i, x), self.p[f"l{i}.norm1"], eps)
                if mlp:
                    x = x + rms_norm(mlp(x), self.p[f"l{i}.norm2"], eps)
            if d["token_side"]:
                n = self.c["token_side"]["dim"]
                x = token_side(x, self.p["side.embed"][tokens][:, i * n:(i + 1) * n], self._sub(f"l{i}.side."), eps)
            if taps is not None:
                taps.append(x)
        return rms_norm(x, self.p["final.norm"], eps) @ self.p["embed" if d["tied"] else "head"].T
