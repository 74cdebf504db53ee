"""Small configurations and random weights of models built from a list of layers, for the tests (the product reads such models from
files).  Weights are drawn so that a fault shows: peaked attention (a wrong or missing key changes the output), decays between
nearly one and a few tokens of memory, norm weights and biases away from one and zero."""
import numpy as np

from sptorch_b200.backend import bf16_bits_to_f32, f32_to_bf16_bits


def bf16(x):
    x = np.asarray(x, np.float32)
    return bf16_bits_to_f32(f32_to_bf16_bits(x)).reshape(x.shape)


def gla(heads=2, dim=24, vdim=40, tau=8.0, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def latent(heads=3, dim=32, vdim=24, kv_rank=56, q_rank=40, rot_dim=16, rope_dims=None, base=5000.0, sharp=1.0, ff=None):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot_dim": rot_dim,
                      "rot": {"base": base, "dims": rot_dim if rope_dims is None else rope_dims}, "scale": sharp * (dim + rot_dim) ** -0.5}}


def window(heads=4, kv_heads=2, dim=32, vdim=24, size=50, conv=3, coef=0.4, every=20, sharp=2.0, ff=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": size}, "q_temp": {"coef": coef, "every": every}, "scale": sharp * dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=72, vocab=150, eps=1e-5):
    return {"architecture": "Tolevik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def parallel_config(layers, width=72, vocab=150, eps=1e-5, side=12, scale=3.0, architecture="Bulidra"):
    return {"architecture": architecture, "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width}


def shapes_of(cfg, decay_rank=7):
    d, parallel, side = cfg["width"], "embedding" in cfg, cfg.get("token_side", {"dim": 0})["dim"]
    s = {"embed": (cfg["vocab"], d)}
    if side and cfg["layers"]:
        s["side.embed"] = (cfg["vocab"], len(cfg["layers"]) * side)
    for i, la in enumerate(cfg["layers"]):
        m, p = la["mixer"], f"l{i}."
        H, D, V = m["heads"], m["dim"], m["vdim"]
        s[p + "norm1"] = (d,)
        if la["mlp"] is not None and not parallel:
            s[p + "norm2"] = (d,)
        if la["type"] == "gla":
            s.update({p + "mix.q": (H * D, d), p + "mix.k": (H * D, d), p + "mix.v": (H * V, d), p + "mix.g": (H * V, d), p + "mix.o": (d, H * V),
                      p + "mix.norm": (V,), p + "mix.a1": (decay_rank, d), p + "mix.a2": (H * D, decay_rank), p + "mix.a2.b": (H * D,)})
        elif la["type"] == "attention":
            rows = {"q": H * D} if "kv_from" in m else {"q": H * D, "k": m["kv_heads"] * D, "v": m["kv_heads"] * V}
            s.update({p + "mix." + n: (r, d) for n, r in rows.items()})
            s.update({p + "mix." + n + ".conv": (r, m["conv"]) for n, r in rows.items()})
            s.update({p + "mix.g": (H * V, d), p + "mix.o": (d, H * V)})
        else:
            R, K, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            s.update({p + "mix.dq": (Q, d), p + "mix.dq.norm": (Q,), p + "mix.uq": (H * (D + R), Q), p + "mix.dkv": (K + R, d), p + "mix.dkv.norm": (K,),
                      p + "mix.uk": (H * D, K), p + "mix.uv": (H * V, K), p + "mix.g": (H, d), p + "mix.o": (d, H * V)})
        if la["mlp"] is not None and parallel:
            F = la["mlp"]["ff"]
            s.update({p + "mlp.gate": (F, d), p + "mlp.up": (F, d), p + "mlp.down": (d, F)})
        elif la["mlp"] is not None:
            F = la["mlp"]["ff"]
            s.update({p + "mlp.gate": (F, d), p + "mlp.gate.b": (F,), p + "mlp.up": (F, d), p + "mlp.up.b": (F,), p + "mlp.down": (d, F), p + "mlp.down.b": (d,)})
        if side:
            s.update({p + "side.gate": (side, d), p + "side.proj": (d, side), p + "side.norm": (d,)})
    s["final.norm"] = (d,)
    if not parallel:
        s["head"] = (cfg["vocab"], d)
    return s


def params(cfg, seed=0, decay_rank=7):
    """{name: f32 array}, every value exact in bf16."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes_of(cfg, decay_rank).items():
        w = rng.standard_normal(shape)
        if name.endswith(".a2.b"):
            w = 1.5 + 2.0 * w                         # slow and fast decays side by side
        elif len(shape) == 1:
            w = 0.3 * w + (0.0 if name.endswith(".b") else 1.0)
        elif name.endswith(".conv"):
            w = 0.4 * w
            w[:, -1] += 1.0
        elif name not in ("embed", "side.embed"):
            w = w * shape[1] ** -0.5
        if name.endswith(("mix.dkv", "mix.dq")):
            w = 2.0 * w
        out[name] = bf16(w.astype(np.float32))
    return out


def row_errors(got, ref):
    """Per position: root mean square over the vocabulary of the difference, mean taken off, against that of the reference."""
    got, ref = np.asarray(got, np.float64).reshape(-1, np.shape(got)[-1]), np.asarray(ref, np.float64).reshape(-1, np.shape(ref)[-1])
    d = got - ref
    d -= d.mean(-1, keepdims=True)
    r = ref - ref.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean())
