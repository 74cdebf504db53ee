"""Models built from a list of layers (architectures "Tolevik" and "Bulidra"): configuration reading and the device model.  The layers
of one model may differ in mixer (gated linear attention, latent attention, window attention), sizes and feed-forward; csrc/layered.cu
runs them."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import numpy as np

from . import _lib
from .backend import BF16, F32, FfiBackend, HalError
from .gpt import GPT, _lib_view

ARCH_LAYERED = 2
MIXERS = {"gla": 0, "latent_attention": 1, "attention": 2}
GLA, LATENT, WINDOW = 0, 1, 2
MLPS = {None: 0, "dense": 1}
POST_NORM, PARALLEL = 0, 1
SILU, RELU = 0, 1


@dataclass(frozen=True)
class Design:
    """What an architecture fixes; everything else is read from its configuration."""
    mixers: tuple
    block: int
    mlp_act: int
    mlp_bias: bool
    tied_head: bool
    token_side: bool = False            # a per-layer token input, of the width config names
    embedding_scale: bool = False
    distance_bias: bool = False         # window attention: geometric slopes
    out_gate: bool = False              # ... sigmoid gate on the heads, element by element


DESIGNS = {
    "Tolevik": Design(("gla", "latent_attention"), POST_NORM, SILU, True, False),
    "Bulidra": Design(("attention",), PARALLEL, RELU, False, True, token_side=True, embedding_scale=True, distance_bias=True, out_gate=True),
}


class ConfigError(ValueError):
    """A configuration this framework cannot run, with the reason."""


def _need(d: dict, key: str, where: str):
    if key not in d:
        raise ConfigError(f"{where}: '{key}' is missing")
    return d[key]


def design_of(config: dict) -> Design:
    arch = config.get("architecture")
    if arch not in DESIGNS:
        raise ConfigError(f"config: architecture {arch!r} is not built from a list of layers")
    return DESIGNS[arch]


def _gla_config(c, m, i, where, shapes):
    c.tau = float(_need(m, "tau", where))
    name = f"l{i}.mix.a1"
    if shapes is not None and name in shapes:
        c.decay_rank = int(shapes[name][0])
    else:
        c.decay_rank = int(_need(m, "decay_rank", where))


def _latent_config(c, m, where):
    rot = _need(m, "rot", where)
    c.kv_rank, c.q_rank, c.rot_dim = (int(_need(m, k, where)) for k in ("kv_rank", "q_rank", "rot_dim"))
    c.rope_dims, c.rope_base = int(_need(rot, "dims", where)), float(_need(rot, "base", where))
    c.scale = float(_need(m, "scale", where))


def _window_config(c, m, i, where, design):
    c.kv_heads, c.scale = int(_need(m, "kv_heads", where)), float(_need(m, "scale", where))
    c.window = int(_need(_need(m, "mask", where), "size", where)) if m.get("mask") is not None else 0
    if m.get("mask") is not None and c.window <= 0:
        raise ConfigError(f"{where}: a window of {c.window} positions")
    c.conv_taps = int(m.get("conv") or 0)
    temp = m.get("q_temp")
    if temp is not None:
        c.q_temp_coef, c.q_temp_every = float(_need(temp, "coef", where)), float(_need(temp, "every", where))
        if c.q_temp_every <= 0:
            raise ConfigError(f"{where}: q_temp.every must be positive")
    if m.get("kv_from") is not None:
        c.kv_shared, c.kv_from = 1, int(m["kv_from"])
        if not 0 <= c.kv_from < i:
            raise ConfigError(f"{where}: reads the keys and values of layer {c.kv_from}, which does not come before it")
    c.distance_bias, c.out_gate = int(design.distance_bias), int(design.out_gate)


def layer_configs(config: dict, shapes: dict | None = None) -> list:
    """config.json's list of layers as the library's structures.  A size the file leaves to a tensor's shape (the rank of the decay
    projection) is taken from ``shapes`` {tensor name: shape}, or from the mixer's own "decay_rank"."""
    design, out = design_of(config), []
    for i, la in enumerate(_need(config, "layers", "config")):
        where = f"layer {i}"
        kind, m = _need(la, "type", where), _need(la, "mixer", where)
        if kind not in design.mixers:
            raise ConfigError(f"{where}: unknown mixer '{kind}'")
        c = _lib.LayerConfig()
        c.mixer = MIXERS[kind]
        c.heads, c.dim, c.vdim = (int(_need(m, k, where)) for k in ("heads", "dim", "vdim"))
        if kind == "gla":
            _gla_config(c, m, i, where, shapes)
        elif kind == "latent_attention":
            _latent_config(c, m, where)
        else:
            _window_config(c, m, i, where, design)
        mlp = la.get("mlp")
        mlp_kind = None if mlp is None else _need(mlp, "kind", where)
        if mlp_kind not in MLPS:
            raise ConfigError(f"{where}: unknown feed-forward '{mlp_kind}'")
        c.mlp = MLPS[mlp_kind]
        c.d_ff = int(_need(mlp, "ff", where)) if mlp is not None else 0
        c.mlp_act, c.mlp_bias = design.mlp_act, int(design.mlp_bias)
        out.append(c)
    return out


def layered_options(config: dict):
    design = design_of(config)
    o = _lib.LayeredOptions()
    o.block, o.tied_head, o.embed_scale = design.block, int(design.tied_head), 1.0
    if design.embedding_scale:
        o.embed_scale = float(_need(_need(config, "embedding", "config"), "scale", "embedding"))
    if design.token_side:
        o.side_dim = int(_need(_need(config, "token_side", "config"), "dim", "token_side"))
    return o


class LayeredGPT(GPT):
    """The device model behind the same surface as GPT: ``forward``, ``generate``, the cache calls and weight files.  A sequence's
    cache holds a row per position for every layer of latent attention and of window attention with keys of its own (and the last
    projected rows its convolutions look back at), and one state matrix per head for every gated linear attention layer, so a prompt
    may arrive in portions of any size (``extend``)."""

    def __init__(self, backend: FfiBackend, config: dict, seq_len: int, dtype: int = BF16, max_batch: int = 1, shapes: dict | None = None):
        self.b, self.config = backend, config
        layers = layer_configs(config, shapes)
        vocab, width = int(_need(config, "vocab", "config")), int(_need(config, "width", "config"))
        self.cfg = dict(vocab=vocab, d_model=width, n_layer=len(layers), seq_len=seq_len)
        self.dtype, self.max_batch, self.arch = dtype, max_batch, ARCH_LAYERED
        self.layers = layers
        c = _lib.GptConfig(vocab, width, len(layers), 1, 1, seq_len, dtype, max_batch, float(_need(_need(config, "norm", "config"), "eps", "norm")), 0, 1, ARCH_LAYERED, 0.0)
        arr = (_lib.LayerConfig * max(len(layers), 1))(*layers)
        self.options = layered_options(config)
        self.h = backend.lib.sptorch_ext_layered_create(C.byref(c), arr, len(layers), C.byref(self.options))
        if not self.h:
            raise HalError("layered_create failed: " + _lib.last_error())
        self.ldl = backend.lib.sptorch_ext_gpt_logits_ld(self.h)
        self.es = 2 if dtype == BF16 else 4
        self._logits = self._ids = self._gen_ctx = None
        self._prompt_len = 0
        self.kv_cache_enabled = False

    def named_parameters(self):
        from .weights import model_parameters
        return model_parameters(self)

    def tap(self, i: int, n_tokens: int) -> np.ndarray:
        """The residual stream (f32 in both dtypes) after the embedding (0) and after layer i - 1, of the last step's tokens."""
        p = self.b.lib.sptorch_ext_gpt_tap(self.h, i)
        if not p:
            raise HalError("taps are not enabled")
        raw = np.empty(n_tokens * self.cfg["d_model"], np.float32)
        self.b._check(self.b.lib.sptorch_ext_copy_d2h_bytes(p, raw.ctypes.data, raw.nbytes), "tap d2h")
        return raw.reshape(n_tokens, -1)

    def forward(self, ids: np.ndarray) -> np.ndarray:
        """ids [B, T] -> logits [B, T, V] float32 on the host; any T up to seq_len."""
        ids = np.asarray(ids)
        B, T = ids.shape
        if T > self.cfg["seq_len"]:
            raise HalError("sequence longer than seq_len")
        d_ids, d_log = self.stage_ids(ids), self.logits_buffer(B * T)
        self.forward_device(d_ids, B, T, d_log)
        return self._read_logits(d_log, B * T).reshape(B, T, -1)

    def decode_logits_from_cache(self, last_ids):
        raise HalError("the recurrent state already holds the last token: its logits cannot be recomputed from the cache")

    def _last_logits_device(self, context):
        """Logits of the last token of ``context`` as a device row: one decode step while the context only grew by one token,
        otherwise a fresh prefill."""
        n = len(context)
        grew_by_one = self._gen_ctx is not None and n == len(self._gen_ctx) + 1 and list(context[:-1]) == self._gen_ctx
        d_log = self.logits_buffer(n)
        if grew_by_one and self.cached_len() == n - 1:
            d_ids, row = self.stage_ids(np.asarray(context[-1:])), 0
            self.b._check(self.b.lib.sptorch_ext_gpt_decode(self.h, d_ids.handle, 1, 1, d_log.handle), "gpt_decode")
        else:
            d_ids, row = self.stage_ids(np.asarray(context)), n - 1
            self.b._check(self.b.lib.sptorch_ext_gpt_prefill(self.h, d_ids.handle, 1, n, d_log.handle), "gpt_prefill")
        self._gen_ctx = list(context)
        return _lib_view(self.b, d_log, row * self.ldl, self.ldl, self.es)
