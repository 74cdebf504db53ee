"""Models built from a list of layers, the parts that need no GPU: configuration reading, the architecture registry, trace replay over a
stand-in model, and the plain implementation's own consistency (its portions and states, known answers of its mechanisms)."""
import io
import json
import os

import numpy as np
import pytest

from layered_models import bf16, config, gla, latent, parallel_config, params, row_errors, shapes_of, window
from oracle import layered as O
from sptorch_b200 import registry, trace
from sptorch_b200.backend import HalError
from sptorch_b200.layered import PARALLEL, RELU, ConfigError, layer_configs, layered_options


def test_layer_configs_read_every_size_and_constant():
    cfg = config([gla(heads=3, dim=20, vdim=28, tau=5.0), latent(heads=5, dim=36, vdim=44, kv_rank=60, q_rank=28, rot_dim=12, rope_dims=8, base=77.0, ff=90)])
    a, b = layer_configs(cfg, {"l0.mix.a1": (11, 72)})
    assert (a.mixer, a.heads, a.dim, a.vdim, a.decay_rank, a.tau, a.mlp) == (0, 3, 20, 28, 11, 5.0, 0)
    assert (b.mixer, b.heads, b.dim, b.vdim, b.kv_rank, b.q_rank, b.rot_dim, b.rope_dims, b.rope_base, b.mlp, b.d_ff) == (1, 5, 36, 44, 60, 28, 12, 8, 77.0, 1, 90)
    assert abs(b.scale - 48 ** -0.5) < 1e-7
    cfg["layers"][0]["mixer"]["decay_rank"] = 4
    assert layer_configs(cfg)[0].decay_rank == 4            # without tensors the configuration may name it


def test_layer_configs_refuse_what_they_do_not_know():
    for change in ({"type": "other"}, {"mlp": {"kind": "sparse", "ff": 8}}, {"mixer": {"heads": 2}}):
        cfg = config([dict(gla(), **change)])
        with pytest.raises(ConfigError):
            layer_configs(cfg, {"l0.mix.a1": (4, 72)})
    with pytest.raises(ConfigError):
        layer_configs(config([gla()]))                      # the decay rank is nowhere


def test_registry_chooses_by_architecture(tmp_path):
    assert set(registry.ARCHITECTURES) == {"GPT", "QwenLikeGPT", "Tolevik", "Bulidra"}
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ConfigError):
        registry.read_config(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps(config([gla()])))
    assert registry.read_config(str(tmp_path))["width"] == 72


class _Recorder:
    """Stands in for a device model: "logits" of a token are (token, position)."""

    def __init__(self):
        self.cfg, self.seen, self.resets = {"vocab": 2}, [], 0

    def enable_kv_cache(self): pass

    def reset_cache(self):
        self.seen, self.resets = [], self.resets + 1

    def extend_device(self, ids):
        start = len(self.seen)
        self.seen += [int(t) for t in ids[0]]
        return np.array([[t, start + i] for i, t in enumerate(ids[0])], np.float32)

    def read_logit_rows(self, rows, want):
        return rows[list(want)].reshape(len(want), 2)


def test_replay_answers_every_step_and_writes_only_what_is_wanted(tmp_path):
    m, said = _Recorder(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [8], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": ["b"]}]
    trace.replay(m, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"]
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32"]
    assert np.fromfile(tmp_path / "0.f32", "<f4").reshape(-1, 2).tolist() == [[5, 0], [7, 2]]
    assert np.fromfile(tmp_path / "2.f32", "<f4").reshape(-1, 2).tolist() == [[9, 0]]      # the second request starts at position 0
    with pytest.raises(HalError):
        trace.replay(m, io.StringIO("".join(json.dumps({"step": i, "entries": [{"id": i, "tokens": [1], "want": []}]}) + "\n" for i in (0, 1))), str(tmp_path), said.append)


def test_plain_implementation_known_answers():
    assert np.allclose(O.rms_norm(np.array([3.0, 4.0]), np.array([1.0, 2.0]), 0.0), np.array([3.0, 8.0]) / np.sqrt(12.5))
    x = np.zeros((2, 1, 6)); x[:, 0, 0] = 1.0; x[:, 0, 3] = 2.0; x[:, 0, 5] = 7.0
    y = O.rotate_pairs(x, [0, 3], 100.0, 4)                  # pairs (0, 1) and (2, 3); the last two entries pass
    assert np.allclose(y[0], x[0]) and np.allclose(y[1, 0], [np.cos(3), np.sin(3), -2 * np.sin(0.3), 2 * np.cos(0.3), 0, 7])
    s = np.zeros((1, 2, 1))
    o = O.gla_recurrence(np.ones((3, 1, 2)), np.array([[[1.0, 0]], [[0, 1.0]], [[0, 0]]]), np.array([[[4.0]], [[8.0]], [[0.0]]]),
                         np.broadcast_to(np.array([0.5, 1.0]), (3, 1, 2)), s)
    assert o[:, 0, 0].tolist() == [4.0, 10.0, 9.0] and s[0, :, 0].tolist() == [1.0, 8.0]
    z = np.array([-30.0, 0.0, 30.0])
    assert np.allclose(O.log_sigmoid(z), [-30.0, np.log(0.5), 0.0], atol=1e-12)


def test_plain_implementation_does_not_depend_on_portions():
    cfg = config([gla(), latent(sharp=3.0, ff=40), gla(ff=24), latent()])
    p = params(cfg, 3)
    ids = np.random.default_rng(0).integers(0, cfg["vocab"], 41)
    whole = O.LayeredOracle(cfg, p).feed(ids)
    m = O.LayeredOracle(cfg, p)
    cut = np.concatenate([m.feed(ids[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 22), (22, 41))])
    assert np.abs(whole - cut).max() < 1e-9
    assert set(shapes_of(cfg)) == set(p) and all(np.array_equal(bf16(v), v) for v in p.values())


def test_window_configs_read_every_size_and_constant():
    cfg = parallel_config([window(heads=6, kv_heads=3, dim=20, vdim=28, size=77, conv=5, coef=0.25, every=33, ff=90), window(heads=6, kv_heads=3, dim=20, vdim=28, size=9, conv=2, kv_from=0)],
                          side=14, scale=2.5)
    a, b = layer_configs(cfg)
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.conv_taps, a.q_temp_coef, a.q_temp_every) == (2, 6, 3, 20, 28, 77, 5, 0.25, 33.0)
    assert (a.mlp, a.d_ff, a.mlp_act, a.mlp_bias, a.kv_shared, a.distance_bias, a.out_gate) == (1, 90, RELU, 0, 0, 1, 1)
    assert (b.window, b.conv_taps, b.mlp, b.kv_shared, b.kv_from) == (9, 2, 0, 1, 0) and abs(b.scale - 2 * 20 ** -0.5) < 1e-7
    o = layered_options(cfg)
    assert (o.block, o.tied_head, o.side_dim, o.embed_scale) == (PARALLEL, 1, 14, 2.5)
    o = layered_options(config([gla()]))
    assert (o.block, o.tied_head, o.side_dim, o.embed_scale) == (0, 0, 0, 1.0)


def test_window_configs_refuse_what_they_do_not_know():
    for layers in ([gla()], [window(kv_from=0)], [window(), window(kv_from=1)], [window(size=0)], [window(every=0)], [dict(window(), mlp={"kind": "dense"})], [dict(window(), mlp={"kind": "sparse", "ff": 3})]):
        with pytest.raises(ConfigError):
            layer_configs(parallel_config(layers))
    for missing in ("heads", "kv_heads", "dim", "vdim", "scale"):
        la = window()
        del la["mixer"][missing]
        with pytest.raises(ConfigError):
            layer_configs(parallel_config([la]))
    for missing in ("embedding", "token_side"):
        cfg = parallel_config([window()])
        del cfg[missing]
        with pytest.raises(ConfigError):
            layered_options(cfg)
    with pytest.raises(ConfigError):
        layer_configs(config([window()]))                   # not one of that design's mixers


def test_plain_window_attention_known_answers():
    y, tail = O.short_convolution(np.array([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]]), np.array([[0.5, 1.0, 2.0], [0.0, 1.0, 0.0]]), np.zeros((2, 2)))
    assert y.tolist() == [[2.0, 0.0], [5.0, 10.0], [8.5, 20.0]] and tail.tolist() == [[2.0, 20.0], [3.0, 30.0]]
    y, tail = O.short_convolution(np.array([[4.0, 40.0]]), np.array([[0.5, 1.0, 2.0], [0.0, 1.0, 0.0]]), tail)
    assert y.tolist() == [[12.0, 30.0]] and tail.tolist() == [[3.0, 30.0], [4.0, 40.0]]
    assert np.allclose(O.query_temperature([0, 6, 7, 14, 15], 0.5, 8), 1 + 0.5 * np.log([1, 1, 2, 2, 3]))
    assert O.distance_slopes(4).tolist() == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8] and np.allclose(O.distance_slopes(3), [2 ** (-8 / 3), 2 ** (-16 / 3), 2.0 ** -8])
    # zero queries: the weights are those of the distance alone, over exactly the window
    v = np.eye(5)[:, None, :]
    o = O.window_attention(np.zeros((2, 2, 3)), np.ones((5, 1, 3)), v, 3, 3, 1.0, np.array([0.0, np.log(2.0)]))
    assert np.allclose(o[0, 0], [0, 1 / 3, 1 / 3, 1 / 3, 0]) and np.allclose(o[1, 0], [0, 0, 1 / 3, 1 / 3, 1 / 3])
    assert np.allclose(o[0, 1], np.array([0, 1, 2, 4, 0]) / 7) and np.allclose(o[1, 1], np.array([0, 0, 1, 2, 4]) / 7)
    # head h reads key/value head h // (H / G)
    o = O.window_attention(np.zeros((1, 4, 1)), np.zeros((1, 2, 1)), np.array([[[1.0], [2.0]]]), 0, 1, 1.0, np.zeros(4))
    assert o[0, :, 0].tolist() == [1, 1, 2, 2]
    x = O.token_side(np.array([[1.0, 2.0]]), np.array([[3.0]]), {"gate": np.array([[0.0, 1.0]]), "proj": np.array([[1.0], [1.0]]), "norm": np.array([1.0, 10.0])}, 0.0)
    assert np.allclose(x, [[2.0, 12.0]])
    assert np.allclose(O.gelu_tanh(np.array([-9.0, 0.0, 9.0])), [0, 0, 9]) and O.relu(np.array([-1.0, 2.0])).tolist() == [0.0, 2.0]


def test_plain_parallel_model_does_not_depend_on_portions():
    cfg = parallel_config([window(ff=24), window(size=9, conv=4), window(kv_from=0, size=80, conv=2, ff=30), window(size=1, conv=1)])
    p = params(cfg, 3)
    ids = np.random.default_rng(0).integers(0, cfg["vocab"], 61)
    whole = O.LayeredOracle(cfg, p).feed(ids)
    m = O.LayeredOracle(cfg, p)
    cut = np.concatenate([m.feed(ids[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 22), (22, 61))])
    assert np.abs(whole - cut).max() < 1e-9
    assert set(shapes_of(cfg)) == set(p) and all(np.array_equal(bf16(v), v) for v in p.values())


@pytest.mark.parametrize("name", ["convolution", "window edge", "distance bias", "temperature", "head groups", "output gate", "key and value source", "token input", "embedding scale"])
def test_every_mechanism_shows(name):
    """A mistake planted in the plain implementation moves the logits by a hundred times the tolerance of the 32-bit device tests (3e-5)."""
    cfg = parallel_config([window(ff=40), window(size=20), window(kv_from=0, coef=0.8)])
    p = params(cfg, 5)
    ids = np.random.default_rng(1).integers(0, cfg["vocab"], 60)
    ref = O.LayeredOracle(cfg, p).feed(ids)
    wrong, q = json.loads(json.dumps(cfg)), dict(p)
    if name == "convolution":
        q["l0.mix.k.conv"] = np.roll(p["l0.mix.k.conv"], 1, 1)
    elif name == "window edge":
        wrong["layers"][1]["mixer"]["mask"]["size"] = 21
    elif name == "distance bias":
        q["l0.mix.q"] = np.concatenate([p["l0.mix.q"][32:64], p["l0.mix.q"][:32], p["l0.mix.q"][64:]])      # heads 0 and 1 exchange slopes
    elif name == "temperature":
        wrong["layers"][2]["mixer"]["q_temp"]["every"] = 21
    elif name == "head groups":
        q["l0.mix.k"] = np.roll(p["l0.mix.k"], 32, 0)
    elif name == "output gate":
        q["l1.mix.g"] = 0 * p["l1.mix.g"]
    elif name == "key and value source":
        wrong["layers"][2]["mixer"]["kv_from"] = 1
    elif name == "token input":
        q["side.embed"] = np.roll(p["side.embed"], 12, 1)
    else:
        wrong["embedding"]["scale"] = 3.3
    moved = row_errors(O.LayeredOracle(wrong, q).feed(ids), ref)
    assert moved.max() > 3e-3
