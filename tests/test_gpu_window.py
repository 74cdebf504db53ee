"""Parallel blocks with window attention, short convolutions, shared keys and values and per-layer token inputs on the device, against the
plain implementation in oracle/layered.py: each mechanism alone, the window's edges, prompts, portions, decoding, batches, reuse of the
cache, sizes the kernels' vectors and tiles do not divide, and generation through the framework's own loop."""
import io
import json

import numpy as np
import pytest

from conftest import parity_record
from layered_models import bf16, config, gla, latent, parallel_config, params, row_errors, shapes_of, window
from oracle import layered as O
from oracle.layered import LayeredOracle
from sptorch_b200 import generate, layered, trace, weights
from sptorch_b200.backend import BF16, EPI_GELU_MUL, EPI_RELU_MUL, F32, MM_BF16, MM_F32, HalError
from sptorch_b200.kv_cache import layer_specs
from sptorch_b200.layered import LayeredGPT
from sptorch_b200.registry import load_model
from weight_files import write_safetensors

pytestmark = pytest.mark.gpu
# per position, against the f64 oracle: f32 is rounding alone, bf16 the rounding of the operands of every product
TOL = {F32: 3e-5, BF16: 4e-2}
DTYPES = [F32, BF16]
IDS = ["f32", "bf16"]


def _model(backend, cfg, p, dtype, seq_len=1024, max_batch=1):
    m = LayeredGPT(backend, cfg, seq_len, dtype=dtype, max_batch=max_batch, shapes=shapes_of(cfg))
    for k, v in p.items():
        m.set_param(k, v)
    m.enable_kv_cache()
    return m


def _ids(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def _check(got, ref, dtype, what, factor=1.0):
    """Every position within the tolerance in f32; in bf16 at least 95 of 100, and none beyond three times."""
    e, tol = row_errors(got, ref), factor * TOL[dtype]
    assert e.max() <= (tol if dtype == F32 else 3 * tol) and np.quantile(e, 0.95) <= tol, f"{what}: {np.quantile(e, 0.95):.3e}, {e.max():.3e} at position {int(e.argmax())}"
    return float(e.max())


def _feed(m, ids, cuts):
    m.reset_cache()
    out, at = [], 0
    for n in cuts:
        out.append(m.extend(np.asarray(ids[at:at + n]).reshape(1, -1))[0])
        at += n
    assert at == len(ids)
    return np.concatenate(out)


# windows of several sizes, two layers on the keys and values of earlier ones, one of them with a wider window than its source
MIXED = parallel_config([window(size=40, ff=88), window(heads=6, kv_heads=2, dim=40, vdim=32, size=130, conv=4, ff=56), window(heads=3, kv_heads=3, dim=24, vdim=16, size=17, conv=2),
                         window(heads=6, kv_heads=2, dim=40, vdim=32, size=300, conv=2, kv_from=1, ff=72), window(heads=3, kv_heads=3, dim=24, vdim=16, size=70, conv=3, kv_from=2)], width=104)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name,layers,extra", [
    ("attention", [window()], {}), ("feed-forward", [window(ff=100)], {}), ("one head", [window(heads=1, kv_heads=1)], {}), ("a key per head", [window(heads=4, kv_heads=4)], {}),
    ("twenty heads on one key", [window(heads=20, kv_heads=1, dim=16, vdim=16)], {}), ("window of one", [window(size=1)], {}), ("window of two", [window(size=2)], {}),
    ("window beyond the prompt", [window(size=4000)], {}), ("window as long as the prompt", [window(size=150)], {}), ("one tap", [window(conv=1)], {}), ("two taps", [window(conv=2)], {}),
    ("six taps", [window(conv=6)], {}), ("hot queries", [window(coef=1.5, every=3)], {}), ("temperature out of reach", [window(coef=5.0, every=1000)], {}), ("peaked", [window(sharp=8.0)], {}),
    ("shared keys and values", [window(), window(kv_from=0)], {}), ("shared, another window", [window(size=9, conv=2), window(size=60, conv=4, kv_from=0, coef=1.0)], {}),
    ("two readers of one layer", [window(), window(size=20), window(kv_from=0, size=30), window(kv_from=0)], {}), ("wide token input", [window()], {"side": 40}),
    ("token input of one", [window()], {"side": 1}), ("embedding scale", [window()], {"scale": 0.5}), ("large eps", [window(ff=40)], {"eps": 0.3}), ("no layer", [], {})])
def test_each_mechanism_alone(backend, dtype, name, layers, extra):
    """The residual stream behind the embedding and behind every layer, and the logits, of one prompt and of a prompt cut in two."""
    cfg = parallel_config(layers, **extra)
    p = params(cfg, 5)
    ids = _ids(cfg, 150)
    taps = []
    ref = LayeredOracle(cfg, p).feed(ids, taps)
    m = _model(backend, cfg, p, dtype)
    m.enable_taps()
    out = m.prefill_kv_cache(ids.reshape(1, -1))[0]
    assert np.array_equal(m.tap(0, len(ids)), (p["embed"][ids] * np.float32(cfg["embedding"]["scale"])).astype(np.float32))
    for i, t in enumerate(taps):
        _check(m.tap(i + 1, len(ids)), t, dtype, f"{name}: layer {i}")
    parity_record(f"window, {name}, {IDS[dtype]}", worst=_check(out, ref, dtype, name))
    m.close()
    m = _model(backend, cfg, p, dtype)                              # without taps, where norms ride along with projections
    _check(m.forward(ids.reshape(1, -1))[0], ref, dtype, f"{name}, without a cache")
    _check(_feed(m, ids, [120, 17, 2, 5] + [1] * 6), ref, dtype, f"{name}, portions")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width,vocab,side,layers", [
    (50, 33, 5, [window(heads=3, kv_heads=3, dim=10, vdim=14, size=25, conv=5, ff=52), window(heads=3, kv_heads=3, dim=10, vdim=14, size=60, kv_from=0)]),
    (33, 130, 3, [window(heads=2, kv_heads=1, dim=7, vdim=5, size=11, conv=2, ff=3), window(heads=1, kv_heads=1, dim=3, vdim=9, size=3, conv=1, ff=1)]),
    (264, 700, 24, [window(heads=5, kv_heads=1, dim=136, vdim=144, size=33, conv=4, ff=136), window(heads=4, kv_heads=2, dim=72, vdim=200, size=77), window(heads=2, kv_heads=1, dim=160, vdim=24, size=128, ff=20)]),
    (88, 96, 8, [window(heads=18, kv_heads=1, dim=8, vdim=8, size=100, ff=8), window(heads=34, kv_heads=2, dim=16, vdim=24, size=31)])])
def test_other_sizes(backend, dtype, width, vocab, side, layers):
    """Sizes that fit no vector, tile or head size the kernels prefer, prompts and decoding."""
    cfg = parallel_config(layers, width=width, vocab=vocab, side=side, eps=1e-3)
    p = params(cfg, 7)
    ids = _ids(cfg, 141)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, dtype, seq_len=141)
    _check(_feed(m, ids, [130] + [1] * 11), ref, dtype, "prompt, then decoding", 1.5)
    _check(_feed(m, ids, [2, 5, 19, 40, 75]), ref, dtype, "portions", 1.5)
    _check(m.forward(ids.reshape(1, -1))[0], ref, dtype, "without a cache", 1.5)
    m.close()


@pytest.mark.parametrize("layer", [
    window(heads=4, kv_heads=2, dim=64, vdim=64, size=200), window(heads=4, kv_heads=1, dim=48, vdim=128, size=129), window(heads=2, kv_heads=2, dim=96, vdim=40, size=128),
    window(heads=8, kv_heads=2, dim=128, vdim=128, size=300), window(heads=2, kv_heads=1, dim=128, vdim=72, size=127), window(heads=2, kv_heads=1, dim=8, vdim=104, size=5),
    window(heads=4, kv_heads=2, dim=64, vdim=64, size=2000), window(heads=4, kv_heads=2, dim=72, vdim=64, size=1), window(heads=3, kv_heads=1, dim=104, vdim=96, size=256, conv=4)])
def test_every_kernel_shape(backend, layer):
    """bf16: every tile shape the fused attention and the decode kernel are built for, over several tiles of keys, as one prompt, behind a
    cached prefix and in decoding."""
    cfg = parallel_config([layer], width=80)
    p = params(cfg, 53)
    ids = _ids(cfg, 660)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, BF16, seq_len=660)
    for cuts in ([660], [300, 200, 2, 3, 16, 33] + [1] * 6 + [100], [129, 383, 148], [256, 17, 128, 129, 130]):
        _check(_feed(m, ids, cuts), ref, BF16, f"portions {cuts}")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_prompt_portions_and_decoding_agree(backend, dtype):
    """The same tokens as one prompt, token by token and in portions of several sizes: each against the oracle at every position."""
    cfg, p = MIXED, params(MIXED, 11)
    ids = _ids(cfg, 300)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, dtype)
    worst = 0.0
    for what, cuts in (("prompt", [300]), ("token by token", [1] * 300), ("twos", [2] * 150), ("threes", [3] * 100), ("sixteens", [16] * 18 + [12]), ("seventeens", [17] * 17 + [11]),
                       ("sixty-fours", [64] * 4 + [44]), ("mixed", [1, 2, 127, 1, 3, 64, 2, 65, 30, 2, 1, 1, 1]), ("tile edges", [127, 2, 126, 2, 43]), ("130s", [130, 130, 40])):
        worst = max(worst, _check(_feed(m, ids, cuts), ref, dtype, what))
    parity_record(f"window, ten ways to cut 300 tokens, {IDS[dtype]}", worst=worst)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_first_tokens(backend, dtype):
    """Sequences of one to seven tokens: the convolutions reach back behind the start of the sequence, the windows are hardly filled."""
    cfg, p = MIXED, params(MIXED, 12)
    m = _model(backend, cfg, p, dtype)
    for n in range(1, 8):
        ids = _ids(cfg, n, 70 + n)
        ref = LayeredOracle(cfg, p).feed(ids)
        _check(_feed(m, ids, [n]), ref, dtype, f"{n} tokens")
        _check(_feed(m, ids, [1] * n), ref, dtype, f"{n} tokens one by one")
        _check(m.forward(ids.reshape(1, -1))[0], ref, dtype, f"{n} tokens without a cache")
    m.close()


def _needle_params(cfg, p, score):
    """Query tokens (1) look along the key of needle tokens (0) in every head of layer 0, whose convolutions only see the current token;
    scores of other pairs stay small."""
    m = cfg["layers"][0]["mixer"]
    x = p["embed"].astype(np.float64) * cfg["embedding"]["scale"]
    h = x / np.sqrt((x * x).mean(-1, keepdims=True) + cfg["norm"]["eps"]) * p["l0.norm1"]
    D, per = m["dim"], m["heads"] // m["kv_heads"]
    for n in ("q", "k", "v"):
        w = np.zeros_like(p[f"l0.mix.{n}.conv"]); w[:, -1] = 1.0
        p[f"l0.mix.{n}.conv"] = w
    # every other token is orthogonal to what makes a needle or a query
    marks = np.linalg.qr(np.stack([h[0], h[1]], 1))[0]
    wq, wk = 0.05 * p["l0.mix.q"].astype(np.float64), 0.05 * p["l0.mix.k"].astype(np.float64)
    wq -= wq @ marks @ marks.T
    wk -= wk @ marks @ marks.T
    dual = np.linalg.pinv(np.stack([h[0], h[1]], 1))                # dual[0] h[0] = 1, dual[0] h[1] = 0
    rng = np.random.default_rng(9)
    for g in range(m["kv_heads"]):
        u = rng.standard_normal(D); u /= np.linalg.norm(u)
        wk[g * D:(g + 1) * D] += np.outer(u, dual[0]) * np.sqrt(score / m["scale"])
        for hd in range(g * per, (g + 1) * per):
            wq[hd * D:(hd + 1) * D] += np.outer(u, dual[1]) * np.sqrt(score / m["scale"])
    p["l0.mix.q"], p["l0.mix.k"] = bf16(wq), bf16(wk)
    p["l0.mix.o"] = 4.0 * p["l0.mix.o"]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("size,dim,vdim", [(128, 64, 64), (141, 32, 24), (200, 128, 128), (50, 10, 12), (300, 64, 96)])
def test_keys_at_the_windows_edge(backend, dtype, size, dim, vdim):
    """A needle just inside and just outside the window of a query, at several distances from tile borders, in a prompt, in a portion behind
    a cached prefix and in decoding.  The needle takes nearly all of the softmax weight when it is seen."""
    cfg = parallel_config([window(heads=4, kv_heads=2, dim=dim, vdim=vdim, size=size, coef=0.1, every=64, sharp=1.0)], width=64, vocab=64)
    p = params(cfg, 13)
    _needle_params(cfg, p, 60.0 + 0.3 * size)                       # the steepest head takes 2^-2 per position off
    m = _model(backend, cfg, p, dtype, seq_len=700)
    rng = np.random.default_rng(3)
    for query in (size + 3, 383, 384, 511, 640):
        n = query + 3
        for distance in (size - 2, size - 1, size, size + 1):
            if distance > query:
                continue
            ids = rng.integers(2, 64, n); ids[query] = 1; ids[query - distance] = 0
            ref = LayeredOracle(cfg, p).feed(ids)
            without = ids.copy(); without[query - distance] = 2
            moved = row_errors(ref[query:query + 1], LayeredOracle(cfg, p).feed(without)[query:query + 1])[0]
            assert (moved > 4 * TOL[BF16]) == (distance < size), "the needle must show exactly when it is inside"
            for cuts in ([n], [query] + [1] * 3, [query - 1, 2, 2], [query - 20, 23], [128, n - 128] if n > 130 else [n]):
                _check(_feed(m, ids, cuts), ref, dtype, f"needle {distance} behind the query at {query}, portions {cuts}")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_far_keys_through_a_shared_layer(backend, dtype):
    """Layer 1 reads layer 0's keys with a wider window of its own: a needle outside layer 0's window and inside layer 1's."""
    cfg = parallel_config([window(heads=2, kv_heads=2, dim=32, vdim=32, size=30, sharp=1.0), window(heads=2, kv_heads=2, dim=32, vdim=32, size=400, kv_from=0, sharp=1.0)], width=64, vocab=64)
    p = params(cfg, 13)
    _needle_params(cfg, p, 120.0)
    p["l1.mix.o"] = p["l0.mix.o"]
    for k in ("l0.mix.o", "l0.side.norm"):
        p[k] = bf16(0.01 * p[k])                                    # layer 1 sees nearly the same stream ...
    p["l1.mix.q"], p["l1.norm1"] = p["l0.mix.q"], p["l0.norm1"]     # ... and asks the same question
    p["l1.mix.q.conv"] = p["l0.mix.q.conv"]
    m = _model(backend, cfg, p, dtype, seq_len=500)
    rng = np.random.default_rng(8)
    for place in (0, 1, 40, 127, 128, 200):
        ids = rng.integers(2, 64, 403); ids[place] = 0; ids[[398, 399, 401]] = 1
        ref = LayeredOracle(cfg, p).feed(ids)
        without = ids.copy(); without[place] = 2
        moved = row_errors(ref, LayeredOracle(cfg, p).feed(without))
        inside = [q for q in (398, 399, 401) if q - place < 400]
        assert moved[inside].min() > 4 * TOL[BF16]
        for cuts in ([403], [400, 1, 1, 1], [397, 2, 2, 2], [130, 260, 13]):
            _check(_feed(m, ids, cuts), ref, dtype, f"needle at {place}, portions {cuts}")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_steep_and_flat_scores(backend, dtype):
    """Raw scores far apart beside distance biases of hundreds: the running maximum of a row rises late, or its nearest keys weigh nothing."""
    cfg = parallel_config([window(heads=2, kv_heads=1, dim=64, vdim=64, size=600, sharp=24.0), window(heads=16, kv_heads=2, dim=16, vdim=16, size=600, sharp=30.0)], width=64, vocab=64)
    p = params(cfg, 15)
    ids = _ids(cfg, 640)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, dtype)
    for cuts in ([640], [500, 139, 1], [620] + [1] * 20, [300, 16, 16, 308]):
        e = row_errors(_feed(m, ids, cuts), ref)
        # operands of 8 bits decide which of two nearly equal keys wins a softmax this sharp: the median says whether the sums are right
        assert np.isfinite(e).all() and (e.max() < 40 * TOL[F32] if dtype == F32 else np.median(e) < TOL[BF16]), f"portions {cuts}: {np.median(e):.3e}, {e.max():.3e}"
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("B", [2, 3, 9, 20])
def test_batch_equals_each_sequence_alone(backend, dtype, B):
    cfg, p = MIXED, params(MIXED, 23)
    T = 160 if B <= 3 else 60
    ids = _ids(cfg, B * T).reshape(B, T)
    m = _model(backend, cfg, p, dtype, max_batch=B, seq_len=256)
    steps = [(0, T - 30), (T - 30, T - 27), (T - 27, T - 6)] + [(t, t + 1) for t in range(T - 6, T)]
    out = np.concatenate([m.extend(ids[:, a:b]) for a, b in steps], axis=1)
    fwd = m.forward(ids)
    for b in sorted({0, 1, B // 2, B - 1}):
        ref = LayeredOracle(cfg, p).feed(ids[b])
        _check(out[b], ref, dtype, f"sequence {b} of the batch")
        _check(fwd[b], ref, dtype, f"sequence {b} of the batch, forward")
    m.close()


def test_decode_batches_of_every_kernel_width(backend):
    """One to 64 sequences at a time: clusters that share a sequence's window, narrow CTAs, projections with and without the norm and the
    activation on the way.  All sequences are alike, so every row must agree with the oracle's one."""
    cfg = parallel_config([window(heads=8, kv_heads=2, dim=64, vdim=64, size=280, ff=96), window(heads=8, kv_heads=2, dim=64, vdim=64, size=70, kv_from=0, ff=40)], width=128)
    p = params(cfg, 25)
    ids = _ids(cfg, 306)
    ref = LayeredOracle(cfg, p).feed(ids)
    for B in (1, 2, 5, 16, 17, 40, 64):
        m = _model(backend, cfg, p, BF16, seq_len=306, max_batch=B)
        m.extend(np.tile(ids[:300], (B, 1)))
        for t in range(300, 306):
            out = m.extend(np.tile(ids[t:t + 1], (B, 1)))[:, 0]
            _check(out, np.tile(ref[t], (B, 1)), BF16, f"{B} sequences, position {t}")
        m.close()


@pytest.mark.parametrize("dim,vdim", [(64, 64), (128, 128), (32, 96), (96, 48)])
def test_more_work_items_than_multiprocessors(backend, dim, vdim):
    """Prompts of a batch large enough that a CTA of the fused kernel goes through several items, with and without a second query tile, with
    windows that begin in the item's first, second or third key tile."""
    for T, size in ((300, 280), (300, 20), (600, 130), (513, 256), (40, 12)):
        cfg = parallel_config([window(heads=8, kv_heads=2, dim=dim, vdim=vdim, size=size)], width=64)
        p = params(cfg, 27)
        ids = _ids(cfg, T)
        ref = LayeredOracle(cfg, p).feed(ids)
        m = _model(backend, cfg, p, BF16, seq_len=T, max_batch=32)
        for b in range(3):
            out = m.forward(np.tile(ids, (32, 1)))
            for i in range(32):
                _check(out[i], ref, BF16, f"{T} tokens, window {size}: sequence {i}")
        m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_cache_is_reused(backend, dtype):
    """A request after others gives the bits it gave on a fresh model: nothing of the earlier ones is left."""
    cfg, p = MIXED, params(MIXED, 29)
    m = _model(backend, cfg, p, dtype, seq_len=400)
    a, b = _ids(cfg, 200, 1), _ids(cfg, 390, 2)
    cuts = [150, 30, 2] + [1] * 18
    first = _feed(m, a, cuts)
    _feed(m, b, [390])
    assert np.array_equal(_feed(m, a, cuts), first)
    _feed(m, b, [7] * 50 + [40])
    assert np.array_equal(_feed(m, a, cuts), first)
    one_by_one = _feed(m, a[:5], [1] * 5)
    _feed(m, b, [390])
    assert np.array_equal(_feed(m, a[:5], [1] * 5), one_by_one)
    m.close()
    m = _model(backend, cfg, p, dtype, seq_len=400)
    assert np.array_equal(_feed(m, a, cuts), first)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding(backend, dtype):
    """Every window passes over decoded tokens alone, several times for the short ones."""
    cfg, p = MIXED, params(MIXED, 31)
    ids = _ids(cfg, 700)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, dtype, seq_len=700)
    parity_record(f"window, 690 decode steps, {IDS[dtype]}", worst=_check(_feed(m, ids, [10] + [1] * 690), ref, dtype, "long decoding"))
    with pytest.raises(HalError):
        m.extend(np.zeros((1, 1), np.int64))                        # the cache is full
    m.close()


def test_decode_does_not_depend_on_graph_replay(backend):
    cfg, p = MIXED, params(MIXED, 37)
    ids = _ids(cfg, 60)
    m = _model(backend, cfg, p, BF16, seq_len=64)
    cuts = [40] + [1] * 20
    a = _feed(m, ids, cuts)
    backend.lib.sptorch_ext_gpt_enable_graphs(m.h, 0)
    assert np.array_equal(_feed(m, ids, cuts), a)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("block", ["parallel", "post"])
def test_any_mixer_in_either_block(backend, dtype, block, monkeypatch):
    """A design that no model folder names: all three mixers in one model, in parallel blocks and with norms behind the sublayers."""
    mixers, parallel = ("gla", "latent_attention", "attention"), block == "parallel"
    monkeypatch.setitem(layered.DESIGNS, "All", layered.Design(mixers, layered.PARALLEL if parallel else layered.POST_NORM, layered.SILU if parallel else layered.RELU, not parallel, parallel,
                                                               token_side=parallel, embedding_scale=parallel, distance_bias=True, out_gate=True))
    monkeypatch.setitem(O.DESIGNS, "All", dict(block=block, act=O.silu if parallel else O.relu, tied=parallel, token_side=parallel, embedding_scale=parallel))
    layers = [gla(ff=40), window(ff=56), latent(ff=64), window(kv_from=1, size=20), gla(), latent()]
    cfg = parallel_config(layers, architecture="All") if parallel else dict(config(layers), architecture="All")
    p = params(cfg, 61)
    ids = _ids(cfg, 150)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, dtype)
    factor = 1.5 if parallel else 3.0                                # six layers; norms behind the sublayers pass rounding on undamped
    for cuts in ([150], [100, 17, 2, 3, 20] + [1] * 8):
        _check(_feed(m, ids, cuts), ref, dtype, f"portions {cuts}", factor)
    _check(m.forward(ids.reshape(1, -1))[0], ref, dtype, "without a cache", factor)
    m.close()


@pytest.mark.parametrize("M", [3, 40, 200])
def test_gated_epilogues(backend, M):
    """out = r * relu(g) and r * gelu(g) of the weight-streaming, tensor-core and f32 products."""
    rng = np.random.default_rng(M)
    x, w, r, b = (bf16(rng.standard_normal(s).astype(np.float32)) for s in ((M, 96), (136, 96), (M, 136), (136,)))
    g = x.astype(np.float64) @ w.T.astype(np.float64) + b
    for epi, ref in ((EPI_RELU_MUL, r * np.maximum(g, 0)), (EPI_GELU_MUL, r * O.gelu_tanh(g))):
        out = np.asarray(backend.linear(x, w, bias=b, residual=r, epilogue=epi, mode=MM_F32)).reshape(M, 136)
        assert np.abs(out - ref).max() <= 1e-5 * np.abs(ref).max()
        out = np.asarray(backend.linear(x, w, bias=b, residual=r, epilogue=epi, mode=MM_BF16)).reshape(M, 136)
        assert np.abs(out - ref).max() <= 8e-3 * np.abs(ref).max()
    with pytest.raises(HalError):
        backend.linear(x, w, epilogue=EPI_RELU_MUL, mode=MM_BF16)


def _save(folder, cfg, p):
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), list(p.items()), dtype="BF16")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_model_folder_generation_and_replay(backend, dtype, tmp_path, capsys):
    """config.json + safetensors through the registry, greedy generation through the framework's own loop, and the same tokens replayed."""
    cfg = MIXED
    p = params(cfg, 41)
    p["final.norm"] = bf16(4.0 * p["final.norm"])
    _save(tmp_path, cfg, p)
    m = load_model(backend, str(tmp_path), seq_len=128, dtype=dtype)
    assert dict(m.named_parameters()) == shapes_of(cfg)
    prompt = [int(t) for t in _ids(cfg, 21, 6)]
    out = m.generate(prompt, 40, top_k=1)
    assert len(out) == 61 and out[:21] == prompt
    logits = LayeredOracle(cfg, p).feed(out)
    agreed = 0
    for i in range(21, 61):
        top = np.sort(logits[i - 1])[-2:]
        if top[1] - top[0] > 4 * TOL[dtype] * logits.std():
            assert out[i] == int(logits[i - 1].argmax()), f"token {i}"
            agreed += 1
    assert agreed >= 10
    assert m.generate(prompt, 40, top_k=1) == out                    # a second request on the same model
    assert generate.main(["--model", str(tmp_path), "--tokens", ",".join(map(str, prompt)), "--max-new-tokens", "40", "--max-context", "128",
                          "--dtype", "float32" if dtype == F32 else "bfloat16"]) == 0
    assert [int(t) for t in capsys.readouterr().out.strip().split(",")] == out
    said = []
    steps = [{"step": 0, "entries": [{"id": "r", "tokens": out[:50], "want": [20, 49]}], "end": []}] + \
            [{"step": i + 1, "entries": [{"id": "r", "tokens": [out[50 + i]], "want": [0]}], "end": []} for i in range(11)]
    steps[-1]["end"] = ["r"]
    trace.replay(m, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(12)]
    got = np.concatenate([np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]) for i in range(12)])
    _check(got, logits[[20, 49] + list(range(50, 61))], dtype, "replayed")
    m.close()


def test_refusals(backend, tmp_path):
    for layers in ([window(), window(kv_from=0, dim=40)], [window(), window(heads=4, kv_heads=4, kv_from=0)], [window(), window(kv_from=0), window(kv_from=1)], [window(heads=4, kv_heads=3)],
                   [window(dim=2000)]):
        with pytest.raises(HalError):
            LayeredGPT(backend, parallel_config(layers), 32)
    cfg, p = MIXED, params(MIXED, 47)
    bad = dict(p)
    bad.pop("l1.mix.k.conv")
    _save(tmp_path, cfg, bad)
    with pytest.raises(weights.WeightsError):
        load_model(backend, str(tmp_path), seq_len=32)
    bad = dict(p, **{"l3.mix.k": p["l1.mix.k"]})                     # a layer on another's keys has none of its own
    _save(tmp_path, cfg, bad)
    m = load_model(backend, str(tmp_path), seq_len=32)
    with pytest.raises(HalError):
        m.set_param("l3.mix.k", p["l1.mix.k"])
    m.close()


def test_cache_specs(backend):
    m = LayeredGPT(backend, MIXED, 48, max_batch=2)
    specs = layer_specs(m)
    assert [(s.layer, s.kind) for s in specs] == [(0, "ring"), (0, "rows"), (1, "ring"), (1, "rows"), (2, "ring"), (2, "rows"), (3, "ring"), (4, "ring")]
    assert specs[1].shape == (2, 48, 2 * (32 + 24)) and specs[0].shape == (2, 3, 4 * 32 + 2 * 32 + 2 * 24) and specs[6].shape == (2, 2, 6 * 40)
    m.close()
