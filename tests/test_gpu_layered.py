"""Models built from a list of layers (gated linear attention, latent attention, norms behind the sublayers) on the device, against the
plain implementation in oracle/layered.py: each mechanism alone, prompts, portions, decoding, batches, reuse of cache and state,
sizes the kernels' vectors and tiles do not divide, and generation through the framework's own loop."""
import io
import json

import numpy as np
import pytest

from conftest import parity_record
from layered_models import bf16, config, gla, latent, params, row_errors, shapes_of
from oracle.layered import LayeredOracle
from sptorch_b200 import generate, trace, weights
from sptorch_b200.backend import BF16, F32, HalError
from sptorch_b200.gpt import GPT
from sptorch_b200.kv_cache import layer_specs
from sptorch_b200.layered import LayeredGPT
from sptorch_b200.registry import load_model
from weight_files import write_safetensors

pytestmark = pytest.mark.gpu
# per position, against the f64 oracle: f32 is rounding alone, bf16 the rounding of the operands of every product
TOL = {F32: 3e-5, BF16: 4e-2}
DTYPES = [F32, BF16]
IDS = ["f32", "bf16"]


def _model(backend, cfg, p, dtype, seq_len=1024, max_batch=1, decay_rank=7):
    m = LayeredGPT(backend, cfg, seq_len, dtype=dtype, max_batch=max_batch, shapes=shapes_of(cfg, decay_rank))
    for k, v in p.items():
        m.set_param(k, v)
    m.enable_kv_cache()
    return m


def _ids(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def _check(got, ref, dtype, what, factor=1.0):
    """Every position within the tolerance in f32.  In bf16 at least 95 of 100, and none beyond three times: a head's output that happens
    to be small before its norm, or two keys with equal scores, turn the rounding of the operands into more than the usual error."""
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


# a model whose two mixers alternate, with and without feed-forwards
MIXED = config([gla(heads=2, dim=40, vdim=48), latent(heads=3, dim=64, vdim=40, rot_dim=32, kv_rank=96, q_rank=72, ff=120),
                latent(heads=2, dim=40, vdim=64, rot_dim=16, kv_rank=64, q_rank=48), gla(heads=3, dim=32, vdim=24, ff=88)], width=104)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name,layers", [
    ("gated linear attention", [gla()]), ("one head, slow decay", [gla(heads=1, dim=64, vdim=64, tau=64.0)]), ("tau 1", [gla(heads=2, dim=16, vdim=16, tau=1.0)]),
    ("wide values", [gla(heads=1, dim=128, vdim=256)]), ("latent attention", [latent()]), ("peaked latent attention", [latent(heads=2, dim=64, vdim=64, sharp=6.0)]),
    ("partly rotated", [latent(rot_dim=24, rope_dims=8)]), ("large heads", [latent(heads=2, dim=128, vdim=128, rot_dim=64, kv_rank=256)]),
    ("feed-forward", [gla(ff=64)]), ("latent and feed-forward", [latent(ff=200)]), ("no layer", [])])
def test_each_mechanism_alone(backend, dtype, name, layers):
    """One layer: the residual stream behind the embedding and behind the layer, and the logits, of one prompt."""
    cfg = config(layers)
    p = params(cfg, 5)
    ids = _ids(cfg, 150)
    taps = []
    ref = LayeredOracle(cfg, p).feed(ids, taps)
    m = _model(backend, cfg, p, dtype)
    m.enable_taps()
    out = m.prefill_kv_cache(ids.reshape(1, -1))[0]
    assert np.array_equal(m.tap(0, len(ids)), p["embed"][ids])
    for i, t in enumerate(taps):
        _check(m.tap(i + 1, len(ids)), t, dtype, f"{name}: layer {i}")
    parity_record(f"layered, {name}, {IDS[dtype]}", worst=_check(out, ref, dtype, name))
    fresh = m.forward(ids.reshape(1, -1))[0]                        # the forward without a cache runs the same layers
    _check(fresh, ref, dtype, name)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width,vocab,layers,rank", [
    (50, 33, [gla(heads=3, dim=10, vdim=14, tau=3.0), latent(heads=3, dim=20, vdim=28, kv_rank=36, q_rank=12, rot_dim=6, rope_dims=4, ff=52)], 5),
    (33, 130, [latent(heads=1, dim=7, vdim=5, kv_rank=9, q_rank=11, rot_dim=2, ff=3), gla(heads=1, dim=3, vdim=7, tau=2.0, ff=1)], 1),
    (264, 700, [latent(heads=5, dim=48, vdim=56, kv_rank=72, q_rank=24, rot_dim=8, base=123.0), gla(heads=4, dim=72, vdim=88, tau=20.0, ff=136), gla(heads=1, dim=136, vdim=40)], 24)])
def test_other_sizes(backend, dtype, width, vocab, layers, rank):
    """Sizes that fit no vector, tile or head size the kernels prefer, prompts and decoding."""
    cfg = config(layers, width=width, vocab=vocab, eps=1e-3)
    p = params(cfg, 7, rank)
    ids = _ids(cfg, 141)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, dtype, seq_len=141, decay_rank=rank)
    _check(_feed(m, ids, [130] + [1] * 11), ref, dtype, "prompt, then decoding", 1.5)
    _check(_feed(m, ids, [2, 5, 19, 40, 75]), ref, dtype, "portions", 1.5)
    m.close()


@pytest.mark.parametrize("layer", [
    latent(heads=2, dim=96, vdim=40, rot_dim=48, sharp=2.0), latent(heads=3, dim=32, vdim=104, rot_dim=64, sharp=2.0), latent(heads=2, dim=128, vdim=128, rot_dim=64, sharp=2.0),
    latent(heads=20, dim=24, vdim=16, kv_rank=400, q_rank=64, rot_dim=24, sharp=2.0), latent(heads=17, dim=16, vdim=32, kv_rank=512, rot_dim=64), latent(heads=1, dim=64, vdim=64, kv_rank=24, rot_dim=8),
    gla(heads=1, dim=32, vdim=120), gla(heads=2, dim=20, vdim=250), gla(heads=2, dim=64, vdim=128), gla(heads=1, dim=60, vdim=200), gla(heads=2, dim=100, vdim=64), gla(heads=1, dim=112, vdim=144)])
def test_every_kernel_shape(backend, layer):
    """bf16: every tile shape the fused attention, the cached-row attention and the chunk kernels are built for, on several tiles of keys
    and chunks, as one prompt, behind a cached prefix and in decoding."""
    cfg = config([layer], width=80)
    p = params(cfg, 53)
    ids = _ids(cfg, 560)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, BF16, seq_len=560)
    for cuts in ([560], [300, 200, 2, 3, 16, 33, 1, 1, 1, 1, 1, 1], [129, 383, 48]):
        _check(_feed(m, ids, cuts), ref, BF16, f"portions {cuts}")
    m.close()


@pytest.mark.parametrize("layer", [latent(heads=20, dim=24, vdim=16, kv_rank=400, q_rank=64, rot_dim=24, sharp=2.0), latent(heads=4, dim=64, vdim=64, rot_dim=32, sharp=3.0),
                                   latent(heads=4, dim=64, vdim=128, rot_dim=32, sharp=3.0), latent(heads=4, dim=128, vdim=64, rot_dim=32, sharp=3.0), latent(heads=4, dim=128, vdim=128, rot_dim=64, sharp=3.0)])
def test_short_portions_behind_long_prefixes(backend, layer):
    """A portion of at most one query tile behind several key tiles, with scores peaked enough that some warps rescale and others do not:
    every position of every portion, none far off."""
    cfg = config([layer], width=80)
    p = params(cfg, 53)
    ids = _ids(cfg, 800)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, BF16, seq_len=800)
    for first in (128, 256, 384, 521, 640):
        for T in (17, 33, 48, 64, 90, 128, 150):
            m.reset_cache()
            m.extend(ids[:first].reshape(1, -1))
            e = row_errors(m.extend(ids[first:first + T].reshape(1, -1))[0], ref[first:first + T])
            assert e.max() <= 2 * TOL[BF16], f"{T} tokens at {first}: {e.max():.3e} at row {int(e.argmax())}"
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
    parity_record(f"layered, ten ways to cut 300 tokens, {IDS[dtype]}", worst=worst)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_far_keys_at_tile_borders(backend, dtype):
    """A marked token at one place and a query for it far behind: the marked key takes nearly all of the softmax weight, so that a key
    that is missing, doubled or shifted by one shows.  Places around every border of the key tiles and of the portions."""
    cfg = config([latent(heads=2, dim=32, vdim=32, rot_dim=16, kv_rank=64, q_rank=64, sharp=1.5)], width=64, vocab=64)
    p = params(cfg, 13)
    # token 0 is the needle: the unrotated queries of token 1 look along its key, for a score of 40
    q = (p["embed"][1] @ p["l0.mix.dq"].T)
    q = q / np.sqrt((q * q).mean() + cfg["norm"]["eps"]) * p["l0.mix.dq.norm"]
    c = (p["embed"][0] @ p["l0.mix.dkv"].T)[:64]
    c = c / np.sqrt((c * c).mean() + cfg["norm"]["eps"]) * p["l0.mix.dkv.norm"]
    for h in range(2):
        kn = p["l0.mix.uk"][h * 32:(h + 1) * 32] @ c
        rows = slice(h * 48, h * 48 + 32)
        p["l0.mix.uq"][rows] += np.outer(40.0 / cfg["layers"][0]["mixer"]["scale"] / (kn @ kn) * kn - p["l0.mix.uq"][rows] @ q, q) / (q @ q)      # unrotated query of token 1 along that key
    p["l0.mix.uq"] = bf16(p["l0.mix.uq"])
    m = _model(backend, cfg, p, dtype)
    rng = np.random.default_rng(3)
    for place in (0, 1, 126, 127, 128, 129, 255, 256, 257, 383):
        ids = rng.integers(2, 64, 402); ids[place] = 0; ids[[390, 399, 401]] = 1
        o = LayeredOracle(cfg, p)
        ref = o.feed(ids)
        without = ids.copy(); without[place] = 2
        moved = row_errors(ref[[399, 401]], LayeredOracle(cfg, p).feed(without)[[399, 401]])
        assert moved.min() > 4 * TOL[BF16], "the needle must matter for the comparison to mean anything"
        for cuts in ([402], [400, 1, 1], [128, 128, 143, 2, 1], [130, 260, 2, 2, 2, 3, 3], [385, 14, 1, 1, 1]):
            got = _feed(m, ids, cuts)
            _check(got, ref, dtype, f"needle at {place}, portions {cuts}")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_state_remembers_across_portions(backend, dtype):
    """A channel that hardly decays (log decay about -5e-5 per token) carries one token over hundreds of others and across every cut."""
    cfg = config([gla(heads=2, dim=16, vdim=32, tau=16.0)], width=64, vocab=64)
    p = params(cfg, 17)
    p["l0.mix.a2.b"] = np.full_like(p["l0.mix.a2.b"], 7.0); p["l0.mix.a2"] *= 0.125
    p["l0.mix.k"] *= 0.0625
    mark = p["embed"][0] / (p["embed"][0] @ p["embed"][0])
    p["embed"][1:] = bf16(p["embed"][1:] - np.outer(p["embed"][1:] @ mark, p["embed"][0]))      # no other token has a part along it
    p["l0.mix.k"] = bf16(p["l0.mix.k"] + 8.0 * np.outer(np.ones(32), mark))         # token 0 writes with a long key
    m = _model(backend, cfg, p, dtype)
    ids = np.random.default_rng(4).integers(1, 64, 500); ids[3] = 0
    ref = LayeredOracle(cfg, p).feed(ids)
    without = ids.copy(); without[3] = 5
    assert row_errors(ref[-1:], LayeredOracle(cfg, p).feed(without)[-1:]).min() > 4 * TOL[BF16]
    for cuts in ([500], [4, 496], [63, 1, 64, 65, 307], [2, 2, 2, 17, 64, 128, 285], [480] + [1] * 20):
        _check(_feed(m, ids, cuts), ref, dtype, f"portions {cuts}")
    m.close()


def test_strong_decay_does_not_overflow(backend):
    """Decays of e^-12 per token and channel beside channels that keep everything: products of decays underflow, nothing may overflow."""
    cfg = config([gla(heads=2, dim=32, vdim=32, tau=1.0)], width=64, vocab=64)
    p = params(cfg, 19)
    b = np.where(np.arange(64) % 2 == 0, -12.0, 9.0)
    p["l0.mix.a2.b"] = bf16(b)
    ids = _ids(cfg, 400)
    ref = LayeredOracle(cfg, p).feed(ids)
    for dtype in DTYPES:
        m = _model(backend, cfg, p, dtype)
        _check(_feed(m, ids, [400]), ref, dtype, "prompt")
        _check(_feed(m, ids, [200, 100, 80, 2] + [1] * 18), ref, dtype, "portions")
        m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_batch_equals_each_sequence_alone(backend, dtype):
    cfg, p = MIXED, params(MIXED, 23)
    B, T = 3, 170
    ids = _ids(cfg, B * T).reshape(B, T)
    m = _model(backend, cfg, p, dtype, max_batch=B, seq_len=256)
    steps = [(0, 140), (140, 143), (143, 164)] + [(t, t + 1) for t in range(164, 170)]
    out = np.concatenate([m.extend(ids[:, a:b]) for a, b in steps], axis=1)
    fwd = m.forward(ids)
    for b in range(B):
        ref = LayeredOracle(cfg, p).feed(ids[b])
        _check(out[b], ref, dtype, f"sequence {b} of the batch")
        _check(fwd[b], ref, dtype, f"sequence {b} of the batch, forward")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_cache_and_state_are_reused(backend, dtype):
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
    m.close()
    m = _model(backend, cfg, p, dtype, seq_len=400)
    assert np.array_equal(_feed(m, a, cuts), first)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding(backend, dtype):
    cfg, p = MIXED, params(MIXED, 31)
    ids = _ids(cfg, 700)
    ref = LayeredOracle(cfg, p).feed(ids)
    m = _model(backend, cfg, p, dtype, seq_len=700)
    parity_record(f"layered, 690 decode steps, {IDS[dtype]}", worst=_check(_feed(m, ids, [10] + [1] * 690), ref, dtype, "long decoding"))
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


def _save(folder, cfg, p):
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), list(p.items()), dtype="BF16")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_model_folder_generation_and_replay(backend, dtype, tmp_path, capsys):
    """config.json + safetensors through the registry, greedy generation through the framework's own loop, and the same tokens replayed."""
    cfg = MIXED
    p = params(cfg, 41)
    p["head"] = bf16(4.0 * p["head"])
    _save(tmp_path, cfg, p)
    m = load_model(backend, str(tmp_path), seq_len=128, dtype=dtype)
    assert [tuple(s) for _, s in m.named_parameters()] == [tuple(s) for s in shapes_of(cfg).values()] and [n for n, _ in m.named_parameters()] == list(shapes_of(cfg))
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


def test_fused_loss_and_greedy_head(backend):
    """The LM head fused with loss and greedy token serves this model as it serves the others."""
    cfg, p = MIXED, params(MIXED, 43)
    m = _model(backend, cfg, p, BF16, seq_len=64)
    ids = _ids(cfg, 64).reshape(1, 64)
    logits = m.forward(ids)[0].astype(np.float64)
    loss, arg = m.forward_loss(ids, np.roll(ids, -1, 1))
    lse = np.log(np.exp(logits - logits.max(-1, keepdims=True)).sum(-1)) + logits.max(-1)
    assert np.array_equal(arg[0], logits.argmax(-1)) and abs(loss - (lse - logits[np.arange(64), np.roll(ids, -1, 1)[0]]).mean()) < 1e-4
    m.close()


def test_refusals(backend, tmp_path):
    cfg, p = MIXED, params(MIXED, 47)
    m = _model(backend, cfg, p, BF16, seq_len=32)
    with pytest.raises(HalError):
        m.append_and_decode([1])                                     # nothing cached yet
    m.extend(np.ones((1, 5), np.int64))
    with pytest.raises(HalError):
        m.decode_logits_from_cache([1])
    with pytest.raises(HalError):
        m.extend(np.ones((1, 28), np.int64))                         # 33 positions in a cache of 32
    m.extend(np.ones((1, 27), np.int64))
    with pytest.raises(HalError):
        m.set_param("l0.mix.nothing", np.zeros(3))
    with pytest.raises(HalError):
        m.set_param("l0.norm1", np.zeros(3))
    m.close()
    bad = dict(p)
    bad.pop("l1.mix.uk")
    _save(tmp_path, cfg, bad)
    with pytest.raises(weights.WeightsError):
        load_model(backend, str(tmp_path), seq_len=32)
    with pytest.raises(HalError):
        LayeredGPT(backend, config([latent(kv_rank=1600)]), 32)
    with pytest.raises(HalError):
        LayeredGPT(backend, config([gla(dim=600)]), 32, shapes={"l0.mix.a1": (4, 72)})


def test_cache_specs(backend):
    m = LayeredGPT(backend, MIXED, 48, max_batch=2, shapes=shapes_of(MIXED))
    specs = layer_specs(m)
    assert [s.kind for s in specs] == ["state", "rows", "rows", "state"]
    assert specs[0].elements() == 2 * 2 * 40 * 48 and specs[0].total_bytes() == 4 * specs[0].elements()
    assert specs[1].elements() == 2 * 48 * (96 + 32) and specs[1].total_bytes() == 2 * specs[1].elements()
    m.close()


def test_other_architectures_through_the_same_calls(backend, tmp_path):
    """extend on a model with a position table: a prefill, then tokens; and a model folder of that architecture."""
    cfg = dict(architecture="GPT", vocab=64, d_model=32, n_head=2, n_layer=2, d_ff=64, seq_len=48)
    m = GPT(backend, 64, 32, 2, 2, 64, 48, dtype=F32)
    rng = np.random.default_rng(0)
    p = [(n, bf16(0.3 * rng.standard_normal(s).astype(np.float32))) for n, s in m.named_parameters()]
    _save(tmp_path, cfg, dict(p))
    m.close()
    m = load_model(backend, str(tmp_path), dtype=F32)
    ids = rng.integers(0, 64, 20)
    ref = m.forward(ids.reshape(1, -1))[0]
    m.enable_kv_cache()
    out = np.concatenate([m.extend(ids[a:b].reshape(1, -1))[0] for a, b in ((0, 12), (12, 15), (15, 16), (16, 20))])
    assert np.abs(out - ref).max() <= 2e-3 * np.abs(ref).max()
    m.close()
