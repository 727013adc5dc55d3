"""GPU tests of the Lotorax design against the plain CPU restatement (oracle/lotorax.py), float64.

Logits are compared row by row: root mean square of the difference over the vocabulary (means taken off) in units of the
logits' spread.  In f32 rounding alone leaves about 1e-6 there, in bf16 about 1e-2; a wrong key or a lost state shows as
0.1 and more.
"""
import os
import subprocess
import sys

import numpy as np
import pytest

import lotorax_cases as cases
import oracle.lotorax as X
from ruai_b200 import __main__ as cli
from ruai_b200 import nn, registry

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 4e-5, "bfloat16": 4e-2}
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def dev():
    assert nn.Device.is_available(), "these tests need a CUDA device"
    return nn.Device.cuda(0)


def build(dev, cfg, w, dtype):
    m = nn.Lotorax(dev, nn.LotoraxConfig(cfg))
    for name, t in w.items():
        m.set_tensor(name, t)
    m.build(dtype)
    return m


def run(m, ids, cuts):
    """Logits of every position, the sequence fed in portions of these sizes (the last one repeats)."""
    m.cache_clear()
    out, p, i = [], 0, 0
    while p < len(ids):
        n = min(cuts[min(i, len(cuts) - 1)], len(ids) - p)
        out.append(m.forward_cached(ids[None, p:p + n], all_positions=True)[0])
        p, i = p + n, i + 1
    return np.concatenate(out)


def check(got, want, dtype, what=""):
    """All rows within the tolerance; of many rows one in fifteen may be up to four times over it (the norms amplify the
    rounding of a result that happens to be small)."""
    e = np.atleast_1d(cases.rel_error(got, want))
    assert (e > TOL[dtype]).sum() <= len(e) // 15 and e.max() <= (4 if len(e) >= 15 else 1) * TOL[dtype], f"{what}: {e.max():.2e} at row {int(e.argmax())}"


MIXED = [cases.delta(mlp=cases.moe(5, 2)), cases.latent(), cases.latent(heads=2, dim=8, rot_dim=4, vdim=20, rank=12, mlp=cases.moe(4, 1)),
         cases.delta(heads=3, kv_heads=3, dim=12, vdim=8, conv=4, mlp=None)]
LOOP = cases.loop(1, 3, 2)


# ---- mechanisms alone ---------------------------------------------------------------------------------------------

MECHANISMS = {
    "latent": [cases.latent()],
    "latent, no feed-forward": [cases.latent(mlp=None)],
    "latent, plain frequencies": [cases.latent(scaling=None)],
    "latent, one head": [cases.latent(heads=1, dim=8, rot_dim=2, vdim=16, rank=8)],
    "latent, nothing rotated": [cases.latent(rot_dim=0, scaling=None)],
    "latent, odd sizes": [cases.latent(heads=5, dim=7, rot_dim=6, vdim=9, rank=11, mlp=cases.dense(21))],
    "latent, rank of one": [cases.latent(heads=2, dim=4, rot_dim=4, vdim=4, rank=1)],
    "latent, 7 heads": [cases.latent(heads=7, dim=12, rot_dim=4, vdim=20, rank=64)],
    "latent, 12 heads": [cases.latent(heads=12, dim=20, rot_dim=16, vdim=8, rank=40)],
    "latent, 16 heads": [cases.latent(heads=16, dim=8, rot_dim=8, vdim=16, rank=128)],
    "latent, large": [cases.latent(heads=4, dim=128, rot_dim=64, vdim=128, rank=256)],
    "latent, larger": [cases.latent(heads=3, dim=64, rot_dim=32, vdim=64, rank=512)],
    "latent, too large for tiles": [cases.latent(heads=2, dim=224, rot_dim=64, vdim=96, rank=96)],
    "latent, wide rank": [cases.latent(heads=2, dim=32, rot_dim=16, vdim=32, rank=1100)],
    "delta": [cases.delta()],
    "delta, no feed-forward": [cases.delta(mlp=None)],
    "delta, heads of their own": [cases.delta(heads=3, kv_heads=3)],
    "delta, one kv head": [cases.delta(heads=6, kv_heads=1)],
    "delta, one head": [cases.delta(heads=1, kv_heads=1, dim=64, vdim=64)],
    "delta, one tap": [cases.delta(conv=1)],
    "delta, two taps": [cases.delta(conv=2)],
    "delta, four taps": [cases.delta(conv=4)],
    "delta, five taps": [cases.delta(conv=5)],
    "delta, many taps": [cases.delta(conv=16)],
    "delta, odd sizes": [cases.delta(heads=6, kv_heads=2, dim=13, vdim=9, mlp=cases.dense(19))],
    "delta, values narrow": [cases.delta(vdim=1)],
    "delta, values wide": [cases.delta(heads=2, kv_heads=1, dim=12, vdim=200)],
    "delta, values wider": [cases.delta(heads=1, kv_heads=1, dim=20, vdim=600)],
    "delta, large": [cases.delta(heads=2, kv_heads=1, dim=128, vdim=128, conv=4)],
    "delta, larger": [cases.delta(heads=2, kv_heads=1, dim=180, vdim=160)],
    "delta, largest": [cases.delta(heads=1, kv_heads=1, dim=256, vdim=256)],
    "dense, odd": [cases.delta(mlp=cases.dense(33))],
    "experts": [cases.delta(mlp=cases.moe())],
    "experts, one used": [cases.latent(mlp=cases.moe(7, 1, 16))],
    "experts, all used": [cases.latent(mlp=cases.moe(3, 3, 16))],
    "experts, odd": [cases.delta(mlp=cases.moe(5, 3, 11))],
    "experts, one": [cases.delta(mlp=cases.moe(1, 1, 40))],
    "experts, many": [cases.delta(mlp=cases.moe(70, 6, 8))],
    "mixed": MIXED,
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_mechanism_whole_and_decoded(dev, name, dtype):
    cfg = cases.config(MECHANISMS[name], width=62 if "odd" in name else 64, vocab=61 if "odd" in name else 60, eps=1e-3 if "one head" in name else 1e-5)
    w, ids = cases.weights(cfg, seed=len(name), settled=dtype == "bfloat16"), cases.tokens(cfg, 150)
    want = X.forward(cfg, w, ids)
    m = build(dev, cfg, w, dtype)
    check(run(m, ids, [150]), want, dtype, "whole")
    check(run(m, ids, [90, 1]), want, dtype, "decoded")
    check(run(m, ids, [1, 1, 1, 60, 2]), want, dtype, "from one token on")


LOOPS = {"none": None, "in the middle": LOOP, "everything": cases.loop(0, 4, 2), "the first": cases.loop(0, 1, 3), "the last": cases.loop(3, 4, 2), "once": cases.loop(1, 4, 1)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", LOOPS)
def test_loops(dev, name, dtype):
    cfg = cases.config(MIXED, LOOPS[name])
    w, ids = cases.weights(cfg, seed=3, settled=dtype == "bfloat16"), cases.tokens(cfg, 60)
    want = X.forward(cfg, w, ids)
    m = build(dev, cfg, w, dtype)
    for cuts in ([60], [30, 1], [2], [9, 20]):
        check(run(m, ids, cuts), want, dtype, f"portions {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_every_size(dev, dtype):
    cfg = cases.config(MIXED, LOOP)
    w, ids = cases.weights(cfg, 3, settled=dtype == "bfloat16"), cases.tokens(cfg, 170)
    want = X.forward(cfg, w, ids)
    m = build(dev, cfg, w, dtype)
    for cuts in ([2], [3], [4, 5], [7], [8], [9], [15, 16, 17, 18], [31, 33, 2], [63, 2, 65], [1, 2, 1, 37], [64], [128, 42]):
        check(run(m, ids, cuts), want, dtype, f"portions {cuts}")
    check(run(m, ids, [1]), want, dtype, "token by token")


def test_long_prompt(dev):
    """Enough tokens for every tile of the experts' rows and for many blocks of the scan."""
    cfg = cases.config([cases.delta(mlp=cases.moe(4, 2)), cases.latent(mlp=cases.moe(9, 2)), cases.delta(heads=2, kv_heads=2, mlp=cases.moe(3, 1))])
    w, ids = cases.weights(cfg, 14), cases.tokens(cfg, 650)
    want = X.forward(cfg, w, ids)
    m = build(dev, cfg, w, "float32")
    for cuts in ([650], [600, 7, 1], [3, 647]):
        check(run(m, ids, cuts), want, "float32", f"portions {cuts}")


def test_residual_stream_layer_by_layer(dev):
    """The stream after each layer run, through models cut short with the identity for a head."""
    cfg = cases.config(MIXED, cases.loop(0, 4, 1), width=64, vocab=64)
    w, ids = cases.weights(cfg, 5), cases.tokens(cfg, 40)
    w["head"] = np.eye(64, dtype=np.float32)
    stream = []
    X.forward(cfg, w, ids, stream)
    for n in range(1, len(MIXED) + 1):
        part = dict(cfg, layers=cfg["layers"][:n], loop=cases.loop(0, n, 1))
        m = build(dev, part, {k: v for k, v in w.items() if not k.startswith("l") or k == "loop.in" or int(k[1:k.index(".")]) < n}, "float32")
        want = X.layer_norm(stream[n - 1], w["final.norm"].astype(np.float64), w["final.norm.b"].astype(np.float64), cfg["norm"]["eps"])
        assert np.abs(run(m, ids, [40]) - want).max() < 3e-5, n


# ---- experts ------------------------------------------------------------------------------------------------------------

def routed_model(experts, top, ff, dtype, seed):
    """One layer whose mixer adds nothing: what a token's experts read depends on the token alone.  With it the tokens whose
    choice no rounding can turn."""
    cfg = cases.config([cases.delta(heads=1, kv_heads=1, dim=4, vdim=4, mlp=cases.moe(experts, top, ff))], vocab=120)
    w = cases.weights(cfg, seed)
    w["l0.mix.o"][:] = 0
    x = w["embed"].astype(np.float64) * cfg["embedding"]["scale"] + w["l0.norm1b.b"]
    h = X.layer_norm(x, w["l0.norm2"].astype(np.float64), w["l0.norm2.b"].astype(np.float64), cfg["norm"]["eps"])
    s = np.sort(X.sigmoid(h @ w["l0.mlp.router"].T.astype(np.float64)) + w["l0.mlp.correction"], axis=-1)
    safe = np.flatnonzero(s[:, -top] - s[:, -top - 1] > (0.02 if dtype == "bfloat16" else 1e-4)).astype(np.int32)
    used = {int(e) for e in X.route(h[safe], {k: v.astype(np.float64) for k, v in w.items()}, "l0.mlp.", top)[0].ravel()}
    return cfg, w, safe, used


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,top,ff", [(4, 1, 24), (6, 2, 32), (16, 4, 8), (40, 3, 16), (130, 5, 10)])
def test_experts_of_many_and_few_tokens(dev, experts, top, ff, dtype):
    cfg, w, safe, used = routed_model(experts, top, ff, dtype, experts)
    assert len(safe) > 20 and len(used) >= min(experts, 4)
    m = build(dev, cfg, w, dtype)
    rng = np.random.default_rng(2)
    for n in (1, 2, 3, 5, 9, 17, 33, 65, 129, 300, 700):
        ids = rng.choice(safe, n).astype(np.int32)
        check(run(m, ids, [n]), X.forward(cfg, w, ids), dtype, f"{n} tokens")


def test_correction_chooses_but_does_not_weigh(dev):
    cfg = cases.config([cases.delta(mlp=cases.moe(8, 2))])
    w, ids = cases.weights(cfg, 21), cases.tokens(cfg, 30)
    w["l0.mlp.correction"] = np.array([0, 3, 0, 0, 0, 0, 2, 0], np.float32)
    want = X.forward(cfg, w, ids)
    other = dict(w)
    other["l0.mlp.correction"] = np.zeros(8, np.float32)
    assert cases.rel_error(X.forward(cfg, other, ids), want).max() > 0.1
    check(run(build(dev, cfg, w, "float32"), ids, [25, 1]), want, "float32")


# ---- far keys, the sink, rotations ----------------------------------------------------------------------------------

def pointed_model(seed=0, n=0, sink=0.0):
    """One attention layer in which token 0's queries are token 399's keys, and nobody else's: the embedding of 399 is that
    of 0 shifted by one channel, the latents' projection the query projection shifted likewise, the keys the latents
    themselves.  Nothing is rotated and the scores are large, so that token 0 attends to 399 and to little else."""
    cfg = cases.config([cases.latent(heads=2, dim=16, rot_dim=4, vdim=12, rank=32, scale=0.55, mlp=None)], vocab=400)
    w = cases.weights(cfg, seed)
    w["embed"][399] = np.roll(w["embed"][0], 1)
    q = w["l0.mix.q"].reshape(2, 20, 64)
    q[:, 16:] = 0
    w["l0.mix.dkv"][:32] = np.roll(q[:, :16].reshape(32, 64), 1, axis=1)
    w["l0.mix.dkv.norm"][:] = 1
    w["l0.mix.uk"] = np.eye(32, dtype=np.float32)
    w["l0.norm1"][:] = 1
    w["l0.norm1.b"][:] = 0
    w["l0.norm1b"][:] = 1.25
    w["l0.mix.sink"] = np.full(2, sink, np.float32)
    ids = np.random.default_rng(n).permutation(np.arange(1, 399))[:n].astype(np.int32)  # no token twice
    return cfg, w, ids


@pytest.mark.parametrize("n", [5, 64, 65, 66, 130, 260, 390])
def test_keys_near_and_far(dev, n):
    cfg, w, base = pointed_model(n=n)
    models = {dtype: build(dev, cfg, w, dtype) for dtype in DTYPES}
    q = n - 1
    for at in {0, 1, 15, 16, 31, 32, 33, 63, 64, 127, 128, q // 2, q - 64, q - 1}:
        if not 0 <= at < q:
            continue
        ids = base.copy()
        ids[at], ids[q] = 399, 0
        want = X.forward(cfg, w, ids)
        without = ids.copy()
        without[at] = base[at]
        assert cases.rel_error(X.forward(cfg, w, without)[q], want[q]) > 3 * TOL["bfloat16"]  # the key matters
        for dtype, m in models.items():
            for cuts in ([q + 1], [q, 1], [max(1, q - 5), 2], [max(1, q - 20), 12]):
                check(run(m, ids, cuts)[q], want[q], dtype, f"query {q}, key {at}, portions {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks(dev, dtype):
    for sink in (-30.0, 0.0, 4.0, 9.0):
        cfg, w, ids = pointed_model(n=90, sink=sink)
        ids[3], ids[89], ids[50] = 399, 0, 0
        want = X.forward(cfg, w, ids)
        m = build(dev, cfg, w, dtype)
        for cuts in ([90], [85, 1], [88, 2]):
            check(run(m, ids, cuts), want, dtype, f"sink {sink}, portions {cuts}")


def test_a_left_out_sink_would_show():
    cfg = cases.config([cases.latent()])
    w, ids = cases.weights(cfg, 2), cases.tokens(cfg, 40)
    w["l0.norm1b"][:] = 1.25
    other = dict(w)
    other["l0.mix.sink"] = np.full(3, -100.0, np.float32)
    assert cases.rel_error(X.forward(cfg, other, ids), X.forward(cfg, w, ids)).max() > 3 * TOL["bfloat16"]


@pytest.mark.parametrize("scaling", [None, {"factor": 2.0, "fast": 32.0, "original": 64, "slow": 1.0}, {"factor": 40.0, "fast": 2.0, "original": 30, "slow": 0.1},
                                     {"factor": 1.0, "fast": 8.0, "original": 100, "slow": 2.0}])
@pytest.mark.parametrize("base,dims", [(10000.0, 16), (50.0, 2), (1e6, 64)])
def test_rotations(dev, scaling, base, dims):
    """The rotated part decides the scores; positions go far beyond the original context."""
    cfg = cases.config([cases.latent(heads=2, dim=4, rot_dim=dims, base=base, scaling=scaling, scale=1.2 / dims, mlp=None)])
    w, ids = cases.weights(cfg, 6), cases.tokens(cfg, 300)
    w["l0.mix.dkv"][20:] *= 2
    want = X.forward(cfg, w, ids)
    m = build(dev, cfg, w, "float32")
    for cuts in ([300], [250, 1], [290, 3]):
        check(run(m, ids, cuts), want, "float32", f"portions {cuts}")


def test_rotated_part_of_the_rotated_part(dev):
    cfg = cases.config([cases.latent(rot_dim=12)])
    cfg["layers"][0]["mixer"]["rot"]["dims"] = 8
    w, ids = cases.weights(cfg, 6), cases.tokens(cfg, 60)
    check(run(build(dev, cfg, w, "float32"), ids, [50, 1]), X.forward(cfg, w, ids), "float32")


def test_far_state_shows(dev):
    """Slow decays: the first tokens still reach the last ones through the state, whole and decoded."""
    cfg = cases.config([cases.delta(heads=2, kv_heads=1, dim=32, vdim=16, mlp=None)])
    w = cases.weights(cfg, 8)
    w["l0.mix.A_log"] = np.full(2, -7.0, np.float32)
    w["l0.mix.b"] *= 0.2
    w["l0.mix.k.conv"][:, -1] = 2
    ids = cases.tokens(cfg, 200)
    other = ids.copy()
    other[:4] = (other[:4] + 7) % 60
    want = X.forward(cfg, w, ids)
    assert cases.rel_error(X.forward(cfg, w, other)[-1], want[-1]) > 1e-3  # the far tokens matter
    m = build(dev, cfg, w, "float32")
    for cuts in ([200], [4, 1], [4, 37], [150, 2]):
        check(run(m, ids, cuts), want, "float32", f"portions {cuts}")


# ---- cache and states ------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
def test_cleared_cache_and_states_leave_nothing(dev, dtype):
    cfg = cases.config(MIXED, LOOP)
    w = cases.weights(cfg, 4, settled=True)
    a, b = cases.tokens(cfg, 90, 1), cases.tokens(cfg, 70, 2)
    m = build(dev, cfg, w, dtype)
    fresh = run(m, b, [50, 1])
    run(m, a, [33, 1])
    assert np.array_equal(run(m, b, [50, 1]), fresh)
    run(m, a, [1])
    assert np.array_equal(run(m, b, [50, 1]), fresh)
    assert m.cache_len() == 70
    check(fresh, X.forward(cfg, w, b), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_grows_the_cache(dev, dtype):
    cfg = cases.config([cases.latent(), cases.delta()], cases.loop(0, 1, 2))
    w, ids = cases.weights(cfg, 6), cases.tokens(cfg, 300)
    m = build(dev, cfg, w, dtype)
    caps = set()
    m.cache_clear()
    rows = []
    for t in ids:
        rows.append(m.forward_cached(np.array([[t]]))[0])
        caps.add(m.cache_capacity())
    assert len(caps) > 3
    want = X.forward(cfg, w, ids)
    check(np.stack(rows), want, dtype)
    m2 = build(dev, cfg, w, dtype)
    m2.cache_reserve(1, 300)
    check(run(m2, ids, [37]), want, dtype, "reserved")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_side_by_side(dev, dtype):
    """Sequences of one length in a batch give what each gives alone; then single-token steps of the batch."""
    cfg = cases.config(MIXED, LOOP)
    w = cases.weights(cfg, 7, settled=dtype == "bfloat16")
    m = build(dev, cfg, w, dtype)
    for B, T in ((3, 45), (18, 10), (2, 5), (70, 3)):
        ids = np.stack([cases.tokens(cfg, T + 6, 10 + b) for b in range(B)])
        m.cache_clear()
        got = [m.forward_cached(ids[:, :T], all_positions=True)]
        for t in range(T, T + 6):
            got.append(m.forward_cached(ids[:, t:t + 1])[:, None])
        got = np.concatenate(got, axis=1)
        for b in {0, 1, B // 2, B - 1}:
            check(got[b], X.forward(cfg, w, ids[b]), dtype, f"sequence {b} of {B}")


@pytest.mark.parametrize("layer", [cases.delta(16, 8, 8, 64, mlp=None), cases.delta(16, 16, 72, 64, mlp=None), cases.delta(8, 2, 128, 128, 4, mlp=None),
                                   cases.delta(12, 3, 144, 40, mlp=None)], ids=["8x64", "72x64", "128x128", "144x40"])
def test_recurrences_of_many_sequences(dev, layer):
    """Batches large enough for every number of value columns per thread."""
    cfg = cases.config([layer])
    w = cases.weights(cfg, 17)
    m = build(dev, cfg, w, "float32")
    for B in (1, 4, 20):
        ids = np.stack([cases.tokens(cfg, 15, 30 + b) for b in range(B)])
        m.cache_clear()
        got = np.concatenate([m.forward_cached(ids[:, :9], all_positions=True), m.forward_cached(ids[:, 9:11], all_positions=True),
                              m.forward_cached(ids[:, 11:12], all_positions=True), m.forward_cached(ids[:, 12:], all_positions=True)], axis=1)
        for b in {0, B // 2, B - 1}:
            check(got[b], X.forward(cfg, w, ids[b]), "float32", f"sequence {b} of {B}")


def test_rows_of_a_step(dev):
    cfg = cases.config(MIXED, LOOP)
    w, ids = cases.weights(cfg, 9), cases.tokens(cfg, 50)
    m = build(dev, cfg, w, "float32")
    full = run(m, ids, [50])
    m.cache_clear()
    assert m.forward_rows(ids[None, :30], []).shape == (0, 60)
    assert np.abs(m.forward_rows(ids[None, 30:49], [18, 0, 7]) - full[[48, 30, 37]]).max() < 1e-4
    assert np.abs(m.forward_rows(ids[None, 49:], [0]) - full[49]).max() < 1e-4
    m.cache_clear()
    assert np.abs(m.forward_cached(ids[None, :])[0] - full[-1]).max() < 1e-4


def test_errors(dev):
    cfg = cases.config([cases.latent(), cases.delta(mlp=cases.moe())])
    w = cases.weights(cfg)
    m = build(dev, cfg, w, "bfloat16")
    with pytest.raises(nn.RuaiError, match="out of range"):
        m.forward_cached(np.full((1, 4), 60, np.int32))
    broken = nn.Lotorax(dev, nn.LotoraxConfig(cfg))
    with pytest.raises(nn.RuaiError, match="does not exist"):
        broken.set_tensor("pos", np.zeros(3))
    with pytest.raises(nn.RuaiError, match="elements"):
        broken.set_tensor("embed", np.zeros(3))
    with pytest.raises(nn.RuaiError, match="was not set"):
        broken.build()
    for layers, loop, what in (([cases.delta(heads=4, kv_heads=3)], None, "multiple of kv_heads"), ([cases.delta(conv=17)], None, "taps"),
                               ([cases.delta(mlp=cases.moe(2, 3))], None, "experts"), ([cases.delta()], cases.loop(0, 2, 1), "loop")):
        with pytest.raises(nn.RuaiError, match=what):
            nn.Lotorax(dev, nn.LotoraxConfig(cases.config(layers, loop)))


# ---- generation through the library's own entry points ------------------------------------------------------------------

def greedy(cfg, w, ids, n):
    """Greedy continuation by the oracle, and the smallest gap between the two best logits on the way."""
    ids, gap = list(ids), np.inf
    for _ in range(n):
        row = X.forward(cfg, w, ids)[-1]
        top = np.sort(row)[-2:]
        gap = min(gap, (top[1] - top[0]) / row.std())
        ids.append(int(row.argmax()))
    return ids, gap


@pytest.mark.parametrize("prompt_len", [1, 2, 13])
def test_greedy_generation(dev, prompt_len):
    cfg = cases.config(MIXED, LOOP)
    w = cases.weights(cfg, 11)
    prompt = cases.tokens(cfg, prompt_len, 3)
    want, gap = greedy(cfg, w, prompt, 24)
    assert gap > 1e-4, "choose another seed: two logits are too close to tell"
    m = build(dev, cfg, w, "float32")
    assert m.generate(prompt, 24).tolist() == want
    assert m.generate_sampled(prompt, 24, 0.0).tolist() == want
    a, b = m.generate_sampled(prompt, 24, 0.8, 20, 0.9, 5), m.generate_sampled(prompt, 24, 0.8, 20, 0.9, 5)
    assert a.tolist() == b.tolist() and len(a) == prompt_len + 24 and 0 <= a.min() and a.max() < 60
    # the step that stays on the device
    m.cache_clear()
    m.forward_cached(prompt[None, :])
    ids = nn.Tensor.from_numpy(dev, np.array(want[prompt_len:prompt_len + 1], np.int32))
    got = [int(m.decode_step(1, ids.ptr)[0])] + [int(m.decode_step(1)[0]) for _ in range(5)]
    assert got == want[prompt_len + 1:prompt_len + 7]


def test_synthetic_weights_and_accounting(dev):
    m = nn.Lotorax(dev, nn.LotoraxConfig(cases.config(MIXED, LOOP)))
    m.load_synthetic(3, "bfloat16")
    out = m.forward_cached(np.arange(12, dtype=np.int32)[None])
    assert np.isfinite(out).all() and out.std() > 0
    m.decode_step(1)
    ms, launches, n = m.time_linears(1, 2)
    assert ms > 0 and m.step_launches() > launches > 0 and m.step_bytes(1, 12) > n > 0


def test_command_line_and_trace_runner(dev, tmp_path, capsys):
    cfg = cases.config(MIXED, LOOP)
    w, ids = cases.weights(cfg, 13, settled=True), cases.tokens(cfg, 40)
    cases.save(tmp_path, cfg, w)
    want = X.forward(cfg, w, ids)
    check(run(registry.load(dev, str(tmp_path)), ids, [31, 1]), want, "bfloat16", "registry")
    assert cli.main(["info", "--model", str(tmp_path)]) == 0 and capsys.readouterr().out.strip() == "lotorax"
    expected, gap = greedy(cfg, w, ids[:9], 8)
    assert gap > 1e-4
    cli.main(["generate", "--model", str(tmp_path), "--ids", ",".join(map(str, ids[:9])), "-n", "8", "--dtype", "float32"])
    assert capsys.readouterr().out.strip() == ",".join(map(str, expected))
    steps = ['{"step": 0, "entries": [{"id": "a", "tokens": %s, "want": [0, 24]}], "end": []}' % ids[:25].tolist(),
             '{"step": 1, "entries": [{"id": "a", "tokens": %s, "want": []}], "end": []}' % ids[25:39].tolist(),
             '{"step": 2, "entries": [{"id": "a", "tokens": %s, "want": [0]}], "end": ["a"]}' % ids[39:].tolist(),
             '{"step": 3, "entries": [{"id": "b", "tokens": %s, "want": [1]}], "end": ["b"]}' % ids[:2].tolist()]
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                           input="\n".join(steps) + "\n", capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
        for step, rows in ((0, [0, 24]), (2, [39]), (3, [1])):
            got = np.fromfile(out / f"{step}.f32", "<f4").reshape(len(rows), -1)
            e = cases.rel_error(np.concatenate([got, want[:20]]), np.concatenate([want[rows], want[:20]]))
            assert e.max() <= TOL[dtype], (dtype, step, e.max())
