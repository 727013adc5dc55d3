"""GPU tests of the Zazasun design against the plain CPU restatement (oracle/zazasun.py), float64.

Logits are compared row by row: root mean square of the difference over the vocabulary (means taken off) in units of the
logits' spread.  In f32 rounding alone leaves about 1e-6 there, in bf16 about 1e-2; a wrong key or a lost state shows as
0.1 and more.
"""
import os
import subprocess
import sys

import numpy as np
import pytest

import oracle.zazasun as Z
import zazasun_cases as cases
from ruai_b200 import __main__ as cli
from ruai_b200 import nn, registry

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 6e-5, "bfloat16": 5e-2}
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def dev():
    assert nn.Device.is_available(), "these tests need a CUDA device"
    return nn.Device.cuda(0)


def build(dev, cfg, w, dtype):
    ranks = [w[f"l{i}.mix.w1"].shape[0] if layer["type"] == "wkv" else 0 for i, layer in enumerate(cfg["layers"])]
    m = nn.Zazasun(dev, nn.ZazasunConfig(cfg, ranks))
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
    """All rows within the tolerance; of many rows one in fifteen may be up to four times over it (the head norms amplify the
    rounding of a head whose output happens to be small)."""
    e = np.atleast_1d(cases.rel_error(got, want))
    assert (e > TOL[dtype]).sum() <= len(e) // 15 and e.max() <= (4 if len(e) >= 15 else 1) * TOL[dtype], f"{what}: {e.max():.2e} at row {int(e.argmax())}"


MIXED = [cases.attention(), cases.wkv(), cases.hgrn2(), cases.wkv(heads=2, dim=24, ff=0), cases.attention(heads=3, kv_heads=1, dim=12, vdim=12, size=17, keep_first=1)]


# ---- unquantized Linears ------------------------------------------------------------------------------------------

@pytest.mark.parametrize("bits,x_dtype", [(16, "bf16"), (16, "f32"), (32, "f32")])
@pytest.mark.parametrize("n,k", [(70, 33), (256, 64), (129, 200), (24, 1032), (520, 2056), (64, 8)])
def test_dense_linear(dev, bits, x_dtype, n, k):
    rng = np.random.default_rng(n + k)
    w = cases.bf16_round(rng.standard_normal((n, k)) / np.sqrt(k))
    bias = rng.standard_normal(n).astype(np.float32)
    qw, bt = nn.QWeight.dense(dev, w, bits), nn.Tensor.from_numpy(dev, bias)
    for m in (1, 2, 3, 4, 7, 16, 17, 33, 64, 100, 300):
        x = cases.bf16_round(rng.standard_normal((m, k)))
        want = x.astype(np.float64) @ w.astype(np.float64).T + bias
        if x_dtype == "bf16":
            raw = (x.view(np.uint32) >> 16).astype(np.uint16)
            got = nn._matmul_q(nn.Tensor.from_numpy(dev, raw, nn.BF16), qw, bt).numpy()
            got = (got.astype(np.uint32) << 16).view(np.float32)
            assert np.abs(got - want).max() <= 5e-3 * (1 + np.abs(want).max()), (m, n, k)
        else:
            got = nn._matmul_q(nn.Tensor.from_numpy(dev, x), qw, bt).numpy()
            assert np.abs(got - want).max() <= 3e-6 * (1 + np.abs(want).max()), (m, n, k)


def test_dense_weights_are_refused_where_only_quantized_ones_fit(dev):
    qw = nn.QWeight.dense(dev, np.ones((8, 16), np.float32), 16)
    with pytest.raises(nn.RuaiError, match="not quantized"):
        dev.check(dev.L.ruai_unpack(dev.ctx, qw.h, b"x" * 64, b"x" * 64))
    x = nn.Tensor.from_numpy(dev, np.ones((1, 8), np.float32))
    with pytest.raises(nn.RuaiError, match="not quantized"):
        nn.matmul_q_grad_input(x, qw)


# ---- mechanisms alone ---------------------------------------------------------------------------------------------

MECHANISMS = {
    "attention": [cases.attention()],
    "attention, no feed-forward": [cases.attention(ff=0)],
    "attention, nothing kept": [cases.attention(size=6, keep_first=0)],
    "attention, window of one": [cases.attention(size=1, keep_first=2)],
    "attention, chunk-sized window": [cases.attention(size=64, keep_first=64)],
    "attention, wide window": [cases.attention(size=500, keep_first=1)],
    "attention, many kept": [cases.attention(size=30, keep_first=70)],
    "attention, one head": [cases.attention(heads=1, kv_heads=1, dim=8, vdim=16)],
    "attention, heads of their own": [cases.attention(heads=3, kv_heads=3, dim=16, vdim=16)],
    "attention, 3 per group": [cases.attention(heads=6, kv_heads=2, dim=20, vdim=12, size=20)],
    "attention, 5 per group": [cases.attention(heads=5, kv_heads=1, dim=4, vdim=8)],
    "attention, 8 per group": [cases.attention(heads=16, kv_heads=2, dim=8, vdim=16)],
    "attention, 12 per group": [cases.attention(heads=12, kv_heads=1, dim=16, vdim=32)],
    "attention, odd sizes": [cases.attention(heads=2, kv_heads=2, dim=10, vdim=7, size=13, keep_first=5, ff=21)],
    "attention, large heads": [cases.attention(heads=4, kv_heads=2, dim=128, vdim=256, size=40)],
    "attention, larger values": [cases.attention(heads=2, kv_heads=1, dim=64, vdim=320, size=40)],
    "wkv": [cases.wkv()],
    "wkv, no feed-forward": [cases.wkv(ff=0)],
    "wkv, one head": [cases.wkv(heads=1, dim=64)],
    "wkv, odd sizes": [cases.wkv(heads=3, dim=13, ff=19)],
    "wkv, large heads": [cases.wkv(heads=2, dim=96)],
    "wkv, larger heads": [cases.wkv(heads=1, dim=180)],
    "wkv, largest heads": [cases.wkv(heads=1, dim=256)],
    "hgrn2": [cases.hgrn2()],
    "hgrn2, no feed-forward": [cases.hgrn2(ff=0)],
    "hgrn2, values wider": [cases.hgrn2(heads=2, dim=12, vdim=40)],
    "hgrn2, values narrow": [cases.hgrn2(heads=4, dim=32, vdim=1)],
    "hgrn2, odd sizes": [cases.hgrn2(heads=3, dim=7, vdim=9, ff=5)],
    "hgrn2, large heads": [cases.hgrn2(heads=1, dim=130, vdim=300)],
    "mixed": MIXED,
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_mechanism_whole_and_decoded(dev, name, dtype):
    cfg = cases.config(MECHANISMS[name], width=62 if "odd" in name else 64, vocab=61 if "odd" in name else 60, eps=1e-3 if "one head" in name else 1e-5)
    w, ids = cases.weights(cfg, seed=len(name), rank=5 if "odd" in name else 8), cases.tokens(cfg, 150)
    want = Z.forward(cfg, w, ids)
    m = build(dev, cfg, w, dtype)
    check(run(m, ids, [150]), want, dtype, "whole")
    check(run(m, ids, [90, 1]), want, dtype, "decoded")
    check(run(m, ids, [1, 1, 1, 60, 2]), want, dtype, "from one token on")


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_every_size(dev, dtype):
    cfg = cases.config(MIXED)
    w, ids = cases.weights(cfg, 3), cases.tokens(cfg, 170)
    want = Z.forward(cfg, w, ids)
    m = build(dev, cfg, w, dtype)
    for cuts in ([2], [3], [4, 5], [7], [8], [9], [15, 16, 17, 18], [31, 33, 2], [63, 2, 65], [1, 2, 1, 37], [64], [128, 42]):
        check(run(m, ids, cuts), want, dtype, f"portions {cuts}")
    check(run(m, ids, [1]), want, dtype, "token by token")


def test_long_prompt(dev):
    """Enough tokens for several per CTA of the norm and for many blocks of the scans."""
    cfg = cases.config(MIXED, max_positions=700)
    w, ids = cases.weights(cfg, 14), cases.tokens(cfg, 650)
    want = Z.forward(cfg, w, ids)
    m = build(dev, cfg, w, "float32")
    for cuts in ([650], [600, 7, 1], [3, 647]):
        check(run(m, ids, cuts), want, "float32", f"portions {cuts}")


def test_residual_stream_layer_by_layer(dev):
    """The stream after each layer, through models cut short with the identity for a head."""
    cfg = cases.config(MIXED, width=64, vocab=64)
    w, ids = cases.weights(cfg, 5), cases.tokens(cfg, 40)
    w["head"] = np.eye(64, dtype=np.float32)
    stream = []
    Z.forward(cfg, w, ids, stream)
    for n in range(1, len(MIXED) + 1):
        part = dict(cfg, layers=cfg["layers"][:n])
        m = build(dev, part, {k: v for k, v in w.items() if not k.startswith("l") or int(k[1:k.index(".")]) < n}, "float32")
        want = Z.rms(stream[n - 1], cfg["norm"]["eps"]) * w["final.norm"]
        assert np.abs(run(m, ids, [40]) - want).max() < 2e-5, n


# ---- edges of the window and of the kept first tokens -----------------------------------------------------------------

def pointed_model(size, keep, seed=0, n=0):
    """One attention layer in which token 0's queries are token 399's keys, and nobody else's: the embedding of 399 is that
    of 0 shifted by one channel, the key projection the query projection shifted likewise.  Positions and shift are off
    and the score scale is large, so that token 0 attends to a visible 399 and to little else."""
    cfg = cases.config([cases.attention(heads=2, kv_heads=2, dim=16, vdim=16, size=size, keep_first=keep, scale=0.8, ff=0)], vocab=400, max_positions=400)
    w = cases.weights(cfg, seed)
    w["embed"][399] = np.roll(w["embed"][0], 1)
    w["l0.mix.k"] = np.roll(w["l0.mix.q"], 1, axis=1)
    w["l0.mix.q.norm"] = w["l0.mix.k.norm"] = np.ones(16, np.float32)
    w["l0.shift"] = np.zeros(64, np.float32)
    w["pos"] = np.zeros_like(w["pos"])
    ids = np.random.default_rng(size).permutation(np.arange(1, 399))[:n].astype(np.int32)  # no token twice
    return cfg, w, ids


@pytest.mark.parametrize("size,keep,n", [(9, 3, 40), (64, 0, 150), (63, 5, 150), (65, 64, 200), (100, 20, 260), (1, 1, 12)])
def test_window_and_kept_edges(dev, size, keep, n):
    cfg, w, base = pointed_model(size, keep, n=n)
    models = {dtype: build(dev, cfg, w, dtype) for dtype in DTYPES}
    for q in {n - 1, min(n - 1, keep + size), min(n - 1, keep + size - 1)}:
        for at in {q - size, q - size + 1, q - size - 1, keep - 1, keep, 0, q // 2}:
            if not 0 <= at < q:
                continue
            ids = base[:q + 1].copy()
            ids[at], ids[q] = 399, 0
            want = Z.forward(cfg, w, ids)
            for dtype, m in models.items():
                for cuts in ([q + 1], [q, 1], [max(1, q - 5), 2]):
                    check(run(m, ids, cuts)[q], want[q], dtype, f"query {q}, key {at}, portions {cuts}")


def test_a_moved_edge_would_show():
    """The cases above tell a window or a kept prefix that is one token off from the right one (checked on the oracle)."""
    size, keep, n = 9, 3, 40
    cfg, w, ids = pointed_model(size, keep, n=n)
    ids[n - 1] = 0
    seen = {}
    for at, d_size, d_keep in ((n - 1 - size, 1, 0), (n - size, -1, 0), (keep - 1, 0, -1), (keep, 0, 1)):
        t = ids.copy()
        t[at] = 399
        right = Z.forward(cfg, w, t)[n - 1]
        wrong = dict(cfg, layers=[cases.attention(heads=2, kv_heads=2, dim=16, vdim=16, size=size + d_size, keep_first=keep + d_keep, scale=0.8, ff=0)])
        seen[(d_size, d_keep)] = cases.rel_error(Z.forward(wrong, w, t)[n - 1], right)
    assert min(seen.values()) > 2 * TOL["bfloat16"], seen


def test_far_state_shows(dev):
    """Slow decays: the first tokens still reach the last ones through the states, whole and decoded."""
    cfg = cases.config([cases.wkv(heads=2, dim=16, ff=0), cases.hgrn2(heads=2, dim=16, vdim=16, ff=0)], max_positions=400)
    w = cases.weights(cfg, 8)
    w["l0.mix.w0"] = np.full(32, -9.0, np.float32)
    w["l1.mix.lower"] = np.full(32, 0.99609375, np.float32)
    ids = cases.tokens(cfg, 300)
    other = ids.copy()
    other[:4] = (other[:4] + 7) % 60
    want = Z.forward(cfg, w, ids)
    assert cases.rel_error(Z.forward(cfg, w, other)[-1], want[-1]) > 1e-3  # the far tokens matter
    m = build(dev, cfg, w, "float32")
    for cuts in ([300], [4, 1], [4, 37], [150, 2]):
        check(run(m, ids, cuts), want, "float32", f"portions {cuts}")


# ---- cache and states ------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
def test_cleared_cache_and_states_leave_nothing(dev, dtype):
    cfg = cases.config(MIXED)
    w = cases.weights(cfg, 4)
    a, b = cases.tokens(cfg, 90, 1), cases.tokens(cfg, 70, 2)
    m = build(dev, cfg, w, dtype)
    fresh = run(m, b, [50, 1])
    run(m, a, [33, 1])
    assert np.array_equal(run(m, b, [50, 1]), fresh)
    run(m, a, [1])
    assert np.array_equal(run(m, b, [50, 1]), fresh)
    assert m.cache_len() == 70
    check(fresh, Z.forward(cfg, w, b), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_grows_the_cache(dev, dtype):
    cfg = cases.config([cases.attention(size=40, keep_first=4), cases.wkv(), cases.hgrn2()], max_positions=300)
    w, ids = cases.weights(cfg, 6), cases.tokens(cfg, 300)
    m = build(dev, cfg, w, dtype)
    caps = set()
    m.cache_clear()
    rows = []
    for t in ids:
        rows.append(m.forward_cached(np.array([[t]]))[0])
        caps.add(m.cache_capacity())
    assert len(caps) > 3
    check(np.stack(rows), Z.forward(cfg, w, ids), dtype)
    m2 = build(dev, cfg, w, dtype)
    m2.cache_reserve(1, 300)
    check(run(m2, ids, [37]), Z.forward(cfg, w, ids), dtype, "reserved")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_side_by_side(dev, dtype):
    """Sequences of one length in a batch give what each gives alone; then single-token steps of the batch."""
    cfg = cases.config(MIXED)
    w = cases.weights(cfg, 7)
    m = build(dev, cfg, w, dtype)
    for B, T in ((3, 45), (18, 10), (2, 5)):
        ids = np.stack([cases.tokens(cfg, T + 6, 10 + b) for b in range(B)])
        want = np.stack([Z.forward(cfg, w, r) for r in ids])
        m.cache_clear()
        got = [m.forward_cached(ids[:, :T], all_positions=True)]
        for t in range(T, T + 6):
            got.append(m.forward_cached(ids[:, t:t + 1])[:, None])
        got = np.concatenate(got, axis=1)
        for b in range(B):
            check(got[b], want[b], dtype, f"sequence {b} of {B}")


@pytest.mark.parametrize("layer", [cases.hgrn2(heads=16, dim=8, vdim=64, ff=0), cases.hgrn2(heads=16, dim=72, vdim=64, ff=0), cases.wkv(heads=16, dim=64, ff=0),
                                   cases.wkv(heads=8, dim=128, ff=0), cases.wkv(heads=12, dim=144, ff=0)], ids=["8x64", "72x64", "64", "128", "144"])
def test_recurrences_of_many_sequences(dev, layer):
    """Batches large enough for every number of value columns per thread."""
    cfg = cases.config([layer], max_positions=40)
    w = cases.weights(cfg, 17)
    m = build(dev, cfg, w, "float32")
    for B in (1, 4, 10):
        ids = np.stack([cases.tokens(cfg, 15, 30 + b) for b in range(B)])
        m.cache_clear()
        got = np.concatenate([m.forward_cached(ids[:, :9], all_positions=True), m.forward_cached(ids[:, 9:11], all_positions=True),
                              m.forward_cached(ids[:, 11:12], all_positions=True), m.forward_cached(ids[:, 12:], all_positions=True)], axis=1)
        for b in {0, B // 2, B - 1}:
            check(got[b], Z.forward(cfg, w, ids[b]), "float32", f"sequence {b} of {B}")


def test_rows_of_a_step(dev):
    cfg = cases.config(MIXED)
    w, ids = cases.weights(cfg, 9), cases.tokens(cfg, 50)
    m = build(dev, cfg, w, "float32")
    full = run(m, ids, [50])
    m.cache_clear()
    assert m.forward_rows(ids[None, :30], []).shape == (0, 60)
    assert np.abs(m.forward_rows(ids[None, 30:49], [18, 0, 7]) - full[[48, 30, 37]]).max() < 1e-4
    assert np.abs(m.forward_rows(ids[None, 49:], [0]) - full[49]).max() < 1e-4
    assert np.abs(run(m, ids, [50])[-1] - m_last(m, ids)).max() < 1e-4
    with pytest.raises(nn.RuaiError, match="row 3"):
        m.forward_rows(ids[None, :3], [3])


def m_last(m, ids):
    m.cache_clear()
    return m.forward_cached(ids[None, :])[0]


def test_errors(dev):
    cfg = cases.config([cases.attention(), cases.wkv()], max_positions=20)
    w = cases.weights(cfg)
    m = build(dev, cfg, w, "bfloat16")
    with pytest.raises(nn.RuaiError, match="max_positions"):
        m.forward_cached(np.zeros((1, 21), np.int32))
    with pytest.raises(nn.RuaiError, match="out of range"):
        m.forward_cached(np.full((1, 4), 60, np.int32))
    m.cache_clear()
    m.forward_cached(np.zeros((1, 20), np.int32))
    with pytest.raises(nn.RuaiError, match="max_positions"):
        m.forward_cached(np.zeros((1, 1), np.int32))
    broken = nn.Zazasun(dev, nn.ZazasunConfig(cfg, 8))
    with pytest.raises(nn.RuaiError, match="does not exist"):
        broken.set_tensor("l0.mix.nothing", np.zeros(3))
    with pytest.raises(nn.RuaiError, match="elements"):
        broken.set_tensor("embed", np.zeros(3))
    with pytest.raises(nn.RuaiError, match="was not set"):
        broken.build()
    with pytest.raises(nn.RuaiError, match="unquantized"):
        nn.Zazasun(dev, nn.ZazasunConfig(cfg, 8)).quantize_int8()
    bad = cases.config([cases.attention(heads=4, kv_heads=3)])
    with pytest.raises(nn.RuaiError, match="multiple of kv_heads"):
        nn.Zazasun(dev, nn.ZazasunConfig(bad))


# ---- generation through the library's own entry points ------------------------------------------------------------------

def greedy(cfg, w, ids, n, limit):
    """Greedy continuation by the oracle, and the smallest gap between the two best logits on the way."""
    ids, gap = list(ids), np.inf
    for _ in range(n):
        row = Z.forward(cfg, w, ids[-limit:])[-1]
        top = np.sort(row)[-2:]
        gap = min(gap, (top[1] - top[0]) / row.std())
        ids.append(int(row.argmax()))
    return ids, gap


@pytest.mark.parametrize("prompt_len", [1, 2, 13])
def test_greedy_generation(dev, prompt_len):
    cfg = cases.config(MIXED, max_positions=64)
    w = cases.weights(cfg, 11)
    prompt = cases.tokens(cfg, prompt_len, 3)
    want, gap = greedy(cfg, w, prompt, 24, 64)
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


def test_generation_slides_past_the_last_position(dev):
    cfg = cases.config([cases.attention(), cases.wkv(), cases.hgrn2()], max_positions=20)
    w = cases.weights(cfg, 12)
    prompt = cases.tokens(cfg, 14, 3)
    want, gap = greedy(cfg, w, prompt, 14, 20)
    assert gap > 1e-4
    assert build(dev, cfg, w, "float32").generate(prompt, 14).tolist() == want


def test_command_line_and_trace_runner(dev, tmp_path, capsys):
    cfg = cases.config(MIXED)
    w, ids = cases.weights(cfg, 13), cases.tokens(cfg, 40)
    cases.save(tmp_path, cfg, w)
    want = Z.forward(cfg, w, ids)
    check(run(registry.load(dev, str(tmp_path)), ids, [31, 1]), want, "bfloat16", "registry")
    assert cli.main(["info", "--model", str(tmp_path)]) == 0 and capsys.readouterr().out.strip() == "zazasun"
    expected, gap = greedy(cfg, w, ids[:9], 8, 300)
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
