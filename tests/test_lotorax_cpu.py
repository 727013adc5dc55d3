"""CPU tests of the Lotorax restatement (oracle/lotorax.py), configuration, registry and loading (no GPU)."""
import numpy as np
import pytest

import lotorax_cases as cases
import oracle.lotorax as X
from ruai_b200 import _lib, checkpoint, nn, registry


def test_layer_norm():
    x = np.random.default_rng(0).standard_normal((5, 9)) * 3 + 2
    y = X.layer_norm(x, np.ones(9), np.zeros(9), 0.0)
    assert np.allclose(y.mean(-1), 0) and np.allclose((y * y).mean(-1), 1)
    assert np.allclose(X.layer_norm(x + 7, np.full(9, 2.0), np.full(9, 3.0), 0.0), 2 * y + 3)


def test_rotation_keeps_lengths_and_depends_on_the_distance():
    rot = {"base": 100.0, "dims": 6, "scaling": None}
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal(6), rng.standard_normal(6)
    assert np.isclose(np.linalg.norm(X.rotate(q, 13, rot)), np.linalg.norm(q))
    assert np.isclose(X.rotate(q, 13, rot) @ X.rotate(k, 4, rot), X.rotate(q, 29, rot) @ X.rotate(k, 20, rot))
    one = X.rotate(np.array([1.0, 0, 0, 0, 0, 0]), 1, rot)
    assert np.allclose(one, [np.cos(1), np.sin(1), 0, 0, 0, 0])


def test_interpolated_frequencies():
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 1.0}}
    f, m = X.frequencies(rot)
    plain, one = X.frequencies(dict(rot, scaling=None))
    assert one == 1.0 and np.isclose(m, 1 + 0.1 * np.log(4))
    ratio = f / plain
    assert np.isclose(ratio[0], 1) and np.isclose(ratio[-1], 0.25) and np.all(np.diff(ratio) <= 1e-12)
    # pairs that turn more than 8 times within the original context keep their frequency, those that turn less than once lose it
    turns = 256 * plain / (2 * np.pi)
    assert np.allclose(ratio[turns > 16], 1) and np.allclose(ratio[turns < 0.5], 0.25)


def test_a_sink_takes_its_share():
    q, k, v = np.zeros((3, 2)), np.zeros((3, 2)), np.ones((3, 1))
    assert np.allclose(X.sink_attention(q, k, v, 1.0, 0.0)[:, 0], [1 / 2, 2 / 3, 3 / 4])
    assert np.allclose(X.sink_attention(q, k, v, 1.0, -200.0), 1.0)


def test_causal_convolution():
    x = np.arange(1.0, 6.0)[:, None]
    assert np.allclose(X.causal_conv(x, np.array([[100.0, 10.0, 1.0]]))[:, 0], [1, 12, 123, 234, 345])


def test_delta_rule_stores_and_overwrites():
    """Without decay and with beta 1 a unit key answers with the last value that was written under it."""
    k = np.array([[1.0, 0], [0, 1], [1, 0], [0.6, 0.8]])
    v = np.array([[3.0], [5], [7], [0]])
    one = np.ones(4)
    o = X.delta_recurrence(k, k, v, one, one)
    assert np.allclose(o[:, 0], [3, 5, 7, 0])
    o = X.delta_recurrence(np.array([[0.0, 1], [1, 0], [0, 1], [1, 0]]), k, v, one, one)
    assert np.allclose(o[:3, 0], [0, 3, 5])
    o = X.delta_recurrence(k, k, v, np.full(4, 0.5), np.zeros(4))
    assert np.allclose(o, 0)


def test_routing_chooses_by_corrected_scores_and_weighs_by_plain_ones():
    w = {"router": np.eye(3), "correction": np.array([0.0, 0.9, 0.0])}
    chosen, weight = X.route(np.array([[2.0, 0.0, 1.0]]), w, "", 2)
    assert chosen.tolist() == [[1, 0]]
    assert np.allclose(weight, X.sigmoid(np.array([[0.0, 2.0]])))


def test_order_of_layers():
    layers = [cases.delta()] * 5
    assert X.schedule(cases.config(layers)) == [(i, False) for i in range(5)]
    assert X.schedule(cases.config(layers, cases.loop(1, 3, 2))) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]
    assert X.schedule(cases.config(layers, cases.loop(0, 5, 1))) == [(0, True)] + [(i, False) for i in range(1, 5)]


def test_a_prefix_does_not_see_what_follows():
    cfg = cases.config([cases.delta(mlp=cases.moe()), cases.latent()], cases.loop(0, 2, 2))
    w, ids = cases.weights(cfg), cases.tokens(cfg, 20)
    assert np.allclose(X.forward(cfg, w, ids)[:13], X.forward(cfg, w, ids[:13]))


def test_configuration_reads_every_size_and_constant():
    cfg = cases.config([cases.latent(5, 10, 6, 14, 33, scale=0.3, base=77.5, scaling={"factor": 3.0, "original": 99, "fast": 7.0, "slow": 0.25}, mlp=cases.moe(9, 4, 13)),
                        cases.delta(6, 3, 12, 7, 5, mlp=None), cases.delta(mlp=cases.dense(17)), cases.latent(scaling=None)],
                       cases.loop(1, 3, 4), vocab=77, width=36, eps=3e-4, scale=1.75)
    c = nn.LotoraxConfig(cfg)
    assert (c.vocab_size, c.width, c.c.num_layers, c.c.block) == (77, 36, 4, _lib.BLOCK_SANDWICH)
    assert (c.c.loop_start, c.c.loop_stop, c.c.loop_times, c.c.embed_scale) == (1, 3, 4, 1.75) and np.isclose(c.c.norm_eps, 3e-4)
    a, d, e, f = c.layers
    assert (a.mixer, a.heads, a.dim, a.rot_dim, a.rot_dims, a.vdim, a.rank) == (_lib.MIX_LATENT, 5, 10, 6, 6, 14, 33)
    assert (a.rot_base, a.yarn_factor, a.yarn_original, a.yarn_fast, a.yarn_slow) == (77.5, 3.0, 99.0, 7.0, 0.25) and np.isclose(a.scale, 0.3)
    assert (a.ff, a.ff_act, a.experts, a.top) == (13, _lib.FF_SILU, 9, 4)
    assert (d.mixer, d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.ff) == (_lib.MIX_DELTA, 6, 3, 12, 7, 5, 0)
    assert (e.ff, e.ff_act, e.experts) == (17, _lib.FF_RELU, 0)
    assert f.yarn_factor == 0.0
    plain = nn.LotoraxConfig(cases.config([cases.delta()]))
    assert plain.c.loop_times == 0
    with pytest.raises(ValueError, match="unknown mixer"):
        nn.LotoraxConfig(cases.config([dict(cases.delta(), type="other")]))
    with pytest.raises(ValueError, match="unknown feed-forward"):
        nn.LotoraxConfig(cases.config([cases.delta(mlp={"kind": "other"})]))


def test_registry_and_file(tmp_path):
    cfg = cases.config([cases.latent(mlp=cases.moe()), cases.delta()], cases.loop(0, 1, 2))
    w = cases.weights(cfg)
    cases.save(tmp_path, cfg, w)
    assert registry.architecture(registry.read_config(tmp_path)) == "lotorax"
    got = checkpoint.load_file(tmp_path / "model.safetensors")
    assert set(got) == set(w)
    assert all(np.array_equal(checkpoint._as_f32(got[n]), w[n]) for n in w)
    with pytest.raises(ValueError, match="unquantized"):
        registry.MODELS["lotorax"](None, cfg, None, "bfloat16", 8, 32)
