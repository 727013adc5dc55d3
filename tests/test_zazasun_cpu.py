"""CPU tests of the Zazasun restatement (oracle/zazasun.py), configuration, registry and loading (no GPU)."""
import json

import numpy as np
import pytest

import oracle.zazasun as Z
import zazasun_cases as cases
from ruai_b200 import checkpoint, nn, registry, trace


def test_window_and_kept_tokens():
    seen = {(i, j) for i in range(12) for j in range(12) if Z.sees(i, j, 4, 2)}
    assert {j for i, j in seen if i == 9} == {0, 1, 6, 7, 8, 9}
    assert {j for i, j in seen if i == 3} == {0, 1, 2, 3}
    assert {j for i, j in seen if i == 0} == {0}
    assert not any(j > i for i, j in seen)


def test_bonus_recurrence_closed_form():
    """o_t = sum_{s<t} (r_t . prod_{s<q<t} w_q k_s) v_s + (r_t . u k_t) v_t."""
    rng = np.random.default_rng(0)
    T, dk, dv = 7, 3, 2
    r, k, w = (rng.standard_normal((T, dk)) for _ in range(3))
    w = 1 / (1 + np.exp(-w))
    v, u = rng.standard_normal((T, dv)), rng.standard_normal(dk)
    got = Z.bonus_recurrence(r, k, v, w, u)
    for t in range(T):
        want = (r[t] @ (u * k[t])) * v[t]
        for s in range(t):
            want = want + (r[t] @ (np.prod(w[s + 1:t], axis=0) * k[s])) * v[s]
        assert np.allclose(got[t], want)


def test_gated_recurrence_keeps_a_constant():
    """With v constant the state is a running mean of it: it tends to v per unit of q."""
    f, q, v = np.full((200, 1), 0.9), np.ones((200, 1)), np.full((200, 1), 3.0)
    got = Z.gated_recurrence(q, f, v)
    assert np.isclose(got[0, 0], 0.3) and np.isclose(got[-1, 0], 3.0, atol=1e-6)


def test_second_map_cancels_the_first():
    a = np.random.default_rng(1).standard_normal((4, 6))
    assert np.allclose(Z.combine_maps(a, a, 1.0, 0.2, 1e-5), 0.0)
    b = Z.combine_maps(a, 0 * a, 0.5, 0.2, 0.0)
    assert np.allclose(np.sqrt((b * b).mean(-1)), 0.8)


def test_a_prefix_does_not_see_what_follows():
    cfg = cases.config([cases.attention(), cases.wkv(), cases.hgrn2()])
    w, ids = cases.weights(cfg), cases.tokens(cfg, 20)
    assert np.allclose(Z.forward(cfg, w, ids)[:13], Z.forward(cfg, w, ids[:13]))


def test_configuration_reads_every_size_and_constant():
    cfg = cases.config([cases.attention(heads=6, kv_heads=3, dim=20, vdim=12, size=5, keep_first=0, scale=0.7, diff=0.1, ff=0), cases.wkv(5, 10), cases.hgrn2(2, 6, 14, 30)],
                       vocab=77, width=36, max_positions=99, eps=3e-4)
    c = nn.ZazasunConfig(cfg, [0, 7, 0])
    assert (c.vocab_size, c.width, c.max_positions) == (77, 36, 99) and np.isclose(c.c.norm_eps, 3e-4) and c.c.num_layers == 3
    a, r, h = c.layers
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first, a.ff) == (0, 6, 3, 20, 12, 5, 0, 0)
    assert np.isclose(a.scale, 0.7) and np.isclose(a.diff, 0.1)
    assert (r.mixer, r.heads, r.dim, r.rank, r.ff) == (1, 5, 10, 7, 40)
    assert (h.mixer, h.heads, h.dim, h.vdim, h.ff) == (2, 2, 6, 14, 30)
    cfg["layers"][1]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        nn.ZazasunConfig(cfg)


def test_registry_chooses_by_configuration(tmp_path):
    assert registry.architecture({"architecture": "Zazasun"}) == "zazasun"
    assert registry.architecture({"architectures": ["LlamaForCausalLM"]}) == "llama"
    assert registry.architecture({"model_type": "gpt2"}) == "gpt2"
    with pytest.raises(ValueError, match="known: gpt2, llama, .*zazasun"):
        registry.architecture({"model_type": "none"})
    with pytest.raises(ValueError, match="dtype"):
        registry.load(None, str(tmp_path), "float16")


def test_checkpoint_round_trip(tmp_path):
    cfg = cases.config([cases.wkv()])
    w = cases.weights(cfg)
    cases.save(tmp_path, cfg, w)
    got = {n: checkpoint._as_f32(t) for n, t in checkpoint.load_file(tmp_path / "model.safetensors").items()}
    assert got.keys() == w.keys() and all(np.array_equal(got[n], w[n]) and got[n].shape == w[n].shape for n in w)
    assert json.load(open(tmp_path / "config.json")) == cfg


class FakeModel:
    vocab = 3

    def __init__(self):
        self.calls = []

    def cache_clear(self):
        self.calls.append("clear")

    def forward_rows(self, ids, rows):
        self.calls.append((ids.tolist(), list(rows)))
        return np.zeros((len(rows), self.vocab), np.float32)


def test_replay_keeps_one_live_request():
    m = FakeModel()
    r = trace.Replay(m)
    assert r.step([{"id": "a", "tokens": [1, 2], "want": [1]}], []).shape == (1, 3)
    assert r.step([{"id": "a", "tokens": [3], "want": []}], ["a"]).shape == (0, 3)
    r.step([{"id": "b", "tokens": [4]}], [])
    with pytest.raises(ValueError, match="before 'b' ended"):
        r.step([{"id": "c", "tokens": [5]}], [])
    with pytest.raises(ValueError, match="one request"):
        r.step([{"id": "b", "tokens": [5]}, {"id": "c", "tokens": [5]}], [])
    assert m.calls == ["clear", ([[1, 2]], [1]), ([[3]], []), "clear", "clear", ([[4]], [])]
