"""Small Lotorax configurations and random weights for the tests (no GPU, no product code)."""
import numpy as np

from zazasun_cases import bf16_round, rel_error, save, tokens  # noqa: F401

YARN = {"factor": 8.0, "fast": 4.0, "original": 40, "slow": 0.5}


def dense(ff=40):
    return {"ff": ff, "kind": "dense"}


def moe(experts=6, top=2, ff=24):
    return {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}


def latent(heads=3, dim=16, rot_dim=8, vdim=12, rank=20, scale=None, base=10000.0, scaling=YARN, mlp=dense()):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale,
                      "rot": {"base": base, "dims": rot_dim, "scaling": scaling}}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, mlp=dense()):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def loop(start, stop, times):
    return {"start": start, "stop": stop, "times": times}


def config(layers, loop=None, vocab=60, width=64, eps=1e-5, scale=3.25):
    c = {"architecture": "Lotorax", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = loop
    return c


def weights(cfg, seed=0, settled=False):
    """Random weights (bf16 values) that keep every branch alive: decays of all lengths, sinks that matter, norms away from 1.
    settled: every token uses the same experts whatever its rounding, so that bf16 can be compared token by token."""
    rng = np.random.default_rng(seed)
    d, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return rng.standard_normal((n, k)) * gain / np.sqrt(k)

    w = {"embed": 0.4 * rng.standard_normal((V, d)), "head": mat(V, d, 2.0)}

    def norm(name, n, low=0.5, high=1.5):
        w[name], w[name + ".b"] = rng.uniform(low, high, n), 0.2 * rng.standard_normal(n)

    norm("final.norm", d)
    if cfg.get("loop"):
        w["loop.in"] = mat(d, 2 * d)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        x, H = p + "mix.", m["heads"]
        norm(p + "norm1", d)
        norm(p + "norm1b", d, 0.2, 0.7)  # a layer adds less than the stream holds: rounding stays small
        if layer["type"] == "delta":
            gk, hv = m["kv_heads"] * m["dim"], H * m["vdim"]
            for n, size in (("q", gk), ("k", gk), ("v", hv)):
                w[x + n], w[x + n + ".conv"] = mat(size, d), rng.uniform(-1, 1, (size, m["conv"]))
            w.update({x + "b": mat(H, d, 1.5), x + "a": mat(H, d), x + "A_log": np.log(rng.uniform(0.02, 4.0, H)), x + "dt_bias": rng.uniform(-4, 1, H),
                      x + "norm": rng.uniform(0.5, 1.5, m["vdim"]), x + "g": mat(hv, d)})
        else:
            r, hv = m["kv_rank"], H * m["vdim"]
            w.update({x + "q": mat(H * (m["dim"] + m["rot_dim"]), d, 2.0), x + "dkv": mat(r + m["rot_dim"], d), x + "dkv.norm": rng.uniform(0.7, 1.5, r),
                      x + "uk": mat(H * m["dim"], r), x + "uv": mat(hv, r), x + "sink": rng.uniform(-1, 3, H), x + "g": mat(H, d, 1.5)})
        w[x + "o"] = mat(d, hv)
        if not mlp:
            continue
        norm(p + "norm2", d)
        norm(p + "norm2b", d, 0.2, 0.7)
        q = p + "mlp."
        if mlp["kind"] == "dense":
            w.update({q + "gate": mat(mlp["ff"], d), q + "up": mat(mlp["ff"], d), q + "down": mat(d, mlp["ff"])})
        else:
            E, f = mlp["router"]["experts"], mlp["expert"]["ff"]
            for e in range(E):
                w.update({f"{q}e{e}.gate": mat(f, d), f"{q}e{e}.up": mat(f, d), f"{q}e{e}.down": mat(d, f)})
            w[q + "router"] = mat(E, d, 1.5)
            w[q + "correction"] = 1.5 * rng.permutation(E) if settled else rng.uniform(-0.4, 0.4, E)
    return {n: bf16_round(a) for n, a in w.items()}
