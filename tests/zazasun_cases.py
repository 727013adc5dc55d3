"""Small Zazasun configurations and random weights for the tests (no GPU, no product code)."""
import json
import struct

import numpy as np


def bf16_round(a):
    """f32 values rounded to the nearest bf16, so that both number formats of the product hold them exactly."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def attention(heads=4, kv_heads=2, dim=16, vdim=24, size=9, keep_first=3, scale=None, diff=0.35, ff=40):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep_first},
                                           "scale": dim ** -0.5 if scale is None else scale, "diff": diff},
            "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def wkv(heads=3, dim=16, ff=40):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def hgrn2(heads=3, dim=16, vdim=8, ff=40):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def config(layers, vocab=60, width=64, max_positions=300, eps=1e-5):
    return {"architecture": "Zazasun", "layers": layers, "max_positions": max_positions, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def weights(cfg, seed=0, rank=8):
    """Random weights (bf16 values) that keep every branch alive: gains away from 1, decays of all lengths, lower bounds up to 0.9."""
    rng = np.random.default_rng(seed)
    d, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return rng.standard_normal((n, k)) * gain / np.sqrt(k)

    w = {"embed": rng.standard_normal((V, d)), "pos": 0.3 * rng.standard_normal((cfg["max_positions"], d)), "final.norm": np.array(1.3), "head": mat(V, d, 2.0)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        w[p + "norm1"] = np.array(rng.uniform(0.7, 1.4))
        w[p + "shift"] = rng.uniform(0, 1, d)
        hk, hv = m["heads"] * m["dim"], m["heads"] * m.get("vdim", m["dim"])
        if layer["type"] == "attention":
            g = m["kv_heads"]
            w.update({x + "q": mat(2 * hk, d), x + "k": mat(2 * g * m["dim"], d), x + "v": mat(g * m["vdim"], d),
                      x + "q.norm": rng.uniform(0.8, 2.0, m["dim"]), x + "k.norm": rng.uniform(0.8, 2.0, m["dim"])})
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[x + n] = 0.3 * rng.standard_normal(m["dim"])
        elif layer["type"] == "wkv":
            for s in "rkvgw":
                w[x + "mu." + s] = rng.uniform(0, 1, d)
            for s in "rkvg":
                w[x + s] = mat(hk, d)
            w.update({x + "w1": mat(rank, d, 2.0), x + "w2": mat(hk, rank), x + "w0": rng.uniform(-5.0, 0.5, hk), x + "u": rng.standard_normal((m["heads"], m["dim"])),
                      x + "norm": rng.uniform(0.5, 1.5, hk)})
        else:
            w.update({x + "q": mat(hk, d), x + "f": mat(hk, d), x + "f.b": rng.uniform(-1, 3, hk), x + "lower": rng.uniform(0, 0.9, hk), x + "v": mat(hv, d),
                      x + "norm": rng.uniform(0.5, 1.5, m["vdim"])})
        w[x + "o"] = mat(d, hv)
        if layer.get("mlp"):
            f = layer["mlp"]["ff"]
            w.update({p + "mlp.gate": mat(f, d), p + "mlp.up": mat(f, d), p + "mlp.down": mat(d, f)})
    return {n: bf16_round(a) for n, a in w.items()}


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


def save(folder, cfg, w):
    """config.json and model.safetensors with bf16 tensors, as a checkpoint holds them."""
    with open(folder / "config.json", "w") as f:
        json.dump(cfg, f)
    head, blob = {}, b""
    for n, a in w.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[n] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    h = json.dumps(head).encode()
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + blob)


def rel_error(got, want):
    """Root mean square of the difference over the vocabulary, row by row, in units of the logits' spread."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()
