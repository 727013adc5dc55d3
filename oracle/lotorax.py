"""Plain, slow CPU restatement of the Lotorax design in float64 numpy: one function per mechanism, token after token where
the mechanism is a recurrence, one (query, head) after the other where it is an attention.  Test infrastructure only; it
shares no code with the product path.

Weights come as a dict name -> float array, the configuration as the dict of a model's config.json.
"""
import math

import numpy as np


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    mean = x.mean(axis=-1, keepdims=True)
    var = ((x - mean) ** 2).mean(axis=-1, keepdims=True)
    return (x - mean) / np.sqrt(var + eps) * w + b


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


# ---- rotation -----------------------------------------------------------------------------------------------------

def frequencies(rot):
    """Angle per position of every pair, and the factor of its cosine and sine, with the frequencies interpolated where a
    pair turns too slowly within the original context (YaRN)."""
    dims, base = rot["dims"], rot["base"]
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def turns(t):  # the (real-valued) pair index that makes t turns within the original context
        return dims * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, position, rot):
    """x [..., n] at one position: neighbouring dimensions are pairs; those past rot["dims"] stay."""
    f, m = frequencies(rot)
    out = np.array(x)
    for i, fi in enumerate(f):
        c, s = m * math.cos(position * fi), m * math.sin(position * fi)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---- latent attention ---------------------------------------------------------------------------------------------

def sink_attention(q, k, v, scale, sink):
    """One head: q, k [T, n], v [T, vdim]; the sink is one more term of the denominator."""
    out = np.zeros((q.shape[0], v.shape[1]))
    for i in range(q.shape[0]):
        s = (k[: i + 1] @ q[i]) * scale
        top = max(s.max(), sink)
        e = np.exp(s - top)
        out[i] = (e / (e.sum() + np.exp(sink - top))) @ v[: i + 1]
    return out


def latent_attention_mixer(h, w, p, m, eps):
    T, H, dim, r, vdim, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, dim + r)
    dkv = h @ w[p + "dkv"].T
    c = rms(dkv[:, :rank], eps) * w[p + "dkv.norm"]
    kr = np.stack([rotate(dkv[t, rank:], t, m["rot"]) for t in range(T)])
    qr = np.stack([rotate(q[t, :, dim:], t, m["rot"]) for t in range(T)])
    k = (c @ w[p + "uk"].T).reshape(T, H, dim)
    v = (c @ w[p + "uv"].T).reshape(T, H, vdim)
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.zeros((T, H, vdim))
    for i in range(H):
        out[:, i] = sink_attention(np.concatenate([q[:, i, :dim], qr[:, i]], 1), np.concatenate([k[:, i], kr], 1), v[:, i], m["scale"], w[p + "sink"][i])
        out[:, i] *= gate[:, i : i + 1]
    return out.reshape(T, H * vdim) @ w[p + "o"].T


# ---- gated delta rule ---------------------------------------------------------------------------------------------

def causal_conv(x, taps):
    """x [T, channels], taps [channels, n]: each channel's own weighted sum of its last n values, the newest last."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return np.stack([(padded[t : t + n] * taps.T).sum(0) for t in range(x.shape[0])])


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_recurrence(q, k, v, decay, beta):
    """One head: q, k [T, dim], v [T, vdim], decay, beta [T].  The state decays, its answer to k moves towards v by beta,
    and q reads what is there then."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(k.shape[0]):
        S = S * decay[t]
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out


def delta_mixer(h, w, p, m, eps):
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q = unit(q.reshape(T, G, dim)) * dim ** -0.5
    k = unit(k.reshape(T, G, dim))
    v = v.reshape(T, H, vdim)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = np.stack([delta_recurrence(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], decay[:, i], beta[:, i]) for i in range(H)], axis=1)
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).reshape(T, H, vdim)
    return o.reshape(T, H * vdim) @ w[p + "o"].T


# ---- feed-forward -------------------------------------------------------------------------------------------------

def gated(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, top):
    """Per token the chosen experts and their weights."""
    s = sigmoid(h @ w[p + "router"].T)
    chosen = np.argsort(-(s + w[p + "correction"]), axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, -1)


def experts(h, w, p, mlp):
    chosen, weight = route(h, w, p, mlp["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t], weight[t]):
            out[t] += a * gated(h[t], w, f"{p}e{e}.", silu)
    return out


def feed_forward(h, w, p, mlp):
    return experts(h, w, p, mlp) if mlp["kind"] == "moe" else gated(h, w, p, lambda z: np.maximum(z, 0.0))


# ---- the model ----------------------------------------------------------------------------------------------------

MIXERS = {"latent_attention": latent_attention_mixer, "delta": delta_mixer}


def schedule(cfg):
    """(layer, whether a pass of the loop begins with it) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    body = [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return [(i, False) for i in range(loop["start"])] + body * loop["times"] + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  layers_out, a list, receives the residual stream after every layer run."""
    w = {n: np.asarray(t, np.float64) for n, t in w.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)

    x = x0 = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, first in schedule(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if first:
            x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T
        x = x + norm(MIXERS[layer["type"]](norm(x, p + "norm1"), w, p + "mix.", layer["mixer"], eps), p + "norm1b")
        if layer.get("mlp"):
            x = x + norm(feed_forward(norm(x, p + "norm2"), w, p + "mlp.", layer["mlp"]), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm(x, "final.norm") @ w["head"].T
