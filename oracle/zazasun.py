"""Plain, slow CPU restatement of the Zazasun design in float64 numpy: one function per mechanism, token after token
where the mechanism is a recurrence, one (query, head) after the other where it is an attention.  Test infrastructure
only; it shares no code with the product path.

Weights come as a dict name -> float array, the configuration as the dict of a model's config.json.
"""
import numpy as np


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def previous(h):
    """Row t of the result is row t - 1 of h; zeros ahead of the first token."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]], axis=0)


def mix_previous(h, mu):
    """Every element moved towards the previous token's by its own share mu."""
    return h + (previous(h) - h) * mu


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def sees(i, j, window, keep_first):
    """Whether position i attends to position j: causal, the last `window` positions (i itself is one) and the kept first ones."""
    return j <= i and (i - j < window or j < keep_first)


def softmax_attention(q, k, v, scale, window, keep_first):
    """q [T, dim], k [T, dim], v [T, vdim] of one head: softmax over the visible keys, position by position."""
    out = np.zeros((q.shape[0], v.shape[1]))
    for i in range(q.shape[0]):
        vis = [j for j in range(i + 1) if sees(i, j, window, keep_first)]
        s = (k[vis] @ q[i]) * scale
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[vis]
    return out


def diff_lambda(w, p, diff):
    """The second map's weight, one number for the layer."""
    return float(np.exp(np.sum(w[p + "lq1"] * w[p + "lk1"])) - np.exp(np.sum(w[p + "lq2"] * w[p + "lk2"])) + diff)


def combine_maps(a1, a2, lam, diff, eps):
    """One head's two map outputs [T, vdim] -> the head's output."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(h, w, p, m, eps):
    """Differential attention: two score maps per head over the same values.  h [T, width], tensors w[p + ...]."""
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T).reshape(T, H, 2, dim), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T).reshape(T, G, 2, dim), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).reshape(T, G, vdim)
    lam = diff_lambda(w, p, m["diff"])
    out = np.zeros((T, H, vdim))
    for i in range(H):
        g = i // (H // G)
        a = [softmax_attention(q[:, i, c], k[:, g, c], v[:, g], m["scale"], m["mask"]["size"], m["mask"]["keep_first"]) for c in (0, 1)]
        out[:, i] = combine_maps(a[0], a[1], lam, m["diff"], eps)
    return out.reshape(T, H * vdim) @ w[p + "o"].T


def bonus_recurrence(r, k, v, decay, u):
    """One head: o_t reads the state before token t plus u-weighted k_t v_t; then the state decays and takes k_t v_t in.
    r, k, decay [T, dim], v [T, dim], u [dim]."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(k.shape[0]):
        kv = np.outer(k[t], v[t])
        out[t] = (S + u[:, None] * kv).T @ r[t]
        S = decay[t][:, None] * S + kv
    return out


def wkv_mixer(h, w, p, m, eps):
    T, H, dim = h.shape[0], m["heads"], m["dim"]
    mix = {s: mix_previous(h, w[p + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].T).reshape(T, H, dim) for s in "rkv")
    gate = silu(mix["g"] @ w[p + "g"].T)
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(T, H, dim)
    o = np.stack([bonus_recurrence(r[:, i], k[:, i], v[:, i], decay[:, i], w[p + "u"][i]) for i in range(H)], axis=1)
    o = rms(o, eps).reshape(T, H * dim) * w[p + "norm"] * gate
    return o @ w[p + "o"].T


def gated_recurrence(q, f, v):
    """One head: the state forgets by f and takes (1 - f) v in, then q reads it.  q, f [T, dim], v [T, vdim]."""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = f[t][:, None] * S + np.outer(1.0 - f[t], v[t])
        out[t] = S.T @ q[t]
    return out


def hgrn2_mixer(h, w, p, m, eps):
    T, H, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, dim)
    v = (h @ w[p + "v"].T).reshape(T, H, vdim)
    low = w[p + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).reshape(T, H, dim)
    o = np.stack([gated_recurrence(q[:, i], f[:, i], v[:, i]) for i in range(H)], axis=1)
    return (rms(o, eps) * w[p + "norm"]).reshape(T, H * vdim) @ w[p + "o"].T


def feed_forward(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"attention": attention_mixer, "wkv": wkv_mixer, "hgrn2": hgrn2_mixer}


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  layers_out, a list, receives the residual stream after every layer."""
    w = {n: np.asarray(t, np.float64) for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = w["embed"][tokens] + w["pos"][: len(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        y = MIXERS[layer["type"]](mix_previous(h, w[p + "shift"]), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + feed_forward(h, w, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
