"""A plain, slow statement of the Tokolorn design in NumPy float64, one function per mechanism.

It shares no code with the package: the tests hold the package's kernels, cache and scheduler to
these functions.  A model is a dict ``config`` (the JSON of config.json) and a dict ``w`` of arrays by
tensor name.  Everything works on one whole sequence (positions 0..T-1); what a cache or a state
would hold is simply recomputed.

Notation: x the residual stream [T, D]; h a sublayer's normed input; H query heads, G key/value heads; d the
query/key size, d_v the value size; S a recurrence's state; t a position.
"""
import math

import numpy as np

F = np.float64


# ------------------------------------------------------------------ elementwise
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def scalar_rms_norm(x, gain, eps):
    """Unit rms over the row, times one number for all its entries."""
    return unit_rms(x, eps) * float(np.asarray(gain).reshape(()))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------ embedding
def pair_rows(tokens, pair):
    """The second table's row for every token: a hash of the token before and the token; the last row at the start."""
    n, a, b = int(pair["buckets"]), int(pair["mul_prev"]), int(pair["mul_cur"])
    return np.array([n if t == 0 else (int(tokens[t - 1]) * a + int(tokens[t]) * b) % n for t in range(len(tokens))])


def embedding(config, tokens, w):
    e = config["embedding"]
    x = w["embed"][np.asarray(tokens, dtype=np.int64)] * float(e["scale"])
    if e.get("bigram"):
        x = x + w["bigram"][pair_rows(tokens, e["bigram"])]
    return x


# ------------------------------------------------------------------ lightning attention
def fading_recurrence(q, k, v, decay):
    """One head: S <- decay S + k v^T, o = S^T q, one constant decay."""
    T, d = q.shape
    S = np.zeros((d, v.shape[1]), dtype=F)
    out = np.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def lightning_mixer(h, m, w, x, eps):
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q = silu(h @ w[x + "q"].T).reshape(T, H, d)
    k = silu(h @ w[x + "k"].T).reshape(T, H, d)
    v = silu(h @ w[x + "v"].T).reshape(T, H, dv)
    o = np.zeros((T, H, dv), dtype=F)
    for a in range(H):
        o[:, a] = fading_recurrence(q[:, a], k[:, a], v[:, a], float(m["decay"][a]))
    o = unit_rms(o.reshape(T, H * dv), eps) * w[x + "norm"] * sigmoid(h @ w[x + "g"].T)
    return o @ w[x + "o"].T


# ------------------------------------------------------------------ attention
def rotate_pairs(y, base, dims):
    """y [T, heads, d]: entries (2i, 2i + 1) of the first ``dims`` turned by t * base^(-2i / dims)."""
    out = y.copy()
    t = np.arange(y.shape[0], dtype=F)
    for i in range(dims // 2):
        angle = (t * base ** (-2.0 * i / dims))[:, None]
        u, v = y[:, :, 2 * i], y[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * np.cos(angle) - v * np.sin(angle)
        out[:, :, 2 * i + 1] = v * np.cos(angle) + u * np.sin(angle)
    return out


def in_window(i, j, size):
    return j <= i and (size is None or i - j < size)


def in_chunk(i, j, size):
    return j <= i and (size is None or i // size == j // size)


def masked_attention(q, k, v, scale, sees, softcap=None, sink=False):
    """One head over the keys that ``sees(i, j)`` shows; a soft cap on the scores; with ``sink`` the denominator has
    one more term, exp(0)."""
    T = q.shape[0]
    out = np.zeros((T, v.shape[1]), dtype=F)
    for i in range(T):
        js = np.array([j for j in range(i + 1) if sees(i, j)])
        s = (k[js] @ q[i]) * scale
        if softcap:
            s = softcap * np.tanh(s / softcap)
        top = max(s.max(), 0.0) if sink else s.max()
        p = np.exp(s - top)
        out[i] = (p / (p.sum() + (math.exp(-top) if sink else 0.0))) @ v[js]
    return out


def attention_mixer(h, m, w, x, eps):
    """Chunks, a sink, keys that are the values, no rotation."""
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    T = h.shape[0]
    size = int(m["mask"]["size"]) if m.get("mask") else None
    q = (h @ w[x + "q"].T).reshape(T, H, d)
    k = (h @ w[x + "k"].T).reshape(T, G, d)
    o = np.zeros((T, H, d), dtype=F)
    for a in range(H):
        g = a // (H // G)
        o[:, a] = masked_attention(q[:, a], k[:, g], k[:, g], float(m["scale"]), lambda i, j: in_chunk(i, j, size), sink=True)
    return o.reshape(T, H * d) @ w[x + "o"].T


def windowed_attention(h, m, w, x):
    """A window, pairs rotated, a soft cap, an output gate per entry."""
    H, G, d, dv = (int(m[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
    T = h.shape[0]
    size = int(m["mask"]["size"]) if m.get("mask") else None
    q = (h @ w[x + "q"].T).reshape(T, H, d)
    k = (h @ w[x + "k"].T).reshape(T, G, d)
    v = (h @ w[x + "v"].T).reshape(T, G, dv)
    if m.get("rot"):
        q, k = (rotate_pairs(y, float(m["rot"]["base"]), int(m["rot"]["dims"])) for y in (q, k))
    o = np.zeros((T, H, dv), dtype=F)
    for a in range(H):
        g = a // (H // G)
        o[:, a] = masked_attention(q[:, a], k[:, g], v[:, g], float(m["scale"]), lambda i, j: in_window(i, j, size),
                                   softcap=m.get("softcap"))
    return (o.reshape(T, H * dv) * sigmoid(h @ w[x + "g"].T)) @ w[x + "o"].T


# ------------------------------------------------------------------ selective scan
def short_convolution(u, taps_of, bias):
    """u [T, C], taps_of [C, taps]: causal, one filter per channel, the last tap on the current token."""
    T, C = u.shape
    n = taps_of.shape[1]
    padded = np.concatenate([np.zeros((n - 1, C), dtype=F), u])
    out = np.zeros((T, C), dtype=F) + bias
    for j in range(n):
        out += padded[j:j + T] * taps_of[:, j]
    return out


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, c], A [c, n], B, C [T, n], D [c]."""
    S = np.zeros(A.shape, dtype=F)
    out = np.zeros(x.shape, dtype=F)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba_mixer(h, m, w, x):
    inner, N, R = int(m["inner"]), int(m["state"]), int(m["dt_rank"])
    u = h @ w[x + "in"].T
    u, z = u[:, :inner], u[:, inner:]
    u = silu(short_convolution(u, w[x + "conv"], w[x + "conv.b"]))
    p = u @ w[x + "x"].T
    dt = softplus(p[:, :R] @ w[x + "dt"].T + w[x + "dt.b"])
    y = selective_scan(u, dt, -np.exp(w[x + "A_log"]), p[:, R:R + N], p[:, R + N:], w[x + "D"])
    return (y * silu(z)) @ w[x + "o"].T


def parallel_mixer(h, m, w, x, eps):
    return (float(m["left_scale"]) * windowed_attention(h, m["left"], w, x + "left.")
            + float(m["right_scale"]) * mamba_mixer(h, m["right"], w, x + "right."))


MIXERS = {"lightning": lightning_mixer, "parallel": parallel_mixer, "attention": attention_mixer}


# ------------------------------------------------------------------ the model
def feed_forward(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def order_of_layers(config):
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def forward(config, w, tokens, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` (a list) receives the stream after every run of a layer."""
    eps = float(config["norm"]["eps"])
    x = embedding(config, tokens, w)
    for i in order_of_layers(config):
        layer, p = config["layers"][i], f"l{i}."
        h = scalar_rms_norm(x, w[p + "norm1"], eps)
        x = x + w[p + "ls1"] * MIXERS[layer["type"]](h, layer["mixer"], w, p + "mix.", eps)
        if layer.get("mlp") is not None:
            x = x + w[p + "ls2"] * feed_forward(scalar_rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.copy())
    return scalar_rms_norm(x, w["final.norm"], eps) @ w["head"].T * float(config["logit_scale"])


# ------------------------------------------------------------------ random weights for tests
def tensor_shapes(config):
    D, V = int(config["width"]), int(config["vocab"])
    shapes = {"embed": (V, D), "final.norm": (), "head": (V, D)}
    if config["embedding"].get("bigram"):
        shapes["bigram"] = (int(config["embedding"]["bigram"]["buckets"]) + 1, D)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        shapes.update({p + "norm1": (), p + "ls1": (D,)})
        if layer["type"] == "lightning":
            H, d, dv = (int(m[n]) for n in ("heads", "dim", "vdim"))
            shapes.update({x + "q": (H * d, D), x + "k": (H * d, D), x + "v": (H * dv, D), x + "g": (H * dv, D),
                           x + "norm": (H * dv,), x + "o": (D, H * dv)})
        elif layer["type"] == "attention":
            H, G, d = (int(m[n]) for n in ("heads", "kv_heads", "dim"))
            shapes.update({x + "q": (H * d, D), x + "k": (G * d, D), x + "o": (D, H * d)})
        else:
            l, r = m["left"], m["right"]
            H, G, d, dv = (int(l[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
            y = x + "left."
            shapes.update({y + "q": (H * d, D), y + "k": (G * d, D), y + "v": (G * dv, D), y + "g": (H * dv, D),
                           y + "o": (D, H * dv)})
            c, N, R, taps = (int(r[n]) for n in ("inner", "state", "dt_rank", "conv"))
            y = x + "right."
            shapes.update({y + "in": (2 * c, D), y + "conv": (c, taps), y + "conv.b": (c,), y + "x": (R + 2 * N, c),
                           y + "dt": (c, R), y + "dt.b": (c,), y + "A_log": (c, N), y + "D": (c,), y + "o": (D, c)})
        if layer.get("mlp") is not None:
            ff = int(layer["mlp"]["ff"])
            shapes.update({p + "norm2": (), p + "ls2": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D),
                           p + "mlp.down": (D, ff)})
    return shapes


def random_weights(config, seed):
    """Weights that bfloat16 holds exactly (the tests write them to a bfloat16 file), sized so that every mechanism
    matters: scores that reach the soft cap and stand out from a sink, decays between nothing and everything, gains and
    layer scales away from one."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2"):
            a = rng.normal(1.0, 0.2, shape)
        elif last in ("ls1", "ls2"):
            a = rng.normal(0.5, 0.2, shape)
        elif last == "conv":
            a = rng.normal(0.0, 0.6, shape)
        elif name.endswith("dt.b"):
            a = rng.uniform(-4.0, 1.0, shape)
        elif last == "A_log":
            a = rng.uniform(-2.0, 2.0, shape)
        elif last == "D":
            a = rng.normal(0.5, 0.5, shape)
        elif name.endswith("conv.b"):
            a = rng.normal(0.0, 0.2, shape)
        elif name in ("embed", "bigram"):
            a = rng.normal(0.0, (1.0 / float(config["embedding"]["scale"])) if name == "embed" else 0.7, shape)
        else:
            wide = 2.0 if last in ("q", "k", "dt", "head") else 1.0
            a = rng.normal(0.0, wide / math.sqrt(shape[-1]), shape)
        out[name] = to_bf16(a)
    return out


def to_bf16(a):
    """To what bfloat16 holds: eight bits of mantissa, ties to even."""
    a = np.asarray(a, dtype=np.float32)
    bits = np.atleast_1d(a).copy().view(np.uint32).astype(np.uint64)
    bits = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16
    return bits.astype(np.uint32).view(np.float32).astype(F).reshape(a.shape)
