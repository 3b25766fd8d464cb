"""A plain, slow statement of the Pelenex design in NumPy float64, one function per mechanism.

It shares no code with the package: the tests hold the package's kernels, cache and scheduler to
these functions.  A model is a dict ``config`` (the JSON of config.json) and a dict ``w`` of arrays by
tensor name.  Everything works on one whole sequence (positions 0..T-1); what a cache or a state
would hold is simply recomputed.

Notation: x the residual stream [T, D]; h a layer's normed stream, which its mixer and its feed-forward both
read; H heads (query or value heads), G key/value heads; d the query/key size, d_v the value size; S a head's
matrix state [d, d_v]; t a position.
"""
import math

import numpy as np

F = np.float64


# ------------------------------------------------------------------ elementwise
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def group_rms_norm(x, weight, groups, eps):
    """The row in ``groups`` consecutive equal parts, each to unit rms by itself, times one weight for the row."""
    T, D = x.shape
    return unit_rms(x.reshape(T, groups, D // groups), eps).reshape(T, D) * weight


def unit_length(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


# ------------------------------------------------------------------ embedding
def sinusoids(T, width):
    """Position vectors: for pair i the sine and the cosine of t * 10000^(-2i / width), side by side."""
    out = np.zeros((T, width), dtype=F)
    t = np.arange(T, dtype=F)
    for c in range(width):
        i = c // 2
        angle = t * 10000.0 ** (-2.0 * i / width)
        out[:, c] = np.sin(angle) if c % 2 == 0 else np.cos(angle)
    return out


def embedding(tokens, w):
    tokens = np.asarray(tokens, dtype=np.int64)
    return w["embed"][tokens] + sinusoids(len(tokens), w["embed"].shape[1])


# ------------------------------------------------------------------ matrix memory with exponential gates
def log_gates(h, m, w, x):
    """(log input gate, log forget gate), [T, H] each."""
    cap = float(m["gate_cap"])
    capped = lambda name: cap * np.tanh((h @ w[x + name].T + w[x + name + ".b"]) / cap)
    return capped("i"), -softplus(-capped("f"))


def mlstm_recurrence(q, k, v, i_log, f_log):
    """One head: q, k [T, d], v [T, d_v], i_log, f_log [T]; the state is kept relative to exp(m), m a running
    maximum that starts at zero."""
    T, d = q.shape
    S, n, m = np.zeros((d, v.shape[1]), dtype=F), np.zeros(d, dtype=F), 0.0
    out = np.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        new = max(f_log[t] + m, i_log[t])
        keep, take = math.exp(f_log[t] + m - new), math.exp(i_log[t] - new)
        S = keep * S + take * np.outer(k[t], v[t])
        n = keep * n + take * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (max(abs(n @ q[t]), math.exp(-m)) + 1e-6)
    return out


def mlstm_mixer(h, m, w, x, eps):
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q = (h @ w[x + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[x + "k"].T).reshape(T, H, d)
    v = (h @ w[x + "v"].T).reshape(T, H, dv)
    i_log, f_log = log_gates(h, m, w, x)
    o = np.zeros((T, H, dv), dtype=F)
    for a in range(H):
        o[:, a] = mlstm_recurrence(q[:, a], k[:, a], v[:, a], i_log[:, a], f_log[:, a])
    o = unit_rms(o, eps).reshape(T, H * dv) * w[x + "norm"] * sigmoid(h @ w[x + "g"].T)
    return o @ w[x + "o"].T


# ------------------------------------------------------------------ attention in a window with kept first tokens
def seen(i, j, mask):
    """Whether position i sees position j."""
    if j > i:
        return False
    if not mask:
        return True
    return i - j < int(mask["size"]) or j < int(mask.get("keep_first") or 0)


def biased_attention(q, k, v, scale, slope, mask):
    """One head: scores scale q . k - slope * distance over what the mask shows, ordinary softmax."""
    T = q.shape[0]
    out = np.zeros((T, v.shape[1]), dtype=F)
    for i in range(T):
        js = np.array([j for j in range(i + 1) if seen(i, j, mask)])
        s = (k[js] @ q[i]) * scale - slope * (i - js)
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[js]
    return out


def attention_mixer(h, m, w, x, eps):
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    T = h.shape[0]
    q = unit_rms((h @ w[x + "q"].T).reshape(T, H, d), eps)
    raw = (h @ w[x + "k"].T).reshape(T, G, d)
    k, v = unit_rms(raw, eps), raw                                 # the values are the projected keys themselves
    o = np.zeros((T, H, d), dtype=F)
    for a in range(H):
        g = a // (H // G)
        o[:, a] = biased_attention(q[:, a], k[:, g], v[:, g], float(m["scale"]), 2.0 ** (-8.0 * (a + 1) / H), m.get("mask"))
    return o.reshape(T, H * d) @ w[x + "o"].T


# ------------------------------------------------------------------ gated linear attention
def linear_recurrence(q, k, v, alpha):
    """One head: S <- diag(alpha_t) S + k v^T, o = S^T q; alpha [T, d]."""
    T, d = q.shape
    S = np.zeros((d, v.shape[1]), dtype=F)
    out = np.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        S = alpha[t][:, None] * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def channel_decays(h, m, w, x):
    """sigmoid(z)^(1 / tau) per head and key channel, z through two matrices and a bias."""
    z = (h @ w[x + "a1"].T) @ w[x + "a2"].T + w[x + "a2.b"]
    return sigmoid(z) ** (1.0 / float(m["tau"]))


def linear_attention_mixer(h, m, w, x, eps):
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q = (h @ w[x + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[x + "k"].T).reshape(T, H, d)
    v = (h @ w[x + "v"].T).reshape(T, H, dv)
    alpha = channel_decays(h, m, w, x).reshape(T, H, d)
    o = np.zeros((T, H, dv), dtype=F)
    for a in range(H):
        o[:, a] = linear_recurrence(q[:, a], k[:, a], v[:, a], alpha[:, a])
    o = rms_norm(o, w[x + "norm"], eps).reshape(T, H * dv) * silu(h @ w[x + "g"].T)
    return o @ w[x + "o"].T


def parallel_mixer(h, m, w, x, eps):
    left = attention_mixer(h, m["left"], w, x + "left.", eps)
    right = linear_attention_mixer(h, m["right"], w, x + "right.", eps)
    return 0.5 * (rms_norm(left, w[x + "left.out"], eps) + rms_norm(right, w[x + "right.out"], eps))


# ------------------------------------------------------------------ the delta rule with a decay per key channel
def short_convolution(u, taps_of):
    """u [T, C], taps_of [C, taps]: causal, one filter per channel, the last tap on the current token."""
    T, C = u.shape
    n = taps_of.shape[1]
    padded = np.concatenate([np.zeros((n - 1, C), dtype=F), u])
    out = np.zeros((T, C), dtype=F)
    for j in range(n):
        out += padded[j:j + T] * taps_of[:, j]
    return out


def delta_recurrence(q, k, v, g, beta):
    """One head: the rows of S decay each by its own number, then S is corrected along k and read with q."""
    T, d = q.shape
    S = np.zeros((d, v.shape[1]), dtype=F)
    out = np.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def delta_decays(h, m, w, x):
    """exp(-exp(A) softplus(z + bias)) per head and key channel, [T, H, d]."""
    H, d = int(m["heads"]), int(m["dim"])
    z = (h @ w[x + "a1"].T) @ w[x + "a2"].T + w[x + "dt_bias"]
    return np.exp(-np.exp(w[x + "A_log"])[:, None] * softplus(z).reshape(-1, H, d))


def delta_mixer(h, m, w, x, eps):
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    conv = lambda name: silu(short_convolution(h @ w[x + name].T, w[x + name + ".conv"]))
    q = unit_length(conv("q").reshape(T, G, d)) * d ** -0.5
    k = unit_length(conv("k").reshape(T, G, d))
    v = conv("v").reshape(T, H, dv)
    beta = sigmoid(h @ w[x + "b"].T)
    g = delta_decays(h, m, w, x)
    o = np.zeros((T, H, dv), dtype=F)
    for a in range(H):
        c = a // (H // G)
        o[:, a] = delta_recurrence(q[:, c], k[:, c], v[:, a], g[:, a], beta[:, a])
    gate = sigmoid((h @ w[x + "g1"].T) @ w[x + "g2"].T)
    o = rms_norm(o, w[x + "norm"], eps).reshape(T, H * dv) * gate
    return o @ w[x + "o"].T


MIXERS = {"mlstm": mlstm_mixer, "parallel": parallel_mixer, "channel_delta": delta_mixer}


# ------------------------------------------------------------------ feed-forward
def gated_ffn(h, w, p):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def routed(h, mlp, w, p):
    """Each token's ``top`` experts by sigmoid score; an expert reads the token times its score."""
    top = int(mlp["router"]["top"])
    scores = sigmoid(h @ w[p + ".router"].T)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e in np.argsort(-scores[t], kind="stable")[:top]:
            out[t] += gated_ffn(scores[t, e] * h[t:t + 1], w, f"{p}.e{e}")[0]
    if mlp.get("shared"):
        out = out + gated_ffn(h, w, p + ".shared")
    return out


def feed_forward(h, mlp, w, p):
    return gated_ffn(h, w, p) if mlp["kind"] == "dense" else routed(h, mlp, w, p)


# ------------------------------------------------------------------ the model
def forward(config, w, tokens, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` (a list) receives the stream after every layer."""
    eps, groups = float(config["norm"]["eps"]), int(config["norm"]["groups"])
    x = embedding(tokens, w)
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = group_rms_norm(x, w[p + "norm1"], groups, eps)
        add = MIXERS[layer["type"]](h, layer["mixer"], w, p + "mix.", eps)
        if layer.get("mlp") is not None:
            add = add + feed_forward(h, layer["mlp"], w, p + "mlp")
        x = x + add
        if layers_out is not None:
            layers_out.append(x.copy())
    logits = group_rms_norm(x, w["final.norm"], groups, eps) @ w["head"].T
    cap = config.get("logit_softcap")
    return float(cap) * np.tanh(logits / float(cap)) if cap else logits


# ------------------------------------------------------------------ random weights for tests
def tensor_shapes(config, rank=None):
    """Names and shapes; ``rank(name)`` gives the inner size of a projection that goes through two matrices (no key
    of the configuration does)."""
    rank = rank or default_rank
    D, V = int(config["width"]), int(config["vocab"])
    shapes = {"embed": (V, D), "final.norm": (D,), "head": (V, D)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        shapes[p + "norm1"] = (D,)
        if layer["type"] == "mlstm":
            H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
            shapes.update({x + "q": (H * d, D), x + "k": (H * d, D), x + "v": (H * dv, D), x + "g": (H * dv, D),
                           x + "o": (D, H * dv), x + "norm": (H * dv,), x + "i": (H, D), x + "i.b": (H,), x + "f": (H, D),
                           x + "f.b": (H,)})
        elif layer["type"] == "channel_delta":
            H, G, d, dv, taps = (int(m[n]) for n in ("heads", "kv_heads", "dim", "vdim", "conv"))
            ra, rg = rank(x + "a"), rank(x + "g")
            shapes.update({x + "q": (G * d, D), x + "q.conv": (G * d, taps), x + "k": (G * d, D), x + "k.conv": (G * d, taps),
                           x + "v": (H * dv, D), x + "v.conv": (H * dv, taps), x + "b": (H, D), x + "A_log": (H,),
                           x + "norm": (dv,), x + "a1": (ra, D), x + "a2": (H * d, ra), x + "dt_bias": (H * d,),
                           x + "g1": (rg, D), x + "g2": (H * dv, rg), x + "o": (D, H * dv)})
        else:
            l, r = m["left"], m["right"]
            H, G, d = int(l["heads"]), int(l["kv_heads"]), int(l["dim"])
            y = x + "left."
            shapes.update({y + "q": (H * d, D), y + "k": (G * d, D), y + "o": (D, H * d), y + "out": (D,)})
            H, d, dv = int(r["heads"]), int(r["dim"]), int(r["vdim"])
            y = x + "right."
            ra = rank(y + "a")
            shapes.update({y + "q": (H * d, D), y + "k": (H * d, D), y + "v": (H * dv, D), y + "g": (H * dv, D),
                           y + "o": (D, H * dv), y + "norm": (dv,), y + "a1": (ra, D), y + "a2": (H * d, ra),
                           y + "a2.b": (H * d,), y + "out": (D,)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        names = [(p + "mlp", mlp.get("ff"))]
        if mlp["kind"] == "moe":
            E = int(mlp["router"]["experts"])
            shapes[p + "mlp.router"] = (E, D)
            names = [(f"{p}mlp.e{e}", mlp["expert"]["ff"]) for e in range(E)]
            if mlp.get("shared"):
                names.append((p + "mlp.shared", mlp["shared"]["ff"]))
        for name, ff in names:
            shapes.update({name + ".gate": (int(ff), D), name + ".up": (int(ff), D), name + ".down": (D, int(ff))})
    return shapes


def default_rank(name):
    """A few sizes, odd ones among them, that follow from the name alone."""
    return (5, 8, 12, 19)[sum(map(ord, name)) % 4]


def random_weights(config, seed, rank=None):
    """Weights that bfloat16 holds exactly (the tests write them to a bfloat16 file), sized so that every mechanism
    matters: decays between nothing and everything, gates on both sides of their caps, norms away from one."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config, rank).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "out"):
            a = rng.normal(1.0, 0.2, shape)
        elif last == "conv":
            a = rng.normal(0.0, 0.6, shape)
        elif last == "A_log":
            a = rng.uniform(-2.0, 1.0, shape)
        elif last == "dt_bias":
            a = rng.uniform(-3.0, 1.0, shape)
        elif name.endswith("f.b"):
            a = rng.uniform(1.0, 5.0, shape)
        elif name.endswith("i.b"):
            a = rng.uniform(-2.0, 1.0, shape)
        elif name.endswith("a2.b"):
            a = rng.uniform(-2.0, 4.0, shape)
        elif name == "embed":
            a = rng.normal(0.0, 1.0, shape)
        else:
            wide = 3.0 if last in ("q", "k", "b", "router") else 2.0 if last in ("a1", "a2", "g1", "g2", "i", "f") else 1.0
            a = rng.normal(0.0, wide / math.sqrt(shape[-1]), shape)
        out[name] = to_bf16(a)
    return out


def to_bf16(a):
    """To what bfloat16 holds: eight bits of mantissa, ties to even."""
    a = np.ascontiguousarray(a, dtype=np.float32)
    bits = a.view(np.uint32).astype(np.uint64)
    bits = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) << 16
    return bits.astype(np.uint32).view(np.float32).astype(F).reshape(a.shape)
