"""A plain, slow implementation of the Nebanex decoder in numpy float64: one function per mechanism, a Python
loop per recurrence, no code shared with the package.  `cfg` is the content of a config.json of this design
(a dict), `w` maps tensor names to float64 arrays.

Notation: h is a sublayer's input (one row per token of ONE sequence, positions from 0), W x a product with a
weight stored [out, in], rms(x) = x / sqrt(mean(x^2) + eps).
"""
import math

import numpy as np

round_inputs = None      # a function that rounds an array as the serving engine's storage type does, or None
route_choices = None     # a dict {(tensor prefix of a routed feed-forward): int array [T, top]}: choices to use instead
                         # of the plain ones (the tests replay the engine's own choices where a call was close)


def product(h, weight, bias=None):
    """h W^T (+ b); with `round_inputs` set, the rows are rounded first: a coarse model of what 16-bit inputs of the
    products do, by which the tests know how far rounding alone moves the logits of a position."""
    y = (round_inputs(h) if round_inputs is not None else h) @ weight.T
    return y if bias is None else y + bias


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, weight, bias, eps):
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * weight + bias


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def log_sigmoid(x):
    return -np.logaddexp(0.0, -x)


def silu(x):
    return x * sigmoid(x)


# ---- the left mixer: attention with a learned bias by distance ------------------------------------------------------

def bucket(n, buckets, furthest):
    """The row of the bias table for a key n >= 0 positions back: the first half of the rows one per distance, the rest
    spaced evenly in ln(n) up to `furthest`, from where on the last row serves.  (A distance that falls on a boundary
    exactly belongs to the upper row; the 1e-9 keeps a logarithm's last bit from deciding that.)"""
    half = buckets // 2
    if buckets < 2:
        return 0
    if n < half:
        return n
    steps = math.log(n / half) / math.log(furthest / half) * (buckets - half)
    return min(buckets - 1, half + int(math.floor(steps + 1e-9)))


def distance_bias(T, table, furthest):
    """[T, T, H]: what head h adds to the score of query i and key j <= i (zero elsewhere)."""
    rows = np.array([bucket(n, table.shape[0], furthest) for n in range(T)])
    back = np.maximum(np.arange(T)[:, None] - np.arange(T)[None, :], 0)
    return table[rows[back]]


def query_factor(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions) + 1) / every) + 1.0)


def softmax_causal(s):
    s = np.where(np.tril(np.ones(s.shape, dtype=bool)), s, -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    return e / e.sum(axis=1, keepdims=True)


def attention(h, w, p, m, eps):
    """q and k normed over all of their rows at once, no rotation, the queries times a factor that grows with the position,
    a bias by distance on the scores, an output gate."""
    T = h.shape[0]
    H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms(product(h, w[p + "q"], w[p + "q.b"]), eps) * w[p + "q.norm"]
    k = rms(product(h, w[p + "k"], w[p + "k.b"]), eps) * w[p + "k.norm"]
    v = product(h, w[p + "v"], w[p + "v.b"])
    if m.get("q_temp"):
        q = q * query_factor(np.arange(T), float(m["q_temp"]["coef"]), float(m["q_temp"]["every"]))[:, None]
    if round_inputs is not None:                 # the queries and the cache are kept in the storage type
        q, k, v = round_inputs(q), round_inputs(k), round_inputs(v)
    q, k, v = q.reshape(T, H, dk), k.reshape(T, G, dk), v.reshape(T, G, dv)
    bias = distance_bias(T, w[p + "rel"], float(m["bias_max"]))
    out = np.zeros((T, H, dv))
    for head in range(H):
        g = head // (H // G)
        out[:, head] = softmax_causal(q[:, head] @ k[:, g].T * float(m["scale"]) + bias[:, :, head]) @ v[:, g]
    out = out.reshape(T, H * dv) * sigmoid(product(h, w[p + "g"]))
    return product(out, w[p + "o"], w[p + "o.b"])


# ---- the right mixer: linear attention with a decay per key channel --------------------------------------------------

def gated_linear_walk(q, k, v, log_decay):
    """q, k, log_decay [T, H, dk], v [T, H, dv]: per head S <- diag(exp(log_decay)) S + k v^T, o = S^T q."""
    T, H, dk = q.shape
    dv = v.shape[2]
    o = np.zeros((T, H, dv))
    for h in range(H):
        S = np.zeros((dk, dv))
        for t in range(T):
            S = np.exp(log_decay[t, h])[:, None] * S + np.outer(k[t, h], v[t, h])
            o[t, h] = S.T @ q[t, h]
    return o


def gated_linear(h, w, p, m, eps):
    T = h.shape[0]
    H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = product(h, w[p + "q"]).reshape(T, H, dk) * dk ** -0.5
    k = product(h, w[p + "k"]).reshape(T, H, dk)
    v = product(h, w[p + "v"]).reshape(T, H, dv)
    z = product(product(h, w[p + "a1"]), w[p + "a2"], w[p + "a2.b"]).reshape(T, H, dk)
    o = gated_linear_walk(q, k, v, log_sigmoid(z) / float(m["tau"]))
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * dv)
    return product(o * silu(product(h, w[p + "g"])), w[p + "o"])


def parallel(h, w, p, m, eps):
    left = attention(h, w, p + "left.", m["left"], eps)
    right = gated_linear(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


# ---- the feed-forward ------------------------------------------------------------------------------------------------

def glu(h, w, p):
    return product(silu(product(h, w[p + "gate"])) * product(h, w[p + "up"]), w[p + "down"])


def route(z, top):
    """z [E] router logits of one token.  Returns (the chosen in order of choice, their weights, the gap between the last
    chosen and the best refused logit)."""
    order = sorted(range(len(z)), key=lambda i: (-z[i], i))
    chosen = order[:top]
    e = np.exp(z[chosen] - z[chosen].max())
    margin = z[order[top - 1]] - z[order[top]] if top < len(z) else np.inf
    return chosen, e / e.sum(), margin


def routed_feed_forward(h, w, p, mlp):
    top = int(mlp["router"]["top"])
    T = h.shape[0]
    z = (round_inputs(h) if round_inputs is not None else h) @ w[p + "router"].T + w[p + "router.b"]
    y = np.zeros((T, h.shape[1]))
    outs = {}
    for t in range(T):
        chosen, weights, _ = route(z[t], top)
        if route_choices is not None and p in route_choices:
            chosen = [int(e) for e in route_choices[p][t]]
            e = np.exp(z[t][chosen] - z[t][chosen].max())
            weights = e / e.sum()
        for e, wt in zip(chosen, weights):
            if e not in outs:
                outs[e] = glu(h, w, f"{p}e{e}.")
            y[t] += wt * outs[e][t]
    if mlp.get("shared"):
        y = y + glu(h, w, p + "shared.")
    return y


# ---- the model -------------------------------------------------------------------------------------------------------

def layer(x, w, cfg, i):
    entry, eps = cfg["layers"][i], float(cfg["norm"]["eps"])
    p = f"l{i}."
    x = x + parallel(layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps), w, p + "mix.", entry["mixer"], eps)
    if entry.get("mlp") is not None:
        x = x + routed_feed_forward(layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), w, p + "mlp.", entry["mlp"])
    return x


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def forward(cfg, w, tokens, trace=None):
    """Logits [T, vocab] of one sequence from its first token.  `trace`: a list that receives the residual stream
    after every layer."""
    x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    for i in range(len(cfg["layers"])):
        x = layer(x, w, cfg, i)
        if trace is not None:
            trace.append(x.copy())
    z = product(layer_norm(x, w["final.norm"], w["final.norm.b"], float(cfg["norm"]["eps"])), w["head"])
    return soft_cap(z, float(cfg["logit_softcap"]))
