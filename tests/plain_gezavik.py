"""A plain, slow implementation of the Gezavik decoder in numpy float64: one function per mechanism, a Python
loop per recurrence, no code shared with the package.  `cfg` is the content of a config.json of this design
(a dict), `w` maps tensor names to float64 arrays.

Notation: h is a sublayer's input (one row per token of ONE sequence, positions from 0), W x a product with a
weight stored [out, in], rms(x) = x / sqrt(mean(x^2) + eps).
"""
import numpy as np

round_inputs = None      # a function that rounds an array as the serving engine's storage type does, or None
route_choices = None     # a dict {(tensor prefix of a routed feed-forward): int array [T, top]}: choices to use instead
                         # of the plain ones (the tests replay the engine's own choices where a call was close)

SLOPE = 1.702            # of the sigmoid in an expert's activation


def product(h, weight):
    """h W^T; with `round_inputs` set, the rows are rounded first: a coarse model of what 16-bit inputs of the
    products do, by which the tests know how far rounding alone moves the logits of a position."""
    return (round_inputs(h) if round_inputs is not None else h) @ weight.T


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def rotate(x, positions, base, dims):
    """x [T, ..., dim]: the first `dims` dims of the last axis turned, dims 2i and 2i + 1 a pair, by the angle
    position * base^(-2i/dims)."""
    f = float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = np.cos(a).reshape(shape), np.sin(a).reshape(shape)
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def short_conv(x, taps_weight, bias):
    """x [T, C], taps_weight [C, taps], bias [C]: causal per channel, the last column weighs the current token, zeros
    before the sequence's start."""
    T, C = x.shape
    taps = taps_weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, C)), x], axis=0)
    y = np.zeros((T, C)) + bias[None, :]
    for j in range(taps):
        y += padded[j:j + T] * taps_weight[:, j][None, :]
    return y


def softmax_rows(s, visible):
    s = np.where(visible, s, -np.inf)
    s = s - s.max(axis=1, keepdims=True)
    e = np.exp(s)
    return e / e.sum(axis=1, keepdims=True)


# ---- mixers ---------------------------------------------------------------------------------------------------

def state_space_walk(x, B, C, dt, a_log, skip):
    """x [T, H, dv], B and C [T, G, N], dt [T, H] (already positive), a_log and skip [H]: per head
    S <- exp(-exp(a_log) dt) S + dt B x^T,  y = S^T C + skip x; head h reads group h // (H / G)."""
    T, H, dv = x.shape
    G, N = B.shape[1:]
    y = np.zeros((T, H, dv))
    for h in range(H):
        g = h // (H // G)
        S = np.zeros((N, dv))
        for t in range(T):
            S = np.exp(-np.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + skip[h] * x[t, h]
    return y


def gated_group_norm(y, z, weight, groups, eps):
    """y silu(z), then each of `groups` equal parts over its own root mean square, then the weight."""
    T, W = y.shape
    return rms((y * silu(z)).reshape(T, groups, W // groups), eps).reshape(T, W) * weight


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, dv, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * dv
    zxbcdt = product(h, w[p + "in"])
    z, xbc, dt = zxbcdt[:, :inner], zxbcdt[:, inner:2 * inner + 2 * G * N], zxbcdt[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    if round_inputs is not None:                 # the convolutions' activated outputs are kept in the storage type
        xbc = round_inputs(xbc)
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    y = state_space_walk(x, B, C, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return product(gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], int(m["norm_groups"]), eps), w[p + "o"])


def latent_attention(h, w, p, m, eps):
    """Attention whose keys and values of every head are products of one small vector per token (the latent), beside one
    rotated key part that all heads share; the queries come through a latent of their own; a sliding window; one sigmoid
    gate per head on the heads' outputs."""
    T = h.shape[0]
    H, dk, dr, dv, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos = np.arange(T)
    q = product(rms(product(h, w[p + "dq"]), eps) * w[p + "dq.norm"], w[p + "uq"]).reshape(T, H, dk + dr)
    ckr = product(h, w[p + "dkv"])
    c = rms(ckr[:, :r], eps) * w[p + "dkv.norm"]
    k_rot = rotate(ckr[:, r:], pos, m["rot"]["base"], int(m["rot"]["dims"]))
    q_plain, q_rot = q[:, :, :dk], rotate(q[:, :, dk:], pos, m["rot"]["base"], int(m["rot"]["dims"]))
    if round_inputs is not None:                 # the cache and the queries are kept in the storage type
        q_plain, q_rot, c, k_rot = (round_inputs(a) for a in (q_plain, q_rot, c, k_rot))
    k = (c @ w[p + "uk"].T).reshape(T, H, dk)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    back = pos[:, None] - pos[None, :]
    visible = back >= 0
    if m.get("mask"):
        visible &= back < int(m["mask"]["size"])
    out = np.zeros((T, H, dv))
    for hh in range(H):
        s = (q_plain[:, hh] @ k[:, hh].T + q_rot[:, hh] @ k_rot.T) * float(m["scale"])
        out[:, hh] = softmax_rows(s, visible) @ v[:, hh]
    out = out * sigmoid(product(h, w[p + "g"]))[:, :, None]
    return product(out.reshape(T, H * dv), w[p + "o"])


MIXERS = {"mamba2": mamba2, "latent_attention": latent_attention}


# ---- feed-forwards ----------------------------------------------------------------------------------------------

def squared_relu_feed_forward(h, w, p):
    return product(np.maximum(product(h, w[p + "up"]), 0.0) ** 2, w[p + "down"])


def clamped_feed_forward(h, w, p, limit):
    g = np.minimum(product(h, w[p + "gate"]), limit)
    u = np.clip(product(h, w[p + "up"]), -limit, limit)
    return product(g * sigmoid(SLOPE * g) * (u + 1.0), w[p + "down"])


def route(z, correction, top):
    """z [E] router logits of one token (experts, then identities).  Returns (the chosen in order of choice, their
    weights, the gap between the last chosen and the best refused choice score)."""
    e = np.exp(z - z.max())
    s = e / e.sum()
    choice = s + correction
    order = sorted(range(len(z)), key=lambda i: (-choice[i], i))
    margin = choice[order[top - 1]] - choice[order[top]] if top < len(z) else np.inf
    return order[:top], s[order[:top]], margin


def routed_feed_forward(h, w, p, mlp):
    """Of the router's outputs the first `experts` are feed-forwards and the rest give back their input."""
    r = mlp["router"]
    E, top = int(r["experts"]), int(r["top"])
    T = h.shape[0]
    hr = round_inputs(h) if round_inputs is not None else h
    z = hr @ w[p + "router"].T
    y = np.zeros((T, h.shape[1]))
    outs = {}
    for t in range(T):
        chosen, weights, _ = route(z[t], w[p + "correction"], top)
        if route_choices is not None and p in route_choices:
            chosen = [int(e) for e in route_choices[p][t]]
            s = np.exp(z[t] - z[t].max())
            weights = (s / s.sum())[chosen]
        for e, wt in zip(chosen, weights):
            if e >= E:
                y[t] += wt * hr[t]
                continue
            if e not in outs:
                outs[e] = clamped_feed_forward(h, w, f"{p}e{e}.", float(mlp["expert"]["limit"]))
            y[t] += wt * outs[e][t]
    if mlp.get("shared"):
        y = y + clamped_feed_forward(h, w, p + "shared.", float(mlp["shared"]["limit"]))
    return y


def feed_forward(h, w, p, mlp):
    if mlp["kind"] == "dense":
        return squared_relu_feed_forward(h, w, p)
    return routed_feed_forward(h, w, p, mlp)


# ---- the model ----------------------------------------------------------------------------------------------------

def layer(x, w, cfg, i):
    """One norm; the mixer and the feed-forward side by side on its output."""
    entry, eps, m = cfg["layers"][i], float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    p = f"l{i}."
    h = rms(x, eps) * w[p + "norm1"]
    y = MIXERS[entry["type"]](h, w, p + "mix.", entry["mixer"], eps)
    if entry.get("mlp") is not None:
        y = y + feed_forward(h, w, p + "mlp.", entry["mlp"])
    return x + m * y


def forward(cfg, w, tokens, trace=None):
    """Logits [T, vocab] of one sequence from its first token.  `trace`: a list that receives the residual stream
    after every layer."""
    x = w["embed"][np.asarray(tokens)]
    for i in range(len(cfg["layers"])):
        x = layer(x, w, cfg, i)
        if trace is not None:
            trace.append(x.copy())
    return product(rms(x, float(cfg["norm"]["eps"])) * w["final.norm"], w["head"])
