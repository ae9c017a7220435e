"""A plain, slow implementation of the Takavik decoder in NumPy float64: whole sequences, no cache,
no batching, one function per mechanism.  It shares no code with the engine and is the oracle its
kernels are compared with.

Notation.  ``W`` of a linear map is stored ``[out, in]`` and applied as ``x @ W.T``.  A sequence is
``T`` tokens at positions ``0 .. T-1``.  A layer reads a weighted sum of several residual streams,
runs a mixer (then a feed-forward) on its norm and writes back into all streams.

* ``rms_norm`` / ``norm_one_plus``  ``x / sqrt(mean(x^2) + eps)`` times ``w`` / times ``1 + w``
* ``stream_read`` / ``stream_write``  the streams' weighted sum; mixing plus the sublayer's result
* ``biased_convolution``    a causal convolution over time per channel with a bias, then SiLU
* ``query_temperature``     ``1 + coef ln(floor((p + 1) / every) + 1)``
* ``head_norm_attention``   grouped-query attention without positions, norms per head, that temperature
* ``selective_scan``        a state per channel whose decay and input weights depend on the token
* ``mamba2``                a state per head with one decay per head and token, gate before a grouped norm
* ``gated_linear``          a state per head with a decay per key channel and token
* ``side_by_side``          half the sum of the two branches' normalised outputs
* ``silu_feed_forward``     ``W_down (silu(W_gate h) * (W_up h))``
"""
from __future__ import annotations

import numpy as np

ROUND = None          # a function applied to activations where a bfloat16 engine rounds; None = exact


def _r(x):
    return x if ROUND is None else ROUND(x)


def round_bf16(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    u = ((u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) >> np.uint32(16)).astype(np.uint32) << 16
    return u.view(np.float32).astype(np.float64)


def round_f32(x):
    return np.asarray(x, dtype=np.float32).astype(np.float64)


def sigmoid(x):
    return np.exp(-np.logaddexp(0.0, -x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def lin(x, W):
    return _r(x) @ np.asarray(W, dtype=np.float64).T


def rms_norm(x, w, eps):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * w


def norm_one_plus(x, w, eps):
    return rms_norm(x, 1.0 + np.asarray(w, dtype=np.float64), eps)


# ----------------------------------------------------------------------------- residual streams

def stream_read(xs, w_in):
    """xs [S, T, H] -> [T, H]."""
    return np.einsum("s,sth->th", w_in, xs)


def stream_write(xs, y, mix, w_out):
    """``x_t <- sum_s mix[s, t] x_s + w_out[t] y`` for all t at once from the old streams."""
    return np.einsum("st,sah->tah", mix, xs) + np.asarray(w_out)[:, None, None] * y


# ----------------------------------------------------------------------------- convolution over time

def biased_convolution(x, w, b):
    """x [T, C], w [C, taps], b [C]: ``silu(b + sum_j w[:, j] x_(t - taps + 1 + j))``, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x) + b
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += x[:T - back] * w[:, j]
    return silu(y)


# ----------------------------------------------------------------------------- softmax attention

def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1.0) / every) + 1.0)


def softmax_attention(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    mask = np.arange(T)[None, :] <= np.arange(T)[:, None]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(mask, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def _heads(x, n):
    return x.reshape(x.shape[0], n, -1)


def head_norm_attention(h, W, c, eps):
    T = h.shape[0]
    H, G = int(c["heads"]), int(c.get("kv_heads") or c["heads"])
    q = rms_norm(_heads(lin(h, W["q"]), H), W["q.norm"], eps)
    k = rms_norm(_heads(lin(h, W["k"]), G), W["k.norm"], eps)
    v = _heads(lin(h, W["v"]), G)
    t = c.get("q_temp")
    if t:
        q = q * query_temperature(np.arange(T), float(t["coef"]), float(t["every"]))[:, None, None]
    o = softmax_attention(_r(q), _r(k), _r(v), float(c["scale"]))
    return lin(o.reshape(T, -1), W["o"])


# ----------------------------------------------------------------------------- recurrences

def selective_scan(h, W, c):
    """``S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n ; y_c = sum_n S[c, n] C_n + D_c x_c``."""
    T = h.shape[0]
    n_in, R, N = int(c["inner"]), int(c["dt_rank"]), int(c["state"])
    xz = lin(h, W["in"])
    x = biased_convolution(xz[:, :n_in], W["conv"], W["conv.b"])
    z = xz[:, n_in:]
    p = lin(x, W["x"])
    dt = softplus(lin(p[:, :R], W["dt"]) + W["dt.b"])
    B, C = p[:, R:R + N], p[:, R + N:]
    A = -np.exp(W["A_log"])
    S = np.zeros((n_in, N))
    y = np.zeros((T, n_in))
    for t in range(T):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + W["D"] * x[t]
    return lin(y * silu(z), W["o"])


def mamba2(h, W, c, eps):
    """``S <- exp(-exp(A_log) dt) S + dt B x^T ; y = S^T C + D x`` per head; the gate stands before the norm."""
    T = h.shape[0]
    H, P, N = int(c["heads"]), int(c["vdim"]), int(c["state"])
    G, NG, taps = int(c.get("groups") or 1), int(c.get("norm_groups") or 1), int(c["conv"])
    assert W["conv"].shape[1] == taps
    inner = H * P
    p = lin(h, W["in"])
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = biased_convolution(xbc, W["conv"], W["conv.b"])
    x, B, C = _heads(xbc[:, :inner], H), _heads(xbc[:, inner:inner + G * N], G), _heads(xbc[:, inner + G * N:], G)
    dt = softplus(dt + W["dt_bias"])
    a = np.exp(-np.exp(W["A_log"]) * dt)
    y = np.zeros((T, H, P))
    for hd in range(H):
        g = hd // (H // G)
        S = np.zeros((N, P))
        for t in range(T):
            S = a[t, hd] * S + dt[t, hd] * np.outer(B[t, g], x[t, hd])
            y[t, hd] = S.T @ C[t, g] + W["D"][hd] * x[t, hd]
    y = y.reshape(T, inner) * silu(z)
    y = rms_norm(y.reshape(T, NG, inner // NG), None, eps).reshape(T, inner) * W["norm"]
    return lin(y, W["o"])


def gated_linear(h, W, c, eps):
    """``S <- diag(alpha) S + k v^T ; o = S^T q`` per head, ``alpha = sigmoid(z)^(1/tau)`` per key channel."""
    T = h.shape[0]
    H, d, tau = int(c["heads"]), int(c["dim"]), float(c["tau"])
    q = _heads(lin(h, W["q"]) * d ** -0.5, H)
    k, v = _heads(lin(h, W["k"]), H), _heads(lin(h, W["v"]), H)
    alpha = _heads(sigmoid(lin(lin(h, W["a1"]), W["a2"]) + W["a2.b"]) ** (1.0 / tau), H)
    o = np.zeros((T, H, v.shape[2]))
    for hd in range(H):
        S = np.zeros((d, v.shape[2]))
        for t in range(T):
            S = alpha[t, hd][:, None] * S + np.outer(k[t, hd], v[t, hd])
            o[t, hd] = S.T @ q[t, hd]
    y = rms_norm(o, W["norm"], eps).reshape(T, -1) * silu(lin(h, W["g"]))
    return lin(y, W["o"])


# ----------------------------------------------------------------------------- the model

def _sub(tensors, prefix):
    n = len(prefix)
    return {k[n:]: np.asarray(v, dtype=np.float64) for k, v in tensors.items() if k.startswith(prefix)}


def side_by_side(h, W, c, eps):
    left = head_norm_attention(h, _sub(W, "left."), c["left"], eps)
    right = selective_scan(h, _sub(W, "right."), c["right"])
    return 0.5 * (rms_norm(left, W["left.out"], eps) + rms_norm(right, W["right.out"], eps))


def mixer_forward(h, layer, W, eps):
    kind, c = layer["type"], layer["mixer"]
    if kind == "parallel":
        return side_by_side(h, W, c, eps)
    if kind == "mamba2":
        return mamba2(h, W, c, eps)
    if kind == "gla":
        return gated_linear(h, W, c, eps)
    raise ValueError(f"unknown layer type {kind}")


def silu_feed_forward(h, W):
    return _r(lin(silu(_r(lin(h, W["gate"]))) * _r(lin(h, W["up"])), W["down"]))


def forward(config, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``tensors``: name -> array.  ``layers_out``: a list that gets
    the sum of the streams after every layer."""
    eps = float(config["norm"]["eps"])
    S = int(config.get("streams") or 0)
    E = np.asarray(tensors["embed"], dtype=np.float64)
    xs = np.repeat(E[np.asarray(tokens)][None], max(S, 1), axis=0)

    def sublayer(xs, p, q, fn):
        hc = _sub(tensors, f"{p}hc{q}.") if S else {"in": np.ones(1), "out": np.ones(1), "mix": np.eye(1)}
        y = fn(norm_one_plus(stream_read(xs, hc["in"]), tensors[f"{p}norm{q}"], eps))
        return stream_write(xs, y, hc["mix"], hc["out"])

    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        xs = sublayer(xs, p, 1, lambda h: mixer_forward(h, layer, _sub(tensors, p + "mix."), eps))
        if layer.get("mlp"):
            xs = sublayer(xs, p, 2, lambda h: silu_feed_forward(h, _sub(tensors, p + "mlp.")))
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return lin(norm_one_plus(xs.sum(0), tensors["final.norm"], eps), E)


def generate(config, tensors, prompt, n):
    seq, out = list(prompt), []
    for _ in range(n):
        out.append(int(np.argmax(forward(config, tensors, seq)[-1])))
        seq.append(out[-1])
    return out
