"""A plain, slow implementation of the Tuzapel decoder in NumPy float64: whole sequences, no cache,
no batching, one function per mechanism.  It shares no code with the engine and is the oracle its
kernels are compared with.

Notation.  ``W`` of a linear map is stored ``[out, in]`` and applied as ``x @ W.T``.  A sequence is
``T`` tokens at positions ``0 .. T-1``.

* ``layer_norm``            ``(x - mean) / sqrt(var + eps) * w``, no bias
* ``rms_norm``              ``x / sqrt(mean(x^2) + eps) * w``
* ``causal_convolution``    over time per channel, no bias, no activation, zeros before the start
* ``frequencies``           ``base^(-2i/dims)``, long wavelengths slowed down, a blend between
* ``rotate``                pairs turned by ``p f_i``; half-split or neighbouring channels
* ``window_mask``           ``0 <= i - j < size``
* ``softmax_with_one``      ``exp(s_j) / (1 + sum exp(s_j))``
* ``conv_attention``        grouped-query attention on convolved projections, norms per head, own or borrowed keys
* ``latent_attention``      attention over a compressed latent, queries through a latent of their own
* ``clamped_gate``          ``g sigmoid(1.702 g) (u + 1)`` of clamped ``g`` and ``u``
* ``choose_experts``        the largest logits (bias included), a softmax over the chosen ones
* ``soft_cap``              ``cap tanh(x / cap)``
"""
from __future__ import annotations

import numpy as np

ROUND = None          # a function applied to activations where a bfloat16 engine rounds; None = exact
GAPS = None           # a list that receives, per router and token, how much the last chosen logit leads the next


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


def lin(x, W):
    return _r(x) @ np.asarray(W, dtype=np.float64).T


# ----------------------------------------------------------------------------- norms

def layer_norm(x, w, eps):
    c = x - np.mean(x, axis=-1, keepdims=True)
    return c / np.sqrt(np.mean(c * c, axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


# ----------------------------------------------------------------------------- time and positions

def causal_convolution(u, w):
    """u [T, C], w [C, taps]: ``y_t = sum_j w[:, j] u_(t - taps + 1 + j)``."""
    T, taps = u.shape[0], w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


def frequencies(dims, base, scaling=None):
    f = np.power(float(base), -2.0 * np.arange(dims // 2) / max(dims, 1))
    if not scaling:
        return f
    factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
    out = np.empty_like(f)
    for i, fi in enumerate(f):
        wavelength = 2.0 * np.pi / fi
        if wavelength < original / high:
            out[i] = fi
        elif wavelength > original / low:
            out[i] = fi / factor
        else:
            s = (original / wavelength - low) / (high - low)
            out[i] = (1.0 - s) * fi / factor + s * fi
    return out


def rotate(x, freqs, layout, positions=None):
    """x [T, heads, d]: the first ``2 len(freqs)`` channels of every head turned by the position."""
    T, n = x.shape[0], len(freqs)
    p = np.arange(T) if positions is None else np.asarray(positions)
    a = p[:, None] * freqs[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    iu = np.arange(n) if layout == "half" else 2 * np.arange(n)
    iv = iu + n if layout == "half" else iu + 1
    y = x.copy()
    u, v = x[..., iu], x[..., iv]
    y[..., iu] = u * c - v * s
    y[..., iv] = v * c + u * s
    return y


# ----------------------------------------------------------------------------- attention

def window_mask(T, size):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < size) if size else True)


def softmax_with_one(s):
    """Over the last axis, one added to the denominator; -inf entries get nothing."""
    m = np.maximum(np.max(s, axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def softmax(s):
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def conv_keys_values(h, w, m, eps):
    """The keys (convolved, normed, rotated) and values (convolved) of a layer that has them."""
    T, G, d, dv = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k, v = lin(h, w["k"]), lin(h, w["v"])
    if m.get("conv"):
        k, v = causal_convolution(k, w["k.conv"]), causal_convolution(v, w["v.conv"])
    k = rms_norm(k.reshape(T, G, d), w["k.norm"], eps)
    return _r(rotate(k, _freqs(m), "half")), _r(v.reshape(T, G, dv))


def _freqs(m):
    rot = m.get("rot") or {}
    return frequencies(rot.get("dims", 0), rot.get("base", 10000.0), rot.get("scaling"))


def conv_attention(h, w, m, eps, kv=None):
    """``kv``: keys and values of another layer; None: the layer's own.  Returns (output, keys and values)."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = lin(h, w["q"])
    if m.get("conv"):
        q = causal_convolution(q, w["q.conv"])
    q = _r(rotate(rms_norm(q.reshape(T, H, d), w["q.norm"], eps), _freqs(m), "half"))
    k, v = kv if kv is not None else conv_keys_values(h, w, m, eps)
    mask = window_mask(T, (m.get("mask") or {}).get("size", 0))
    out = np.empty((T, H, m["vdim"]))
    for n in range(H):
        g = n // (H // G)
        s = np.where(mask, q[:, n] @ k[:, g].T * m["scale"], -np.inf)
        out[:, n] = softmax_with_one(s) @ v[:, g]
    return lin(out.reshape(T, -1), w["o"]), (k, v)


def latent_attention(h, w, m, eps):
    T, H, d, r, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    f = frequencies(m["rot"]["dims"], m["rot"]["base"])
    q = lin(rms_norm(_r(lin(h, w["dq"])), w["dq.norm"], eps), w["uq"]).reshape(T, H, d + r)
    qn, qr = _r(q[..., :d]), rotate(q[..., d:], f, "pairs")
    ckv = _r(lin(h, w["dkv"]))
    c = _r(rms_norm(ckv[:, :rank], w["dkv.norm"], eps))
    kr = _r(rotate(ckv[:, None, rank:], f, "pairs"))[:, 0]
    kn, v = lin(c, w["uk"]).reshape(T, H, d), lin(c, w["uv"]).reshape(T, H, m["vdim"])
    mask = window_mask(T, 0)
    out = np.empty((T, H, m["vdim"]))
    for n in range(H):
        s = (qn[:, n] @ kn[:, n].T + qr[:, n] @ kr.T) * m["scale"]
        out[:, n] = softmax(np.where(mask, s, -np.inf)) @ v[:, n]
    return lin(out.reshape(T, -1), w["o"])


# ----------------------------------------------------------------------------- feed-forwards

def clamped_gate(g, u, limit):
    g = np.minimum(g, limit)
    u = np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def clamped_feed_forward(h, gate, up, down, limit):
    return lin(clamped_gate(_r(lin(h, gate)), _r(lin(h, up)), limit), down)


def choose_experts(z, top):
    """z [T, E] -> weights [T, E], zero where an expert is not chosen."""
    out = np.zeros_like(z)
    if GAPS is not None and top < z.shape[1]:
        s = -np.sort(-z, axis=-1)
        GAPS.extend(s[:, top - 1] - s[:, top])
    for t in range(z.shape[0]):
        best = np.argsort(-z[t], kind="stable")[:top]
        out[t, best] = softmax(z[t, best])
    return out


def mixture(h, w, mlp):
    weights = choose_experts(lin(h, w["router"]) + w["router.b"], mlp["router"]["top"])
    y = np.zeros((h.shape[0], w["e0.down"].shape[0]))
    for e in range(mlp["router"]["experts"]):
        rows = np.nonzero(weights[:, e])[0]
        if len(rows):
            y[rows] += weights[rows, e, None] * clamped_feed_forward(h[rows], w[f"e{e}.gate"], w[f"e{e}.up"],
                                                                     w[f"e{e}.down"], mlp["expert"].get("limit", np.inf))
    return y


def soft_cap(x, cap):
    return cap * np.tanh(x / cap) if cap else x


# ----------------------------------------------------------------------------- the model

def _under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = np.asarray(w["embed"], dtype=np.float64)[np.asarray(tokens)]
    stored = {}
    for i, layer in enumerate(cfg["layers"]):
        lw, m = _under(w, f"l{i}."), layer["mixer"]
        h, mw = layer_norm(x, lw["norm1"], eps), _under(lw, "mix.")
        if layer["type"] == "latent_attention":
            y = latent_attention(h, mw, m, eps)
        else:
            src = m.get("kv_from")
            y, stored[i] = conv_attention(h, mw, m, eps, None if src is None else stored[src])
        x = x + layer_norm(_r(y), lw["norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h, fw = layer_norm(x, lw["norm2"], eps), _under(lw, "mlp.")
            y = (mixture(h, fw, mlp) if mlp["kind"] == "moe"
                 else clamped_feed_forward(h, fw["gate"], fw["up"], fw["down"], mlp.get("limit", np.inf)))
            x = x + layer_norm(_r(y), lw["norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return soft_cap(lin(layer_norm(x, w["final.norm"], eps), w["embed"]), cfg.get("logit_softcap"))


def generate(cfg, w, tokens, n):
    """``n`` greedy tokens after ``tokens``."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(np.argmax(forward(cfg, w, seq)[-1])))
    return seq[len(tokens):]
