"""Small Takavik configurations that differ in every size and option, random weights for them (made
here, not by the engine's random-weights mode) and model folders written by the tests' own writer."""
from __future__ import annotations

import copy

import numpy as np

from helpers import bf16_round, write_model_dir

RANK = "decay_rank"     # the low rank of a gla layer's decay: in the tensors' shapes, not in config.json


def attention(heads, kv, dim, vdim, scale, temp=None):
    a = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if temp is not None:
        a["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return a


def scan(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def _par(left, right):
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def _mamba2(heads, vdim, state, groups, norm_groups, conv):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                        "norm_groups": norm_groups, "conv": conv}}


def _gla(heads, dim, vdim, tau, rank):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, RANK: rank}}


def _with(layer, ff):
    return dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


# odd sizes everywhere: heads of 10, 6 and 14 channels, values wider and narrower than keys, states that are no
# multiple of four, two and five taps, an uneven step of the temperature, a layer without a feed-forward
TK_A = {"architecture": "Takavik", "vocab": 101, "width": 40, "streams": 2, "norm": {"eps": 1e-5},
        "layers": [_with(_gla(3, 10, 6, 7.0, 5), 28),
                   _with(_par(attention(6, 3, 12, 20, 0.3, (0.7, 9)), scan(36, 10, 5, 2)), 12),
                   _with(_mamba2(6, 10, 14, 3, 5, 5), None),
                   _with(_par(attention(4, 1, 20, 6, 0.25, (-0.2, 5)), scan(22, 19, 3, 3)), 20),
                   _with(_gla(1, 14, 22, 3.0, 2), 8)]}
# everything that can be 1, equal or absent: one residual stream without connections, one head, one group, a
# convolution of one tap, one state per channel, tau 1, no temperature, a temperature that steps at every token
TK_B = {"architecture": "Takavik", "vocab": 64, "width": 32, "norm": {"eps": 1e-6},
        "layers": [_with(_mamba2(1, 16, 16, 1, 1, 1), 16),
                   _with(_par(attention(1, 1, 16, 16, 0.25), scan(16, 1, 1, 1)), None),
                   _with(_gla(1, 16, 16, 1.0, 1), 16),
                   _with(_par(attention(2, 2, 8, 8, 0.35, (0.3, 1)), scan(32, 16, 2, 1)), 8),
                   _with(_mamba2(4, 8, 8, 4, 4, 2), None)]}
# still small, with the sizes the tensor-core attention, the few-row product and the wide pieces of the recurrences
# take: head sizes 64 and 128, values narrower than keys, states of 128 and 160 rows (more than a block's), a rank
# from which the step sizes are a product, prompts of hundreds of tokens (recurrences in segments)
TK_C = {"architecture": "Takavik", "vocab": 320, "width": 192, "streams": 4, "norm": {"eps": 1e-6},
        "layers": [_with(_mamba2(4, 64, 128, 2, 2, 4), 256),
                   _with(_gla(2, 160, 64, 16.0, 16), 256),
                   _with(_par(attention(4, 2, 64, 64, 0.125, (0.4, 100)), scan(256, 16, 32, 4)), 384),
                   _with(_par(attention(4, 1, 128, 64, 0.09, (0.2, 48)), scan(192, 64, 8, 3)), None),
                   _with(_mamba2(6, 32, 64, 1, 3, 3), 256)]}
CONFIGS = {"A": TK_A, "B": TK_B, "C": TK_C}


def random_config(seed, big):
    """A configuration drawn from a seed: two to five layers of the three types with sizes, ranks, taps and
    constants drawn apart.  ``big``: sizes that come in whole pieces among others; else small and odd ones."""
    rng = np.random.default_rng(seed)
    pick = lambda xs: xs[int(rng.integers(len(xs)))]

    def layer():
        r = rng.random()
        if r < 0.4:
            kv = pick([1, 2, 3])
            dim = pick([32, 64, 96, 128] if big else [4, 8, 12, 20])
            left = attention(kv * pick([1, 2, 4]), kv, dim, pick([dim, dim // 2, 64] if big else [dim, 6, 10]),
                             float(pick([0.05, 0.125, 0.2, dim ** -0.5])), pick([None, (0.5, 17), (0.1, 64), (1.0, 3)]))
            right = scan(pick([64, 128, 320] if big else [12, 20, 36]), pick([8, 16, 24, 48, 128] if big else [1, 3, 12]),
                         pick([4, 33, 64] if big else [1, 3, 6]), pick([1, 2, 3, 4, 5]))
            return _par(left, right)
        if r < 0.7:
            g = pick([1, 2])
            heads = g * pick([1, 2, 3])
            return _mamba2(heads, pick([16, 32, 64, 100] if big else [4, 6, 10]), pick([16, 48, 64, 128, 200] if big else [3, 8, 14]),
                           g, pick([1, heads]), pick([1, 2, 3, 4]))
        return _gla(pick([1, 2, 4]), pick([16, 32, 64, 128, 192] if big else [4, 6, 10]),
                    pick([16, 32, 64, 160] if big else [4, 6, 14]), float(pick([1.0, 4.0, 16.0])), pick([1, 3, 16, 40]))

    width = pick([64, 96, 128, 192, 256] if big else [24, 40, 56, 72])
    ffs = [64, 128, 320] if big else [8, 12, 20]
    layers = [_with(layer(), None if rng.random() < 0.2 else pick(ffs)) for _ in range(int(rng.integers(2, 6)))]
    cfg = {"architecture": "Takavik", "vocab": int(pick([50, 101, 256, 1000])), "width": width,
           "norm": {"eps": float(pick([1e-6, 1e-5, 1e-4]))}, "layers": layers}
    s = pick([0, 1, 2, 4, 5])
    return dict(cfg, streams=s) if s else cfg


def tensor_shapes(cfg):
    H, S = cfg["width"], cfg.get("streams", 0)
    out = [("embed", (cfg["vocab"], H))]
    for i, layer in enumerate(cfg["layers"]):
        p, m, kind, mlp = f"l{i}.", layer["mixer"], layer["type"], layer["mlp"]
        q = p + "mix."
        out.append((p + "norm1", (H,)))
        if kind == "mamba2":
            inner, nh = m["heads"] * m["vdim"], m["heads"]
            C = inner + 2 * m["groups"] * m["state"]
            out += [(q + "in", (inner + C + nh, H)), (q + "conv", (C, m["conv"])), (q + "conv.b", (C,)), (q + "dt_bias", (nh,)),
                    (q + "A_log", (nh,)), (q + "D", (nh,)), (q + "norm", (inner,)), (q + "o", (H, inner))]
        elif kind == "gla":
            n, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out += [(q + "q", (n, H)), (q + "k", (n, H)), (q + "v", (nv, H)), (q + "g", (nv, H)), (q + "o", (H, nv)),
                    (q + "norm", (m["vdim"],)), (q + "a1", (m[RANK], H)), (q + "a2", (n, m[RANK])), (q + "a2.b", (n,))]
        else:
            a, r = m["left"], m["right"]
            out += [(q + "left.q", (a["heads"] * a["dim"], H)), (q + "left.k", (a["kv_heads"] * a["dim"], H)),
                    (q + "left.v", (a["kv_heads"] * a["vdim"], H)), (q + "left.q.norm", (a["dim"],)),
                    (q + "left.k.norm", (a["dim"],)), (q + "left.o", (H, a["heads"] * a["vdim"])), (q + "left.out", (H,))]
            n = r["inner"]
            out += [(q + "right.in", (2 * n, H)), (q + "right.conv", (n, r["conv"])), (q + "right.conv.b", (n,)),
                    (q + "right.x", (r["dt_rank"] + 2 * r["state"], n)), (q + "right.dt", (n, r["dt_rank"])),
                    (q + "right.dt.b", (n,)), (q + "right.A_log", (n, r["state"])), (q + "right.D", (n,)),
                    (q + "right.o", (H, n)), (q + "right.out", (H,))]
        if mlp:
            out += [(p + "norm2", (H,)), (p + "mlp.gate", (mlp["ff"], H)), (p + "mlp.up", (mlp["ff"], H)),
                    (p + "mlp.down", (H, mlp["ff"]))]
        if S:
            for hc in ("hc1", "hc2") if mlp else ("hc1",):
                out += [(f"{p}{hc}.in", (S,)), (f"{p}{hc}.out", (S,)), (f"{p}{hc}.mix", (S, S))]
    out.append(("final.norm", (H,)))
    return out


def random_weights(cfg, seed, qk_gain=1.0):
    """float32 arrays, exact in bfloat16.  ``qk_gain`` scales the attention's query and key norm weights so that
    the softmax is peaked and a wrong or missing key shows.  Step sizes and decays are spread so that
    some states forget within a few tokens and some keep for hundreds."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg):
        n = lambda std, mean=0.0: (mean + rng.standard_normal(shape) * std).astype(np.float32)
        parts = name.split(".")
        leaf = parts[-1]
        if name == "embed":
            a = n(0.5)
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            a = n(0.2)                          # stored around zero: 1 + w multiplies
        elif leaf == "norm" and parts[-2] in ("q", "k"):
            a = n(0.1, 1.0) * np.float32(qk_gain)
        elif leaf in ("norm", "out") and len(shape) == 1 and parts[-2] not in ("hc1", "hc2"):
            a = n(0.1, 1.0)
        elif leaf == "mix":
            a = np.eye(shape[0], dtype=np.float32) + n(0.15)
        elif leaf in ("in", "out") and parts[-2] in ("hc1", "hc2"):
            a = n(0.2, 1.0 / shape[0] if leaf == "in" else 1.0)
        elif leaf == "conv":
            a = n(0.5)
        elif leaf == "A_log":
            a = n(1.0, 0.3)
        elif leaf == "D":
            a = n(0.3, 0.8)
        elif leaf == "dt_bias" or parts[-2:] == ["dt", "b"]:
            a = n(1.3, -2.5)
        elif parts[-2:] == ["a2", "b"]:
            a = n(1.5, 1.0)
        elif leaf == "b":
            a = n(0.3)
        else:
            a = n(1.2 / np.sqrt(shape[-1]))
        w[name] = bf16_round(a.astype(np.float32))
    return w


def make_model(tmp_path, which, seed=0, qk_gain=1.0):
    cfg = CONFIGS[which]
    w = random_weights(cfg, seed, qk_gain)
    d = write_model_dir(str(tmp_path / f"takavik_{which}_{seed}_{qk_gain}"), file_config(cfg), w, "bfloat16")
    return d, cfg, {k: v.astype(np.float64) for k, v in w.items()}


def file_config(cfg):
    """The configuration as a file has it: without the sizes that only the tensors' shapes say."""
    c = copy.deepcopy(cfg)
    for layer in c["layers"]:
        if layer["type"] == "gla":
            layer["mixer"].pop(RANK, None)
    return c


def prompt(cfg, n, seed):
    return np.random.default_rng(9000 + seed).integers(0, cfg["vocab"], size=n).tolist()
