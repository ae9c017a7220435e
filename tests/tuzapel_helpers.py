"""Small Tuzapel configurations that differ in every size and option, random weights for them (made
here, not by the engine's random-weights mode) and model folders written by the tests' own writer."""
from __future__ import annotations

import numpy as np

from helpers import bf16_round, write_model_dir


def scaling(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def attention(heads, kv, dim, vdim, scale, window, conv, rot, kv_from=None):
    """``rot``: (dims, base, scaling or None), or None."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if conv:
        m["conv"] = conv
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if rot[2]:
            m["rot"]["scaling"] = rot[2]
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "scale": scale, "rot": {"base": base, "dims": rot_dim}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _att(m, mlp):
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _lat(m, mlp):
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


BANDS = scaling(6.0, 1.0, 3.0, 120)       # some waves kept, some blended, some slowed down at small sizes
# odd sizes everywhere: heads of 12 and 10 channels, values wider and narrower than keys, two and five taps, a
# layer without a feed-forward, keys and values lent to a layer that sees further and to one that sees less far
TZ_A = {"architecture": "Tuzapel", "vocab": 101, "width": 40, "norm": {"eps": 1e-5}, "logit_softcap": 7.0,
        "layers": [_att(attention(6, 3, 12, 20, 0.5, 11, 5, (8, 500.0, BANDS)), dense(28, 0.7)),
                   _lat(latent(3, 10, 6, 14, 18, 22, 0.3, 900.0), moe(5, 3, 12, 1.5)),
                   _att(attention(6, 3, 12, 20, 0.4, 23, 2, (8, 500.0, BANDS), kv_from=0), None),
                   _att(attention(6, 3, 12, 20, 0.6, 7, 3, (8, 500.0, BANDS), kv_from=0), moe(7, 2, 10, 0.8)),
                   _lat(latent(1, 6, 2, 8, 5, 9, 0.4, 50.0), dense(13, 2.0))]}
# everything that can be 1, equal or absent: one head, one tap or none, a window of one token, no window, no
# scaling, no rotation, one expert, all experts chosen, no soft cap, no clamp
TZ_B = {"architecture": "Tuzapel", "vocab": 64, "width": 32, "norm": {"eps": 1e-6},
        "layers": [_att(attention(1, 1, 16, 16, 0.25, 0, 1, (16, 10000.0, None)), moe(1, 1, 16, 1.0)),
                   _att(attention(2, 2, 8, 8, 0.35, 1, 2, (8, 100.0, None)), dense(16, 1.0)),
                   _lat(latent(1, 16, 16, 16, 16, 16, 0.2, 10000.0), {"kind": "dense", "ff": 16}),
                   _att(attention(1, 1, 16, 16, 0.25, 5, 0, (16, 10000.0, None), kv_from=0), moe(4, 4, 8, 3.0)),
                   _att(attention(4, 1, 8, 8, 0.3, 9, 4, None), None)]}
# still small, with the sizes the tensor-core attention, the few-row product and the fused preparation take:
# heads of 64 and 128 channels, values narrower than keys, a latent of 96 + 32, prompts of hundreds of tokens
TZ_C = {"architecture": "Tuzapel", "vocab": 320, "width": 192, "norm": {"eps": 1e-6}, "logit_softcap": 20.0,
        "layers": [_att(attention(4, 2, 64, 64, 0.125, 70, 4, (32, 20000.0, scaling(8.0, 1.0, 4.0, 256))), dense(256, 1.2)),
                   _lat(latent(4, 48, 32, 64, 80, 96, 0.11, 10000.0), moe(8, 2, 64, 1.7)),
                   _att(attention(6, 3, 128, 48, 0.09, 33, 3, (128, 5000.0, None)), moe(8, 3, 32, 2.5)),
                   _att(attention(6, 3, 128, 48, 0.09, 130, 4, (128, 5000.0, None), kv_from=2), dense(320, 0.9)),
                   _att(attention(4, 2, 64, 64, 0.1, 70, 4, (32, 20000.0, scaling(8.0, 1.0, 4.0, 256)), kv_from=0), dense(128, 1.0))]}
CONFIGS = {"A": TZ_A, "B": TZ_B, "C": TZ_C}


def random_config(seed, big):
    """A configuration drawn from a seed: two to six layers of the two types with sizes, taps, windows and
    constants drawn apart; some read an earlier layer's keys and values.  ``big``: sizes that come in whole
    pieces among others; else small and odd ones."""
    rng = np.random.default_rng(seed)
    pick = lambda xs: xs[int(rng.integers(len(xs)))]
    layers = []

    def mlp():
        limit = float(pick([0.5, 1.0, 2.0, 7.0]))
        if rng.random() < 0.15:
            return None
        if rng.random() < 0.5:
            return dense(pick([64, 128, 320] if big else [8, 12, 21]), limit)
        E = pick([4, 8, 16] if big else [2, 3, 7])
        return moe(E, int(rng.integers(1, min(E, 5) + 1)), pick([32, 64, 96] if big else [6, 10, 16]), limit)

    for i in range(int(rng.integers(2, 7))):
        owners = [j for j, l in enumerate(layers) if l["type"] == "attention" and "kv_from" not in l["mixer"]]
        r = rng.random()
        if r < 0.3 and owners:
            src = pick(owners)
            m = dict(layers[src]["mixer"], kv_from=src, scale=float(pick([0.1, 0.2, 0.4])))
            m["mask"] = {"size": int(pick([1, 6, 16, 40, 97]))}
            layers.append(_att(m, mlp()))
        elif r < 0.65 or not i:
            kv = pick([1, 2, 3])
            dim = pick([32, 48, 64, 128] if big else [4, 8, 14, 20])
            dims = pick([dim, dim // 2 // 2 * 2])
            sc = pick([None, BANDS, scaling(4.0, 1.0, 4.0, 512), scaling(2.0, 2.0, 2.0, 64)])
            layers.append(_att(attention(kv * pick([1, 2, 4]), kv, dim, pick([dim, 16, 64] if big else [dim, 6, 10]),
                                         float(pick([0.1, 0.25, dim ** -0.5])), int(pick([2, 9, 17, 40, 64, 100])),
                                         int(pick([1, 2, 3, 4, 5])), (dims, float(pick([100.0, 10000.0, 250000.0])), sc)), mlp()))
        else:
            rot = pick([16, 32] if big else [2, 4, 8])
            layers.append(_lat(latent(pick([1, 2, 4]), pick([16, 32, 64] if big else [5, 8, 12]), rot,
                                      pick([16, 48, 64] if big else [6, 9, 12]), pick([24, 64, 100] if big else [7, 16]),
                                      pick([32, 64, 128] if big else [8, 13]), float(pick([0.1, 0.2, 0.3])),
                                      float(pick([50.0, 10000.0]))), mlp()))
    cfg = {"architecture": "Tuzapel", "vocab": int(pick([50, 101, 256, 1000])),
           "width": pick([64, 96, 128, 192] if big else [24, 40, 56, 72]), "norm": {"eps": float(pick([1e-6, 1e-5, 1e-4]))},
           "layers": layers}
    cap = pick([None, 5.0, 30.0])
    return dict(cfg, logit_softcap=cap) if cap else cfg


def tensor_shapes(cfg):
    H = cfg["width"]
    out = [("embed", (cfg["vocab"], H))]
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        q = p + "mix."
        out += [(p + "norm1", (H,)), (p + "norm1b", (H,))]
        if layer["type"] == "latent_attention":
            nh, r = m["heads"], m["rot_dim"]
            out += [(q + "dq", (m["q_rank"], H)), (q + "dq.norm", (m["q_rank"],)), (q + "uq", (nh * (m["dim"] + r), m["q_rank"])),
                    (q + "dkv", (m["kv_rank"] + r, H)), (q + "dkv.norm", (m["kv_rank"],)), (q + "uk", (nh * m["dim"], m["kv_rank"])),
                    (q + "uv", (nh * m["vdim"], m["kv_rank"])), (q + "o", (H, nh * m["vdim"]))]
        else:
            rows = {"q": m["heads"] * m["dim"]}
            if "kv_from" not in m:
                rows.update(k=m["kv_heads"] * m["dim"], v=m["kv_heads"] * m["vdim"])
            for r, n in rows.items():
                out.append((q + r, (n, H)))
                if m.get("conv"):
                    out.append((q + r + ".conv", (n, m["conv"])))
                if r != "v":
                    out.append((q + r + ".norm", (m["dim"],)))
            out.append((q + "o", (H, m["heads"] * m["vdim"])))
        if mlp:
            out += [(p + "norm2", (H,)), (p + "norm2b", (H,))]
            one = lambda e, ff: [(p + f"mlp.{e}gate", (ff, H)), (p + f"mlp.{e}up", (ff, H)), (p + f"mlp.{e}down", (H, ff))]
            if mlp["kind"] == "dense":
                out += one("", mlp["ff"])
            else:
                E = mlp["router"]["experts"]
                out += [(p + "mlp.router", (E, H)), (p + "mlp.router.b", (E,))]
                for e in range(E):
                    out += one(f"e{e}.", mlp["expert"]["ff"])
    out.append(("final.norm", (H,)))
    return out


def random_weights(cfg, seed, qk_gain=1.0):
    """float32 arrays, exact in bfloat16.  ``qk_gain`` scales the query and key norm weights so that the softmax
    is peaked and a wrong or missing key shows.

    A choice of experts that hangs on the last bit would flip under rounding and hide every other difference, so
    the first channels of the stream hold a code of the token (one of a few classes) that no sublayer writes to,
    and the routers read mostly that: which experts a token takes varies from token to token, by clear margins."""
    rng = np.random.default_rng(seed)
    w = {}
    K = min(6, cfg["width"] // 4)
    for name, shape in tensor_shapes(cfg):
        n = lambda std, mean=0.0: (mean + rng.standard_normal(shape) * std).astype(np.float32)
        leaf = name.split(".")[-1]
        if name == "embed":
            a = n(0.5)
            a[:, :K] = 0.0
            a[np.arange(len(a)), np.arange(len(a)) % K] = 2.0
        elif leaf in ("norm1b", "norm2b"):
            a = n(0.1, 0.5)
            a[:K] = 0.0
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            a = n(0.15, 1.0)
        elif leaf == "norm":
            a = n(0.1, 1.0) * np.float32(qk_gain if name.split(".")[-2] in ("q", "k", "dq") else 1.0)
        elif leaf == "conv":
            a = n(0.5)
        elif leaf == "b":
            a = n(0.15)
        elif leaf == "router":
            a = n(0.1 / np.sqrt(shape[-1]))
            for c in range(K):
                a[:, c] = 0.4 * (rng.permutation(shape[0]) - (shape[0] - 1) / 2)
        else:
            a = n(1.2 / np.sqrt(shape[-1]))
        w[name] = bf16_round(a.astype(np.float32))
    return w


def make_model(tmp_path, which, seed=0, qk_gain=1.0):
    cfg = CONFIGS[which]
    w = random_weights(cfg, seed, qk_gain)
    d = write_model_dir(str(tmp_path / f"tuzapel_{which}_{seed}_{qk_gain}"), cfg, w, "bfloat16")
    return d, cfg, {k: v.astype(np.float64) for k, v in w.items()}


def prompt(cfg, n, seed):
    return np.random.default_rng(9000 + seed).integers(0, cfg["vocab"], size=n).tolist()
