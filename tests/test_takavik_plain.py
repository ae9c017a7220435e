"""The plain Takavik implementation against closed forms, and what needs no GPU of the engine's side:
the configuration reader, the tensor lists, the cache layout, how a portion is cut into segments."""
import copy
import json
import math
from types import SimpleNamespace

import numpy as np
import pytest

import plain_takavik as P
from takavik_helpers import CONFIGS, RANK, TK_A, TK_B, TK_C, file_config, random_config, random_weights, tensor_shapes

RNG = np.random.default_rng(5)


def r(*shape, std=1.0):
    return RNG.standard_normal(shape) * std


# ----------------------------------------------------------------------------- the oracle's mechanisms

def test_norms_and_streams():
    x = r(5, 6)
    assert np.allclose(P.norm_one_plus(x, np.zeros(6), 1e-5), P.rms_norm(x, None, 1e-5))
    assert np.allclose(P.norm_one_plus(x, np.full(6, 0.5), 0.0), 1.5 * x / np.sqrt((x * x).mean(1, keepdims=True)))
    xs, y = r(3, 5, 6), r(5, 6)
    assert np.allclose(P.stream_read(xs, np.array([0.0, 2.0, 0.0])), 2.0 * xs[1])
    mix = np.zeros((3, 3))
    mix[0, 2] = 1.0                                        # [from, to]: stream 0 flows into stream 2 alone
    out = P.stream_write(xs, y, mix, np.array([0.0, 1.0, 0.0]))
    assert np.allclose(out[0], 0) and np.allclose(out[1], y) and np.allclose(out[2], xs[0])
    assert np.allclose(P.stream_write(xs[:1], y, np.ones((1, 1)), np.ones(1))[0], xs[0] + y)


def test_convolution_by_hand():
    x, w, b = r(5, 3), r(3, 3), r(3)
    y = P.biased_convolution(x, w, b)
    assert np.allclose(y[0], P.silu(b + w[:, 2] * x[0]))
    assert np.allclose(y[1], P.silu(b + w[:, 2] * x[1] + w[:, 1] * x[0]))
    assert np.allclose(y[4], P.silu(b + w[:, 2] * x[4] + w[:, 1] * x[3] + w[:, 0] * x[2]))


def test_query_temperature_steps_where_the_next_position_divides():
    t = P.query_temperature(np.arange(9), 0.5, 4)
    assert np.allclose(t[:3], 1.0) and np.allclose(t[3:7], 1 + 0.5 * math.log(2)) and np.allclose(t[7:], 1 + 0.5 * math.log(3))
    assert np.allclose(P.query_temperature(np.arange(3), 1.0, 1), 1 + np.log(np.arange(3) + 2.0))


def test_attention_by_hand():
    H, c = 5, {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 2, "scale": 0.7, "q_temp": {"coef": 0.9, "every": 2}}
    W = {"q": r(12, H), "k": r(6, H), "v": r(4, H), "q.norm": 1 + 0.1 * r(3), "k.norm": 1 + 0.1 * r(3), "o": np.eye(8)}
    h = r(4, H)
    out = P.head_norm_attention(h, W, c, 1e-5)
    v = (h @ W["v"].T).reshape(4, 2, 2)
    assert np.allclose(out[0], np.concatenate([v[0, 0], v[0, 0], v[0, 1], v[0, 1]]))     # alone: its own value
    q = P.rms_norm((h @ W["q"].T).reshape(4, 4, 3), W["q.norm"], 1e-5)
    k = P.rms_norm((h @ W["k"].T).reshape(4, 2, 3), W["k.norm"], 1e-5)
    s = q[3, 2] @ k[:, 1].T * 0.7 * (1 + 0.9 * math.log(2 + 1))       # head 2 reads key head 1; position 3, steps of 2
    p = np.exp(s - s.max())
    assert np.allclose(out[3, 4:6], (p / p.sum()) @ v[:, 1])


def test_recurrences_by_hand():
    H = 5
    h = r(4, H)
    # selective scan: one channel's sum over the past with the products of its decays
    c = {"inner": 3, "state": 2, "dt_rank": 2, "conv": 2}
    W = {"in": r(6, H), "conv": r(3, 2), "conv.b": r(3), "x": r(6, 3), "dt": r(3, 2), "dt.b": r(3), "A_log": r(3, 2), "D": r(3),
         "o": np.eye(3)}
    out = P.selective_scan(h, W, c)
    xz = h @ W["in"].T
    x = P.biased_convolution(xz[:, :3], W["conv"], W["conv.b"])
    p = x @ W["x"].T
    dt = P.softplus(p[:, :2] @ W["dt"].T + W["dt.b"])
    y = 0.0
    for j in range(4):
        decay = np.exp(-np.exp(W["A_log"][1]) * dt[j + 1:, 1].sum())
        y = y + (decay * dt[j, 1] * x[j, 1] * p[j, 2:4] * p[3, 4:6]).sum()
    want = (y + W["D"][1] * x[3, 1]) * P.silu(xz[3, 4])
    assert np.allclose(out[3, 1], want)
    # mamba2: the same with one decay per head; gate before a norm in two parts
    c = {"heads": 2, "vdim": 2, "state": 3, "groups": 1, "norm_groups": 2, "conv": 1}
    W = {"in": r(4 + 4 + 6 + 2, H), "conv": np.ones((10, 1)), "conv.b": np.zeros(10), "dt_bias": r(2), "A_log": r(2), "D": r(2),
         "norm": 1 + 0.1 * r(4), "o": np.eye(4)}
    out = P.mamba2(h, W, c, 1e-5)
    p = h @ W["in"].T
    xbc = P.silu(p[:, 4:14])
    dt = P.softplus(p[:, 14:] + W["dt_bias"])
    y = np.zeros(4)
    for hd in range(2):
        for j in range(4):
            decay = np.exp(-np.exp(W["A_log"][hd]) * dt[j + 1:, hd].sum())
            y[2 * hd:2 * hd + 2] += decay * dt[j, hd] * (xbc[j, 4:7] @ xbc[3, 7:10]) * xbc[j, 2 * hd:2 * hd + 2]
        y[2 * hd:2 * hd + 2] += W["D"][hd] * xbc[3, 2 * hd:2 * hd + 2]
    y = y * P.silu(p[3, :4])
    want = np.concatenate([y[:2] / np.sqrt((y[:2] ** 2).mean() + 1e-5), y[2:] / np.sqrt((y[2:] ** 2).mean() + 1e-5)]) * W["norm"]
    assert np.allclose(out[3], want)
    # gated linear attention: a decay per key channel
    c = {"heads": 1, "dim": 3, "vdim": 2, "tau": 4.0}
    W = {"q": r(3, H), "k": r(3, H), "v": r(2, H), "g": r(2, H), "a1": r(2, H), "a2": r(3, 2), "a2.b": r(3),
         "norm": 1 + 0.1 * r(2), "o": np.eye(2)}
    out = P.gated_linear(h, W, c, 1e-5)
    a = P.sigmoid(h @ W["a1"].T @ W["a2"].T + W["a2.b"]) ** 0.25
    q, k, v = (h @ W[n].T for n in "qkv")
    o = sum(((q[3] * 3 ** -0.5) * np.prod(a[j + 1:], axis=0) * k[j]).sum() * v[j] for j in range(4))
    want = P.rms_norm(o, W["norm"], 1e-5) * P.silu(h[3] @ W["g"].T)
    assert np.allclose(out[3], want)


def test_side_by_side_is_half_the_sum_of_normalised_branches():
    cfg = TK_A
    W = {k[len("l1.mix."):]: v.astype(np.float64) for k, v in random_weights(cfg, 3).items() if k.startswith("l1.mix.")}
    h, c = r(6, 40), cfg["layers"][1]["mixer"]
    zero_left = dict(W, **{"left.out": np.zeros(40)})
    zero_right = dict(W, **{"right.out": np.zeros(40)})
    right, left = P.side_by_side(h, zero_left, c, 1e-5), P.side_by_side(h, zero_right, c, 1e-5)
    assert np.allclose(P.side_by_side(h, W, c, 1e-5), left + right)
    assert np.allclose(((right / (0.5 * W["right.out"])) ** 2).mean(1), 1.0, atol=1e-2)


@pytest.mark.parametrize("which", list(CONFIGS))
def test_the_model_runs_and_prefixes_agree(which):
    cfg = CONFIGS[which]
    w = {k: v.astype(np.float64) for k, v in random_weights(cfg, 1).items()}
    toks = np.random.default_rng(3).integers(0, cfg["vocab"], size=12).tolist()
    layers = []
    full = P.forward(cfg, w, toks, layers)
    assert full.shape == (12, cfg["vocab"]) and len(layers) == len(cfg["layers"]) and np.isfinite(full).all()
    assert np.allclose(P.forward(cfg, w, toks[:7]), full[:7])         # causal throughout


# ----------------------------------------------------------------------------- the engine's side, without a GPU

class _RT:
    precise = True
    device = "cpu"
    stream_max_rows = 16

    def __init__(self):
        import torch
        self.dtype = torch.float32

    def buffer(self, *a, **k):
        raise AssertionError("no scratch at build time")


def _model(cfg):
    from mlxforge_b200.config import config_from_json
    from mlxforge_b200.config.registry import get_architecture
    from mlxforge_b200.models.decoder import DecoderModel
    c = config_from_json(json.loads(json.dumps(file_config(cfg)))).with_tensor_shapes(dict(tensor_shapes(cfg)))
    return c, DecoderModel(get_architecture("Takavik").build_spec(c), _RT())


def test_config_reader_defaults_errors_and_round_trip():
    from mlxforge_b200.config import config_from_json
    from mlxforge_b200.config.model_config import ConfigError
    from mlxforge_b200.config.registry import registered_architectures
    assert "Takavik" in registered_architectures()
    c = config_from_json(json.loads(json.dumps(TK_B)))
    assert c.streams == 0 and c.layers[1]["mixer"]["left"]["q_temp"] is None and c.layers[1]["mlp"] is None
    bare = copy.deepcopy(TK_B)
    for k in ("groups", "norm_groups"):
        bare["layers"][0]["mixer"].pop(k)
    bare["layers"][2]["mixer"].pop("vdim")
    for k in ("kv_heads", "vdim", "scale"):
        bare["layers"][1]["mixer"]["left"].pop(k)
    b = config_from_json(bare)
    assert (b.layers[0]["mixer"]["groups"], b.layers[0]["mixer"]["norm_groups"], b.layers[2]["mixer"]["vdim"]) == (1, 1, 16)
    left = b.layers[1]["mixer"]["left"]
    assert (left["kv_heads"], left["vdim"], left["scale"]) == (1, 16, 0.25)
    a = config_from_json(json.loads(json.dumps(TK_A)))
    again = config_from_json(json.loads(json.dumps(a.to_json())))
    assert again.layers == a.layers and (again.vocab, again.width, again.streams, again.norm_eps) == (101, 40, 2, 1e-5)

    def broken(edit, text):
        j = copy.deepcopy(TK_A)
        edit(j)
        with pytest.raises(ConfigError, match=text):
            config_from_json(j)
    broken(lambda j: j.pop("width"), "missing required field 'width'")
    broken(lambda j: j.update(streams=9), "between 1 and 8")
    broken(lambda j: j["layers"][0].update(type="mamba"), "is not supported")
    broken(lambda j: j["layers"][0]["mixer"].update(tau=0.0), "must be positive")
    broken(lambda j: j["layers"][1]["mixer"]["left"].update(kv_heads=4), "multiple of")
    broken(lambda j: j["layers"][1]["mixer"]["left"]["q_temp"].update(every=0), "must be positive")
    broken(lambda j: j["layers"][1]["mixer"]["right"].pop("state"), "missing required field 'layers\\[1\\].mixer.right.state'")
    broken(lambda j: j["layers"][2]["mixer"].update(groups=4), "multiple of")
    broken(lambda j: j["layers"][2]["mixer"].update(norm_groups=7), "multiple of")
    broken(lambda j: j["layers"][0]["mlp"].update(kind="moe"), "is not supported")


@pytest.mark.parametrize("cfg", [TK_A, TK_B, TK_C])
def test_tensor_lists_agree_with_the_description(cfg):
    from mlxforge_b200.config.registry import get_architecture
    c, model = _model(cfg)
    specs = {k: tuple(v.shape) for k, v in model.tensor_specs().items()}
    assert specs == {n: tuple(s) for n, s in tensor_shapes(cfg)}
    listed = {n: tuple(s) for n, s, _ in get_architecture("Takavik").random_tensors(c)}
    assert listed == specs
    assert model.graph_safe and model.spec.streams == (cfg.get("streams") or 1)
    assert [l["mixer"][RANK] for l in c.layers if l["type"] == "gla"] == [l["mixer"][RANK] for l in cfg["layers"] if l["type"] == "gla"]


def test_cache_layout_pages_beside_states():
    import torch
    from mlxforge_b200.cache.manager import CacheManager
    from mlxforge_b200.parts.base import FixedState, PagedKV
    _, model = _model(TK_A)
    layout = model.cache_layout
    assert {(g.need, g.n_lanes) for g in layout.paged} == {(PagedKV(3, 12, v_head_dim=20), 1), (PagedKV(1, 20, v_head_dim=6), 1)}
    up4 = lambda n: (n + 3) // 4 * 4
    tags = sorted((g.need.tag, g.need.shape[0]) for g in layout.state)
    assert tags == sorted([("gated_linear", 3 * 10 * 6), ("selective_scan", up4(36 * 10 + 36)),
                           ("mamba2", up4(6 * 14 * 10 + 4 * (60 + 2 * 3 * 14))),
                           ("selective_scan", up4(up4(22 * 19) + 2 * 22)), ("gated_linear", 14 * 22)])
    assert [w[0] for w in layout.item_lane[1]] == ["paged", "state"] and layout.item_lane[0][0] == "state"
    cache = CacheManager(layout, page_size=16, max_tokens=128, max_seqs=2, dtype=torch.float32, device="cpu")
    lanes = cache.lane(1)
    assert isinstance(lanes, tuple) and isinstance(lanes[1].need, FixedState)
    seq = cache.open_sequence()
    cache.reserve([(seq, 50)])
    cache.commit(seq, 50)
    assert [len(b) for b in seq.blocks] == [4, 4]
    cache.close(seq)
    cache.check()


def test_how_a_portion_is_cut_into_segments():
    from mlxforge_b200.csrc.ops import SCAN_MAX_FLOATS, scan_segments
    b = lambda *lens: SimpleNamespace(q_len=list(lens), n_seqs=len(lens))
    held = (300, 600)
    assert scan_segments(b(1, 1, 1), 4, held, 1000, 64) == (1, 1)     # a decode step runs in one piece
    assert scan_segments(b(127, 1), 4, held, 1000, 64) == (1, 127)
    for lens, blocks, least in (((2048,), 32, 64), ((300, 1, 129), 3, 64), ((45, 23), 2, 8), ((1000,), 100, 64)):
        n, length = scan_segments(b(*lens), blocks, held, 1000, least)
        assert n > 1 and n * length >= max(lens) > (n - 1) * length and length % 8 == 0 and length >= least
    assert scan_segments(b(2048), 300, held, 1000, 64) == (1, 2048)   # the GPU is full without
    assert scan_segments(b(2048), 4, (0, 0), 1000, 64) == (1, 2048)   # how full it is cannot be had
    n, _ = scan_segments(b(4096), 1, held, SCAN_MAX_FLOATS // 8, 64)
    assert n <= 8                                                     # within the scratch for start states


def test_configurations_drawn_at_random_are_read():
    for seed in range(40):
        cfg = random_config(seed, seed % 2 == 0)
        _, model = _model(cfg)
        assert {k: tuple(v.shape) for k, v in model.tensor_specs().items()} == {n: tuple(s) for n, s in tensor_shapes(cfg)}
