"""The plain Tuzapel implementation against closed forms and hand-worked cases, the configuration
reader, the model description and the cache layout.  No GPU."""
import copy
import json
import math

import numpy as np
import pytest

import plain_tuzapel as P
from tuzapel_helpers import (BANDS, CONFIGS, TZ_A, TZ_B, TZ_C, attention, prompt, random_config, random_weights,
                             tensor_shapes)


# ----------------------------------------------------------------------------- the oracle's mechanisms

def test_layer_norm_takes_the_mean_off_and_has_no_bias():
    x = np.array([[1.0, 3.0, 5.0, 7.0]])
    want = np.array([-3.0, -1.0, 1.0, 3.0]) / math.sqrt(5.0 + 0.25)
    assert np.allclose(P.layer_norm(x, np.array([1.0, 2.0, 1.0, 0.5]), 0.25), want * [1.0, 2.0, 1.0, 0.5])
    assert np.allclose(P.layer_norm(x + 100.0, np.ones(4), 0.25), want)          # a shift changes nothing
    assert np.allclose(P.rms_norm(np.array([[3.0, 4.0]]), 1.0, 0.0), np.array([3.0, 4.0]) / math.sqrt(12.5))


def test_convolution_ends_at_its_own_token():
    u = np.zeros((6, 1))
    u[2] = 1.0
    y = P.causal_convolution(u, np.array([[5.0, 7.0, 11.0]]))[:, 0]
    assert y.tolist() == [0, 0, 11, 7, 5, 0]           # the last tap reads the token itself
    assert P.causal_convolution(u, np.array([[2.0]]))[2] == 2.0


def test_frequencies_keep_blend_and_slow_down():
    f, g = P.frequencies(8, 500.0), P.frequencies(8, 500.0, BANDS)
    waves = 2 * np.pi / f
    for w, a, b in zip(waves, f, g):
        if w < 40:
            assert b == a
        elif w > 120:
            assert b == a / 6
        else:
            s = (120 / w - 1) / 2
            assert a / 6 <= b <= a and np.isclose(b, (1 - s) * a / 6 + s * a)
    assert {bool(w < 40) for w in waves} == {True, False} and waves.max() > 120
    assert np.isclose(P.frequencies(2, 10.0)[0], 1.0) and P.frequencies(0, 10.0).shape == (0,)


@pytest.mark.parametrize("layout", ["half", "pairs"])
def test_rotation_turns_pairs_and_passes_the_rest(layout):
    x = np.zeros((4, 1, 6))
    x[:, 0] = [1, 0, 0, 0, 9, 8]
    y = P.rotate(x, np.array([0.5, 0.1]), layout)
    partner = 2 if layout == "half" else 1
    for p in range(4):
        assert np.isclose(y[p, 0, 0], math.cos(0.5 * p)) and np.isclose(y[p, 0, partner], math.sin(0.5 * p))
        assert y[p, 0, 4:].tolist() == [9, 8]
    # scores depend on the distance alone
    q, k = np.random.default_rng(0).standard_normal((2, 4))
    turn = lambda v, p: P.rotate(v[None, None], np.array([0.5, 0.1]), layout, [p])[0, 0]
    assert np.isclose(turn(q, 7) @ turn(k, 4), turn(q, 3) @ turn(k, 0))


def test_window_counts_the_token_itself():
    m = P.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[1].tolist() == [True, True] + [False] * 4
    assert np.array_equal(P.window_mask(4, 1), np.eye(4, dtype=bool)) and P.window_mask(5, 0).sum() == 15


def test_softmax_with_one_in_the_denominator():
    s = np.array([[0.0, math.log(2.0), -np.inf]])
    assert np.allclose(P.softmax_with_one(s), [[0.25, 0.5, 0.0]])
    assert np.allclose(P.softmax_with_one(np.array([[-800.0, -900.0]])), 0.0)      # nothing relevant: no attention
    assert np.allclose(P.softmax_with_one(np.array([[800.0, 700.0]])), [[1.0, 0.0]])


def test_clamped_gate():
    lim = 2.0
    for g, u in ((5.0, 9.0), (-7.0, -9.0), (0.5, -0.25)):
        a, b = min(g, lim), max(-lim, min(u, lim))
        assert np.isclose(P.clamped_gate(np.array(g), np.array(u), lim), a / (1 + math.exp(-1.702 * a)) * (b + 1))
    assert P.clamped_gate(np.array(-7.0), np.array(0.0), lim) > -1e-4             # the gate has no lower clamp: it closes


def test_experts_are_weighted_by_the_softmax_over_the_chosen():
    z = np.array([[1.0, 3.0, 2.0, -5.0], [0.0, 0.0, 0.0, 0.0]])
    w = P.choose_experts(z, 2)
    e = math.exp(1.0)
    assert np.allclose(w[0], [0, e / (1 + e), 1 / (1 + e), 0]) and np.allclose(w[1], [0.5, 0.5, 0, 0])
    assert np.allclose(P.choose_experts(z, 4)[0], P.softmax(z[0]))


def test_borrowed_keys_see_the_readers_window():
    """A reader with a window larger than the owner's sees keys that the owner no longer does."""
    rng = np.random.default_rng(2)
    m = attention(2, 1, 4, 4, 0.5, 3, 2, (4, 100.0, None))
    w = {"q": rng.standard_normal((8, 6)), "k": rng.standard_normal((4, 6)), "v": rng.standard_normal((4, 6)),
         "o": np.eye(8)[:6], "q.norm": np.ones(4), "k.norm": np.ones(4), "q.conv": rng.standard_normal((8, 2)),
         "k.conv": rng.standard_normal((4, 2)), "v.conv": rng.standard_normal((4, 2))}
    h = rng.standard_normal((9, 6))
    own, kv = P.conv_attention(h, w, m, 1e-6)
    assert np.allclose(P.conv_attention(h, w, m, 1e-6, kv)[0], own)
    wide = dict(m, mask={"size": 9})
    moved = h.copy()
    moved[0] += 1.0
    kv2 = P.conv_keys_values(moved, w, m, 1e-6)
    far = lambda mm, t: P.conv_attention(h, w, mm, 1e-6, t)[0][8]
    assert np.allclose(far(m, kv2), far(m, kv)) and not np.allclose(far(wide, kv2), far(wide, kv))


def test_latent_attention_is_ordinary_attention_over_expanded_keys():
    rng = np.random.default_rng(3)
    m = {"heads": 2, "dim": 3, "rot_dim": 2, "vdim": 4, "q_rank": 5, "kv_rank": 6, "scale": 0.7, "rot": {"base": 20.0, "dims": 2}}
    n = lambda *s: rng.standard_normal(s)
    w = {"dq": n(5, 7), "dq.norm": n(5), "uq": n(10, 5), "dkv": n(8, 7), "dkv.norm": n(6), "uk": n(6, 6), "uv": n(8, 6),
         "o": np.eye(8)}
    h = n(5, 7)
    y = P.latent_attention(h, w, m, 1e-6)
    cq = P.rms_norm(h @ w["dq"].T, w["dq.norm"], 1e-6) @ w["uq"].T
    ckv = h @ w["dkv"].T
    c = P.rms_norm(ckv[:, :6], w["dkv.norm"], 1e-6)
    for i in (0, 4):
        for hd in range(2):
            def turned(v, p):
                return np.array([v[0] * math.cos(p) - v[1] * math.sin(p), v[1] * math.cos(p) + v[0] * math.sin(p)])
            q = cq[i, hd * 5:hd * 5 + 5]
            s = [0.7 * (q[:3] @ (w["uk"][hd * 3:hd * 3 + 3] @ c[j]) + turned(q[3:], i) @ turned(ckv[j, 6:], j))
                 for j in range(i + 1)]
            p = np.exp(s) / np.sum(np.exp(s))
            want = sum(pj * (w["uv"][hd * 4:hd * 4 + 4] @ c[j]) for j, pj in enumerate(p))
            assert np.allclose(y[i, hd * 4:hd * 4 + 4], want)


def test_soft_cap():
    assert np.isclose(P.soft_cap(3.0, 2.0), 2 * math.tanh(1.5)) and P.soft_cap(3.0, None) == 3.0


def test_a_prefix_does_not_see_what_follows():
    for cfg in CONFIGS.values():
        w = {k: v.astype(np.float64) for k, v in random_weights(cfg, 1).items()}
        toks = prompt(cfg, 30, 0)
        assert np.allclose(P.forward(cfg, w, toks)[:17], P.forward(cfg, w, toks[:17]))


# ----------------------------------------------------------------------------- configuration and description

class _RT:
    """What the parts need of a runtime to be built (nothing is run)."""

    def __init__(self):
        import torch
        self.dtype, self.device, self.precise = torch.float32, torch.device("cpu"), True


def _model(cfg):
    from mlxforge_b200.config import config_from_json
    from mlxforge_b200.config.registry import get_architecture
    from mlxforge_b200.models.decoder import DecoderModel
    c = config_from_json(json.loads(json.dumps(cfg)))
    return c, DecoderModel(get_architecture("Tuzapel").build_spec(c), _RT())


def test_config_reader_defaults_errors_and_round_trip():
    from mlxforge_b200.config import config_from_json
    from mlxforge_b200.config.model_config import ConfigError
    from mlxforge_b200.config.registry import registered_architectures
    assert "Tuzapel" in registered_architectures()
    c = config_from_json(json.loads(json.dumps(TZ_B)))
    assert c.logit_softcap == 0.0 and c.layers[0]["mixer"]["window"] == 0 and c.layers[2]["mlp"]["limit"] is None
    assert c.layers[3]["mixer"]["conv"] == 0 and c.layers[4]["mixer"]["rot"] is None and c.layers[4]["mlp"] is None
    bare = copy.deepcopy(TZ_B)
    for k in ("kv_heads", "vdim", "scale"):
        bare["layers"][0]["mixer"].pop(k)
        bare["layers"][2]["mixer"].pop(k, None)
    bare["layers"][0]["mixer"]["rot"].pop("dims")
    b = config_from_json(bare)
    m = b.layers[0]["mixer"]
    assert (m["kv_heads"], m["vdim"], m["scale"], m["rot"]["dims"]) == (1, 16, 0.25, 16)
    assert b.layers[2]["mixer"]["vdim"] == 16 and np.isclose(b.layers[2]["mixer"]["scale"], 32 ** -0.5)
    for cfg in CONFIGS.values():
        a = config_from_json(json.loads(json.dumps(cfg)))
        again = config_from_json(json.loads(json.dumps(a.to_json())))
        assert again == a and again.layers == a.layers

    def broken(edit, text):
        j = copy.deepcopy(TZ_A)
        edit(j)
        with pytest.raises(ConfigError, match=text):
            config_from_json(j)
    mix = lambda j, i: j["layers"][i]["mixer"]
    broken(lambda j: j.pop("vocab"), "missing required field 'vocab'")
    broken(lambda j: j.update(logit_softcap=-1), "must not be negative")
    broken(lambda j: j["layers"][0].update(type="mamba2"), "is not supported")
    broken(lambda j: mix(j, 0).update(kv_heads=4), "multiple of")
    broken(lambda j: mix(j, 0)["rot"].update(dims=14), "between 0 and 12")
    broken(lambda j: mix(j, 0)["rot"]["scaling"].pop("low"), "missing required field 'layers\\[0\\].mixer.rot.scaling.low'")
    broken(lambda j: mix(j, 0)["rot"]["scaling"].update(high=0.5), "must not be below")
    broken(lambda j: mix(j, 0).update(conv=-1), "must not be negative")
    broken(lambda j: mix(j, 1).pop("q_rank"), "missing required field 'layers\\[1\\].mixer.q_rank'")
    broken(lambda j: mix(j, 1)["rot"].update(scaling=BANDS), "not supported in this mixer")
    broken(lambda j: mix(j, 2).update(kv_from=1), "must name an earlier attention layer")
    broken(lambda j: mix(j, 3).update(kv_from=2), "must name an earlier attention layer")
    broken(lambda j: mix(j, 2).update(kv_from=3), "must name an earlier attention layer")
    broken(lambda j: mix(j, 2).update(vdim=8), "differs from layer 0")
    broken(lambda j: j["layers"][0]["mlp"].update(limit=0), "must be positive")
    broken(lambda j: j["layers"][1]["mlp"]["router"].update(top=6), "cannot give a token 6")
    broken(lambda j: j["layers"][0]["mlp"].update(kind="gated"), "is not supported")


@pytest.mark.parametrize("which", list(CONFIGS))
def test_tensor_lists_agree_with_the_description(which):
    from mlxforge_b200.config.registry import get_architecture
    c, model = _model(CONFIGS[which])
    specs = {k: tuple(v.shape) for k, v in model.tensor_specs().items()}
    assert specs == {n: tuple(s) for n, s in tensor_shapes(CONFIGS[which])}
    assert {n: tuple(s) for n, s, _ in get_architecture("Tuzapel").random_tensors(c)} == specs
    assert model.graph_safe
    assert [s.cache_of for s in model.spec.schedule] == [l["mixer"].get("kv_from") for l in CONFIGS[which]["layers"]]


def test_cache_layout_lent_pages_last_for_the_widest_reader():
    import torch
    from mlxforge_b200.cache.manager import CacheManager
    from mlxforge_b200.parts.base import PagedKV
    _, model = _model(TZ_A)
    layout = model.cache_layout
    # layer 0 sees 11 tokens, its readers 23 and 7: its pages stay for 23; the readers have none of their own
    assert {(g.need, g.n_lanes) for g in layout.paged} == {
        (PagedKV(3, 12, 23, v_head_dim=20), 1), (PagedKV(1, 28, v_head_dim=22, values_in_keys=True), 1),
        (PagedKV(1, 11, v_head_dim=9, values_in_keys=True), 1)}
    # convolution state: taps - 1 rows of every projected channel, queries alone for the readers
    q, k, v = 6 * 12, 3 * 12, 3 * 20
    assert sorted(g.need.shape[0] for g in layout.state) == sorted([4 * (q + k + v), 1 * q, 2 * q])
    assert [w[0] for w in layout.item_lane[0]] == ["paged", "state"]
    for reader in (2, 3):
        assert layout.item_lane[reader][0] == layout.item_lane[0][0] and layout.item_lane[reader][1] != layout.item_lane[0][1]
    assert layout.item_lane[1][0] == "paged"
    _, b = _model(TZ_B)
    # a causal owner stays causal; one tap, or no convolution, keeps nothing
    assert b.cache_layout.item_lane[0][0] == "paged" and b.cache_layout.item_lane[3] == b.cache_layout.item_lane[0]
    assert b.cache_layout.paged[b.cache_layout.item_lane[0][1]].need.window == 0
    cache = CacheManager(layout, page_size=16, max_tokens=128, max_seqs=2, dtype=torch.float32, device="cpu")
    seq = cache.open_sequence()
    win = [g for g, gl in enumerate(layout.paged) if gl.need.window][0]
    for n in (50, 4, 1):
        cache.reserve([(seq, n)])
        cache.commit(seq, n)
    # the query at position 55 sees back to 33 through the widest reader: pages 0 and 1 are given back, 2 is not
    assert seq.length == 55 and [p < 0 for p in seq.blocks[win]] == [True, True, False, False]
    cache.close(seq)
    cache.check()


def test_pages_of_an_owner_whose_reader_has_no_window_are_never_given_back():
    cfg = copy.deepcopy(TZ_A)
    cfg["layers"][2]["mixer"].pop("mask")
    _, model = _model(cfg)
    assert all(g.need.window == 0 for g in model.cache_layout.paged)


def test_configurations_drawn_at_random_are_read():
    for seed in range(40):
        cfg = random_config(seed, seed % 2 == 0)
        _, model = _model(cfg)
        assert {k: tuple(v.shape) for k, v in model.tensor_specs().items()} == {n: tuple(s) for n, s in tensor_shapes(cfg)}


@pytest.mark.parametrize("dims,base,sc", [(8, 500.0, BANDS), (64, 10000.0, BANDS), (2, 3.0, None), (0, 100.0, None)])
def test_banded_frequencies_of_the_engine(dims, base, sc):
    from mlxforge_b200.parts.rope import banded_inverse_wavelengths
    f32, f64 = banded_inverse_wavelengths(dims, base, sc, "cpu")
    assert np.allclose(f64.numpy(), P.frequencies(dims, base, sc), rtol=1e-14) and f32.dtype.itemsize == 4


def test_plain_generation_is_greedy():
    w = {k: v.astype(np.float64) for k, v in random_weights(TZ_C, 2).items()}
    toks = prompt(TZ_C, 5, 1)
    out = P.generate(TZ_C, w, toks, 3)
    assert out[2] == int(np.argmax(P.forward(TZ_C, w, toks + out[:2])[-1]))
