"""The Takavik parts and models on the GPU against the plain implementation (plain_takavik.py).

Mechanism by mechanism (each part built from its registry with its own sizes, given a runtime, a
step batch and a cache lane, run over portions and single tokens of two sequences with pools full
of NaN; the recurrences in one piece and in segments), far keys and far states made to decide, then
whole models of three configurations and of random ones through the trace replayer's functions -- whole
prompts, the last tokens decoded one by one, portions down to two tokens, mixed batches on a pool
so small that pages and slots are used again, every request decoded from its first token -- in
float32 and bfloat16, and greedy generation through the engine's entry point and scheduler."""
import io

import numpy as np
import pytest

import plain_takavik as P
import trace_tools as TT
from helpers import bf16_round
from takavik_helpers import CONFIGS, attention, file_config, make_model, prompt, scan
from test_notirax_gpu import Harness, dev, host, rand, tdt, tol
from test_rabapel_gpu import build, launched

pytestmark = pytest.mark.gpu

LONG = [150, 70]
LONG_STEPS = [(90, 0), (40, 33), (1, 30), (17, 1), (1, 1), (1, 5)]
SHORT_STEPS = [(20, 0), (2, 5), (1, 1), (0, 15), (21, 1), (1, 1)]
H = 40


def f64(w, cut=2):
    return {k[cut:]: v.astype(np.float64) for k, v in w.items()}


def as32(w):
    return {k: np.asarray(v, np.float32) for k, v in w.items()}


# ----------------------------------------------------------------------------- streams and their norm

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("S,width,T", [(1, 40, 5), (3, 33, 4), (2, 192, 7), (5, 2304, 3), (4, 2048, 1)])
def test_stream_write_of_two_normalised_branches(dtype, S, width, T):
    """``x_t <- sum mix x + out (s1 rms(y1) w1 + s2 rms(y2) w2)``, the next read and its norm around zero, one
    kernel; with rows selected the streams stay."""
    from mlxforge_b200.engine.runtime import Runtime
    from mlxforge_b200.parts.base import NormedPair
    from mlxforge_b200.parts.connections import StreamWrite
    rng = np.random.default_rng(S * 1000 + width)
    rt = Runtime(tdt(dtype))
    w = {"m.weight": rand(rng, width, std=0.2)}
    norm = build("NORMS", "group_rmsnorm", {"size": width, "eps": 1e-5, "streams": S, "one_plus": True}, rt, w)
    xs, y1, y2 = rand(rng, T, S, width), rand(rng, T, width, std=3.0), rand(rng, T, width, std=0.2)
    w1, w2 = rand(rng, width), rand(rng, width)
    mix, w_out, w_in = rand(rng, S, S), rand(rng, S), rand(rng, S)
    f = lambda a: a.astype(np.float64)
    y = 0.5 * P.rms_norm(f(y1), f(w1), 1e-4) - 1.5 * P.rms_norm(f(y2), f(w2), 1e-4)
    new = P.stream_write(f(xs).transpose(1, 0, 2), y, f(mix), f(w_out))
    want = P.norm_one_plus(P.stream_read(new, f(w_in)), w["m.weight"], 1e-5)
    for branch in ("float32", dtype):
        pair = NormedPair(dev(y1, tdt(branch)), dev(w1), 0.5, dev(y2, tdt(branch)), dev(w2), -1.5, 1e-4)
        write = StreamWrite(pair, None, dev(mix), dev(w_out))
        streams = dev(xs.reshape(T, S * width))
        rows = dev(np.array([T - 1, 0], dtype=np.int32))
        picked = host(norm.add_forward(streams, write, rows=rows, read=dev(w_in)))
        assert np.array_equal(host(streams), f(xs).reshape(T, -1))
        out = host(norm.add_forward(streams, write, read=dev(w_in)))
        assert np.max(np.abs(out - want)) < tol(dtype, np.abs(want).max())
        assert np.max(np.abs(picked - want[[T - 1, 0]])) < tol(dtype, np.abs(want).max())
        assert np.max(np.abs(host(streams).reshape(T, S, width).transpose(1, 0, 2) - new)) < 1e-5 * np.abs(new).max()


# ----------------------------------------------------------------------------- the convolution

@pytest.mark.parametrize("out2", [None, "bfloat16", "float32"])
@pytest.mark.parametrize("C,taps,extra", [(40, 4, 8), (33, 2, 0), (256, 3, 4), (64, 1, 0), (24, 6, 3), (20, 4, 1)])
def test_convolution_over_portions_and_single_tokens(out2, C, taps, extra):
    """Columns of wider rows, with a bias and SiLU, the last inputs kept in the slot between steps (portions
    shorter than the taps among them); a long portion in runs of several tokens a thread."""
    import torch
    from mlxforge_b200.csrc import ops
    from mlxforge_b200.parts.base import FixedState
    rng = np.random.default_rng(C + taps)
    off = 8
    h = Harness("float32", FixedState((off + (taps - 1) * C + (-(taps - 1) * C) % 4,)), lengths=[345, 23],
                steps=[(20, 0), (2, 5), (1, 1), (0, 15), (21, 1), (300, 0), (1, 1)], max_tokens=512)
    w, b = as32({"w": rand(rng, C, taps, std=0.5), "b": rand(rng, C, std=0.5)}).values()
    wd, bd = dev(w), dev(b)
    xs = [rand(rng, n, C + extra).astype(np.float32) for n in h.lengths]
    got = [np.zeros((n, C)) for n in h.lengths]
    lane = h.cache.lane(0)
    for batch, rows in h.steps():
        x = dev(np.stack([xs[s][p] for s, p in rows]))
        out = torch.empty((len(rows), C), dtype=torch.float32, device="cuda")
        second = None if out2 is None else torch.empty((len(rows), C), dtype=tdt(out2), device="cuda")
        ops.conv_act(x, C + extra, wd, bd, True, lane.tensor, off, batch, out, second)
        if second is not None:
            assert np.array_equal(host(second), host(out.to(second.dtype)))
        o = host(out)
        for i, (s, p) in enumerate(rows):
            got[s][p] = o[i]
    for x, g in zip(xs, got):
        want = P.biased_convolution(x[:, :C].astype(np.float64), w.astype(np.float64), b.astype(np.float64))
        assert np.max(np.abs(g - want)) < 1e-5 * max(1.0, np.abs(want).max())


# ----------------------------------------------------------------------------- attention with norms per head

ATTN_CASES = {
    # heads, kv, dim, vdim, coef, every
    "odd": (6, 3, 12, 20, 0.7, 9),
    "narrow": (4, 1, 20, 6, -0.3, 5),
    "ones": (1, 1, 16, 16, 0.0, 1),
    "every_token": (2, 2, 8, 8, 0.4, 1),
    "tc64": (4, 2, 64, 64, 0.5, 33),
    "tc96": (6, 3, 96, 96, 0.4, 40),
    "tc128": (4, 1, 128, 128, 0.3, 50),
    "tc128v64": (4, 2, 128, 64, 0.3, 50),
    "wide_values": (2, 1, 48, 80, 0.3, 50),
}


def attention_part(case, rt, rng, width=H, scale=0.35):
    nh, kv, d, dv, coef, every = ATTN_CASES[case]
    w = as32({"m.q": rand(rng, nh * d, width, std=width ** -0.5), "m.k": rand(rng, kv * d, width, std=width ** -0.5),
              "m.v": rand(rng, kv * dv, width, std=width ** -0.5), "m.q.norm": 1.4 + 0.2 * rand(rng, d),
              "m.k.norm": 1.4 + 0.2 * rand(rng, d), "m.o": rand(rng, width, nh * dv, std=(nh * dv) ** -0.5)})
    temp = {"coef": coef, "every": every} if coef else None
    params = {"hidden_size": width, "n_heads": nh, "n_kv_heads": kv, "head_dim": d, "v_head_dim": dv, "softmax_scale": scale,
              "qk_norm": "head", "query_temperature": temp, "eps": 1e-5, "out_f32": True}
    return build("MIXERS", "normed_attention", params, rt, w), w, attention(nh, kv, d, dv, scale, (coef, every) if coef else None)


def kv_need(case):
    from mlxforge_b200.parts.base import PagedKV
    _, kv, d, dv, _, _ = ATTN_CASES[case]
    return PagedKV(kv, d, 0, v_head_dim=0 if dv == d else dv)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(ATTN_CASES))
def test_attention_with_norms_per_head_and_query_temperature(dtype, case):
    from mlxforge_b200.csrc import binding
    rng = np.random.default_rng(len(case))
    big = case.startswith("tc")
    h = Harness(dtype, kv_need(case), lengths=LONG if big else [45, 23], steps=LONG_STEPS if big else SHORT_STEPS)
    part, w, c = attention_part(case, h.rt, rng)
    assert part.cache_need() == h.cache.layout.paged[0].need
    xs = [rand(rng, n, H) for n in h.lengths]
    before = binding.kernel_launches()
    got = h.run_mixer(part, xs, dtype)
    ran = launched(before)
    for x, g in zip(xs, got):
        want = P.head_norm_attention(x.astype(np.float64), f64(w), c, 1e-5)
        assert np.max(np.abs(g - want)) < tol(dtype, np.abs(want).max()), (case, np.max(np.abs(g - want)))
        if dtype == "float32" and c.get("q_temp") and c["q_temp"]["every"] < len(x):       # the check has teeth
            for every in (c["q_temp"]["every"] + 1, 10 ** 6):
                other = P.head_norm_attention(x.astype(np.float64), f64(w), dict(c, q_temp=dict(c["q_temp"], every=every)), 1e-5)
                assert np.max(np.abs(other - want)) > 2 * tol(dtype, np.abs(want).max()), "the temperature does nothing here"
    assert ran.get("qk_norm_rope", 0) > 0
    if dtype == "bfloat16" and big:
        assert "attn_generic" not in ran, ran
        assert sum(v for k, v in ran.items() if k.startswith("attn_prefill")) and sum(v for k, v in ran.items() if k.startswith("attn_decode")), ran


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["odd", "tc64", "tc96", "tc128", "tc128v64", "wide_values"])
def test_far_keys_decide(dtype, case):
    """Every query prefers marked keys: one hundreds of tokens back, the first token and both sides of page borders.
    What they carry is large, so one key too few shows.  Prompt portions, then decoding."""
    width, n = 8, 400
    rng = np.random.default_rng(7)
    h = Harness(dtype, kv_need(case), lengths=[n], steps=[(n - 70,), (49,)] + [(1,)] * 21, max_tokens=512)
    part, w, c = attention_part(case, h.rt, rng, width=width, scale=0.25)
    nh, kv, d = c["heads"], c["kv_heads"], c["dim"]
    wq, wk = np.zeros_like(w["m.q"]), 0.01 * w["m.k"]
    for hh in range(nh):
        wq[hh * d + d - 1, 0] = 1.0               # a query has its whole norm in the last channel
    for g in range(kv):
        wk[g * d + d - 1] = 0.0
        wk[g * d + d - 1, 1] = 1.0                # a marked key too, an unmarked one has nothing there
    one = np.ones_like(w["m.q.norm"])
    w = dict(w, **{"m.q": wq, "m.k": wk, "m.q.norm": one, "m.k.norm": one})
    part.bind({k: dev(v) for k, v in w.items()})
    x = rand(rng, n, width)
    x[:, 0], x[:, 1] = 1.0, 0.0
    marked = [0, 15, 16, 63, 64, 127, 128, n - 300]
    for i, j in enumerate(marked):
        x[j, 1] = 3.0
        x[j, 2:] = np.roll(np.linspace(-4, 4, width - 2), i)
    x = bf16_round(x.astype(np.float32))
    got = h.run_mixer(part, [x], dtype)[0]
    want = P.head_norm_attention(x.astype(np.float64), f64(w), c, 1e-5)
    for j in (0, 16, n - 300):
        x2 = x.copy()
        x2[j, 1] = 0.0
        other = P.head_norm_attention(x2.astype(np.float64), f64(w), c, 1e-5)
        assert np.max(np.abs(other[-22:] - want[-22:])) > 1.5 * tol(dtype, np.abs(want).max()), j
    assert np.max(np.abs(got - want)) < tol(dtype, np.abs(want).max()), np.argmax(np.abs(got - want).max(axis=1))


# ----------------------------------------------------------------------------- the recurrent mixers

SCAN_CASES = {  # inner, state, dt_rank, taps
    "odd": (36, 10, 5, 2), "ones": (16, 1, 1, 1), "uneven": (22, 19, 3, 3), "rank": (64, 16, 40, 4), "two_lanes": (128, 32, 8, 4),
    "many_states": (40, 128, 4, 5), "most_states": (12, 500, 2, 3)}
MAMBA2_CASES = {  # heads, vdim, state, groups, norm_groups, taps
    "odd": (6, 10, 14, 3, 5, 5), "ones": (1, 16, 16, 1, 1, 1), "small": (2, 32, 32, 1, 2, 4), "wide": (4, 64, 128, 2, 1, 4),
    "mid": (3, 64, 64, 3, 3, 2), "parts": (2, 48, 200, 1, 1, 3), "uneven_parts": (1, 70, 131, 1, 2, 2)}
GLA_CASES = {  # heads, dim, vdim, tau, rank
    "odd": (3, 10, 6, 7.0, 5), "ones": (1, 16, 16, 1.0, 1), "small": (4, 32, 64, 16.0, 16), "wide": (2, 128, 128, 16.0, 16),
    "mid": (2, 48, 20, 4.0, 33), "parts": (1, 160, 40, 8.0, 3), "uneven_parts": (1, 133, 35, 2.0, 2)}


def scan_part(case, rt, rng, **kw):
    n, N, R, taps = SCAN_CASES[case]
    w = as32({"m.in": rand(rng, 2 * n, H, std=H ** -0.5), "m.conv": rand(rng, n, taps, std=0.5), "m.conv.b": rand(rng, n, std=0.3),
              "m.x": rand(rng, R + 2 * N, n, std=1.5 * n ** -0.5), "m.dt": rand(rng, n, R, std=R ** -0.5),
              "m.dt.b": rand(rng, n, std=1.0) - 2.0, "m.A_log": rand(rng, n, N, std=0.8), "m.D": rand(rng, n),
              "m.o": rand(rng, H, n, std=n ** -0.5)})
    params = dict({"hidden_size": H, "inner": n, "state": N, "dt_rank": R, "conv": taps, "out_f32": True}, **kw)
    c = scan(n, N, R, taps)
    return build("MIXERS", "selective_scan", params, rt, w), w, lambda x, W: P.selective_scan(x, W, c)


def mamba2_part(case, rt, rng, **kw):
    nh, dv, N, G, NG, taps = MAMBA2_CASES[case]
    inner, C = nh * dv, nh * dv + 2 * G * N
    w = as32({"m.in": rand(rng, inner + C + nh, H, std=1.5 * H ** -0.5), "m.conv": rand(rng, C, taps, std=0.5),
              "m.conv.b": rand(rng, C, std=0.3), "m.dt_bias": rand(rng, nh) - 1.0, "m.A_log": rand(rng, nh, std=0.8),
              "m.D": rand(rng, nh), "m.norm": 1 + 0.1 * rand(rng, inner), "m.o": rand(rng, H, inner, std=inner ** -0.5)})
    params = dict({"hidden_size": H, "n_heads": nh, "head_dim": dv, "state": N, "n_groups": G, "norm_groups": NG, "conv": taps,
                   "eps": 1e-5, "out_f32": True}, **kw)
    c = {"heads": nh, "vdim": dv, "state": N, "groups": G, "norm_groups": NG, "conv": taps}
    return build("MIXERS", "mamba2", params, rt, w), w, lambda x, W: P.mamba2(x, W, c, 1e-5)


def gla_part(case, rt, rng, **kw):
    nh, d, dv, tau, R = GLA_CASES[case]
    n, nv = nh * d, nh * dv
    w = as32({"m.q": rand(rng, n, H, std=H ** -0.5), "m.k": rand(rng, n, H, std=H ** -0.5), "m.v": rand(rng, nv, H, std=H ** -0.5),
              "m.g": rand(rng, nv, H, std=H ** -0.5), "m.a1": rand(rng, R, H, std=H ** -0.5), "m.a2": rand(rng, n, R, std=R ** -0.5),
              "m.a2.b": rand(rng, n), "m.norm": 1 + 0.1 * rand(rng, dv), "m.o": rand(rng, H, nv, std=nv ** -0.5)})
    params = dict({"hidden_size": H, "n_heads": nh, "head_dim": d, "v_head_dim": dv, "tau": tau, "decay_rank": R, "eps": 1e-5,
                   "out_f32": True}, **kw)
    c = {"heads": nh, "dim": d, "vdim": dv, "tau": tau}
    return build("MIXERS", "gated_linear", params, rt, w), w, lambda x, W: P.gated_linear(x, W, c, 1e-5)


MAKERS = {"selective_scan": (scan_part, SCAN_CASES), "mamba2": (mamba2_part, MAMBA2_CASES), "gated_linear": (gla_part, GLA_CASES)}
RECURRENT = [(k, c) for k, (_, cases) in MAKERS.items() for c in cases]


def state_need(kind, case, rng_seed=0):
    from mlxforge_b200.engine.runtime import Runtime
    return MAKERS[kind][0](case, Runtime(tdt("float32")), np.random.default_rng(rng_seed))[0].cache_need()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,case", RECURRENT)
@pytest.mark.parametrize("least", [64, 8])
def test_recurrent_mixers(dtype, kind, case, least):
    """In one piece (portions below the least segment) and cut into segments of eight tokens and more, beside
    single tokens and portions shorter than the convolution's taps."""
    from mlxforge_b200.csrc import binding
    rng = np.random.default_rng(len(case))
    h = Harness(dtype, state_need(kind, case), lengths=[104, 43], steps=[(40, 0), (2, 5), (1, 1), (0, 35), (60, 1), (1, 1)])
    part, w, oracle = MAKERS[kind][0](case, h.rt, rng, scan_min_tokens=least)
    assert part.cache_need() == h.cache.layout.state[0].need
    xs = [rand(rng, n, H, std=1.5) for n in h.lengths]
    before = binding.kernel_launches()
    got = h.run_mixer(part, xs, dtype)
    ran = launched(before)
    local = "scan_local" if kind == "selective_scan" else "decay_local"
    assert (ran.get(local, 0) > 0) == (least == 8) and (ran.get("scan_combine", 0) > 0) == (least == 8), ran
    for x, g in zip(xs, got):
        want = oracle(x.astype(np.float64), f64(w))
        assert np.max(np.abs(g - want)) < tol(dtype, np.abs(want).max()), (case, np.max(np.abs(g - want)), np.abs(want).max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(MAKERS))
@pytest.mark.parametrize("least", [64, 16])
def test_a_far_token_that_only_an_intact_state_returns(kind, least, dtype):
    """Nothing decays; one early token is large, hundreds of small ones follow (in portions and segments, the
    last ones decoded one by one).  A state lost, zeroed or mixed on the way would not return it."""
    case = {"selective_scan": "odd", "mamba2": "small", "gated_linear": "small"}[kind]
    rng = np.random.default_rng(11)
    n = 360
    h = Harness(dtype, state_need(kind, case), lengths=[n], steps=[(100,), (37,), (2,), (201,)] + [(1,)] * 20, max_tokens=512)
    part, w, oracle = MAKERS[kind][0](case, h.rt, rng, scan_min_tokens=least)
    keep = {"m.A_log": -9.0, "m.a2.b": 9.0, "m.dt.b": 1.0, "m.dt_bias": 1.0}
    w = {k: (np.full_like(v, keep[k]) if k in keep else v) for k, v in w.items()}
    part.bind({k: dev(v) for k, v in w.items()})
    x = rand(rng, n, H, std=0.12)
    x[5] = rand(rng, H, std=4.0)
    got = h.run_mixer(part, [x], dtype)[0]
    want = oracle(x.astype(np.float64), f64(w))
    x2 = x.copy()
    x2[5] = 0.0
    other = oracle(x2.astype(np.float64), f64(w))
    late = slice(n - 22, n)
    limit = tol(dtype, np.abs(want).max()) if dtype == "float32" else 0.1 * np.max(np.abs(want[late]))
    assert np.max(np.abs(other[late] - want[late])) > 3 * limit, "the far token leaves no trace in this set-up"
    assert np.max(np.abs(got[late] - want[late])) < limit


def test_segments_change_a_result_by_rounding_only():
    """The same portion in one piece and in segments of several lengths, and the state it leaves."""
    for kind, case in (("mamba2", "wide"), ("gated_linear", "mid"), ("selective_scan", "two_lanes")):
        outs, states = [], []
        for least in (1000, 64, 24, 8):
            rng = np.random.default_rng(3)
            h = Harness("float32", state_need(kind, case), lengths=[200, 7], steps=[(199, 7), (1, 0)])
            part, w, _ = MAKERS[kind][0](case, h.rt, rng, scan_min_tokens=least)
            xs = [rand(rng, n, H, std=1.5) for n in h.lengths]
            outs.append(h.run_mixer(part, xs, "float32"))
            states.append(host(h.cache.lane(0).tensor)[[s.slot for s in h.seqs]])
        for o, s in zip(outs[1:], states[1:]):
            assert max(np.max(np.abs(a - b)) for a, b in zip(o, outs[0])) < 1e-5 * max(np.abs(outs[0][0]).max(), 1.0), kind
            assert np.nanmax(np.abs(s - states[0])) < 1e-5 * max(np.nanmax(np.abs(states[0])), 1.0), kind


@pytest.mark.parametrize("wdtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,R,n,tau", [(1, 1, 7, None), (8, 16, 128, 16.0), (64, 5, 33, 3.0), (65, 16, 96, 1.0), (300, 7, 40, None),
                                       (70, 130, 64, 8.0), (9, 600, 40, None), (130, 700, 33, None)])
def test_narrow_product_and_its_decay(wdtype, T, R, n, tau):
    import torch
    from mlxforge_b200.csrc import ops
    rng = np.random.default_rng(T + R)
    low, wt, b = rand(rng, T, R + 3).astype(np.float32), rand(rng, R, n, std=2.0 * R ** -0.5), rand(rng, n, std=3.0).astype(np.float32)
    out = torch.empty((T, n), dtype=torch.float32, device="cuda")
    ops.low_rank(dev(low), R + 3, dev(wt, tdt(wdtype)), dev(b), out, decay_tau=tau)
    z = low[:, :R].astype(np.float64) @ wt.astype(np.float64) + b
    want = z if tau is None else P.sigmoid(z) ** (1.0 / tau)
    assert np.max(np.abs(host(out) - want)) < 2e-6 * max(1.0, np.abs(want).max()) * max(1, R // 100)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("first", [True, False])
@pytest.mark.parametrize("parts,T,width,groups,shared", [(1, 5, 64, 4, True), (3, 2, 30, 3, False), (2, 7, 1024, 1, False),
                                                         (1, 3, 4096, 2, False), (1, 9, 33, 1, False), (2, 4, 1200, 2, True),
                                                         (1, 6, 602, 1, False)])
def test_gate_and_grouped_norm(dtype, first, parts, T, width, groups, shared):
    import torch
    from mlxforge_b200.csrc import ops
    rng = np.random.default_rng(width)
    x, g = rand(rng, parts, T, width).astype(np.float32), rand(rng, T, width + 4, std=2.0).astype(np.float32)
    w = (1 + 0.2 * rand(rng, width // groups if shared else width)).astype(np.float32)
    out = torch.empty((T, width), dtype=tdt(dtype), device="cuda")
    ops.gated_norm(dev(x), dev(g)[:, 4:], width + 4, dev(w), 1e-5, out, groups, first)
    y, s = x.astype(np.float64).sum(0), P.silu(g[:, 4:].astype(np.float64))
    y = y * s if first else y
    y = P.rms_norm(y.reshape(T, groups, -1), None, 1e-5).reshape(T, width) * np.tile(w, groups if shared else 1)
    want = y if first else y * s
    assert np.max(np.abs(host(out) - want)) < tol(dtype, np.abs(want).max())


# ----------------------------------------------------------------------------- whole models

REQUEST_LENGTHS = {"A": [45, 23, 1, 60, 37, 2], "B": [40, 18, 33, 1], "C": [300, 150, 1, 260, 90]}
PORTIONS = {"A": (7, 2, 5, 3, 2, 11, 4, 2, 16, 1, 9), "B": (2, 3, 16, 2, 1, 17), "C": (150, 2, 64, 3, 70, 1, 16)}
PEAKED = {"A": 3.0, "B": 3.0, "C": 2.0}


def _oracle(cfg, w, reqs):
    expected = {rid: P.forward(cfg, w, toks) for rid, toks in reqs.items()}
    noise = {}
    for name, fn in (("bfloat16", P.round_bf16), ("float32", P.round_f32)):
        P.ROUND = fn
        try:
            noise[name] = max(float(np.max(np.abs(P.forward(cfg, w, toks) - expected[rid]))) for rid, toks in reqs.items())
        finally:
            P.ROUND = None
    scale = max(float(np.max(np.abs(e))) for e in expected.values())
    # 32-bit: 1e-4 of the logits' scale, unless the design itself is ill-conditioned somewhere (a read-out that is
    # nearly zero before it is normalised): then twenty times what rounding to 32-bit does to the plain implementation
    return expected, {"float32": max(1e-4 * max(1.0, scale), 20.0 * noise["float32"]), "bfloat16": 3.0 * noise["bfloat16"]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("takavik")
    out = {}
    for which in CONFIGS:
        for peaked in (False, True):
            d, cfg, w = make_model(tmp, which, seed=ord(which), qk_gain=PEAKED[which] if peaked else 1.0)
            reqs = {f"r{i}": prompt(cfg, n, i) for i, n in enumerate(REQUEST_LENGTHS[which])}
            expected, tols = _oracle(cfg, w, reqs)
            out[(which, peaked)] = (d, cfg, reqs, expected, tols, w)
    return out


def _replay(model_dir, dtype, trace, tmp_path, max_tokens=None, max_seqs=4):
    from mlxforge_b200.csrc import binding
    from mlxforge_b200.engine.replay import make_runner, replay
    runner = make_runner(model_dir, dtype, max_tokens or trace.live_tokens_rounded(), max_seqs=max_seqs)
    for pool in runner.cache._k + runner.cache._v + runner.cache._state:
        pool.fill_(float("nan"))
    out_dir = str(tmp_path / "out")
    before = binding.kernel_launches()
    replay(runner, trace.lines(), out_dir, done=io.StringIO())
    runner.cache.check()
    assert runner.cache.free_pages() == runner.cache.total_pages() and runner.cache.slots.n_free == max_seqs
    return out_dir, launched(before)


def _compare(got, expected, tol_, dtype, what):
    assert got, "the trace asked for nothing"
    worst, where = TT.worst(got, expected)
    if dtype == "float32":
        assert worst <= tol_, (what, worst, tol_, where, TT.first_bad(got, expected, tol_))
        return
    # bfloat16: the limit is three times what rounding did to ONE run of the plain implementation, so a
    # place may pass it by chance; none passes one and a half times the limit and at most one place in
    # fifty (or one) passes the limit itself
    assert worst <= 1.5 * tol_, (what, worst, tol_, where, TT.first_bad(got, expected, 1.5 * tol_))
    over = sum(1 for (rid, pos), row in got.items() if not np.max(np.abs(row.astype(np.float64) - expected[rid][pos])) <= tol_)
    assert over <= max(1, len(got) // 50), (what, over, len(got), tol_, TT.first_bad(got, expected, tol_))


def _check(models, which, peaked, dtype, trace, tmp_path, **kw):
    d, cfg, reqs, expected, tols, _ = models[(which, peaked)]
    out_dir, ran = _replay(d, dtype, trace, tmp_path, **kw)
    _compare(TT.read_outputs(trace, out_dir, cfg["vocab"]), expected, tols[dtype], dtype, (which, peaked, dtype))
    return ran


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CONFIGS))
def test_sum_of_the_streams_after_every_layer(models, which, dtype):
    from mlxforge_b200.engine.replay import make_runner
    from mlxforge_b200.engine.step import StepEntry
    d, cfg, reqs, _, tols, w = models[(which, False)]
    toks = reqs["r0"]
    layers, rounded = [], []
    P.forward(cfg, w, toks, layers)
    P.ROUND = P.round_bf16
    try:
        P.forward(cfg, w, toks, rounded)
    finally:
        P.ROUND = None
    runner = make_runner(d, dtype, 512)
    S, width = cfg.get("streams") or 1, cfg["width"]
    got = []

    def probe(i, streams, pending):
        moved = streams.clone()
        runner.model.final_norm.add_forward(moved, pending)         # the pending write, into a copy
        got.append(host(moved).reshape(len(toks), S, width).sum(1))
    runner.model.probe = probe
    seq = runner.cache.open_sequence()
    runner.step([StepEntry(seq, toks, [0])])
    assert len(got) == len(layers)
    for i, (g, want) in enumerate(zip(got, layers)):
        limit = 1e-5 * np.abs(want).max() if dtype == "float32" else 4.0 * np.max(np.abs(rounded[i] - want))
        assert np.max(np.abs(g - want)) < limit, (i, np.max(np.abs(g - want)), limit)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("peaked", [False, True])
@pytest.mark.parametrize("which", list(CONFIGS))
def test_whole_prompts_and_decoded_tails(models, which, peaked, dtype, tmp_path):
    reqs = models[(which, peaked)][2]
    _check(models, which, peaked, dtype, TT.whole(reqs), tmp_path)
    _check(models, which, peaked, dtype, TT.decode_tail(reqs, tail=40), tmp_path / "tail")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CONFIGS))
def test_portions_down_to_two_tokens(models, which, dtype, tmp_path):
    reqs = models[(which, True)][2]
    _check(models, which, True, dtype, TT.portions(reqs, PORTIONS[which]), tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CONFIGS))
def test_mixed_batches_on_a_pool_where_pages_and_slots_are_used_again(models, which, dtype, tmp_path):
    reqs = models[(which, True)][2]
    trace = TT.mixed(reqs, max_live=3, seed=3, decode_last=6, max_portion=9 if which != "C" else 200)
    assert trace.live_tokens_rounded() < sum((len(t) + 63) // 64 * 64 for t in reqs.values())
    _check(models, which, True, dtype, trace, tmp_path, max_seqs=3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CONFIGS))
def test_every_request_decoded_from_its_first_token(models, which, dtype, tmp_path):
    """Long decoding (300 steps for C) in a batch that shrinks: the first tokens of a sequence, page borders and
    the decode kernel's splits met token by token, decode steps replayed from graphs."""
    reqs = models[(which, False)][2]
    _check(models, which, False, dtype, TT.lockstep(reqs), tmp_path, max_seqs=len(reqs))


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Sizes, layer orders and constants drawn from a seed: whole prompts, portions and a mixed batch with reused
    pages, both dtypes, against the plain implementation."""
    from helpers import write_model_dir
    from takavik_helpers import random_config, random_weights
    big = seed % 2 == 0
    cfg = random_config(200 + seed, big)
    w = random_weights(cfg, seed)
    d = write_model_dir(str(tmp_path / "model"), file_config(cfg), w, "bfloat16")
    w64 = {k: v.astype(np.float64) for k, v in w.items()}
    reqs = {f"r{i}": prompt(cfg, n, i) for i, n in enumerate([200 + 9 * seed, 170] if big else [97 + seed, 40, 61])}
    reqs.update({"one": prompt(cfg, 1, 8), "two": prompt(cfg, 2, 9)})
    expected, tols = _oracle(cfg, w64, reqs)
    traces = (TT.whole(reqs), TT.portions(reqs), TT.mixed(reqs, max_live=3, seed=seed, decode_last=6, max_portion=50))
    for i, trace in enumerate(traces):
        for dtype in ("float32", "bfloat16"):
            out_dir, _ = _replay(d, dtype, trace, tmp_path / f"{i}{dtype}", max_seqs=3 if i == 2 else 4)
            got = TT.read_outputs(trace, out_dir, cfg["vocab"])
            assert len(got) > 100
            _compare(got, expected, tols[dtype], dtype, (cfg, i, dtype))


def test_batch_and_cut_do_not_change_a_position(models, tmp_path):
    """float32: a request inside a mixed batch, cut into portions, and alone and whole agree to rounding."""
    for which in ("A", "C"):
        d, cfg, reqs, *_ = models[(which, True)]
        a_dir, _ = _replay(d, "float32", TT.whole(reqs), tmp_path / (which + "whole"))
        t_mixed = TT.mixed(reqs, max_live=3, seed=11, decode_last=5, max_portion=9 if which == "A" else 180)
        b_dir, _ = _replay(d, "float32", t_mixed, tmp_path / (which + "mixed"), max_seqs=3)
        a = TT.read_outputs(TT.whole(reqs), a_dir, cfg["vocab"])
        b = TT.read_outputs(t_mixed, b_dir, cfg["vocab"])
        assert set(a) == set(b)
        scale = max(float(np.abs(v).max()) for v in a.values())
        assert max(float(np.max(np.abs(a[k] - b[k]))) for k in a) < 2e-5 * max(1.0, scale)


def test_serving_shapes_take_the_fast_kernels(models, tmp_path):
    """Configuration C in bfloat16: which kernels its prompts and its decoding go through."""
    reqs = models[("C", False)][2]
    ran = _check(models, "C", False, "bfloat16", TT.decode_tail(reqs, tail=8), tmp_path)
    for k in ("embed_positions", "hyper_norm", "conv_act", "decay_recurrence", "decay_local", "scan_combine", "gated_norm",
              "selective_scan", "scan_local", "low_rank", "qk_norm_rope", "attn_prefill_mma", "attn_decode", "stream_tmap"):
        assert ran.get(k, 0) > 0, (k, ran)
    assert "attn_generic" not in ran and "gemm_f32" not in ran, ran


# ----------------------------------------------------------------------------- generation through the entry point

@pytest.mark.parametrize("which", ["A", "C"])
def test_greedy_generation_through_the_engine(models, which):
    import mlxforge_b200 as mf
    d, cfg, reqs, expected, _, w = models[(which, False)]
    prompts = [reqs["r1"], reqs["r4"], reqs["r3"][:50]]
    # portions of at most 16 tokens under a budget of 24: prompts are cut and run beside decoding
    eng = mf.Engine(model_spec=d, dtype="float32", kv_pool_tokens=1024, prefill_chunk=16, token_budget=24, max_running=4)
    got = eng.generate(prompts, max_tokens=6)
    clear = agree = 0
    for p, g in zip(prompts, got):
        seq = list(p)
        for t in g:
            row = P.forward(cfg, w, seq)[-1]
            top2 = np.sort(row)[-2:]
            if top2[1] - top2[0] > 1e-3:
                clear += 1
                agree += int(t == int(np.argmax(row)))
            seq.append(t)
    assert clear >= 10 and agree == clear, (got, clear, agree)
    assert eng.metrics()["completed"] == 3
    eng16 = mf.Engine(model_spec=d, dtype="bfloat16", kv_pool_tokens=1024, max_running=4)
    out16 = eng16.generate(prompts, max_tokens=6)
    assert all(len(o) == 6 for o in out16)


def test_cli_generate_and_trace_run_for_takavik(models, tmp_path, capsys):
    from mlxforge_b200 import cli
    from mlxforge_b200.engine import replay as R
    d, cfg, reqs, expected, tols, w = models[("B", False)]
    prompt_ids = reqs["r2"][:20]
    capsys.readouterr()
    assert cli.main(["generate", d, ",".join(map(str, prompt_ids)), "5", "--dtype", "float32"]) == 0
    got = [int(t) for t in capsys.readouterr().out.split()]
    assert got == P.generate(cfg, w, prompt_ids, 5), got
    trace = TT.mixed(reqs, max_live=4, seed=1, decode_last=4)
    out_dir = tmp_path / "out"
    import sys
    old = sys.stdin
    sys.stdin = trace.lines()
    try:
        assert R.main(["--model", d, "--dtype", "float32", "--out", str(out_dir), "--max-tokens",
                       str(trace.live_tokens_rounded())]) == 0
    finally:
        sys.stdin = old
    capsys.readouterr()
    worst, where = TT.worst(TT.read_outputs(trace, str(out_dir), cfg["vocab"]), expected)
    assert worst <= tols["float32"], (worst, where)


def test_random_weights_mode_writes_a_model_that_loads(tmp_path):
    """The engine's own random-weights mode for this architecture, then a step through the model it wrote."""
    import json
    from mlxforge_b200.config import config_from_json
    from mlxforge_b200.engine.replay import make_runner
    from mlxforge_b200.engine.step import StepEntry
    from mlxforge_b200.weights.random_init import write_random_model
    from takavik_helpers import TK_A
    d = write_random_model(str(tmp_path / "m"), config_from_json(json.loads(json.dumps(TK_A))), seed=5, norm_std=0.1)
    runner = make_runner(d, "bfloat16", 64)
    seq = runner.cache.open_sequence()
    logits = runner.step([StepEntry(seq, [1, 2, 3, 4, 5], [4])])
    assert logits.shape == (1, 101) and bool(np.isfinite(host(logits)).all())
