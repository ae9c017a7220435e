"""``Takavik``: a decoder over several residual streams (hyper-connections, pre-norm with weights stored around
zero) whose layers are, in an order that config.json gives, softmax attention beside a selective scan
(``parallel``: half the sum of the two branches' normalised outputs; the attention has norms per head, no
rotation and a query temperature that grows with the position), a Mamba-2 recurrence (``mamba2``) or gated linear
attention (``gla``), each followed by a SiLU-gated feed-forward, or by nothing.  The head is the embedding table.
Described as data: every part is a registry kind that gets its sizes and constants as parameters.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.norm1|norm2``, ``l<i>.hc1|hc2.in|out|mix``,
``l<i>.mlp.gate|up|down``, and behind ``l<i>.mix.``: ``left.q|k|v|o|q.norm|k.norm``,
``right.in|conv|conv.b|x|dt|dt.b|A_log|D|o``, ``left.out``, ``right.out`` (parallel);
``in|conv|conv.b|dt_bias|A_log|D|norm|o`` (mamba2); ``q|k|v|g|o|norm|a1|a2|a2.b`` (gla).
"""
from __future__ import annotations

from typing import Iterator, Tuple

from ..config.registry import register_architecture
from ..config.takavik_config import TakavikConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleItem

DEFAULT_DECAY_RANK = 16      # of a configuration that does not name it (random weights)


def _mixer(cfg: TakavikConfig, layer, prefix: str) -> PartSpec:
    H, m, eps = cfg.width, layer["mixer"], cfg.norm_eps
    if layer["type"] == "mamba2":
        return PartSpec("mamba2", {
            "hidden_size": H, "n_heads": m["heads"], "head_dim": m["vdim"], "state": m["state"], "n_groups": m["groups"],
            "norm_groups": m["norm_groups"], "conv": m["conv"], "eps": eps, "out_f32": True}, prefix=prefix)
    if layer["type"] == "gla":
        return PartSpec("gated_linear", {
            "hidden_size": H, "n_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "tau": m["tau"],
            "decay_rank": m["decay_rank"] or DEFAULT_DECAY_RANK, "eps": eps, "out_f32": True}, prefix=prefix)
    a, r = m["left"], m["right"]
    left = PartSpec("normed_attention", {
        "hidden_size": H, "n_heads": a["heads"], "n_kv_heads": a["kv_heads"], "head_dim": a["dim"],
        "v_head_dim": a["vdim"], "softmax_scale": a["scale"], "qk_norm": "head", "query_temperature": a["q_temp"],
        "eps": eps, "out_f32": True}, prefix=prefix + "left.")
    right = PartSpec("selective_scan", {
        "hidden_size": H, "inner": r["inner"], "state": r["state"], "dt_rank": r["dt_rank"], "conv": r["conv"],
        "out_f32": True}, prefix=prefix + "right.")
    return PartSpec("side_by_side", {
        "hidden_size": H, "left": left, "right": right, "left_scale": 0.5, "right_scale": 0.5,
        "out_norm": {"eps": eps, "left": "left.out", "right": "right.out"}}, prefix=prefix)


def build_takavik_spec(cfg: TakavikConfig) -> ModelSpec:
    H, S = cfg.width, cfg.streams or 1

    def norm(name: str) -> PartSpec:
        i = name.rindex(".") + 1
        return PartSpec("group_rmsnorm", {"size": H, "eps": cfg.norm_eps, "streams": S, "tensor": name[i:],
                                          "one_plus": True}, prefix=name[:i])

    layers = []
    for i, layer in enumerate(cfg.layers):
        p, mlp, ff = f"l{i}.", layer["mlp"], None
        extra = [("mixer_connection", "connection", PartSpec("hyper", {"streams": S}, prefix=p + "hc1."))]
        if mlp is not None:
            ff = PartSpec("swiglu", {"hidden_size": H, "intermediate_size": mlp["ff"], "activation": "silu",
                                     "names": {"gate": "gate", "up": "up", "down": "down"}}, prefix=p + "mlp.")
            extra.append(("feed_forward_connection", "connection", PartSpec("hyper", {"streams": S}, prefix=p + "hc2.")))
        layers.append(LayerSpec(block="stream_prenorm", mixer=_mixer(cfg, layer, p + "mix."), mixer_norm=norm(p + "norm1"),
                                feed_forward=ff, feed_forward_norm=norm(p + "norm2") if ff is not None else None,
                                extra=tuple(extra) if cfg.streams else ()))
    return ModelSpec(
        hidden_size=H, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": H, "tensor": "embed"}),
        layers=tuple(layers), schedule=tuple(ScheduleItem(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": H, "tensor": "embed"}),
        streams=S,
    )


def takavik_random_tensors(cfg: TakavikConfig) -> Iterator[Tuple[str, Tuple[int, ...], object]]:
    """Names, shapes and kinds of a checkpoint of this configuration, in file order."""
    H, S = cfg.width, cfg.streams
    yield "embed", (cfg.vocab, H), "matrix"
    for i, layer in enumerate(cfg.layers):
        p, m, kind, mlp = f"l{i}.", layer["mixer"], layer["type"], layer["mlp"]
        q = p + "mix."
        yield p + "norm1", (H,), (0.0, 0.1)
        if kind == "mamba2":
            inner, bc, nh = m["heads"] * m["vdim"], m["groups"] * m["state"], m["heads"]
            C = inner + 2 * bc
            yield q + "in", (inner + C + nh, H), "matrix"
            yield q + "conv", (C, m["conv"]), (0.0, 0.5)
            yield q + "conv.b", (C,), (0.0, 0.1)
            yield q + "dt_bias", (nh,), (-3.0, 1.0)
            yield q + "A_log", (nh,), (1.0, 0.7)
            yield q + "D", (nh,), (1.0, 0.1)
            yield q + "norm", (inner,), "norm"
            yield q + "o", (H, inner), "matrix"
        elif kind == "gla":
            rank, n, nv = m["decay_rank"] or DEFAULT_DECAY_RANK, m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for t, rows in (("q", n), ("k", n), ("v", nv), ("g", nv)):
                yield q + t, (rows, H), "matrix"
            yield q + "o", (H, nv), "matrix"
            yield q + "norm", (m["vdim"],), "norm"
            yield q + "a1", (rank, H), "matrix"
            yield q + "a2", (n, rank), (0.0, 0.3)
            yield q + "a2.b", (n,), (1.0, 1.0)
        else:
            a, r = m["left"], m["right"]
            for t, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                yield q + "left." + t, (rows, H), "matrix"
            yield q + "left.q.norm", (a["dim"],), "norm"
            yield q + "left.k.norm", (a["dim"],), "norm"
            yield q + "left.o", (H, a["heads"] * a["vdim"]), "matrix"
            n = r["inner"]
            yield q + "right.in", (2 * n, H), "matrix"
            yield q + "right.conv", (n, r["conv"]), (0.0, 0.5)
            yield q + "right.conv.b", (n,), (0.0, 0.1)
            yield q + "right.x", (r["dt_rank"] + 2 * r["state"], n), "matrix"
            yield q + "right.dt", (n, r["dt_rank"]), (0.0, 0.1)
            yield q + "right.dt.b", (n,), (-3.0, 1.0)
            yield q + "right.A_log", (n, r["state"]), (1.0, 0.7)
            yield q + "right.D", (n,), (1.0, 0.1)
            yield q + "right.o", (H, n), "matrix"
            yield q + "left.out", (H,), "norm"
            yield q + "right.out", (H,), "norm"
        if mlp is not None:
            yield p + "norm2", (H,), (0.0, 0.1)
            yield p + "mlp.gate", (mlp["ff"], H), "matrix"
            yield p + "mlp.up", (mlp["ff"], H), "matrix"
            yield p + "mlp.down", (H, mlp["ff"]), "matrix"
        if S:
            for hc in ("hc1",) + (("hc2",) if mlp is not None else ()):
                yield f"{p}{hc}.in", (S,), (1.0 / S, 0.05)
                yield f"{p}{hc}.out", (S,), (1.0, 0.05)
                yield f"{p}{hc}.mix", (S, S), ("eye", 0.05)
    yield "final.norm", (H,), (0.0, 0.1)


register_architecture("Takavik", TakavikConfig, build_takavik_spec, takavik_random_tensors, replace=True)
