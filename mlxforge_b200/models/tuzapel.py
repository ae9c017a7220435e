"""``Tuzapel``: a decoder with a layer norm before and behind every sublayer
(``x += norm1b(mixer(norm1(x))); x += norm2b(ff(norm2(x)))``).  The mixer is, in an order that config.json
gives, attention over a compressed latent (queries through a latent of their own, neighbouring channels
rotated), or grouped-query attention within a window whose projections pass a short causal convolution, with
norms per head, a rotation of the first channels by a table that slows long waves down, one added to the
softmax denominator, and keys and values of its own or of an earlier layer.  The feed-forward is a clamped
gated one, dense or a mixture of experts (weights: the softmax over the chosen logits), or absent.  The head is
the embedding table, its logits under a soft cap.  Described as data: every part is a registry kind that gets
its sizes and constants as parameters.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.norm1|norm1b|norm2|norm2b``, behind ``l<i>.mix.``
``dq|dq.norm|uq|dkv|dkv.norm|uk|uv|o`` (latent) or ``q|k|v|o|q.norm|k.norm|q.conv|k.conv|v.conv`` (attention;
without the keys' and values' where another layer's are read), ``l<i>.mlp.gate|up|down`` (dense) or
``l<i>.mlp.router|router.b|e<j>.gate|up|down``.
"""
from __future__ import annotations

from typing import Iterator, Tuple

from ..config.registry import register_architecture
from ..config.tuzapel_config import TuzapelConfig
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleItem

GATE_ALPHA, GATE_UP_OFFSET = 1.702, 1.0       # g sigmoid(1.702 g) (u + 1)
SINK = 0.0                                    # exp(0) = 1 joins every softmax denominator of an attention layer


def _mixer(cfg: TuzapelConfig, layer, prefix: str) -> PartSpec:
    m = layer["mixer"]
    common = {"hidden_size": cfg.width, "n_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
              "softmax_scale": m["scale"], "eps": cfg.norm_eps}
    if layer["type"] == "latent_attention":
        rot = m["rot"] or {"base": 10000.0, "dims": 0}
        return PartSpec("latent_attention", dict(
            common, rot_dim=m["rot_dim"], q_rank=m["q_rank"], kv_rank=m["kv_rank"], rope_base=rot["base"],
            rot_dims=rot["dims"], pairing="pairs", gate=False), prefix=prefix)
    return PartSpec("normed_attention", dict(
        common, n_kv_heads=m["kv_heads"], qk_norm="head", rotary=m["rot"], window=m["window"], conv=m["conv"], sink=SINK,
        shares_cache=m["kv_from"] is not None), prefix=prefix)


def _feed_forward(cfg: TuzapelConfig, mlp, prefix: str) -> PartSpec:
    size = {"hidden_size": cfg.width, "intermediate_size": mlp["ff"]}
    if mlp["kind"] == "dense":
        return PartSpec("swiglu", dict(
            size, activation={"limit": mlp["limit"], "alpha": GATE_ALPHA, "up_offset": GATE_UP_OFFSET},
            names={"gate": "gate", "up": "up", "down": "down"}), prefix=prefix)
    # the softmax over all logits, divided by the sum of the chosen ones, is the softmax over the chosen ones
    return PartSpec("routed_experts", dict(
        size, n_experts=mlp["experts"], top=mlp["top"], scoring="softmax", renormalize=True, logit_bias="router.b",
        limit=mlp["limit"], alpha=GATE_ALPHA, up_offset=GATE_UP_OFFSET), prefix=prefix)


def build_tuzapel_spec(cfg: TuzapelConfig) -> ModelSpec:
    H = cfg.width

    def norm(name: str) -> PartSpec:
        i = name.rindex(".") + 1
        return PartSpec("layernorm", {"size": H, "eps": cfg.norm_eps, "tensor": name[i:]}, prefix=name[:i])

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, mlp = f"l{i}.", layer["mlp"]
        extra = [("mixer_post_norm", "norm", norm(p + "norm1b"))]
        if mlp is not None:
            extra.append(("feed_forward_post_norm", "norm", norm(p + "norm2b")))
        layers.append(LayerSpec(block="sandwich_norm", mixer=_mixer(cfg, layer, p + "mix."), mixer_norm=norm(p + "norm1"),
                                feed_forward=_feed_forward(cfg, mlp, p + "mlp.") if mlp is not None else None,
                                feed_forward_norm=norm(p + "norm2") if mlp is not None else None, extra=tuple(extra)))
        schedule.append(ScheduleItem(i, cache_of=layer["mixer"].get("kv_from")))
    return ModelSpec(
        hidden_size=H, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": H, "tensor": "embed"}),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": H, "tensor": "embed",
                                      "softcap": cfg.logit_softcap}),
    )


def tuzapel_random_tensors(cfg: TuzapelConfig) -> Iterator[Tuple[str, Tuple[int, ...], object]]:
    """Names, shapes and kinds of a checkpoint of this configuration, in file order."""
    H = cfg.width
    yield "embed", (cfg.vocab, H), "matrix"
    for i, layer in enumerate(cfg.layers):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp is not None else ()):
            yield p + n, (H,), "norm"
        q = p + "mix."
        nh, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "latent_attention":
            yield q + "dq", (m["q_rank"], H), "matrix"
            yield q + "dq.norm", (m["q_rank"],), "norm"
            yield q + "uq", (nh * (d + m["rot_dim"]), m["q_rank"]), "matrix"
            yield q + "dkv", (m["kv_rank"] + m["rot_dim"], H), "matrix"
            yield q + "dkv.norm", (m["kv_rank"],), "norm"
            yield q + "uk", (nh * d, m["kv_rank"]), "matrix"
            yield q + "uv", (nh * dv, m["kv_rank"]), "matrix"
        else:
            rows = {"q": nh * d, "k": m["kv_heads"] * d, "v": m["kv_heads"] * dv}
            for r in ("q",) if m["kv_from"] is not None else ("q", "k", "v"):
                yield q + r, (rows[r], H), "matrix"
                if m["conv"]:
                    yield q + r + ".conv", (rows[r], m["conv"]), (0.0, 0.5)
                if r != "v":
                    yield q + r + ".norm", (d,), "norm"
        yield q + "o", (H, nh * dv), "matrix"
        if mlp is None:
            continue
        q = p + "mlp."
        if mlp["kind"] == "moe":
            yield q + "router", (mlp["experts"], H), "matrix"
            yield q + "router.b", (mlp["experts"],), (0.0, 0.1)
        for e in ("",) if mlp["kind"] == "dense" else [f"e{k}." for k in range(mlp["experts"])]:
            yield q + e + "gate", (mlp["ff"], H), "matrix"
            yield q + e + "up", (mlp["ff"], H), "matrix"
            yield q + e + "down", (H, mlp["ff"]), "matrix"
    yield "final.norm", (H,), "norm"


register_architecture("Tuzapel", TuzapelConfig, build_tuzapel_spec, tuzapel_random_tensors, replace=True)
