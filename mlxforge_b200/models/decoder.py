"""The model every architecture becomes: parts built from a ``ModelSpec`` and run
in the order its schedule gives.  Nothing here knows Llama; the layer loop is
the reference's (src/model/decoder_model.cpp:330-351: embed, blocks, final norm,
head) with the head applied only to the rows whose logits were asked for.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Dict, List, Optional

import torch

from ..cache.manager import CacheLayout, GroupLayout
from ..parts.base import (EMBEDDINGS, HEADS, NORMS, FixedState, ModelSpec, PagedKV, TensorSpec, build_layer, build_part,
                          flatten_needs)
from ..weights.loader import WeightError, load_tensors


class DecoderModel:
    def __init__(self, spec: ModelSpec, runtime):
        self.spec = spec
        self.rt = runtime
        self.embedding = build_part(EMBEDDINGS, spec.embedding, runtime)
        self.blocks = [build_layer(ls, runtime) for ls in spec.layers]
        self.final_norm = build_part(NORMS, spec.final_norm, runtime)
        self.head = build_part(HEADS, spec.head, runtime)
        for i, item in enumerate(spec.schedule):
            if not (0 <= item.layer < len(self.blocks)):
                raise ValueError(f"schedule item {i} names layer {item.layer}, the model has {len(self.blocks)}")
            if item.cache_of is not None and not (0 <= item.cache_of < i):
                raise ValueError(f"schedule item {i} reads the cache of item {item.cache_of}, which does not run before it")
        self.cache_layout = self._layout()
        # called after every run of a layer with (item, stream tensor, pending write), if set: how a
        # test reads the residual stream between layers
        self.probe = None

    # ------------------------------------------------------------------ weights
    def parts(self):
        yield self.embedding
        for b in self.blocks:
            yield from b.parts()
        yield self.final_norm
        yield self.head

    @property
    def graph_safe(self) -> bool:
        """Whether every part (the attention mixers' position encodings included) can be
        recorded into a CUDA graph."""
        for p in self.parts():
            if not getattr(p, "graph_safe", False):
                return False
            pos = getattr(p, "position", None)
            if pos is not None and not getattr(pos, "graph_safe", False):
                return False
        return True

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        specs: Dict[str, TensorSpec] = {}
        for p in self.parts():
            for name, s in p.tensor_specs().items():
                old = specs.get(name)
                if old is not None and tuple(old.shape) != tuple(s.shape):
                    raise ValueError(f"tensor '{name}' is declared with shapes {old.shape} and {s.shape}")
                # a tensor is optional only if every part that reads it says so
                specs[name] = s if old is None else TensorSpec(s.shape, old.optional and s.optional, s.role)
        return specs

    def load(self, model_dir: str) -> None:
        tensors = load_tensors(model_dir, self.tensor_specs(), self.rt.device, exact=self.rt.precise)
        self.bind(tensors)

    def bind(self, tensors) -> None:
        for p in self.parts():
            p.bind(tensors)

    def weight_bytes(self) -> int:
        """Bytes of weights that one step reads: every part once per run of its layer."""
        total = self.final_norm.weight_bytes() + self.head.weight_bytes()
        for item in self.spec.schedule:
            total += sum(p.weight_bytes() for p in self.blocks[item.layer].parts())
        return total

    # ------------------------------------------------------------------ cache
    def _needs(self) -> List[tuple]:
        """What every item of the schedule keeps per request, as a flat tuple.  Items that read another's cache
        may see further back than it does: the owner's pages are then kept for the widest of them."""
        needs = [flatten_needs(self.blocks[item.layer].cache_need()) for item in self.spec.schedule]
        for i, item in enumerate(self.spec.schedule):
            if item.cache_of is None:
                continue
            root = item.cache_of
            while self.spec.schedule[root].cache_of is not None:
                root = self.spec.schedule[root].cache_of
            own = [n for n in needs[i] if isinstance(n, PagedKV)]
            src = [k for k, n in enumerate(needs[root]) if isinstance(n, PagedKV)]
            if len(src) != 1:
                raise ValueError(f"schedule item {i} reads the cache of item {item.cache_of}, which has none to share")
            need = needs[root][src[0]]
            if len(own) != 1 or (own[0].n_kv_heads, own[0].head_dim, own[0].value_dim, own[0].values_in_keys) != (
                    need.n_kv_heads, need.head_dim, need.value_dim, need.values_in_keys):
                raise ValueError(f"schedule item {i} cannot read a cache of another geometry")
            window = 0 if 0 in (own[0].window, need.window) else max(own[0].window, need.window)
            widened = list(needs[root])
            widened[src[0]] = replace(need, window=window, chunk=need.chunk if own[0].chunk == need.chunk else 0,
                                      keep_first=max(own[0].keep_first, need.keep_first))
            needs[root] = tuple(widened)
        return needs

    def _layout(self) -> CacheLayout:
        paged: List[list] = []     # [need, lanes]
        state: List[list] = []
        item_lane: List[Optional[tuple]] = []

        def place(need, layer: int) -> tuple:
            """The group and lane of one need: a lane more in the group of equal needs, or a new group."""
            if isinstance(need, PagedKV):
                groups, kind = paged, "paged"
            elif isinstance(need, FixedState):
                groups, kind = state, "state"
            else:
                raise TypeError(f"mixer of layer {layer} declares an unknown cache need {need!r}")
            for g, (n, lanes) in enumerate(groups):
                if n == need:
                    groups[g][1] += 1
                    return (kind, g, lanes)
            groups.append([need, 1])
            return (kind, len(groups) - 1, 0)

        for i, (item, needs) in enumerate(zip(self.spec.schedule, self._needs())):
            # an item that reads another's cache has the owner's pages in place of its own, and its own state
            lanes = tuple(self._paged_lane(item_lane[item.cache_of])
                          if item.cache_of is not None and isinstance(n, PagedKV) else place(n, item.layer) for n in needs)
            # several needs: the item's lanes are a tuple in the order of the needs
            item_lane.append(None if not lanes else lanes[0] if len(lanes) == 1 else lanes)
        return CacheLayout(tuple(GroupLayout(n, l) for n, l in paged), tuple(GroupLayout(n, l) for n, l in state),
                           tuple(item_lane))

    @staticmethod
    def _paged_lane(where) -> tuple:
        """The lane of pages among an item's lanes."""
        return next(w for w in (where if isinstance(where[0], tuple) else (where,)) if w[0] == "paged")

    # ------------------------------------------------------------------ forward
    def forward(self, batch, cache) -> Optional[torch.Tensor]:
        """Run the tokens of ``batch`` through every item of the schedule, writing
        the cache, and return float32 logits [n_wanted, vocab] (None if nothing
        was asked for)."""
        rt = self.rt
        T = batch.n_tokens
        residual = rt.buffer("residual", (T, self.spec.streams * self.spec.hidden_size), torch.float32)
        self.embedding.embed(batch, residual, self.spec.streams)
        pending = None
        for i, item in enumerate(self.spec.schedule):
            residual, pending = self.blocks[item.layer].forward(
                residual, pending, batch, cache.lane(i), writes_cache=item.cache_of is None)
            if self.probe is not None:
                self.probe(i, residual, pending)
        if batch.n_wanted == 0:
            return None
        hn = self.final_norm.add_forward(residual, pending, rows=batch.want_rows,
                                         out=rt.buffer("final.norm", (batch.n_wanted, self.spec.hidden_size)))
        logits = rt.buffer("logits", (batch.n_wanted, self.spec.vocab_size), torch.float32)
        return self.head.forward(hn, logits)
