"""A mixture of experts without a router: a table [vocab, top] names each token id's experts.

    y = 1 / top * sum over the experts e of the token's row:  W_down,e (g sigmoid(alpha g) (u + 1)),
        g = min(W_gate,e h, limit),  u = clamp(W_up,e h, -limit, limit)

Tensors: ``.table`` (integers; a row's entries differ), ``.e<i>.gate`` / ``.up`` [F, E], ``.e<i>.down`` [E, F], stacked when they are
bound as ``parts/moe.py`` stacks them.

What runs depends on the token ids alone, so it is settled before the first layer: ``TableRouting``, which all such
feed-forwards of a model share, sorts the rows of every layer's table in one launch per step, and runs of a layer that a
schedule repeats use the same result.  Because the places are known before the layer's norm, the norm's kernel writes its rows straight
into the experts' tiles, and the next one adds a token's experts up: between them stand the two grouped products and nothing else.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional

import torch

from .. import ops
from ..weights import INT_TABLE, TensorSpec
from .base import Part, register_part


class TableRouting:
    """The tables of all layers of a model, and per step where every (token, expert) row goes."""

    def __init__(self):
        self.vocab, self._tables, self._shapes = 0, [], []
        self.flat = self.desc = None

    def add(self, table: torch.Tensor, n_experts: int) -> int:
        """One more table (at binding time); its number."""
        vocab, top = table.shape
        if self._tables and vocab != self.vocab:
            raise ValueError(f"expert tables of {self.vocab} and {vocab} token ids in one model")
        if int(table.min()) < 0 or int(table.max()) >= n_experts:
            raise ValueError(f"an expert table names experts {int(table.min())} .. {int(table.max())}, there are {n_experts}")
        self.vocab = vocab
        self._tables.append(table)
        self._shapes.append((int(n_experts), int(top)))
        self.flat = None
        return len(self._tables) - 1

    def _finish(self):
        at, rows = 0, []
        for t, (n_experts, top) in zip(self._tables, self._shapes):
            rows.append((n_experts, top, at))
            at += t.numel()
        if at >= 1 << 31:
            raise ValueError("the expert tables hold more entries than an int32 counts")
        device = self._tables[0].device
        self.flat = torch.cat([t.reshape(-1) for t in self._tables]).contiguous()
        self.desc = torch.tensor(rows, dtype=torch.int32, device=device)

    def begin(self, rt, batch) -> None:
        """At the start of a step, before any layer."""
        if not self._tables:
            return
        if self.flat is None:
            self._finish()
        batch.shared[self] = ops.table_route(batch.token_ids, self.vocab, self.flat, self.desc, self._shapes)

    def of(self, batch, number: int) -> "ops.TableRoute":
        return batch.shared[self][number]


@dataclass
class ExpertTiles:
    """Where a step's rows go for one layer's experts: the tiles and every row's place among them (tiles None: the row form,
    which reads the rows as they are)."""

    route: "ops.TableRoute"
    tiles: Optional[torch.Tensor] = None

    @property
    def places(self):
        return self.route.places if self.tiles is not None else None


class TableExperts(Part):
    graph_safe = True
    routes_ahead = True         # a block asks ``route`` before its norm and hands the result to ``forward``

    def __init__(self, width: int, inner: int, n_experts: int, top: int, vocab: int, limit: float, routing: TableRouting, alpha: float = 1.702):
        if not 0 < top <= n_experts:
            raise ValueError(f"{top} of {n_experts} experts cannot be chosen")
        self.width, self.inner, self.n_experts, self.top, self.vocab = width, inner, n_experts, top, vocab
        self.clamp = (float(alpha), float(limit))
        self.routing, self.number = routing, None
        self.w_gu = self.wd = None

    def tensor_specs(self, prefix) -> List[TensorSpec]:
        E, F = self.width, self.inner
        specs = [TensorSpec(prefix + ".table", (self.vocab, self.top), INT_TABLE, below=self.n_experts)]
        for e in range(self.n_experts):
            specs += [TensorSpec(f"{prefix}.e{e}.gate", (F, E)), TensorSpec(f"{prefix}.e{e}.up", (F, E)), TensorSpec(f"{prefix}.e{e}.down", (E, F))]
        return specs

    def bind(self, prefix, tensors, rt):
        pair = lambda e: torch.stack([tensors[f"{prefix}.e{e}.gate"], tensors[f"{prefix}.e{e}.up"]], dim=1).reshape(2 * self.inner, self.width)
        self.w_gu = torch.stack([pair(e) for e in range(self.n_experts)], dim=0).contiguous()
        self.wd = torch.stack([tensors[f"{prefix}.e{e}.down"] for e in range(self.n_experts)], dim=0).contiguous()
        for e in range(self.n_experts):      # the stacked copies are what runs
            for name in ("gate", "up", "down"):
                tensors.pop(f"{prefix}.e{e}.{name}", None)
        self.number = self.routing.add(tensors[prefix + ".table"], self.n_experts)

    def route(self, rt, batch) -> ExpertTiles:
        route = self.routing.of(batch, self.number)
        if not rt.experts_in_tiles(route.ids.numel(), self.w_gu):
            return ExpertTiles(route)
        return ExpertTiles(route, torch.empty((route.max_tiles * route.tile_rows, self.width), dtype=rt.dtype, device=route.ids.device))

    def forward(self, rt, h, routed: ExpertTiles):
        """float32 [tokens, width], or ``ops.ExpertRows`` that the next norm adds up."""
        if routed.tiles is None:
            return ops.moe_experts_rows(h, routed.route.ids, None, self.w_gu, self.wd, clamp=self.clamp)
        y = ops.moe_tile_products(routed.tiles, routed.route.tiles, self.w_gu, self.wd, rt.status, clamp=self.clamp)
        return ops.ExpertRows(y, routed.route.places, 1.0 / self.top)


register_part("feed_forward", "table_experts", TableExperts)
