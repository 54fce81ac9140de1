"""A model: embedding, layers, the order they run in, final norm, output head.

CodeClaper/tinyllama.c's architecture file builds one static node list per model
(falcon_h1.c:256-417) and the executor walks it (graph.c:1278-1302), evaluating the
output head for the last row only (graph.c:1282-1283).  Here the walk is over
``schedule``, a list of (layer, cache) pairs that is data of the model, and the head
runs on the rows whose logits are wanted.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from .. import ops
from ..parts.base import (ChunkRequest, KVRequest, LayerCache, LayerRun, LayerSpec, Part, PartSpec, StateRequest, StepInfo, WeightSpec,
                          step_scratch)
from ..parts.block import Block
from ..parts.feed_forward import MoEFeedForward
from ..parts.linear import StackedLinear, matrix_dtype


class Model:
    def __init__(self, config, layer_specs: Sequence[LayerSpec], schedule: Optional[Sequence[LayerRun]],
                 final_norm: PartSpec, embed_name: str, head_name: Optional[str], vocab: int, hidden: int,
                 embed_scale: float = 1.0, head_scale: float = 1.0, logit_softcap: float = 0.0,
                 row_tables: Optional[Dict[str, int]] = None, unused_tensors: Sequence[str] = ()):
        """unused_tensors: names that a model folder may hold although this model reads none of them (the loader does not
        call them unexpected).  row_tables: learned tables [rows, hidden] by tensor name -> number of rows; an entry of the run order may name a
        row that is added to the residual stream before it runs (LayerRun.add)."""
        self.config = config
        self.vocab, self.hidden = int(vocab), int(hidden)
        self.layers: List[Block] = [Block(s) for s in layer_specs]
        self.schedule: List[LayerRun] = list(schedule) if schedule is not None \
            else [LayerRun(i) for i in range(len(self.layers))]
        for r, run in enumerate(self.schedule):
            if not (0 <= run.layer < len(self.layers)):
                raise ValueError(f"run-order entry {r} names layer {run.layer}, which does not exist")
            if run.cache is not None and not (0 <= run.cache < len(self.schedule) and self.schedule[run.cache].cache is None):
                raise ValueError(f"run-order entry {r} reads the cache of entry {run.cache}, which has none of its own")
            if run.cache is not None and any(isinstance(q, StateRequest) for q in self.layers[run.layer].cache_requests()):
                raise ValueError(f"run-order entry {r} reads the cache of entry {run.cache} but layer {run.layer} has a "
                                 f"mixer with state of its own: only keys and values can be read without storing")
            if run.add is not None and not (row_tables and run.add[0] in row_tables and 0 <= run.add[1] < row_tables[run.add[0]]):
                raise ValueError(f"run-order entry {r} adds row {run.add!r}, which no table of the model has")
            if run.kv_cache is not None:
                # keys and values of an EARLIER entry with a cache of its own: its rows of this step are stored
                # before this entry reads them
                if run.cache is not None or not (0 <= run.kv_cache < r) or self.schedule[run.kv_cache].cache is not None \
                        or self.schedule[run.kv_cache].kv_cache is not None:
                    raise ValueError(f"run-order entry {r} reads the keys and values of entry {run.kv_cache}, which must be "
                                     f"an earlier entry that stores its own")
        # chunk lengths that parts want the step function to cut sequences into (one table each, every step)
        # as (rows, from how many rows of a sequence the table is wanted): the smallest threshold asked for a length
        asked: Dict[int, int] = {}
        for layer in self.layers:
            for q in layer.step_requests():
                if isinstance(q, ChunkRequest):
                    start = q.rows if q.from_rows is None else min(q.rows, q.from_rows)
                    asked[q.rows] = min(asked.get(q.rows, start), start)
        self.chunk_rows = tuple(sorted(asked))
        self.chunk_from = dict(asked)               # chunk length -> rows a sequence must exceed for the table to be made
        self.final_norm = final_norm.build()
        self.embed_name, self.head_name = embed_name, head_name            # head_name None: tied (core.c:1246-1249)
        self.embed_scale = float(embed_scale)
        self.logit_softcap = float(logit_softcap)          # > 0: logits <- cap * tanh(logits / cap)
        self.head = StackedLinear(hidden)
        self.head.add(head_name or embed_name, vocab, None, 1.0, head_scale)
        self.unused_tensors = frozenset(unused_tensors)
        self.row_tables = {k: int(v) for k, v in (row_tables or {}).items()}
        self.rows_of: Dict[str, torch.Tensor] = {}
        self.embed_table: Optional[torch.Tensor] = None
        self.by_table: List[MoEFeedForward] = []
        self.dtype: Optional[torch.dtype] = None
        self.device: Optional[torch.device] = None

    # ---- declarations ----------------------------------------------------------------------
    def weight_specs(self) -> List[WeightSpec]:
        specs = [WeightSpec(self.embed_name, (self.vocab, self.hidden), "normal")]
        if self.head_name:
            specs.append(WeightSpec(self.head_name, (self.vocab, self.hidden), "normal"))
        for layer in self.layers:
            specs += layer.weight_specs()
        specs += self.final_norm.weight_specs()
        specs += [WeightSpec(name, (rows, self.hidden), "normal") for name, rows in self.row_tables.items()]
        seen, out = set(), []
        for s in specs:
            if s.name not in seen:
                seen.add(s.name)
                out.append(s)
        return out

    def adopt_shapes(self, shapes: Dict[str, tuple]) -> None:
        """Before the tensors are checked: a part with a size that no configuration key gives (shapes_from) reads it off
        the stored tensors' shapes."""
        for layer in self.layers:
            for part in layer.parts():
                if hasattr(part, "shapes_from"):
                    part.shapes_from(shapes)

    def cache_requests(self) -> Dict[int, list]:
        """Cache needs per entry of the run order that owns a cache (key: its index)."""
        out = {}
        for r, run in enumerate(self.schedule):
            if run.cache is None:
                reqs = self.layers[run.layer].cache_requests()
                if run.kv_cache is not None:          # its keys and values are another entry's
                    reqs = [q for q in reqs if not isinstance(q, KVRequest)]
                out[r] = reqs
        return out

    def bind(self, tensors: Dict[str, torch.Tensor], dtype: torch.dtype, device) -> None:
        self.dtype, self.device = dtype, torch.device(device)
        for layer in self.layers:
            layer.bind(tensors, dtype, device)
        self.final_norm.bind(tensors, dtype, device)
        self.by_table = [l.ffn for l in self.layers if isinstance(l.ffn, MoEFeedForward) and l.ffn.table is not None] \
            if self.device.type == "cuda" else []
        self.expert_tables = ops.ExpertTables([p.table_entry() for p in self.by_table]) if self.by_table else None
        self.rows_of = {name: tensors[name].to(device=device, dtype=torch.float32).contiguous() for name in self.row_tables}
        emb = tensors[self.embed_name]
        self.embed_table = emb.to(device=device, dtype=matrix_dtype(emb.dtype, dtype)).contiguous()
        if self.head_name is None:
            self.head.bind({self.embed_name: self.embed_table}, dtype, device)     # shares the table's storage
        else:
            self.head.bind(tensors, dtype, device)

    # ---- forward ------------------------------------------------------------------------------
    def forward(self, step: StepInfo, cache, want_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """Runs the step's rows through every scheduled layer; returns float32 logits
        [n_wanted, vocab] for the packed rows in want_rows (None: no logits).

        The embedding is the step's first kernel and is launched with a full dependency on everything
        before it on the stream: kernels of this step may therefore fetch, ahead of their own dependency
        wait, what earlier steps left in the cache (never what a kernel of this step writes)."""
        x = torch.empty((step.n_rows, self.hidden), dtype=torch.float32, device=self.device)
        ops.embed(step.tokens, self.embed_table, self.embed_scale, x)
        if self.by_table:                              # experts that token ids choose: all layers' routing at once
            MoEFeedForward.route_step(self.by_table, self.expert_tables, step)
        with step_scratch(step):                       # the layers share the step's temporaries
            ready = False                              # whether a layer left the next one's input (Block.entry)
            for r, run in enumerate(self.schedule):
                if run.add is not None:            # a learned row joins the stream before this entry (a pass of a repeated range)
                    ops.add_row(x, self.rows_of[run.add[0]][run.add[1]])
                    ready = False
                if run.add_embedding:              # or the embedding output does
                    ops.embed_add(step.tokens, self.embed_table, self.embed_scale, x)
                    ready = False
                nxt = self.schedule[r + 1] if r + 1 < len(self.schedule) else None
                wanted = self.layers[nxt.layer].entry if nxt is not None and nxt.add is None and not nxt.add_embedding else None
                ready = self.layers[run.layer].forward(x, step, cache.layer_view(r if run.cache is None else run.cache, run.writes,
                                                                                 run.kv_cache), ready, wanted)
        if want_rows is None or want_rows.numel() == 0:
            return None
        n = want_rows.numel()
        normed = torch.empty((n, self.hidden), dtype=self.dtype, device=self.device)
        self.final_norm.forward(x, normed, want_rows)
        logits = torch.empty((n, self.vocab), dtype=torch.float32, device=self.device)
        self.head.forward(normed, logits)
        if self.logit_softcap > 0:
            ops.softcap(logits, self.logit_softcap)
        return logits
