"""Retention mixer: linear attention with one fixed decay per head and no softmax or denominator.

Projections of the mixer's input h: queries and keys (H heads of dk values), values and a gate (H heads of dv), stacked
into one product.  Queries and keys are rotated (split halves of the leading dimensions), the key is then multiplied by
dk ** -0.5.  Per head, with the head's decay a (a constant of the layer) and the state S, a matrix that starts at zero:

    S <- a S + k v^T;    o = S^T q;    y = o / sqrt(mean(o^2) + eps) * silu(W_g h)

and W_o maps the heads' results back.  S is kept per sequence between steps, 32-bit, value by value ([H, dv, dk]);
everything between the projections and the output projection is 32-bit.

One-token steps run one kernel between the two products.  Prompts of a bfloat16 run are cut into chunks whose products run
on the tensor cores, every 32-bit operand as a pair of TF32 numbers.  Everything else (32-bit runs, short portions, head
sizes the chunk kernels are not built for) runs the selective scan's 32-bit kernels: with a step size of one, the decay as a
step's factor and k and q as its input and output vectors that recurrence is this one.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ... import ops
from ..base import ChunkRequest, LayerCache, Part, PartSpec, StateRequest, StepInfo, WeightSpec, register_mixer, scratch_buf
from ..linear import StackedLinear


@register_mixer("retention")
class RetentionMixer(Part):
    def __init__(self, hidden: int, n_heads: int, key_dim: int, v_dim: int, decay: Sequence[float], eps: float, position: PartSpec,
                 names: Dict[str, str], cache_key: str = "retention", scan_chunk: int = ops.RETENTION_CHUNK):
        """decay: one number per head.  eps: of the heads' norm.  names: tensor names of q, k, v, g, o.  scan_chunk: rows of a
        chunk of the parallel scan of prompts (the result does not depend on it: the state is linear in its initial value)."""
        self.hidden, self.H, self.dk, self.dv = int(hidden), int(n_heads), int(key_dim), int(v_dim)
        if not (1 <= self.dk <= ops.MAX_RETENTION_KEY_DIM) or not (1 <= self.dv <= ops.MAX_RETENTION_VALUE_DIM):
            raise ValueError(f"retention: heads of {key_dim} x {v_dim} are outside what the kernels are built for "
                             f"({ops.MAX_RETENTION_KEY_DIM} x {ops.MAX_RETENTION_VALUE_DIM})")
        if self.H > ops.MAX_HEADS:
            raise ValueError(f"retention: {n_heads} heads exceed the kernels' limit of {ops.MAX_HEADS}")
        self.decay = tuple(float(a) for a in decay)
        if len(self.decay) != self.H:
            raise ValueError(f"retention: {len(self.decay)} decays for {self.H} heads")
        self.eps, self.k_scale = float(eps), self.dk ** -0.5
        self.cache_key, self.scan_chunk = cache_key, int(scan_chunk)
        self.position = position.build()
        if getattr(self.position, "layout", None) != "split_half" or (getattr(self.position, "scaling", None) or {}).get("kind") == "ramp":
            raise ValueError("retention: the kernels of this mixer rotate split-half pairs, cosines and sines as they are")
        self.proj = StackedLinear(hidden)
        self.q_off = self.proj.add(names["q"], self.H * self.dk)
        self.k_off = self.proj.add(names["k"], self.H * self.dk)
        self.v_off = self.proj.add(names["v"], self.H * self.dv)
        self.g_off = self.proj.add(names["g"], self.H * self.dv)
        self.o = StackedLinear(self.H * self.dv)
        self.o.add(names["o"], hidden)
        self.dtype: Optional[torch.dtype] = None

    def weight_specs(self) -> List[WeightSpec]:
        return self.proj.weight_specs() + self.o.weight_specs() + self.position.weight_specs()

    def cache_requests(self) -> list:
        return [StateRequest(self.cache_key, (self.H, self.dv, self.dk))]

    CHUNKS_FROM_ROWS = 32          # sequences of more rows are scanned in chunks side by side

    def step_requests(self) -> list:
        return [ChunkRequest(self.scan_chunk, min(self.scan_chunk, self.CHUNKS_FROM_ROWS))]

    def bind(self, tensors: Dict[str, torch.Tensor], dtype, device) -> None:
        self.dtype = dtype
        self.proj.bind(tensors, dtype, device)
        self.o.bind(tensors, dtype, device)
        self.position.bind(tensors, dtype, device)
        self.decays = torch.tensor(self.decay, dtype=torch.float32, device=device)
        self._no_skip = torch.zeros(self.H, dtype=torch.float32, device=device)
        self._one = torch.ones(self.H * self.dv, dtype=torch.float32, device=device)

    def forward(self, normed: torch.Tensor, step: StepInfo, cache: LayerCache, residual: torch.Tensor, accumulate: bool = True) -> None:
        proj = scratch_buf(f"retention.{self.cache_key}.proj", (step.n_rows, self.proj.out_features), torch.float32, normed.device)
        self.proj.forward(normed, proj)
        self.o.forward(self.mix(proj, step, cache), residual, accumulate=accumulate)

    def mix(self, proj: torch.Tensor, step: StepInfo, cache: LayerCache) -> torch.Tensor:
        """Everything between the projections (float32 [T, q | k | v | g]) and the output projection: [T, H * dv]."""
        if not cache.writes:
            raise ValueError("retention: a recurrent mixer cannot run on another layer's cache without storing "
                             "(its state would advance twice in one step)")
        T, dev, f32 = step.n_rows, proj.device, torch.float32
        new = lambda tag, shape, dt: scratch_buf(f"retention.{self.cache_key}.{tag}", shape, dt, dev)
        H, dk, dv = self.H, self.dk, self.dv
        gated = new("gated", (T, H * dv), self.dtype)
        state, table = cache.state[self.cache_key], self.position.rotation_table()
        if step.max_new == 1:
            ops.retention_decode(proj, self.q_off, self.k_off, self.v_off, self.g_off, table, self.decays, self.k_scale, self.eps, state,
                                 step, H, dk, dv, gated)
            return gated
        chunks = step.chunks.get(self.scan_chunk)
        if self.dtype == torch.bfloat16 and chunks is not None and ops.retention_chunked_ok(
                proj, (self.q_off, self.k_off, self.v_off, self.g_off), dk, dv, 2 * table.numel(), self.scan_chunk):
            ops.retention_chunked(proj, self.q_off, self.k_off, self.v_off, self.g_off, table, self.decays, self.k_scale, self.eps, state,
                                  step, chunks, self.scan_chunk, H, dk, dv, gated)
            return gated
        vkq = new("vkq", (T, H * (dv + 2 * dk)), f32)
        ones, decays = new("ones", (T, H), f32), new("decays", (T, H), f32)
        ops.retention_prepare(proj, self.q_off, self.k_off, self.v_off, table, step.positions, self.decays, self.k_scale, H, dk, dv,
                              vkq, ones, decays)
        y = new("y", (T, H * dv), f32)
        ops.ssm_scan(vkq, ones, decays, self._no_skip, state, step.cu_seqlens, step.slots, step.start_pos, y, H, dv, dk, H,
                     step.chunks.get(self.scan_chunk))
        ops.gated_rmsnorm(y, proj[:, self.g_off:self.g_off + H * dv], self._one, self.eps, H, True, gated)
        return gated
