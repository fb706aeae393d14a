"""Retention, as the mixer of a layer: linear attention with one fixed decay per head and no denominator.

Per head the mixer keeps a matrix S [dim, vdim] per sequence (32-bit) instead of keys and values:
    S <- decay S + k v^T;  o = S^T q
with q = rot(W_q h), k = rot(W_k h) dim^-1/2 (rot turns q and k by the token's position where the layer has a position
encoding), v = W_v h and a constant decay per head.  What is read out is brought to unit root mean square per head,
without a weight, multiplied by SiLU(W_g h), and projected back.  The reference has no such mixer (src/model/llama.rs
has attention only).

q, k, v and g are one matrix after loading (each part starting at a multiple of 8 rows), so one product reads h once.
Angles, rotated rows, decays and the state are 32-bit (csrc/retention.cu: prompts in chunks on the tensor cores, single tokens in
one pass over S, other cases by a walk over the tokens).  The part may stand beside another mixer that
reads the same rows (parts/pair.py).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import kernels
from ..cache.cache import KVSpec
from ..weights.loader import TensorRequest, WeightStore
from .base import Part, RunView, StepContext
from .linear import Linear
from .registry import register_mixer


@register_mixer("retention")
class Retention(Part):
    """params: hidden_size, heads, dim, vdim, decay (a list of one number per head), eps (of the read-out's norm).
    tensors: q, k [heads*dim, E], v, g [heads*vdim, E], o [E, heads*vdim]."""

    NAMES = ("q", "k", "v", "g", "o")

    def __init__(self, spec, dtype, device, position=None):
        super().__init__(spec, dtype, device)
        p = self.p
        self.H, self.D, self.Dv = p["heads"], p["dim"], p["vdim"]
        if len(p["decay"]) != self.H:
            raise ValueError(f"retention: {len(p['decay'])} decays for {self.H} heads")
        if position is not None and getattr(position, "gain", 1.0) != 1.0:
            raise ValueError("retention: a rotation whose sine and cosine carry a factor is not supported here")
        self.position = position

    def kv_spec(self) -> Optional[KVSpec]:
        return None

    def state_spec(self) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        return {"S": ((self.H, self.D, self.Dv), "float32")}

    def tensor_requests(self) -> List[TensorRequest]:
        E, t, n, nv = self.p["hidden_size"], self.spec.tensors, self.H * self.D, self.H * self.Dv
        return [TensorRequest(t["q"], (n, E)), TensorRequest(t["k"], (n, E)), TensorRequest(t["v"], (nv, E)),
                TensorRequest(t["g"], (nv, E)), TensorRequest(t["o"], (E, nv))]

    def load(self, store: WeightStore) -> None:
        w = {local: store.get(r) for local, r in zip(self.NAMES, self.tensor_requests())}
        dt, dev = w["q"].dtype, w["q"].device
        self.off, rows = {}, 0
        for name in ("q", "k", "v", "g"):
            self.off[name] = rows
            rows = (rows + w[name].shape[0] + 7) // 8 * 8
        proj = torch.zeros(rows, w["q"].shape[1], dtype=dt, device=dev)
        for name, at in self.off.items():
            proj[at:at + w[name].shape[0]] = w[name].to(dt)
        self.proj = Linear(proj, name="retention.proj")
        self.o = Linear(w["o"], name="retention.o")
        decay = torch.tensor(self.p["decay"], dtype=torch.float64)
        self.decay = decay.to(torch.float32).to(dev)
        # the chunked form takes powers of the decay
        self.log2_decay = torch.log2(decay).to(torch.float32).to(dev) if bool(((decay > 0) & (decay <= 1)).all()) else None
        self._norm_weights = {}

    accepts_residual = True
    graph_class = ()              # grids depend on the batch size only

    def give_projections(self) -> Tuple[Linear, Linear]:
        """For a mixer that runs this one beside another: hands its first and last product over (the caller then gives
        `mix_rows` what the first gives, and multiplies by the last itself)."""
        both, self.proj, self.o = (self.proj, self.o), None, None
        return both

    def absorb_input_norm(self, weight: torch.Tensor) -> bool:
        if not self.proj.tensor_core():
            return False
        self.proj.fold_input_scale(weight)
        return True

    def _norm_weight(self, scale: float, device) -> torch.Tensor:
        """The read-out's norm has no weight: its kernel gets a constant one, which carries the result's factor."""
        if scale not in self._norm_weights:
            self._norm_weights[scale] = torch.full((self.Dv,), scale, dtype=torch.float32, device=device)
        return self._norm_weights[scale]

    def mix_rows(self, proj, ctx: StepContext, run: RunView, out, out_scale: float = 1.0) -> torch.Tensor:
        """proj: what the first product gives; out [T, heads*vdim]: the gated rows times out_scale, for the last."""
        H, D, Dv, off, pos = self.H, self.D, self.Dv, self.off, self.position
        T = proj.shape[0]
        q, k, v = proj[:, off["q"]:off["q"] + H * D], proj[:, off["k"]:off["k"] + H * D], proj[:, off["v"]:off["v"] + H * Dv]
        gate, state, eps, k_scale = proj[:, off["g"]:off["g"] + H * Dv], ctx.state(f"run{run.index}.S"), self.p["eps"], D ** -0.5
        inv_freq, rot, pairing = (None, 0, 0) if pos is None else (pos.inv_freq, pos.rotary_dim, pos.pairing)
        if ctx.decode and max(D, Dv) <= 2048:
            kernels.retention_step(q, k, v, gate, inv_freq, rot, pairing, k_scale, self.decay, state, out, ctx, H, D, Dv, eps, out_scale)
            ctx.mark("recurrence")
            return out
        if self.log2_decay is not None and kernels.retention_chunks_supported(q, D, Dv):
            kernels.retention_chunks(q, k, v, gate, inv_freq, pairing, k_scale, self.log2_decay, state, out, ctx, H, D, eps, out_scale)
            ctx.mark("recurrence")
            return out
        read = ctx.ws.get("retention.read", (T, H * Dv), torch.float32)
        kernels.retention(q, k, v, inv_freq, rot, pairing, k_scale, self.decay, state, read, ctx, H, D, Dv)
        ctx.mark("recurrence")
        kernels.gated_head_norm(read, gate, self._norm_weight(out_scale, proj.device), eps, out, H, Dv, gate_function="silu")
        ctx.mark("head_norm")
        return out

    def forward(self, h, ctx: StepContext, run: RunView, residual=None) -> Optional[torch.Tensor]:
        proj = self.proj(h, ctx)
        ctx.mark("projections")
        out = self.mix_rows(proj, ctx, run, ctx.ws.get("retention.rows", (h.shape[0], self.H * self.Dv), ctx.dtype))
        term = self.o(out, ctx, residual=residual, out_dtype=torch.float32)
        ctx.mark("o")
        return term
