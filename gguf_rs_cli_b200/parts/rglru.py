"""A recurrent block around a real-gated linear recurrent unit, as the mixer of a layer (the recurrent block of Griffin).

Two branches of `width` channels read the layer's row h: y = gelu_tanh(W_y h + b_y), and u = conv(W_x h + b_x), a short
causal convolution per channel with a bias and no activation.  u is cut into `blocks` equal parts, each of which has a
square matrix for each of two gates, r = sigmoid(R_b u_b + b_r) and i = sigmoid(I_b u_b + b_i).  Per channel the mixer keeps
one number S per sequence (32-bit):
    log a = -8 r softplus(lam);   S <- a S + sqrt(1 - a^2) i u
and gives W_o (S y).  The convolution's last taps - 1 inputs are per-sequence state beside S.  The reference has no such
mixer (src/model/llama.rs has attention only).

y and x are one product.  The gates' products keep 32-bit results; gates, decays with their logarithms and exponentials
and the state are 32-bit (csrc/rglru.cu).  The gates' products are part of the recurrence's kernels, for prompts in bfloat16
on the tensor cores and for single tokens on the CUDA cores; other cases make them first.
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

RATE = 8.0                       # what the gated softplus of lam is multiplied by


@register_mixer("rglru")
class GatedLinearRecurrence(Part):
    """params: hidden_size, width, blocks, conv (taps).
    tensors: y, x [width, E] with y_bias, x_bias; conv [width, taps], conv_bias; ra, ri [blocks, n, n] with ra_bias, ri_bias
    [blocks, n] (n = width / blocks); lam [width]; o [E, width]."""

    NAMES = ("y", "y_bias", "x", "x_bias", "conv", "conv_bias", "ra", "ra_bias", "ri", "ri_bias", "lam", "o")

    def __init__(self, spec, dtype, device, position=None):
        super().__init__(spec, dtype, device)
        p = self.p
        self.W, self.blocks, self.K = int(p["width"]), int(p["blocks"]), int(p["conv"])
        if self.W % self.blocks:
            raise ValueError(f"rglru: {self.W} channels do not form {self.blocks} equal blocks")
        if not 1 <= self.K <= 16:
            raise ValueError(f"rglru: a convolution of {self.K} taps is not supported (1..16)")
        self.n = self.W // self.blocks

    def kv_spec(self) -> Optional[KVSpec]:
        return None

    def state_spec(self) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        spec = {"S": ((self.W,), "float32")}
        if self.K > 1:
            spec["conv"] = ((self.K - 1, self.W), "float32")
        return spec

    def tensor_requests(self) -> List[TensorRequest]:
        E, t, W, B, n = self.p["hidden_size"], self.spec.tensors, self.W, self.blocks, self.n
        shapes = {"y": (W, E), "y_bias": (W,), "x": (W, E), "x_bias": (W,), "conv": (W, self.K), "conv_bias": (W,), "ra": (B, n, n),
                  "ra_bias": (B, n), "ri": (B, n, n), "ri_bias": (B, n), "lam": (W,), "o": (E, W)}
        inits = {"conv": "uniform:-0.6:0.6", "lam": "uniform:-6:-2"}
        return [TensorRequest(t[name], shapes[name], init=inits.get(name, "normal")) for name in self.NAMES]

    def load(self, store: WeightStore) -> None:
        w = {local: store.get(r) for local, r in zip(self.NAMES, self.tensor_requests())}
        dt, dev, W, n = w["y"].dtype, w["y"].device, self.W, self.n
        # y and x as one matrix, x starting at a multiple of 8 rows
        self.off_x = (W + 7) // 8 * 8
        rows = (self.off_x + W + 7) // 8 * 8
        proj, bias = torch.zeros(rows, w["y"].shape[1], dtype=dt, device=dev), torch.zeros(rows, dtype=torch.float32, device=dev)
        for name, at in (("y", 0), ("x", self.off_x)):
            proj[at:at + W] = w[name].to(dt)
            bias[at:at + W] = w[name + "_bias"].to(torch.float32)
        self.proj = Linear(proj, bias, name="rglru.proj")
        self.taps = w["conv"].to(dt).contiguous()
        self.taps_t = self.taps.t().contiguous() if dt == torch.bfloat16 else None      # tap by tap, for 16-byte loads
        self.conv_bias = w["conv_bias"].to(dt).contiguous()
        # the gates' matrices of a block as one [2n, n], r's rows in front of i's
        self.gates = torch.cat([w["ra"].to(dt), w["ri"].to(dt)], dim=1).contiguous()
        self.gates_in = self.gates.transpose(1, 2).contiguous() if n <= self.HEAD_PRODUCT else None
        self.r_bias, self.i_bias = (w[k].to(torch.float32).reshape(W).contiguous() for k in ("ra_bias", "ri_bias"))
        lam = w["lam"].to(torch.float64)
        self.rate = (RATE * torch.nn.functional.softplus(lam, threshold=50.0)).to(torch.float32).contiguous()
        self.o = Linear(w["o"], name="rglru.o")

    HEAD_PRODUCT = 1024           # inputs per block up to which the per-head product kernel takes the gates
    accepts_residual = True
    graph_class = ()              # grids depend on the batch size only

    def absorb_input_norm(self, weight: torch.Tensor) -> bool:
        if not self.proj.tensor_core():
            return False
        self.proj.fold_input_scale(weight)
        return True

    def _gates(self, u, ctx: StepContext) -> torch.Tensor:
        """The gates' products [T, 2 width], 32-bit results: block by block its r columns, then its i columns."""
        T, n = u.shape[0], self.n
        z = ctx.ws.get("rglru.gates", (T, 2 * self.W), torch.float32)
        if self.gates_in is not None:
            return kernels.head_matmul(u, n, self.gates_in, z, 2 * n)
        for b in range(self.blocks):
            kernels.gemm(u[:, b * n:(b + 1) * n], self.gates[b], None, z[:, 2 * b * n:2 * (b + 1) * n])
        return z

    def forward(self, h, ctx: StepContext, run: RunView, residual=None) -> Optional[torch.Tensor]:
        W, T = self.W, h.shape[0]
        proj = self.proj(h, ctx)
        ctx.mark("projections")
        u = ctx.ws.get("rglru.conv", (T, W), ctx.dtype)
        carried = ctx.state(f"run{run.index}.conv") if self.K > 1 else None
        kernels.short_conv(proj[:, self.off_x:self.off_x + W], self.taps, carried, ctx, u, taps_t=self.taps_t, bias=self.conv_bias)
        ctx.mark("conv")
        rows = ctx.ws.get("rglru.rows", (T, W), ctx.dtype)
        y, S, rates = proj[:, :W], ctx.state(f"run{run.index}.S"), (self.r_bias, self.i_bias, self.rate)
        if ctx.decode and self.gates_in is not None:
            kernels.rglru_step(u, y, self.gates_in, *rates, S, rows, ctx, self.blocks)
        elif kernels.rglru_fused_supported(u, self.n):
            kernels.rglru_fused(u, y, self.gates, *rates, S, rows, ctx, self.blocks)
        else:
            kernels.rglru(u, y, self._gates(u, ctx), *rates, S, rows, ctx, self.blocks)
        ctx.mark("recurrence")
        term = self.o(rows, ctx, residual=residual, out_dtype=torch.float32)
        ctx.mark("o")
        return term
