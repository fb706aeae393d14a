"""Two mixers side by side as the mixer of a layer: both read the same rows.  The branches are parts of the mixer
registry; cache and state are theirs (at most one of them may keep keys and values).  Two ways of joining them:

`pair`: each result is brought to unit root mean square over the model's width and multiplied by a weight of its own,
and the mixer gives `mix` times their sum (mix 0.5: their mean).

`weighted_pair`: a constant times the one plus a constant times the other.  Because both are products of rows with an
output matrix, the sum is one product: the branches' rows, each times its constant, side by side against the two matrices
side by side.  The first products, which read the same rows, are one too.  So the pair costs two launches of products
where the branches apart cost four, and its result can be added to the stream in the last one's epilogue.

The reference has no such arrangement.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import kernels
from ..cache.cache import KVSpec
from ..config.specs import PartSpec
from ..weights.loader import TensorRequest, WeightStore
from .base import Blend, HostBatch, Part, RunView, StepContext, plan_key_of
from .linear import Linear
from .registry import MIXERS, register_mixer


def _round8(n: int) -> int:
    return (n + 7) // 8 * 8


class _Prefixed:
    """A run as a branch sees it: its states are named <branch>.<name> in the layer's run."""

    def __init__(self, run: RunView, prefix: str):
        self._run, self._prefix = run, prefix

    def __getattr__(self, name):
        return getattr(self._run, name)

    @property
    def index(self):
        return f"{self._run.index}.{self._prefix}"


class SideBySide(Part):
    """What both ways have in common.  params: left, right (PartSpecs of two mixers), position_of ("left" by default, or
    "right": the branch that gets the layer's position encoding)."""

    def __init__(self, spec, dtype, device, position=None):
        super().__init__(spec, dtype, device)
        p = self.p
        at = p.get("position_of", "left")
        self.left = MIXERS.get(p["left"].kind)(p["left"], dtype, device, position=position if at == "left" else None)
        self.right = MIXERS.get(p["right"].kind)(p["right"], dtype, device, position=position if at == "right" else None)
        self.branches = (("left", self.left), ("right", self.right))
        if sum(b.kv_spec() is not None for _, b in self.branches) > 1:
            raise ValueError("pair: at most one of two mixers side by side may keep keys and values")
        if p["left"].kind == p["right"].kind:
            raise ValueError("pair: two mixers of one kind would write their results into the same buffers of the step")
        if any(getattr(b, "shares_kv", False) for _, b in self.branches):
            raise ValueError("pair: a branch cannot read another run's keys and values")

    def kv_spec(self) -> Optional[KVSpec]:
        for _, b in self.branches:
            if b.kv_spec() is not None:
                return b.kv_spec()
        return None

    def reads_kv_spec(self) -> Optional[KVSpec]:
        return self.kv_spec()

    def state_spec(self) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        return {f"{name}.{k}": v for name, b in self.branches for k, v in b.state_spec().items()}

    def tensor_requests(self) -> List[TensorRequest]:
        return [r for _, b in self.branches for r in b.tensor_requests()]

    def load(self, store: WeightStore) -> None:
        for _, b in self.branches:
            b.load(store)

    # ---- planning and capture: the branches'
    def plan_key(self):
        return ("pair",) + tuple(plan_key_of(b) for _, b in self.branches)

    def plan(self, batch: HostBatch):
        out = {}
        for name, b in self.branches:
            if hasattr(b, "plan"):
                out.update({f"{name}.{k}": v for k, v in b.plan(batch).items()})
        return out

    def graph_class(self, batch: HostBatch):
        classes = []
        for _, b in self.branches:
            gc = getattr(b, "graph_class", None)
            c = gc(batch) if callable(gc) else gc
            if c is None:
                return None
            classes.append(c)
        return tuple(classes)

    def _branch_view(self, name: str, branch, ctx: StepContext, run: RunView) -> _Prefixed:
        """The run as the branch sees it; the branch finds its own index arrays under its own key."""
        if hasattr(branch, "plan"):
            mine = {k[len(name) + 1:]: v for k, v in ctx.plan_of(self).items() if k.startswith(name + ".")}
            ctx.plans[plan_key_of(branch)] = mine
        return _Prefixed(run, name)


@register_mixer("pair")
class MixerPair(SideBySide):
    """params: hidden_size, eps, mix (default 0.5), left, right.  tensors: left_out [E], right_out [E] (plain weights)."""

    def __init__(self, spec, dtype, device, position=None):
        super().__init__(spec, dtype, device, position)
        self.mix = float(self.p.get("mix", 0.5))

    def tensor_requests(self) -> List[TensorRequest]:
        E, t = self.p["hidden_size"], self.spec.tensors
        return super().tensor_requests() + [TensorRequest(t["left_out"], (E,), init="ones"), TensorRequest(t["right_out"], (E,), init="ones")]

    def load(self, store: WeightStore) -> None:
        super().load(store)
        wl, wr = (store.get(r) for r in self.tensor_requests()[-2:])
        self.weights = (wl, wr if wr.dtype == wl.dtype else wr.to(wl.dtype))

    def forward_blend(self, h, ctx: StepContext, run: RunView) -> Blend:
        terms = []
        for name, b in self.branches:
            term = b.forward(h, ctx, self._branch_view(name, b, ctx, run))
            if term is None or term.dim() != 2:
                raise RuntimeError("pair: a branch must give one term [tokens, width]")
            terms.append(term)
        return Blend(terms[0], terms[1], self.weights, self.mix, float(self.p["eps"]))

    def forward(self, h, ctx: StepContext, run: RunView) -> torch.Tensor:
        """The blended term itself, for arrangements that do not finish it in their own kernel."""
        b = self.forward_blend(h, ctx, run)
        out = ctx.ws.get("pair.out", b.a.shape, torch.float32)
        kernels.norm_sandwich(None, b.a, None, b.eps, y2=b.b, inner_weights=b.weights, mix=b.mix, u_out=out)
        return out


@register_mixer("weighted_pair")
class WeightedPair(SideBySide):
    """left_scale * left + right_scale * right.  Both branches must hand their first and last products over
    (`give_projections`, `mix_rows`).  params: hidden_size, left, right, left_scale, right_scale, position_of."""

    accepts_residual = True

    def __init__(self, spec, dtype, device, position=None):
        super().__init__(spec, dtype, device, position)
        self.scales = (float(self.p["left_scale"]), float(self.p["right_scale"]))
        for name, b in self.branches:
            if not hasattr(b, "give_projections"):
                raise ValueError(f"weighted_pair: a mixer of kind {b.spec.kind!r} cannot hand its products over")

    def load(self, store: WeightStore) -> None:
        super().load(store)
        ins, outs, self.in_cols, self.out_cols = [], [], [], []
        rows = cols = 0
        biased = None
        for name, b in self.branches:
            got = b.give_projections()
            if got is None:
                raise ValueError(f"weighted_pair: the {name} branch cannot hand its products over with these options")
            first, last = got
            if last.bias is not None:
                raise ValueError("weighted_pair: a bias behind a branch's output matrix is not supported")
            ins.append((rows, first))
            outs.append((cols, last))
            self.in_cols.append((rows, rows + first.out_features))
            self.out_cols.append((cols, cols + last.in_features))
            rows, cols = _round8(rows + first.out_features), _round8(cols + last.in_features)
            biased = biased or first.bias is not None
        w0 = ins[0][1].weight
        # each branch's rows (and columns) from a multiple of 8 on, zeros between
        w_in = torch.zeros(rows, w0.shape[1], dtype=w0.dtype, device=w0.device)
        bias = torch.zeros(rows, dtype=torch.float32, device=w0.device) if biased else None
        w_out = torch.zeros(outs[0][1].out_features, cols, dtype=w0.dtype, device=w0.device)
        for (at, first), (to, last) in zip(ins, outs):
            w_in[at:at + first.out_features] = first.weight.to(w0.dtype)
            if first.bias is not None:
                bias[at:at + first.out_features] = first.bias.to(torch.float32)
            w_out[:, to:to + last.in_features] = last.weight.to(w0.dtype)
        self.proj, self.o = Linear(w_in, bias, name="pair.proj"), Linear(w_out, name="pair.o")

    def absorb_input_norm(self, weight: torch.Tensor) -> bool:
        """Multiplies the weight of the norm in front of this mixer into the first product's matrix, where the tensor-core
        product (which can apply the norm's per-token scale) will run it."""
        if not self.proj.tensor_core():
            return False
        self.proj.fold_input_scale(weight)
        return True

    def forward(self, h, ctx: StepContext, run: RunView, residual=None) -> Optional[torch.Tensor]:
        proj = self.proj(h, ctx)
        ctx.mark("projections")
        # columns that no branch writes stay zero (their rows of the matrix are zero as well)
        rows = ctx.ws.get("pair.rows", (h.shape[0], self.o.in_features), ctx.dtype, zeroed=True)
        for (name, b), (i0, i1), (o0, o1), scale in zip(self.branches, self.in_cols, self.out_cols, self.scales):
            b.mix_rows(proj[:, i0:i1], ctx, self._branch_view(name, b, ctx, run), rows[:, o0:o1], out_scale=scale)
        term = self.o(rows, ctx, residual=residual, out_dtype=torch.float32)
        ctx.mark("o")
        return term
