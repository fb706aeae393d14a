"""Latent attention as the mixer of a layer: keys and values of all heads are products of one latent row
per position, c = rms_norm(W_dkv h)[:kv_rank] * w, plus one rotated key part of rot_dim entries that all
heads share; only these kv_rank + rot_dim numbers per position are cached.

Per head the score is (q_plain . W_uk c + q_rot . k_rot) * scale and the value W_uv c.  The products
with W_uk and W_uv are moved to the query's side: q' = W_uk^T q_plain lives in the latent's space, so a
head's score is [q', q_rot] . [c, k_rot], the mix of values is the mix of latent rows, and W_uv is applied
to that mix once per token.  The attention kernel then sees one key/value head of kv_rank + rot_dim entries
whose first kv_rank entries are also its values.  Scores, softmax and mix run in 32-bit.

Prompts that start their sequences take the other order where the sizes allow it (bfloat16, dim + rot_dim
= vdim = 64 or 128): the step's latent rows are multiplied with W_uk and W_uv in one tensor-core product,
the per-head keys [W_uk c, k_rot] and values are laid out as pages of the step's own, and the tiled
attention kernel runs over them with 32-bit weights; the cache still receives the latent rows only.

Options: a window of the last `window` positions (the cache then keeps a ring of pages); a sink, one more key without a
value in the softmax's denominator whose score is a learned number per head, not scaled (`sink="learned"`, tensor `sink`
[heads]); one sigmoid gate per head on the heads' results, from a projection of the mixer's input (`out_gate="head"`,
tensor `g` [heads, E]; a number per head commutes with W_uv, so it is applied to the mix of latent rows).  The rotation
pairs neighbours or halves, as the position table says, and its sine and cosine may carry a factor.

Further options: queries that go through a latent of their own, c_q = rms_norm(W_dq h) * w, q = W_uq c_q (`q_rank`); a gate
per entry of the heads' results, sigmoid(W_g h) with a row for every value entry (`out_gate=True`; applied behind W_uv); and
layers that read another run's latent rows instead of making their own (`shares_kv`: no W_dkv; prompts on the tiled kernel
find the step's rows where the other layer left them).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import kernels
from ..cache.cache import KVSpec
from ..weights.loader import TensorRequest, WeightStore
from .base import HostBatch, Part, RunView, StepContext
from .linear import Linear
from .registry import register_mixer


@register_mixer("latent_attention")
class LatentAttention(Part):
    """params: hidden_size, heads, dim (unrotated q/k entries per head), rot_dim (rotated ones, behind them), vdim,
    kv_rank, scale, eps (of the latents' norms), window (default None), sink (default None; "learned"), out_gate (default
    None; "head", or True: a gate per entry), q_rank (default None), shares_kv (default False),
    term_f32 (default False: the result, which is added to the residual stream, in 32-bit also in bfloat16 mode).  position: a rotary table over the rot_dim part (its first rotary_dim entries are rotated, in the
    table's pairing).
    tensors: q [heads*(dim+rot_dim), E], or with q_rank dq [q_rank, E], dq_norm [q_rank], uq [heads*(dim+rot_dim), q_rank];
    unless shares_kv dkv [kv_rank+rot_dim, E], dkv_norm [kv_rank]; uk [heads*dim, kv_rank], uv [heads*vdim, kv_rank],
    o [E, heads*vdim]; with a sink `sink` [heads]; with a gate g [heads, E], per entry [heads*vdim, E]."""

    def __init__(self, spec, dtype, device, position=None):
        super().__init__(spec, dtype, device)
        p = self.p
        self.H, self.D, self.R, self.Dv, self.C = p["heads"], p["dim"], p["rot_dim"], p["vdim"], p["kv_rank"]
        self.position = position
        if self.R % 2:
            raise ValueError(f"latent_attention: rot_dim {self.R} must be even")
        if position is not None and position.rotary_dim > self.R:
            raise ValueError("latent_attention: the rotation must fit into rot_dim")
        self.halves = position is not None and position.pairing == 0
        self.window = p.get("window") or None
        if p.get("sink") not in (None, False, "learned") or p.get("out_gate") not in (None, False, True, "head"):
            raise ValueError("latent_attention: sink is None or 'learned', out_gate None, True or 'head'")
        self.sink = p.get("sink") == "learned"
        self.gate_per_head = p.get("out_gate") == "head"
        self.gate_rows = 0 if not p.get("out_gate") else self.H if self.gate_per_head else self.H * self.Dv
        self.q_rank = int(p.get("q_rank") or 0)
        self.shares_kv = bool(p.get("shares_kv", False))
        self.term_dtype = torch.float32 if p.get("term_f32") else None

    def kv_spec(self) -> Optional[KVSpec]:
        return None if self.shares_kv else self.reads_kv_spec()

    def reads_kv_spec(self) -> KVSpec:
        return KVSpec(1, self.C + self.R, self.window, 0)

    def state_spec(self) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        return {}

    def _requests(self) -> Dict[str, TensorRequest]:
        E, t = self.p["hidden_size"], self.spec.tensors
        H, D, R, Dv, C = self.H, self.D, self.R, self.Dv, self.C
        shapes = {"dq": (self.q_rank, E), "dq_norm": (self.q_rank,), "uq": (H * (D + R), self.q_rank)} if self.q_rank \
            else {"q": (H * (D + R), E)}
        if not self.shares_kv:
            shapes.update(dkv=(C + R, E), dkv_norm=(C,))
        shapes.update(uk=(H * D, C), uv=(H * Dv, C), o=(E, H * Dv))
        if self.sink:
            shapes["sink"] = (H,)
        if self.gate_rows:
            shapes["g"] = (self.gate_rows, E)
        init = {"dq_norm": "ones", "dkv_norm": "ones", "sink": "uniform:-1:1"}
        return {n: TensorRequest(t[n], shape, init=init.get(n, "normal")) for n, shape in shapes.items()}

    def tensor_requests(self) -> List[TensorRequest]:
        return list(self._requests().values())

    def load(self, store: WeightStore) -> None:
        got = {n: store.get(r) for n, r in self._requests().items()}
        H, D, R, Dv, C = self.H, self.D, self.R, self.Dv, self.C
        self.sink_values = got["sink"].to(torch.float32).contiguous() if self.sink else None
        # the products of the mixer's input as one matrix: the queries (or their latent), the down-projection and the gate,
        # each part starting at a multiple of 8 rows
        parts, rows, self.off = [], 0, {}
        first = got["dq" if self.q_rank else "q"]
        for name in ("dq", "q", "dkv", "g"):
            if name not in got:
                continue
            m, at = got[name], (rows + 7) // 8 * 8
            if at > rows:
                parts.append(torch.zeros(at - rows, m.shape[1], dtype=first.dtype, device=m.device))
            self.off[name] = at
            parts.append(m.to(first.dtype))
            rows = at + m.shape[0]
        if rows % 8:                      # rows of the result that start on 16 bytes, whatever the parts' sizes
            parts.append(torch.zeros(8 - rows % 8, first.shape[1], dtype=first.dtype, device=first.device))
        self.proj = Linear(torch.cat(parts, dim=0).contiguous(), name="latent.proj")
        self.uq = Linear(got["uq"], name="latent.q") if self.q_rank else None
        self.q_norm, self.norm_weight = got.get("dq_norm"), got.get("dkv_norm")
        uk, uv = got["uk"], got["uv"]
        self.uk = uk.reshape(H, D, C).contiguous()                           # q' = q_plain W_uk[h]: [in D, out C]
        self.uv_t = uv.reshape(H, Dv, C).transpose(1, 2).contiguous()        # value = mix W_uv[h]^T: [in C, out Dv]
        self.kv_up = Linear(torch.cat([uk, uv.to(uk.dtype)], dim=0).contiguous(), name="latent.kv") if self._tiled() else None
        self.o = Linear(got["o"], name="latent.o")

    def _tiled(self) -> bool:
        """Whether prompts can take the tiled attention kernel over per-head keys and values."""
        return self.dtype == torch.bfloat16 and self.D + self.R == self.Dv and self.Dv in (64, 128)

    # ---- planning on the host
    def plan_key(self):
        return ("latent_attention", self.H, self.D, self.R, self.Dv, self.C, self._tiled(), self.window, self.sink)

    def plan(self, batch: HostBatch):
        """Prompts that start their sequences, where the tiled kernel fits: its list of query tiles, and a page table
        of the step's own (sequence b's tokens lie in pages of their own, numbered from 0 on across the step)."""
        if batch.decode or not self._tiled() or any(batch.starts):
            return {}
        width = max((n + 63) // 64 for n in batch.qlens)
        table, base = [], 0
        for n in batch.qlens:
            pages = (n + 63) // 64
            table += list(range(base, base + pages)) + [0] * (width - pages)
            base += pages
        return {"tiles": kernels.attention_prefill_tiles(batch.qlens), "pages": table, "n_pages": [base]}

    accepts_residual = True

    def _fast_decode(self) -> bool:
        """Whether single tokens take the kernel that serves all heads from one pass over the latent rows."""
        return kernels.latent_decode_supported(self.H, self.C, self.R, self.dtype)

    def graph_class(self, batch: HostBatch):
        """The decode kernel splits each token's keys by a rule of the longest sequence; the general kernel launches one
        block per token and head whatever the lengths."""
        seen = min(batch.max_kv, self.window + 31) if self.window else batch.max_kv
        return ("latent", kernels.latent_decode_class(seen)) if self._fast_decode() else ()

    def _queries(self, proj, ctx: StepContext) -> torch.Tensor:
        """The heads' queries [T, H*(D + R)], not rotated yet."""
        if not self.q_rank:
            return proj[:, :self.H * (self.D + self.R)]
        cq = ctx.ws.get("latent.cq", (proj.shape[0], self.q_rank), ctx.dtype)
        kernels.rms_rows(proj[:, :self.q_rank], self.q_norm, self.p["eps"], cq)
        return self.uq(cq, ctx)

    def forward(self, h, ctx: StepContext, run: RunView, residual=None) -> Optional[torch.Tensor]:
        H, D, R, Dv, C = self.H, self.D, self.R, self.Dv, self.C
        T = h.shape[0]
        proj = self.proj(h, ctx)
        dkv = None if self.shares_kv else proj[:, self.off["dkv"]:self.off["dkv"] + C + R]
        gate = proj[:, self.off["g"]:self.off["g"] + self.gate_rows] if self.gate_rows else None
        q = self._queries(proj, ctx)
        ctx.mark("projections")
        table, pos, plan = ctx.tables[run.group], self.position, ctx.plan_of(self)
        rotation = dict(rot_dims=0 if pos is None else pos.rotary_dim, inv_freq=None if pos is None else pos.inv_freq,
                        halves=self.halves, gain=1.0 if pos is None else pos.gain)

        def prepare(qa, row_out):
            kernels.latent_prep(q, dkv, H, D, R, C, weight=self.norm_weight, eps=self.p["eps"], qa=qa, seq_of=ctx.seq_of, pos=ctx.pos,
                                table=table, ring_pages=run.ring_pages, cache=run.k, row_out=row_out, **rotation)

        # this step's latent rows side by side, for the tiled kernel's products: made here, or left by the run whose rows
        # this layer reads; a run with readers leaves them in a buffer of its own
        tiled = not ctx.decode and "pages" in plan and kernels.attention_prefill_supported(q, run.k, D + R)
        key = f"latent.row{run.source}"
        row = None
        if self.shares_kv:
            row = ctx.shared.get(key)
            tiled = tiled and row is not None
        elif tiled or (run.has_readers and not ctx.decode):
            row = ctx.ws.get(key if run.has_readers else "latent.row", (T, C + R), ctx.dtype)
            if run.has_readers:
                ctx.shared[key] = row
        own_row = None if self.shares_kv else row
        if tiled:
            # per-head keys and values of this step's tokens as pages of the step's own
            prepare(None, own_row)
            kv = self.kv_up(row[:, :C], ctx)
            own = plan["pages"].view(ctx.B, -1)
            n_pages = sum((n + 63) // 64 for n in ctx.host["qlens"])
            k_pages = ctx.ws.get("latent.k_pages", (n_pages, H, 64, D + R), ctx.dtype)
            v_pages = ctx.ws.get("latent.v_pages", (n_pages, H, 64, Dv), ctx.dtype)
            kernels.pack_latent_heads(kv, row, H, D, R, Dv, C, ctx.seq_of, ctx.pos, own, k_pages, v_pages)
            values = ctx.ws.get("latent.values", (T, H * Dv), ctx.dtype)
            kernels.attention_prefill(q, values, H, H, D + R, plan["tiles"], ctx.cu, ctx.starts, ctx.qlens, own, 1 << 20,
                                      k_pages, v_pages, self.window or 0, float(self.p["scale"]), tc=False, exact=True, gate=gate,
                                      sink_values=self.sink_values)
            ctx.mark("attention")
            term = self.o(values, ctx, residual=residual, out_dtype=self.term_dtype)
            ctx.mark("o")
            return term
        qa = ctx.ws.get("latent.qa", (T, H * (C + R)), ctx.dtype)
        prepare(qa, own_row)
        kernels.head_matmul(q, D + R, self.uk, qa, C + R)
        mix = ctx.ws.get("latent.mix", (T, H * C), ctx.dtype)
        more = dict(gate=gate if self.gate_per_head else None, sink_values=self.sink_values)
        if ctx.decode and self._fast_decode():
            kernels.latent_decode(qa, mix, H, C, R, ctx, table, run.ring_pages, run.k, float(self.p["scale"]), window=self.window or 0,
                                  **more)
        else:
            kernels.attention_generic(qa, mix, H, 1, C + R, ctx.seq_of, ctx.pos, table, run.ring_pages, run.k, None,
                                      self.window or 0, float(self.p["scale"]), v_dim=C, **more)
        ctx.mark("attention")
        values = ctx.ws.get("latent.values", (T, H * Dv), ctx.dtype)
        kernels.head_matmul(mix, C, self.uv_t, values, Dv, gate=None if self.gate_per_head else gate)
        term = self.o(values, ctx, residual=residual, out_dtype=self.term_dtype)
        ctx.mark("o")
        return term
