"""Tukevik in the package against the plain implementation (tests/plain_tukevik.py), in 32-bit and in bfloat16: every
mechanism alone, whole prompts against token-by-token decoding, prompts cut into portions down to two tokens, unequal
batches against each request alone, slots and pages that are used again, keys far back, at page borders and just inside
and outside every chunk, the first tokens of a sequence, long decoding through rings of pages that go round, sizes that
fit no fast kernel, and greedy generation through the package's entry point.

A router's choice is discrete: where two logits are closer than bfloat16's rounding, bfloat16 takes another expert than
the float64 oracle.  So whole models run with their routers in 32-bit, and in bfloat16 as twins in which every expert is
chosen (the same weights; `all_chosen`); the routed kernels themselves are tested in bfloat16 with the choice given."""
import copy
import json
import math

import pytest
import torch

from tests import plain_tukevik as P
from tests.gpu_util import TOL
from tests.tukevik_util import CONFIGS, all_chosen, as_plain, build, config, llm, make_weights, new_engine, plain_logits, tokens_of, weights

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = ["float32", "bfloat16"]
NAMES = ["small", "wide"]


def assert_close(got, want, dtype, what="", tol=None):
    """32-bit: the largest error against the largest value of the compared block.  bfloat16, row by row: the root mean
    square of a row's error is held to 5% of the block's root mean square for a mechanism alone, to 10% for whole models,
    where one row in twenty may be off further: what retention reads out is normed, so a sum that happens to be close to
    zero (a first token's q.k) passes its rounding on enlarged.  The 32-bit runs are the sharper test of those."""
    got, want = got.detach().float().cpu(), want.detach().float().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} != {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    err, ref = float((got - want).abs().max()), max(float(want.abs().max()), 1e-6)
    if dtype == "float32":
        assert err <= (tol or TOL[dtype]) * ref, f"{what}: max error {err:.3e} against max |ref| {ref:.3e} ({dtype})"
        return
    g2, w2 = got.reshape(-1, got.shape[-1]), want.reshape(-1, want.shape[-1])
    rms_ref = max(float(w2.pow(2).mean().sqrt()), 1e-6)
    rows = (g2 - w2).pow(2).mean(-1).sqrt().sort().values / rms_ref
    limit, spared = (0.05, 0) if tol is None else (0.1, rows.numel() // 20)
    worst = float(rows[rows.numel() - 1 - spared])
    assert worst <= limit, f"{what}: a row is off by {worst:.3f} of {rms_ref:.3e} (max error {err:.3e}, {dtype})"


def assert_model(got, want, dtype, what=""):
    assert_close(got, want, dtype, what, tol=2e-4)


def entry(slot, tokens, want):
    from gguf_rs_cli_b200.engine.step import Entry
    return Entry(slot, tokens, want)


def tdtype(name):
    return {"float32": torch.float32, "bfloat16": torch.bfloat16}[name]


def dense(dtype):
    """bfloat16 runs the twin in which every expert is chosen."""
    return dtype == "bfloat16"


def plan_for(eng, lens, slots=None):
    slots = slots or [eng.open() for _ in lens]
    ctx, _, _ = eng.plan([entry(s, [1] * n, ()) for s, n in zip(slots, lens)])
    return ctx, slots


def run_steps(lens, steps, make):
    """Runs make(ctx, rows) for steps that bring a number of tokens of each sequence (0: none); rows are, in the step's
    packing, (sequence, first position, number).  Returns what it gave, sequence by sequence."""
    eng = new_engine("small", "float32", n_tokens=4096, n_slots=6)
    for _ in range(2):
        eng.open()                                     # the sequences' slots are not their numbers
    slots, at = [eng.open() for _ in lens], [0] * len(lens)
    got = [[] for _ in lens]
    for step in steps:
        live = [(i, n) for i, n in enumerate(step) if n]
        ctx, _, _ = eng.plan([entry(slots[i], [1] * n, ()) for i, n in live])
        out = make(ctx, [(i, at[i], n) for i, n in live]).float().cpu()
        eng.cache.advance([slots[i] for i, _ in live], [n for _, n in live])
        r = 0
        for i, n in live:
            got[i].append(out[r:r + n])
            r += n
            at[i] += n
    assert at == lens
    return [torch.cat(g) for g in got]


# ------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,routed", [(5, True), (72, False), (72, True), (1000, True), (2048, False), (4096, True), (9000, True), (12304, False),
                                      (20000, True)])
def test_norm_behind_a_factor_and_a_mixtures_gated_sum(E, routed, dtype):
    from gguf_rs_cli_b200 import kernels
    g = torch.Generator().manual_seed(E)
    T, eps, td, top, m = 7, 1e-3, tdtype(dtype), 3, 0.7
    x, y, w = torch.randn(T, E, generator=g), (torch.randn(T, E, generator=g) * 2).to(td), (1 + 0.3 * torch.randn(E, generator=g)).to(td)
    gate, z, wz = torch.rand(T, generator=g), torch.randn(T * top, E, generator=g), torch.rand(T, top, generator=g)
    place = torch.randperm(T * top, generator=g)
    mixed = (wz.double()[:, :, None] * z.double()[place].view(T, top, E)).sum(1)
    v = x.double() + m * ((gate.double()[:, None] if routed else 1.0) * y.double() + (mixed if routed else 0.0))
    want = P.rms_norm(v, w.double(), eps)
    xd, h = x.to(DEV), torch.empty(T, E, dtype=td, device=DEV)
    kw = dict(y_gate=gate.to(DEV), routed=(z.to(DEV), wz.to(DEV), place.to(torch.int32).to(DEV))) if routed else {}
    kernels.add_rmsnorm_terms(xd, y.to(DEV), w.to(DEV), eps, h, scale=m, **kw)
    assert_close(xd, v.float(), "float32", "the new x")
    assert_close(h, want.float(), dtype, "normed")
    # chosen rows only, x left as it is; rows in the pairs' own order, nothing beside them
    xd, rows = x.to(DEV), torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
    h = torch.empty(3, E, dtype=td, device=DEV)
    kernels.add_rmsnorm_terms(xd, None, w.to(DEV), eps, h, scale=m, routed=(z[place].contiguous().to(DEV), wz.to(DEV), None), rows=rows, write_x=False)
    assert_close(h, P.rms_norm(x.double() + m * mixed, w.double(), eps)[[4, 0, 4]].float(), dtype, "chosen rows")
    assert torch.equal(xd.cpu(), x)


@pytest.mark.parametrize("T", [1, 9, 64, 100])
def test_factor_in_the_residual_epilogue_of_a_product(T):
    from gguf_rs_cli_b200 import kernels
    g = torch.Generator().manual_seed(T)
    N, K = 264, 200
    x, w, r = torch.randn(T, K, generator=g).to(torch.bfloat16), (torch.randn(N, K, generator=g) / 14).to(torch.bfloat16), torch.randn(T, N, generator=g)
    rd, xb, ssq = r.to(DEV), torch.empty(T, N, dtype=torch.bfloat16, device=DEV), torch.empty(3, T, device=DEV)
    kernels.gemm_tc(x.to(DEV), w.to(DEV), None, None, resid_x=rd, resid_xb=xb, ssq_out=ssq, resid_scale=0.6)
    want = r.double() + 0.6 * (x.double() @ w.double().T)
    assert_close(rd, want.float(), "float32", "the new x")
    assert torch.equal(xb, rd.to(torch.bfloat16))
    assert_close(ssq.sum(0), want.pow(2).sum(-1).float(), "float32", "sums of squares")


@pytest.mark.parametrize("dtype,H,G,D,Dv,chunk,cap", [
    ("float32", 6, 2, 24, 24, 13, 5.0), ("float32", 3, 3, 5, 9, None, 2.0), ("float32", 4, 1, 96, 96, 64, None), ("bfloat16", 4, 2, 64, 64, 70, 5.0),
    ("bfloat16", 4, 1, 96, 96, 64, 30.0), ("bfloat16", 3, 3, 96, 96, None, None), ("bfloat16", 4, 1, 128, 128, None, 3.0),
    ("bfloat16", 8, 8, 64, 64, 96, None), ("bfloat16", 5, 5, 48, 48, 40, 4.0), ("bfloat16", 3, 1, 20, 12, 9, 4.0), ("bfloat16", 2, 1, 96, 96, 1, 8.0)])
def test_softcap_sink_chunks_and_factor_on_every_attention_kernel(dtype, H, G, D, Dv, chunk, cap):
    from gguf_rs_cli_b200 import kernels
    T, td, scale, eps, factor = 200, tdtype(dtype), 6.0 / D, 1e-3, 0.7
    g = torch.Generator().manual_seed(D + H)
    buf, gate = torch.randn(T, H * D + G * (D + Dv), generator=g).to(td), torch.randn(T, H, generator=g).to(td)
    q, k, v = buf[:, :H * D].double().view(T, H, D), buf[:, H * D:(H + G) * D].double().view(T, G, D), buf[:, (H + G) * D:].double().view(T, G, Dv)
    o = P.sink_attention(P.unit_rms(q, eps), P.unit_rms(k, eps), v, scale, cap, P.visible(T, chunk))
    want = (factor * o * torch.sigmoid(gate.double())[:, :, None]).reshape(T, H * Dv).float()
    pages = (T + 63) // 64
    table = torch.randperm(pages, generator=torch.Generator().manual_seed(1)).to(torch.int32).to(DEV)[None, :].contiguous()
    kc, vc = torch.zeros(pages, G, 64, D, dtype=td, device=DEV), torch.zeros(pages, G, 64, Dv, dtype=td, device=DEV)
    bd, pos, seq = buf.to(DEV), torch.arange(T, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV)
    q, k, v, ones = bd[:, :H * D], bd[:, H * D:(H + G) * D], bd[:, (H + G) * D:], torch.ones(D, device=DEV)
    kernels.head_prep_kv_write(q, k, v, H, G, D, Dv, ones, ones, eps, None, 0, 0, None, 0.0, None, seq, pos, table, pages, 0, kc, vc)
    kw = dict(gate=gate.to(DEV), sink=True, chunk=chunk or 0, softcap=cap or 0.0, out_scale=factor)
    out = torch.empty(T, H * Dv, dtype=td, device=DEV)
    kernels.attention_generic(q, out, H, G, D, seq, pos, table, pages, kc, vc, 0, scale, v_dim=Dv, **kw)
    assert_close(out, want, dtype, "general kernel")
    if dtype == "float32" or D != Dv:
        return
    if kernels.attention_prefill_supported(q, kc, D) and q.stride(0) % 8 == 0:
        assert D in (64, 96, 128)
        meta = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)                            # noqa: E731
        got = torch.empty_like(out)
        kernels.attention_prefill(q, got, H, G, D, meta(*kernels.attention_prefill_tiles([T])), meta(0, T), meta(0), meta(T), table, pages, kc, vc,
                                  0, scale, tc=False, exact=True, **kw)
        assert_close(got, want, dtype, "tiled kernel")
        assert_close(got, out.cpu(), dtype, "tiled against general kernel")
    if kernels.attention_decode_supported(q, kc, D):
        for splits in (1, 3):
            got = torch.empty_like(out)
            kernels.attention_decode(q, got, H, G, D, seq, pos, table, pages, kc, vc, 0, scale, mma=False, max_kv=T, splits=splits, **kw)
            assert_close(got, want, dtype, f"single tokens, {splits} splits")


def test_plain_attention_weights_for_heads_of_96():
    """The tiled kernel without 32-bit weights at the head size it gained (a model of rotated heads of 96 takes it)."""
    from gguf_rs_cli_b200 import kernels
    H, G, D, T = 2, 1, 96, 150
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(T, n * D, generator=g).to(torch.bfloat16) for n in (H, G, G))
    want = torch.zeros(T, H, D, dtype=P.F64)
    for h in range(H):
        s = (q.double()[:, h * D:(h + 1) * D] @ k.double().T / 10).masked_fill(~P.visible(T, None), -math.inf)
        want[:, h] = torch.softmax(s, -1) @ v.double()
    pad = torch.zeros(192 - T, D, dtype=torch.bfloat16)
    kc, vc = (torch.cat([t, pad]).view(3, 1, 64, D).contiguous().to(DEV) for t in (k, v))
    meta = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)                                # noqa: E731
    out = torch.empty(T, H * D, dtype=torch.bfloat16, device=DEV)
    kernels.attention_prefill(q.to(DEV), out, H, G, D, meta(*kernels.attention_prefill_tiles([T])), meta(0, T), meta(0), meta(T), meta(0, 1, 2)[None],
                              3, kc, vc, 0, 0.1, tc=False)
    assert_close(out, want.reshape(T, H * D).float(), "bfloat16")


@pytest.mark.parametrize("n,top,sg", [(5, 3, True), (12, 2, False), (1, 1, True), (40, 8, True), (3, 3, False)])
def test_router_with_a_bias_and_the_shared_experts_gate(n, top, sg):
    from gguf_rs_cli_b200 import kernels
    g = torch.Generator().manual_seed(n)
    T, K = 9, 24
    h, w, b = torch.randn(T, K, generator=g), torch.randn(n + sg, K, generator=g), torch.randn(n, generator=g)
    z = h.double() @ w[:n].double().T + b.double()
    ids_want = torch.topk(z, top, dim=-1).indices
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    gate = torch.empty(T, device=DEV) if sg else None
    kernels.moe_router(h.to(DEV), w.to(DEV), 1, 1, top, 1.0, ids, wts, softmax=True, bias=b.to(DEV), gate=gate)
    assert ids.cpu().tolist() == ids_want.tolist()
    assert_close(wts, torch.softmax(torch.gather(z, 1, ids_want), -1).float(), "float32", "weights")
    if sg:
        assert_close(gate, torch.sigmoid(h.double() @ w[n].double()).float(), "float32", "gate")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [1, 2])
@pytest.mark.parametrize("T,by_expert", [(3, False), (50, False), (50, True)])
def test_experts_for_a_given_choice_summed_here_and_there(T, by_expert, layer, dtype):
    """Token by token, in sorted tiles and expert by expert; with a gated shared expert and without; summed by the part, and
    left to the norm behind it: the same x either way."""
    from gguf_rs_cli_b200.parts.base import RoutedRows, Stream
    if by_expert and dtype == "float32":
        pytest.skip("expert by expert is a bfloat16 path")
    name = "wide"
    cfg, w = config(name), weights(name)
    mlp, p = cfg["layers"][layer]["mlp"], f"l{layer}.mlp."
    model = llm(name, dtype).model
    ff, norm = model.layers[layer].feed_forward, model.layers[layer].norms["feed_forward"]
    g = torch.Generator().manual_seed(T)
    h = torch.randn(T, cfg["width"], generator=g).to(torch.bfloat16).float()
    ctx, _ = plan_for(new_engine(name, dtype), [T])
    hd = h.to(tdtype(dtype)).to(DEV)
    try:
        if by_expert:
            ff.BY_EXPERT, ff.BY_EXPERT_ENTRIES = 0, 0
        got = ff.forward(hd, ctx).clone()
        ids = ctx.ws.get("moe.ids", (T, ff.top), torch.int32).cpu().long()
        want = P.moe(mlp, as_plain(w), p, h.double(), ids=ids)
        assert_close(got, want.float(), dtype, f"{T} tokens")
        rows = ff.forward(hd, ctx, unsummed=True)
        assert isinstance(rows, RoutedRows) and (rows.base is None) == (layer == 2) == (rows.base_gate is None)
        x = torch.randn(T, cfg["width"], generator=g)
        a, b = Stream(x.to(DEV)), Stream(x.to(DEV))
        a.pending, a.pending_scale, b.pending, b.pending_scale = rows, 0.5, got, 0.5
        ha = norm.apply(a, ctx, buffer="test.a").clone()
        hb = norm.apply(b, ctx, buffer="test.b")
        assert_close(a.x, b.x.cpu(), "float32", "summed behind the norm's back and by the part")
        assert_close(ha, hb.cpu(), dtype, "normed")
        assert a.pending is None and a.pending_scale == 1.0
    finally:
        ff.__dict__.pop("BY_EXPERT", None)
        ff.__dict__.pop("BY_EXPERT_ENTRIES", None)


STEPS = ([300, 41], [[300, 41]]), ([300, 41], [[130, 2], [2, 0], [64, 38], [100, 0], [1, 1], [3, 0]]), ([70, 5], [[1, 1]] * 5 + [[65, 0]]), \
    ([200, 129], [[128, 129], [72, 0]])


@pytest.mark.parametrize("lens,steps", STEPS)
@pytest.mark.parametrize("dtype,H,D,Dv,rot", [("float32", 3, 12, 18, (100.0, 8)), ("float32", 1, 5, 3, None), ("float32", 2, 64, 64, (1e4, 64)),
                                              ("bfloat16", 3, 64, 64, (1e4, 64)), ("bfloat16", 2, 128, 128, (500.0, 96)), ("bfloat16", 4, 32, 32, (1e3, 20)),
                                              ("bfloat16", 1, 96, 96, None), ("bfloat16", 2, 96, 96, (1e4, 6)), ("bfloat16", 2, 24, 40, (10.0, 2))])
def test_retention_in_portions_batches_and_single_tokens(dtype, H, D, Dv, rot, lens, steps):
    """The walk, the chunked form and the pass of single tokens, each as the part takes them; two sequences side by side."""
    from gguf_rs_cli_b200.config import PartSpec
    from gguf_rs_cli_b200.parts import MIXERS, POSITIONS
    td, eps, factor = tdtype(dtype), 1e-4, 0.7
    decay = [0.5, 0.998046875, 1.0, 0.96875][:H]
    g = torch.Generator().manual_seed(D + H)
    round8 = lambda n: (n + 7) // 8 * 8                                                             # noqa: E731
    sizes = [("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)]
    total = sum(round8(n) for _, n in sizes)
    proj = [torch.randn(n, total, generator=g).to(td) for n in lens]
    off, o = {}, 0
    for name, n in sizes:
        off[name], o = (o, o + n), o + round8(n)
    want = []
    for p in proj:
        x = {name: p[:, a:b].double() for name, (a, b) in off.items()}
        T, pos = p.shape[0], torch.arange(p.shape[0])
        q, k, v = x["q"].view(T, H, D), x["k"].view(T, H, D), x["v"].view(T, H, Dv)
        if rot:
            q, k = P.rotate(q, pos, {"base": rot[0], "dims": rot[1]}), P.rotate(k, pos, {"base": rot[0], "dims": rot[1]})
        r = P.unit_rms(P.retention(q, k * D ** -0.5, v, decay), eps)
        want.append((factor * r.reshape(T, H * Dv) * P.silu(x["g"])).float())
    position = None if rot is None else POSITIONS.get("rope")(PartSpec("rope", dict(head_dim=D, rotary_dim=rot[1], theta=rot[0], pairing="half")), td, DEV)
    part = MIXERS.get("retention")(PartSpec("retention", dict(hidden_size=8, heads=H, dim=D, vdim=Dv, decay=decay, eps=eps),
                                            {n: n for n in ("q", "k", "v", "g", "o")}), td, DEV, position=position)

    class Store:
        @staticmethod
        def get(r):
            return torch.zeros(r.shape, dtype=td, device=DEV)
    part.load(Store)
    assert part.off == {name: a for name, (a, _) in off.items()}
    state = torch.zeros(6, H, D, Dv, device=DEV)

    def make(ctx, rows):
        class Run:
            index = 0
        ctx.state = lambda name: state
        packed = torch.cat([proj[i][a:a + n] for i, a, n in rows]).to(DEV)
        return part.mix_rows(packed, ctx, Run, torch.empty(packed.shape[0], H * Dv, dtype=td, device=DEV), out_scale=factor)

    for a, b in zip(run_steps(lens, steps, make), want):
        assert_close(a, b, dtype)


@pytest.mark.parametrize("lens,steps", STEPS)
@pytest.mark.parametrize("dtype,W,blocks", [("float32", 60, 3), ("float32", 7, 7), ("float32", 130, 1), ("bfloat16", 128, 1), ("bfloat16", 240, 3),
                                            ("bfloat16", 512, 4), ("bfloat16", 64, 8), ("bfloat16", 24, 2), ("bfloat16", 272, 1)])
def test_gated_linear_recurrence_in_portions_batches_and_single_tokens(dtype, W, blocks, lens, steps):
    """Gates, walk, segments and single tokens, each by the kernels that the part takes for them."""
    from gguf_rs_cli_b200 import kernels
    td, n = tdtype(dtype), W // blocks
    g = torch.Generator().manual_seed(W)
    w = {"ra": torch.randn(blocks, n, n, generator=g) * 1.5 / n ** 0.5, "ri": torch.randn(blocks, n, n, generator=g) * 1.5 / n ** 0.5}
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    w.update({"ra.b": torch.randn(blocks, n, generator=g), "ri.b": torch.randn(blocks, n, generator=g), "lam": -9.0 + 9.0 * torch.rand(W, generator=g)})
    u, y = ([torch.randn(m, W, generator=g).to(td) for m in lens] for _ in range(2))
    want = []
    for uu, yy in zip(u, y):
        a, b = P.recurrence_coefficients({k: v.double() for k, v in w.items()}, "", uu.double())
        S, rows = torch.zeros(W, dtype=P.F64), []
        for t in range(uu.shape[0]):
            S = a[t] * S + b[t]
            rows.append(S)
        want.append((torch.stack(rows) * P.gelu_tanh(yy.double())).float())
    gates = torch.cat([w["ra"], w["ri"]], dim=1).to(td).to(DEV)
    gates_in = gates.transpose(1, 2).contiguous()
    rates = (w["ra.b"].reshape(-1).to(DEV), w["ri.b"].reshape(-1).to(DEV), (8.0 * P.softplus(w["lam"].double())).float().to(DEV))
    state, used = torch.zeros(6, W, device=DEV), set()

    def make(ctx, rows):
        uu, yy = (torch.cat([x[i][a:a + m] for i, a, m in rows]).to(DEV) for x in (u, y))
        out = torch.empty_like(uu)
        if ctx.decode:
            used.add("single")
            return kernels.rglru_step(uu, yy, gates_in, *rates, state, out, ctx, blocks)
        if kernels.rglru_fused_supported(uu, n):
            used.add("fused")
            return kernels.rglru_fused(uu, yy, gates, *rates, state, out, ctx, blocks)
        used.add("general")
        z = kernels.head_matmul(uu, n, gates_in, torch.empty(uu.shape[0], 2 * W, device=DEV), 2 * n)
        return kernels.rglru(uu, yy, z, *rates, state, out, ctx, blocks)

    for a, b in zip(run_steps(lens, steps, make), want):
        assert_close(a, b, dtype)
    assert (("fused" in used) if dtype == "bfloat16" and n % 8 == 0 else ("general" in used))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,K", [(40, 4), (24, 2), (9, 16), (16, 1), (64, 3)])
def test_convolution_with_a_bias_and_no_activation(C, K, dtype):
    from gguf_rs_cli_b200 import kernels
    td, g = tdtype(dtype), torch.Generator().manual_seed(C)
    lens, steps = [30, 20], [[5, 1], [1, 1], [1, 0], [2, 17], [1, 1], [20, 0]]
    x = [torch.randn(n, C, generator=g).to(td) for n in lens]
    taps, bias = torch.randn(C, K, generator=g).to(td), torch.randn(C, generator=g).to(td)
    want = [P.causal_conv(v.double(), taps.double(), bias.double()).float() for v in x]
    state = torch.zeros(6, K - 1, C, device=DEV) if K > 1 else None

    def make(ctx, rows):
        xx = torch.cat([x[i][a:a + n] for i, a, n in rows]).to(DEV)
        return kernels.short_conv(xx, taps.to(DEV), state, ctx, torch.empty_like(xx), bias=bias.to(DEV),
                                  taps_t=taps.t().contiguous().to(DEV) if dtype == "bfloat16" else None)

    for a, b in zip(run_steps(lens, steps, make), want):
        assert_close(a, b, dtype)


def test_a_decay_next_to_one_keeps_its_digits():
    """Thousands of tokens with a decay whose rounding to 32 bits would show: single tokens and segments alike."""
    from gguf_rs_cli_b200 import kernels
    W, T = 32, 3000
    lam = torch.linspace(-16.0, -8.0, W)
    one = torch.zeros(1, W, W, dtype=torch.float64)
    u = torch.randn(T, W, generator=torch.Generator().manual_seed(5)) + 0.5
    W64 = {"ra": one, "ri": one, "ra.b": torch.full((1, W), 3.0, dtype=P.F64), "ri.b": torch.zeros(1, W, dtype=P.F64), "lam": lam.double()}
    a, b = P.recurrence_coefficients(W64, "", u.double())
    S, rows = torch.zeros(W, dtype=P.F64), []
    for t in range(T):
        S = a[t] * S + b[t]
        rows.append(S)
    want = torch.stack(rows)
    rates = (torch.full((W,), 3.0, device=DEV), torch.zeros(W, device=DEV), (8.0 * P.softplus(lam.double())).float().to(DEV))
    gates_in = torch.zeros(1, W, 2 * W, device=DEV)
    big = torch.full((T, W), 20.0, device=DEV)                # gelu_tanh(20) = 20
    state = torch.zeros(6, W, device=DEV)

    def make(ctx, rows):
        (i, at, n), = rows
        uu, out = u[at:at + n].to(DEV), torch.empty(n, W, device=DEV)
        if ctx.decode:
            return kernels.rglru_step(uu, big[:n], gates_in, *rates, state, out, ctx, 1)
        return kernels.rglru(uu, big[:n], torch.zeros(n, 2 * W, device=DEV), *rates, state, out, ctx, 1)

    got = run_steps([T], [[2000]] + [[60]] * 5 + [[1]] * 700, make)[0].double() / 20.0
    err = ((got - want).abs().max(0).values / want.abs().max(0).values).max()
    assert float(err) < 3e-6, float(err)


# ------------------------------------------------------------ whole models
def with_pending(stream):
    """x with the term that the next norm will add."""
    from gguf_rs_cli_b200.parts.base import RoutedRows
    t = stream.pending
    if t is None:
        return stream.x.clone()
    if isinstance(t, RoutedRows):
        T, top = t.weights.shape
        rows = t.rows if t.place_of is None else t.rows[t.place_of.long()]
        base = 0.0 if t.base is None else t.base if t.base_gate is None else t.base_gate[:, None] * t.base
        t = base + (t.weights[:, :, None] * rows.view(T, top, -1)).sum(1)
    return stream.x + stream.pending_scale * t.float()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_request_alone(name, dtype):
    for n, seed in ((1, 1), (2, 2), (150, 3), (400, 4)):
        eng = new_engine(name, dtype, dense(dtype))
        s = eng.open()
        got = eng.step([entry(s, tokens_of(name, n, seed), range(n))])
        assert_model(got, plain_logits(name, n, seed, dense(dtype)), dtype, f"{name}: prompt of {n}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_stream_after_every_layer(name, dtype):
    cfg = all_chosen(CONFIGS[name]) if dense(dtype) else CONFIGS[name]
    toks, want = tokens_of(name, 90, 7), []
    P.forward(cfg, as_plain(weights(name)), toks, layers_out=want)
    model = llm(name, dtype, dense(dtype)).model
    eng = new_engine(name, dtype, dense(dtype))
    got, undo = [], []
    for layer in model.layers:
        orig = layer.block.forward
        undo.append((layer.block, orig))

        def fwd(stream, ctx, run, orig=orig):
            orig(stream, ctx, run)
            got.append(with_pending(stream))
        layer.block.forward = fwd
    try:
        eng.step([entry(eng.open(), toks, [0])])
    finally:
        for block, orig in undo:
            block.forward = orig
    assert len(got) == len(want)
    for i, (a, b) in enumerate(zip(got, want)):
        assert_model(a, b.float(), dtype, f"{name}: stream after layer {i}")


def test_a_step_that_asks_for_no_logits_and_chosen_rows():
    eng = new_engine("small", "float32")
    toks, want = tokens_of("small", 40, 5), plain_logits("small", 40, 5)
    s = eng.open()
    assert eng.step([entry(s, toks[:20], [])]) is None
    got = eng.step([entry(s, toks[20:], [19, 0, 7])])
    assert_model(got, want[[39, 20, 27]], "float32", "rows in the order asked for")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_from_the_first(name, dtype):
    n = 45
    toks, want = tokens_of(name, n, 11), plain_logits(name, n, 11, dense(dtype))
    eng = new_engine(name, dtype, dense(dtype))
    s = eng.open()
    got = torch.cat([eng.step([entry(s, [t], [0])]).clone() for t in toks])
    assert_model(got, want, dtype, f"{name}: decoded from the first token")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_in_portions(name, dtype):
    n = 333
    toks, want = tokens_of(name, n, 12), plain_logits(name, n, 12, dense(dtype))
    for cuts in ([2, 2, 60, 5, 64, 128, 70, 2], [1, 63, 64, 65, 3, 137], [300, 33]):
        eng = new_engine(name, dtype, dense(dtype))
        s, at, got = eng.open(), 0, []
        for c in cuts:
            got.append(eng.step([entry(s, toks[at:at + c], range(c))]).clone())
            at += c
        assert at == n
        assert_model(torch.cat(got), want, dtype, f"{name}: portions {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_slots_and_pages_used_again(name, dtype):
    """Three requests of unequal lengths start together and are decoded together, the shortest ends early; then new requests
    fill the slots and pages that were given back, and a step mixes first tokens with later ones."""
    eng = new_engine(name, dtype, dense(dtype), n_tokens=1024, n_slots=3)
    lens, extra = [70, 3, 131], 9
    seqs = [tokens_of(name, n + extra, 20 + i) for i, n in enumerate(lens)]
    wants = [plain_logits(name, n + extra, 20 + i, dense(dtype)) for i, n in enumerate(lens)]
    slots = [eng.open() for _ in lens]
    gots = [eng.step([entry(s, q[:n], [n - 1]) for s, q, n in zip(slots, seqs, lens)]).clone()]
    rows = [torch.stack([w[n - 1] for w, n in zip(wants, lens)])]
    for j in range(extra):
        live = [i for i in range(3) if not (i == 1 and j >= 4)]            # the short request ends early
        gots.append(eng.step([entry(slots[i], [seqs[i][lens[i] + j]], [0]) for i in live]).clone())
        rows.append(torch.stack([wants[i][lens[i] + j] for i in live]))
        if j == 3:
            eng.close(slots[1])
    assert_model(torch.cat(gots), torch.cat(rows), dtype, f"{name}: prompts together, then decoded together")
    eng.close(slots[0])
    eng.close(slots[2])
    eng.check()
    for rounds in range(2):
        lens2 = [200, 64, 65]
        seqs2 = [tokens_of(name, n, 40 + i) for i, n in enumerate(lens2)]
        wants2 = [plain_logits(name, n, 40 + i, dense(dtype)) for i, n in enumerate(lens2)]
        slots2 = [eng.open() for _ in lens2]
        got = eng.step([entry(slots2[0], seqs2[0][:150], [0, 149])]).clone()
        assert_model(got, wants2[0][[0, 149]], dtype, f"{name}: slots and pages used again")
        got = eng.step([entry(slots2[0], seqs2[0][150:], [0, 49]), entry(slots2[1], seqs2[1], [0, 63]), entry(slots2[2], seqs2[2], [0, 64])])
        want = torch.cat([wants2[0][[150, 199]], wants2[1][[0, 63]], wants2[2][[0, 64]]])
        assert_model(got, want, dtype, f"{name}: a later portion beside two prompts")
        for s in slots2:
            eng.close(s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_long_decoding_through_rings_that_go_round(name, dtype):
    """Steps of at most 16 tokens keep the rings of the windowed layers short: 260 decoded tokens take every ring round."""
    n0, n = 50, 310
    toks, want = tokens_of(name, n, 31), plain_logits(name, n, 31, dense(dtype))
    eng = new_engine(name, dtype, dense(dtype), max_step_tokens=16)
    s = eng.open()
    for at in range(0, n0 - 2, 16):
        eng.step([entry(s, toks[at:at + 16], [])])
    got = [eng.step([entry(s, toks[48:50], [0, 1])]).clone()]
    got += [eng.step([entry(s, [toks[i]], [0])]).clone() for i in range(n0, n)]
    assert_model(torch.cat(got), want[48:], dtype, f"{name}: long decoding")


ODD = {
    "architecture": "Tukevik", "vocab": 91, "width": 50, "norm": {"eps": 1e-4}, "residual_mult": 1.0,
    "layers": [
        {"type": "parallel", "mlp": {"kind": "moe", "router": {"experts": 1, "top": 1}, "expert": {"ff": 7}},
         "mixer": {"left": {"heads": 5, "kv_heads": 5, "dim": 6, "vdim": 6, "scale": 1.0, "softcap": 1.0, "mask": {"size": 1}},
                   "right": {"heads": 1, "dim": 2, "vdim": 1, "decay": [1.0], "rot": {"base": 10.0, "dims": 2}}, "left_scale": 1.0, "right_scale": 1.0}},
        {"type": "rglru", "mixer": {"width": 9, "blocks": 9, "conv": 1},
         "mlp": {"kind": "moe", "router": {"experts": 2, "top": 2}, "expert": {"ff": 3}, "shared": {"ff": 5}}},
        {"type": "rglru", "mixer": {"width": 51, "blocks": 1, "conv": 16}, "mlp": {"kind": "dense", "ff": 1}},
        {"type": "parallel", "mlp": None,
         "mixer": {"left": {"heads": 7, "kv_heads": 1, "dim": 10, "vdim": 3, "scale": 0.3, "softcap": 50.0, "mask": {"size": 2}},
                   "right": {"heads": 3, "dim": 5, "vdim": 7, "decay": [0.999, 0.25, 0.0]}, "left_scale": 2.0, "right_scale": 0.5}},
        {"type": "parallel", "mlp": {"kind": "dense", "ff": 9},
         "mixer": {"left": {"heads": 1, "kv_heads": 1, "dim": 256, "vdim": 256, "scale": 0.02, "softcap": 8.0, "mask": {"size": 64}},
                   "right": {"heads": 1, "dim": 130, "vdim": 130, "decay": [0.97], "rot": {"base": 100.0, "dims": 130}},
                   "left_scale": 0.7, "right_scale": 0.7}},
        {"type": "rglru", "mixer": {"width": 1, "blocks": 1, "conv": 3}, "mlp": None},
    ],
}


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_that_fit_no_fast_kernel_and_values_of_one(dtype):
    """A width that is no multiple of 8, one head and one expert, chunks of one position and of two, a factor of 1, a decay
    of 0 and of 1, a convolution of one tap and of 16, blocks of one channel, one channel."""
    cfg = copy.deepcopy(ODD)
    w = make_weights(cfg, seed=9)
    if dtype == "bfloat16":                      # rows of one entry, normed, are a sign, which a rounding can turn
        cfg["layers"][0]["mixer"]["right"]["vdim"] = 6
        w = make_weights(cfg, seed=9)
    model = build(cfg, w, dtype).model
    from gguf_rs_cli_b200.engine.step import Engine
    toks = torch.randint(0, cfg["vocab"], (150,), generator=torch.Generator().manual_seed(2)).tolist()
    want = P.forward(cfg, as_plain(w), toks).float()
    for cuts in ([150], [70, 2, 1, 77], [1] * 40):
        eng = Engine(model, n_tokens=1024, n_slots=2)
        s, at, got = eng.open(), 0, []
        for c in cuts:
            got.append(eng.step([entry(s, toks[at:at + c], range(c))]).clone())
            at += c
        assert_model(torch.cat(got), want[:at], dtype, f"odd sizes, portions {cuts[:4]}")


# ------------------------------------------------------------ keys that stand out
def spike_model(chunk, D, heads, cap):
    """Attention that is decided by one key: token t + 1024 is the partner of token t; its query is the key of t (behind an
    orthogonal map S of the rows; the partner's row is S^T times the row of t), so a partner's score with its token's key
    is large and all others are a few units.  The partner's result is then the value of t if it may see t, and else
    something else altogether.  The retention beside it reads with a small factor."""
    g = torch.Generator().manual_seed(7)
    E, V = 64, 2048
    S, _ = torch.linalg.qr(torch.randn(E, E, generator=g))
    base = torch.randn(1024, E, generator=g)
    base = base / base.pow(2).mean(-1, keepdim=True).sqrt()
    k = torch.randn(D, E, generator=g) / E ** 0.5
    w = {"embed": torch.cat([base, base @ S]), "l0.norm1": torch.ones(E), "final.norm": torch.ones(E)}
    p = "l0.mix.left."
    w[p + "q"], w[p + "k"], w[p + "v"] = torch.cat([k @ S] * heads), k, torch.randn(D, E, generator=g) / E ** 0.5 * 2
    w[p + "q.b"], w[p + "k.b"], w[p + "v.b"] = torch.zeros(heads * D), torch.zeros(D), torch.zeros(D)
    w[p + "g"], w[p + "o"] = torch.zeros(heads, E), torch.randn(E, heads * D, generator=g) / (heads * D) ** 0.5 * 6
    p = "l0.mix.right."
    for n in ("q", "k", "v", "g"):
        w[p + n] = torch.randn(32, E, generator=g) / E ** 0.5
    w[p + "o"] = torch.randn(E, 32, generator=g) / 6
    left = {"heads": heads, "kv_heads": 1, "dim": D, "vdim": D, "scale": 60.0 / D, **({"softcap": cap} if cap else {}),
            **({"mask": {"size": chunk}} if chunk else {})}
    right = {"heads": 1, "dim": 32, "vdim": 32, "decay": [0.96875], "rot": {"base": 100.0, "dims": 32}}
    cfg = {"architecture": "Tukevik", "vocab": V, "width": E, "norm": {"eps": 1e-6}, "residual_mult": 0.9,
           "layers": [{"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 1.0, "right_scale": 0.1}, "mlp": None}]}
    return cfg, {n: t.to(torch.bfloat16).float() for n, t in w.items()}


@pytest.mark.parametrize("chunk,D,heads,cap", [(70, 24, 2, 40.0), (70, 64, 2, None), (90, 128, 4, 30.0), (64, 96, 2, 30.0), (None, 64, 2, 50.0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_that_stand_out_at_every_edge_in_prompt_and_decode(dtype, chunk, D, heads, cap):
    """All tokens differ; for chosen pairs (i, j) position i holds the partner of the token at position j, whose key then
    takes all of i's attention if and only if i may see j.  Pairs: j the first position of i's chunk and the last of the
    chunk before, i the first and the last of a chunk, across page borders, at the sequence's first positions, and hundreds
    of positions back."""
    cfg, w = spike_model(chunk, D, heads, cap)
    n, c = 700, chunk or 70
    toks = torch.randperm(1024, generator=torch.Generator().manual_seed(1))[:n].tolist()
    pairs = [(2 * c + 5, 2 * c), (2 * c + 6, 2 * c - 1), (3 * c, 3 * c - 1), (4 * c - 1, 3 * c + 1), (c - 1, 0), (c + 1, 2), (c + 2, c), (5 * c + 3, 4 * c - 3),
             (192, 191), (193, 130), (650, 3), (660, 660 // c * c), (671, 671 // c * c - 1), (699, 699 // c * c + 1), (5, 1), (4, 0)]
    pairs = [(i, j) for k, (i, j) in enumerate(pairs) if i not in {x for x, _ in pairs[:k]}]
    sources = {j for _, j in pairs}
    pairs = [(i, j) for i, j in pairs if i not in sources]
    assert len(pairs) >= 12
    for i, j in pairs:
        toks[i] = toks[j] + 1024
    pw = as_plain(w)
    want = P.forward(cfg, pw, toks).float()
    top = float(want.abs().max())
    # the pairs do decide the logits: other chunk borders, or another token in the far key's place, move them far
    other, moved = copy.deepcopy(cfg), list(toks)
    if chunk:
        other["layers"][0]["mixer"]["left"]["mask"]["size"] = chunk - 1
    else:
        moved[3] = 1000 if toks[3] != 1000 else 1001
    rows = sorted({i for i, _ in pairs})
    change = (P.forward(other, pw, moved).float() - want)[rows].abs().max(-1).values
    assert int((change > 0.15 * top).sum()) >= (3 if chunk else 1)
    model = build(cfg, w, dtype).model
    from gguf_rs_cli_b200.engine.step import Engine
    for max_step, cuts in [(None, [n]), (None, [190, 12, 2, 96, 400]), (64, [64] * 10 + [60])]:
        eng = Engine(model, n_tokens=2048, n_slots=2, max_step_tokens=max_step)
        s, at = eng.open(), 0
        for k in cuts:
            wanted = [r - at for r in rows if at <= r < at + k]
            got = eng.step([entry(s, toks[at:at + k], wanted)])
            if wanted:
                assert_model(got, want[[at + x for x in wanted]], dtype, f"portion {at}..{at + k} of {cuts}")
            at += k
        eng.close(s)
    # decoded one by one from position 180 on, in a cache whose ring goes round; and from the very first token
    for start in (180, 0):
        eng = Engine(model, n_tokens=2048, n_slots=2, max_step_tokens=32)
        s = eng.open()
        for at in range(0, start - 20, 32):
            eng.step([entry(s, toks[at:at + 32], [])])
        if start:
            eng.step([entry(s, toks[160:180], [])])
        for i in range(start, n if start else 150):
            got = eng.step([entry(s, [toks[i]], [0])])
            if i in rows:
                assert_model(got[0], want[i], dtype, f"position {i} decoded alone")
        eng.close(s)


@pytest.mark.parametrize("dtype", DTYPES)
def test_states_carry_the_first_tokens_far(dtype):
    """Long memories (a decay of 1, and recurrences whose decay is near it): the sequence's first tokens show hundreds of
    positions on, and a sequence in a slot that another has used before starts from nothing."""
    cfg = {"architecture": "Tukevik", "vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "layers": [
        {"type": "parallel", "mlp": None, "mixer": {
            "left": {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.2, "softcap": 5.0, "mask": {"size": 8}},
            "right": {"heads": 2, "dim": 32, "vdim": 32, "decay": [1.0, 0.9990234375]}, "left_scale": 0.5, "right_scale": 1.5}},
        {"type": "rglru", "mlp": None, "mixer": {"width": 64, "blocks": 2, "conv": 4}}]}
    w = make_weights(cfg, seed=3)
    w["l1.mix.lam"] = torch.full((64,), -9.0)
    toks = torch.randint(0, 64, (400,), generator=torch.Generator().manual_seed(1)).tolist()
    other = [(t + 17) % 64 for t in toks[:40]] + toks[40:]
    pw = as_plain(w)
    want, want2 = P.forward(cfg, pw, toks).float(), P.forward(cfg, pw, other).float()
    assert float((want - want2)[-20:].pow(2).mean().sqrt()) > 0.1 * float(want[-20:].pow(2).mean().sqrt())
    from gguf_rs_cli_b200.engine.step import Engine
    eng = Engine(build(cfg, w, dtype).model, n_tokens=1024, n_slots=1)
    for seq, ref, cuts in ((toks, want, [380] + [1] * 20), (other, want2, [39, 2, 200, 139, 20]), (toks, want, [1] * 60 + [340])):
        s, at, got = eng.open(), 0, []
        for c in cuts:
            got.append(eng.step([entry(s, seq[at:at + c], range(c))]).clone())
            at += c
        eng.close(s)
        assert_model(torch.cat(got), ref, dtype, f"portions {cuts[:3]}")


def test_fast_paths_agree_with_the_general_kernels():
    """The wide model in bfloat16 twice: with the tiled attention of prompts, the decode kernel of single tokens, the chunked
    retention and the fused recurrence where its layers take them, and with the general kernels in their place."""
    from gguf_rs_cli_b200 import kernels
    name = "wide"
    model = llm(name, "bfloat16", True).model
    fast = [l.mixer.left for l in model.layers if l.mixer.spec.kind == "weighted_pair"]
    assert [m._exact_tiled() for m in fast] == [True, True, True, False] and all(m._exact_decode() == (m.hd == m.vd) for m in fast)
    toks, results = tokens_of(name, 260, 77), []
    saved = kernels.retention_chunks_supported, kernels.rglru_fused_supported
    for use_fast in (True, False):
        if not use_fast:
            for m in fast:
                m._fast_masks = lambda: False
            kernels.retention_chunks_supported = lambda *a: False
            kernels.rglru_fused_supported = lambda *a: False
        try:
            eng = new_engine(name, "bfloat16", True)
            s = eng.open()
            out = [eng.step([entry(s, toks[:200], range(200))]).clone(), eng.step([entry(s, toks[200:230], range(30))]).clone()]
            out += [eng.step([entry(s, [t], [0])]).clone() for t in toks[230:]]
            results.append(torch.cat(out))
        finally:
            kernels.retention_chunks_supported, kernels.rglru_fused_supported = saved
            for m in fast:
                m.__dict__.pop("_fast_masks", None)
    assert_model(results[0], results[1].cpu(), "bfloat16", "fast against general paths")


# ------------------------------------------------------------ generation
def plain_greedy(name, prompt, max_tokens):
    cfg, w = CONFIGS[name], as_plain(weights(name))
    seq, out = list(prompt), []
    for _ in range(max_tokens):
        out.append(int(P.forward(cfg, w, seq)[-1].argmax()))
        seq.append(out[-1])
    return out


def test_greedy_generation_float32_equals_plain():
    from gguf_rs_cli_b200.api import generate
    prompts = [tokens_of("small", n, 50 + n) for n in (5, 1, 13, 66)]
    got = generate(llm("small", "float32"), prompts, max_tokens=10, temperature=0.0, stop_token_ids=[])
    assert got == [plain_greedy("small", p, 10) for p in prompts]
    # more requests than the batch holds: one batch after another through the same slots
    got2 = generate(llm("small", "float32"), prompts, max_tokens=10, temperature=0.0, stop_token_ids=[], max_batch=2)
    assert got2 == got


def test_bfloat16_greedy_follows_plain_until_a_near_tie():
    from gguf_rs_cli_b200.api import generate
    cfg, w = all_chosen(CONFIGS["wide"]), as_plain(weights("wide"))
    prompts = [tokens_of("wide", n, 80 + n) for n in (3, 40)]
    got = generate(llm("wide", "bfloat16", True), prompts, max_tokens=12, temperature=0.0, stop_token_ids=[])
    for p, g in zip(prompts, got):
        seq = list(p)
        for tok in g:
            logits = P.forward(cfg, w, seq)[-1]
            assert float(logits[tok]) >= float(logits.max()) - 0.05 * float(logits.abs().max())
            seq.append(tok)


def test_decode_steps_run_as_captured_graphs():
    """The generation loop captures decode steps of this design as of the others: every part declares its class."""
    assert llm("wide", "bfloat16", True).model.capturable and llm("small", "float32").model.capturable


def test_command_line_with_random_weights(tmp_path, capsys):
    from gguf_rs_cli_b200.cli import main
    path = tmp_path / "config.json"
    path.write_text(json.dumps(config("small")))
    assert main(["--random", str(path), "-p", "1,2,3", "-p", "9", "-n", "5", "-t", "0", "--no-eos"]) == 0
    lines = capsys.readouterr().out.strip().splitlines()
    assert len(lines) == 2 and all(len(l.split(",")) == 5 for l in lines)


def test_trace_replay_of_a_model_folder(tmp_path):
    """bin/trace_run on a Tukevik folder: two requests together, decoded together, the rest alone."""
    from gguf_rs_cli_b200.weights import write_safetensors
    from tests.test_trace_run_gpu import Replay
    name = "small"
    cfg, w, V = config(name), weights(name), config(name)["vocab"]
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), [(k, v.to(torch.bfloat16)) for k, v in w.items()])
    a, b = tokens_of(name, 40, 1), tokens_of(name, 23, 2)
    wa, wb = plain_logits(name, 40, 1), plain_logits(name, 23, 2)
    run = Replay(str(folder), "float32", str(tmp_path / "out"), 256)
    got = torch.from_numpy(run.step([("a", a[:30], [0, 29]), ("b", b[:20], [19])])).view(3, V)
    assert_model(got, torch.stack([wa[0], wa[29], wb[19]]), "float32", "two prompts together")
    assert run.step([("a", [a[30]], []), ("b", [b[20]], [])]) is None
    for j in range(1, 3):
        got = torch.from_numpy(run.step([("a", [a[30 + j]], [0]), ("b", [b[20 + j]], [0])], ["b"] if j == 2 else [])).view(2, V)
        assert_model(got, torch.stack([wa[30 + j], wb[20 + j]]), "float32", f"decoded together, step {j}")
    got = torch.from_numpy(run.step([("a", a[33:], [6])], ["a"])).view(1, V)
    assert_model(got, wa[39:40], "float32", "the rest alone")
    run.finish()
