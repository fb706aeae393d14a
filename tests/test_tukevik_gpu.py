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
    square of a row's error is held to 5% of the block's root mean square for a mechanism alone, to 10% for whole models
    (peaked softmaxes pass a rounding on enlarged, from layer to layer; the 32-bit runs are the sharper test of those)."""
    got, want = got.detach().float().cpu(), want.detach().float().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} != {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    err, ref = float((got - want).abs().max()), max(float(want.abs().max()), 1e-6)
    if dtype == "float32":
        assert err <= (tol or TOL[dtype]) * ref, f"{what}: max error {err:.3e} against max |ref| {ref:.3e} ({dtype})"
        return
    g2, w2 = got.reshape(-1, got.shape[-1]), want.reshape(-1, want.shape[-1])
    rms_ref = max(float(w2.pow(2).mean().sqrt()), 1e-6)
    worst, limit = float((g2 - w2).pow(2).mean(-1).sqrt().max()) / rms_ref, 0.05 if tol is None else 0.1
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
