"""Betirax in the package against the plain implementation (tests/plain_betirax.py), in 32-bit and in bfloat16: every
mechanism alone, whole prompts against token-by-token decoding, prompts cut into portions down to two tokens, unequal
batches against each request alone, slots and pages that are used again, keys far back, at page borders and just inside
and outside every window, the first tokens of a sequence, long decoding through rings of pages that go round, sizes that
fit no fast kernel, and greedy generation through the package's entry point.

A router's choice is discrete: where two logits are closer than bfloat16's rounding, bfloat16 takes another expert than
the float64 oracle.  So whole models run with their routers in 32-bit, and in bfloat16 as twins in which every expert is
chosen (the same weights; `all_chosen`); the routed kernels themselves are tested in bfloat16 with the choice given."""
import copy
import json

import pytest
import torch

from tests import plain_betirax as P
from tests.betirax_util import CONFIGS, all_chosen, as_plain, build, config, llm, make_weights, new_engine, plain_logits, tokens_of, weights
from tests.gpu_util import TOL

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


# ------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,routed", [(5, True), (72, False), (72, True), (1000, True), (2048, False), (4096, True), (9000, True), (12304, False),
                                      (20000, True)])
def test_layer_norm_of_a_sum_with_a_mixtures_rows(E, routed, dtype):
    from gguf_rs_cli_b200 import kernels
    g = torch.Generator().manual_seed(E)
    T, eps, td, top, alpha = 7, 1e-3, tdtype(dtype), 3, 1.8
    x, y, w = torch.randn(T, E, generator=g) + 0.7, (torch.randn(T, E, generator=g) * 2).to(td), (1 + 0.3 * torch.randn(E, generator=g)).to(td)
    z, wz = torch.randn(T * top, E, generator=g), torch.rand(T, top, generator=g)
    place = torch.randperm(T * top, generator=g)
    v = alpha * x.double() + y.double()
    if routed:
        v = v + (wz.double()[:, :, None] * z.double()[place].view(T, top, E)).sum(1)
    want = P.layer_norm(v, w.double(), eps).float()
    xd, xb, h = x.to(DEV), torch.empty(T, E, dtype=torch.bfloat16, device=DEV), torch.empty(T, E, dtype=td, device=DEV)
    kernels.layernorm(xd, y.to(DEV), w.to(DEV), eps, alpha=alpha, h=h, xb=xb,
                      routed=(z.to(DEV), wz.to(DEV), place.to(torch.int32).to(DEV)) if routed else None)
    assert_close(xd, want, "float32", "the new x")
    assert torch.equal(xb, xd.to(torch.bfloat16)) and torch.equal(h, xd.to(td))
    if routed:      # rows in the pairs' own order, nothing beside them
        xd = x.to(DEV)
        kernels.layernorm(xd, None, w.to(DEV), eps, routed=(z[place].contiguous().to(DEV), wz.to(DEV), None))
        v = x.double() + (wz.double()[:, :, None] * z.double()[place].view(T, top, E)).sum(1)
        assert_close(xd, P.layer_norm(v, w.double(), eps).float(), "float32", "rows in their own order")
    # chosen rows only, x left as it is
    xd, rows = x.to(DEV), torch.tensor([4, 0, 4], dtype=torch.int32, device=DEV)
    h = torch.empty(3, E, dtype=td, device=DEV)
    kernels.layernorm(xd, None, w.to(DEV), eps, rows=rows, h=h, write_x=False)
    assert_close(h, P.layer_norm(x.double(), w.double(), eps)[[4, 0, 4]].float(), dtype, "chosen rows")
    assert torch.equal(xd.cpu(), x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,lead", [(1, 0), (17, 3), (96, 8), (768, 16)])
def test_norm_of_the_query_latent_in_a_block_of_columns(C, lead, dtype):
    from gguf_rs_cli_b200 import kernels
    g = torch.Generator().manual_seed(C)
    td, buf = tdtype(dtype), torch.randn(9, lead + C + 5, generator=g).to(tdtype(dtype))
    w = (1 + 0.3 * torch.randn(C, generator=g)).to(td)
    out = kernels.rms_rows(buf.to(DEV)[:, lead:lead + C], w.to(DEV), 1e-2, torch.empty(9, C, dtype=td, device=DEV))
    assert_close(out, P.rms_norm(buf[:, lead:lead + C].double(), w.double(), 1e-2).float(), dtype)


def attention_case(dtype, H, G, D, T, window, seed, temp=None):
    """q, k (which is v) of one sequence through head_prep_kv_write into a cache of its own."""
    g = torch.Generator().manual_seed(seed)
    td = tdtype(dtype)
    qk = torch.randn(T, (H + G) * D, generator=g).to(td)
    wq, wk = (1 + 0.3 * torch.randn(D, generator=g)).to(td), (1 + 0.3 * torch.randn(D, generator=g)).to(td)
    gate = torch.randn(T, H * D, generator=g).to(td)
    scale, eps = 9.0 / D, 1e-3
    q, k = qk[:, :H * D].double().view(T, H, D), qk[:, H * D:].double().view(T, G, D)
    qn = P.rms_norm(q, wq.double(), eps)
    if temp:
        qn = qn * P.query_temperature(torch.arange(T), temp)[:, None, None]
    o = P.softmax_attention(qn, P.rms_norm(k, wk.double(), eps), k, scale, P.visible(T, window), P.head_slopes(H)).reshape(T, H * D)
    want = (o * torch.sigmoid(gate.double())).float()
    return qk, wq, wk, gate, scale, eps, want


@pytest.mark.parametrize("dtype,H,G,D,window", [("float32", 6, 2, 24, 13), ("float32", 3, 3, 5, None), ("bfloat16", 4, 2, 64, 70), ("bfloat16", 4, 1, 128, None),
                                                ("bfloat16", 8, 8, 64, 96), ("bfloat16", 5, 5, 48, 40), ("bfloat16", 3, 1, 20, 9)])
def test_distance_bias_keys_as_values_and_temperature_on_every_attention_kernel(dtype, H, G, D, window):
    from gguf_rs_cli_b200 import kernels
    T, temp, td = 200, {"coef": 0.3, "every": 16}, tdtype(dtype)
    qk, wq, wk, gate, scale, eps, want = attention_case(dtype, H, G, D, T, window, D + H, temp)
    slopes = torch.tensor(P.head_slopes(H), dtype=torch.float32, device=DEV)
    pages = (T + 63) // 64
    table = torch.randperm(pages, generator=torch.Generator().manual_seed(1)).to(torch.int32).to(DEV)[None, :].contiguous()
    kc, vc = torch.zeros(pages, G, 64, D, dtype=td, device=DEV), torch.zeros(pages, G, 64, D, dtype=td, device=DEV)
    buf, pos = qk.to(DEV), torch.arange(T, dtype=torch.int32, device=DEV)
    seq = torch.zeros(T, dtype=torch.int32, device=DEV)
    q, k = buf[:, :H * D], buf[:, H * D:]
    kernels.head_prep_kv_write(q, k, k, H, G, D, D, wq.to(DEV), wk.to(DEV), eps, None, 0, 0, None, 0.0, None, seq, pos, table, pages, 0, kc, vc,
                               temp_coef=temp["coef"], temp_every=temp["every"])
    gd, win = gate.to(DEV), window or 0
    assert torch.equal(vc[table[0, 1].item(), G - 1, 5].cpu(), qk[69, (H + G - 1) * D:])          # the key as projected is the value
    out = torch.empty(T, H * D, dtype=td, device=DEV)
    kernels.attention_generic(q, out, H, G, D, seq, pos, table, pages, kc, vc, win, scale, gate=gd, slopes=slopes)
    assert_close(out, want, dtype, "general kernel")
    if dtype == "float32":
        return
    if kernels.attention_prefill_supported(q, kc, D) and q.stride(0) % 8 == 0:
        meta = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)                            # noqa: E731
        got = torch.empty_like(out)
        kernels.attention_prefill(q, got, H, G, D, meta(*kernels.attention_prefill_tiles([T])), meta(0, T), meta(0), meta(T), table, pages, kc, vc,
                                  win, scale, tc=False, exact=True, gate=gd, slopes=slopes)
        assert_close(got, want, dtype, "tiled kernel")
        assert_close(got, out.cpu(), dtype, "tiled against general kernel")
    if kernels.attention_decode_supported(q, kc, D):
        for splits in (1, 3):
            got = torch.empty_like(out)
            kernels.attention_decode(q, got, H, G, D, seq, pos, table, pages, kc, vc, win, scale, mma=False, max_kv=T, splits=splits, gate=gd,
                                     slopes=slopes)
            assert_close(got, want, dtype, f"single tokens, {splits} splits")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("reads", [False, True])
def test_latent_rows_and_queries_with_a_gain_on_the_rotation(reads, dtype):
    """Both halves of the preparation: the row that goes into the cache and the queries' rotated parts; a layer that reads
    another's rows rotates its queries only and leaves the cache as it is."""
    from gguf_rs_cli_b200 import kernels
    H, D, R, C, T = 3, 10, 12, 36, 9
    rot = CONFIGS["small"]["layers"][0]["mixer"]["rot"]
    td, g = tdtype(dtype), torch.Generator().manual_seed(2)
    q, dkv, w = torch.randn(T, H * (D + R), generator=g).to(td), torch.randn(T, C + R, generator=g).to(td), (1 + 0.3 * torch.randn(C, generator=g)).to(td)
    pos = torch.arange(60, 60 + T)
    qw = q.double().view(T, H, D + R)
    want_q = P.rotate(qw[..., D:], pos, rot).float()
    want_row = torch.cat([P.rms_norm(dkv[:, :C].double(), w.double(), 1e-4), P.rotate(dkv[:, None, C:].double(), pos, rot)[:, 0]], dim=-1).float()
    cache = torch.full((2, 1, 64, C + R), 7.0, dtype=td, device=DEV)
    table = torch.tensor([[1, 0]], dtype=torch.int32, device=DEV)
    qa, row = torch.zeros(T, H * (C + R), dtype=td, device=DEV), torch.empty(T, C + R, dtype=td, device=DEV)
    freq = P.rotary_frequencies(rot).float().to(DEV)
    kernels.latent_prep(q.to(DEV), None if reads else dkv.to(DEV), H, D, R, C, 12, freq, w.to(DEV), 1e-4, qa, torch.zeros(T, dtype=torch.int32, device=DEV),
                        pos.to(torch.int32).to(DEV), table, 2, cache, row_out=None if reads else row, halves=True, gain=P.rotary_gain(rot))
    assert_close(qa.view(T, H, C + R)[..., C:], want_q, dtype, "queries")
    flat = torch.cat([cache[1, 0], cache[0, 0]])
    if reads:
        assert bool((cache == 7.0).all())
    else:
        assert_close(flat[60:60 + T], want_row, dtype, "cached rows")
        assert torch.equal(row, flat[60:60 + T]) and bool((flat[:60] == 7.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
def test_product_per_head_with_a_gate_per_entry(dtype):
    from gguf_rs_cli_b200 import kernels
    g, td = torch.Generator().manual_seed(3), tdtype(dtype)
    H, I, O, T = 3, 36, 28, 11
    x, w, gate = torch.randn(T, H * I, generator=g).to(td), (torch.randn(H, I, O, generator=g) / 6).to(td), torch.randn(T, H * O + 4, generator=g).to(td)
    out = kernels.head_matmul(x.to(DEV), I, w.to(DEV), torch.empty(T, H * O, dtype=td, device=DEV), O, gate=gate.to(DEV)[:, 4:])
    want = torch.einsum("thi,hio->tho", x.double().view(T, H, I), w.double()).reshape(T, H * O) * torch.sigmoid(gate[:, 4:].double())
    assert_close(out, want.float(), dtype)


@pytest.mark.parametrize("n,top", [(5, 3), (12, 2), (1, 1), (40, 8), (3, 3)])
def test_router_weighs_by_the_softmax_of_the_chosen_logits(n, top):
    from gguf_rs_cli_b200 import kernels
    g = torch.Generator().manual_seed(n)
    T, K = 9, 24
    h, w = torch.randn(T, K, generator=g), torch.randn(n, K, generator=g)
    h[0] *= 20.0                                     # logits that lie far apart
    ids_want, w_want = P.route({"router": {"experts": n, "top": top}}, {"m.router": w.double()}, "m.", h.double())
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    kernels.moe_router(h.to(DEV), w.to(DEV), 1, 1, top, 1.0, ids, wts, softmax=True)
    assert ids.cpu().tolist()[1:] == ids_want.tolist()[1:] and ids[0, 0].item() == int(ids_want[0, 0])
    assert_close(wts, w_want.float(), "float32", "weights")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [1, 2])
@pytest.mark.parametrize("T,by_expert", [(3, False), (50, False), (50, True)])
def test_experts_with_the_plain_unit_for_a_given_choice(T, by_expert, layer, dtype):
    """Token by token, in sorted tiles and expert by expert; with a shared expert and without; summed by the part, and left
    to the norm behind it: the same x either way."""
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
        assert isinstance(rows, RoutedRows) and (rows.base is None) == (layer == 2) and (rows.place_of is not None) == by_expert
        x = torch.randn(T, cfg["width"], generator=g)
        a, b = Stream(x.to(DEV)), Stream(x.to(DEV))
        norm.norm_sum(a, rows, ctx, 1.5)
        norm.norm_sum(b, got, ctx, 1.5)
        assert_close(a.x, b.x.cpu(), "float32", "summed behind the norm's back and by the part")
    finally:
        ff.__dict__.pop("BY_EXPERT", None)
        ff.__dict__.pop("BY_EXPERT_ENTRIES", None)


@pytest.mark.parametrize("n", [8, 4096, 77])
def test_activation_of_whole_rows(n):
    from gguf_rs_cli_b200 import kernels
    x = torch.randn(3, n, generator=torch.Generator().manual_seed(n)).to(torch.bfloat16)
    for name, f in (("gelu_tanh", P.gelu_tanh), ("silu", P.silu)):
        got = kernels.unary_act_(x.to(DEV), name)
        assert_close(got, f(x.double()).float(), "bfloat16", name)
        assert torch.equal(kernels.unary_act_(x.to(DEV)[:, 1:], name), got[:, 1:]) if n > 8 else True


# ------------------------------------------------------------ whole models
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
            got.append(stream.x.clone())
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


ODD_ROT = {"base": 10.0, "dims": 2, "scaling": {"factor": 3.0, "original": 9, "fast": 2.0, "slow": 0.1}}
ODD = {
    "architecture": "Betirax", "vocab": 91, "width": 50, "norm": {"eps": 1e-4}, "postln_alpha": 1.0, "embedding": {"scale": 1.0},
    "layers": [
        {"type": "attention", "mixer": {"heads": 5, "kv_heads": 5, "dim": 6, "vdim": 6, "scale": 1.0, "mask": {"size": 1}},
         "mlp": {"kind": "moe", "router": {"experts": 1, "top": 1}, "expert": {"ff": 7}}},
        {"type": "latent_attention", "mixer": {"heads": 1, "dim": 10, "rot_dim": 2, "vdim": 9, "kv_rank": 7, "q_rank": 3, "scale": 0.3, "rot": ODD_ROT},
         "mlp": {"kind": "moe", "router": {"experts": 2, "top": 2}, "expert": {"ff": 3}, "shared": {"ff": 5}}},
        {"type": "latent_attention", "mixer": {"heads": 17, "dim": 1, "rot_dim": 2, "vdim": 1, "kv_rank": 7, "q_rank": 1, "scale": 1.0, "kv_from": 1,
                                               "rot": ODD_ROT}, "mlp": {"kind": "dense", "ff": 1}},
        {"type": "attention", "mixer": {"heads": 7, "kv_heads": 1, "dim": 10, "vdim": 10, "scale": 0.3, "mask": {"size": 2},
                                        "q_temp": {"coef": 1.5, "every": 1}}, "mlp": None},
        {"type": "latent_attention", "mixer": {"heads": 2, "dim": 8, "rot_dim": 4, "vdim": 8, "kv_rank": 700, "q_rank": 5, "scale": 0.3,
                                               "rot": {"base": 100.0, "dims": 4}}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 1, "kv_heads": 1, "dim": 256, "vdim": 256, "scale": 0.1, "q_temp": {"coef": 0.2, "every": 1000}},
         "mlp": {"kind": "dense", "ff": 9}},
    ],
}


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_that_fit_no_fast_kernel_and_values_of_one(dtype):
    """A width that is no multiple of 8, one head and 17 on one latent row, one expert, windows of one and of two positions,
    query latents of one entry, latent rows longer than the general attention kernel's middle instance takes."""
    cfg = copy.deepcopy(ODD)
    if dtype == "bfloat16":
        cfg["layers"][2]["mixer"]["q_rank"] = 6       # a query latent of one entry is a sign, which a rounding can turn
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
def spike_model(kind, size, dims=(24, 24), heads=2):
    """Attention that is decided by one key: token t + 1024 is the partner of token t; its query is the key of t (behind an
    orthogonal map S of the rows; the partner's row is S^T times the row of t), so a partner's score with its token's key
    is large and all others are a few units.  The partner's result is then the value of t if it may see t, and else
    something else altogether.  With `reader` a second layer reads the first one's latent rows."""
    g = torch.Generator().manual_seed(7)
    E, V = 64, 2048
    D, Dv = dims
    S, _ = torch.linalg.qr(torch.randn(E, E, generator=g))
    base = torch.randn(1024, E, generator=g)
    base = base / base.pow(2).mean(-1, keepdim=True).sqrt()
    k = torch.randn(D, E, generator=g) / E ** 0.5
    w = {"embed": torch.cat([base, base @ S]), "l0.norm1": torch.ones(E), "final.norm": torch.ones(E)}
    p = "l0.mix."
    if kind == "latent_attention":
        mixer = {"heads": heads, "dim": D, "rot_dim": 4, "vdim": Dv, "kv_rank": D, "q_rank": E, "scale": 40.0 / D,
                 "rot": {"base": 10.0, "dims": 4, "scaling": {"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0}}}
        w[p + "dq"], w[p + "dq.norm"] = S, torch.ones(E)
        w[p + "uq"] = torch.cat([torch.cat([k, torch.zeros(4, E)])] * heads)
        w[p + "dkv"], w[p + "dkv.norm"] = torch.cat([k, torch.zeros(4, E)]), torch.ones(D)
        w[p + "uk"], w[p + "uv"] = torch.cat([torch.eye(D)] * heads), torch.randn(heads * Dv, D, generator=g) / D ** 0.5 * 3
        w[p + "g"], w[p + "o"] = torch.zeros(heads * Dv, E), torch.randn(E, heads * Dv, generator=g) / 4
    else:
        mixer = {"heads": heads, "kv_heads": 1, "dim": D, "vdim": D, "scale": 60.0 / D, **({"mask": {"size": size}} if size else {})}
        w[p + "q"], w[p + "k"] = torch.cat([k @ S] * heads), k
        w[p + "q.b"], w[p + "k.b"], w[p + "o.b"] = torch.zeros(heads * D), torch.zeros(D), torch.zeros(E)
        w[p + "q.norm"], w[p + "k.norm"] = torch.ones(D), torch.ones(D)
        w[p + "g"], w[p + "o"] = torch.zeros(heads * D, E), torch.randn(E, heads * D, generator=g)
    cfg = {"architecture": "Betirax", "vocab": V, "width": E, "norm": {"eps": 1e-6}, "postln_alpha": 1.0, "embedding": {"scale": 1.0},
           "layers": [{"type": kind, "mixer": mixer, "mlp": None}]}
    return cfg, {n: t.to(torch.bfloat16).float() for n, t in w.items()}


def add_reader(cfg, w, dims):
    """A second layer that reads the first one's latent rows with queries and values of its own."""
    _, w2 = spike_model("latent_attention", None, (cfg["layers"][0]["mixer"]["dim"], dims[1]))
    second = copy.deepcopy(cfg["layers"][0])
    second["mixer"].update(kv_from=0, vdim=dims[1])
    cfg["layers"].append(second)
    for n in ("dq", "dq.norm", "uq", "uk", "uv", "g", "o"):
        w["l1.mix." + n] = w2["l0.mix." + n]
    w["l1.norm1"] = w["l0.norm1"]


@pytest.mark.parametrize("kind,size,dims,heads", [("attention", 70, (24, 24), 2), ("attention", 70, (64, 64), 2), ("attention", 90, (128, 128), 4),
                                                  ("attention", None, (64, 64), 2), ("latent_attention", None, (24, 16), 2),
                                                  ("latent_attention", None, (60, 64), 2), ("latent_attention reader", None, (60, 64), 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_that_stand_out_at_every_edge_in_prompt_and_decode(dtype, kind, size, dims, heads):
    """All tokens differ; for chosen pairs (i, j) position i holds the partner of the token at position j, whose key then
    takes all of i's attention if and only if i may see j (and, with the distance bias, only in the heads whose slope lets
    it).  Pairs: j just inside and just outside the window, across page borders, at the sequence's first positions, and
    hundreds of positions back."""
    cfg, w = spike_model(kind.split()[0], size, dims, heads)
    if "reader" in kind:
        add_reader(cfg, w, dims)
    n, edge = 700, size or 70
    toks = torch.randperm(1024, generator=torch.Generator().manual_seed(1))[:n].tolist()
    pairs = [(200, 200 - edge + 1), (210, 210 - edge), (edge - 1, 0), (edge, 0), (edge + 2, 3), (64 + edge - 1, 64), (64 + edge + 3, 65),
             (128, 127), (129, 66), (650, 3), (660, 660 - edge + 1), (670, 670 - edge), (699, 699 - edge + 1), (690, 690 - edge), (5, 0), (1, 0)]
    assert not {i for i, _ in pairs} & {j for _, j in pairs}
    for i, j in pairs:
        toks[i] = toks[j] + 1024
    pw = as_plain(w)
    want = P.forward(cfg, pw, toks).float()
    top = float(want.abs().max())
    # the pairs do decide the logits
    if size:                         # a mask one position longer moves the second pair far
        longer = copy.deepcopy(cfg)
        longer["layers"][0]["mixer"]["mask"]["size"] = size + 1
        assert float((P.forward(longer, pw, toks[:211]).float()[210] - want[210]).abs().max()) > 0.2 * top
    else:                            # another token in the far key's place moves its partner far
        other = list(toks)
        other[3] = 1000 if toks[3] != 1000 else 1001
        assert float((P.forward(cfg, pw, other).float()[650] - want[650]).abs().max()) > 0.2 * top
    rows = sorted({i for i, _ in pairs})
    model = build(cfg, w, dtype).model
    from gguf_rs_cli_b200.engine.step import Engine
    for max_step, cuts in [(None, [n]), (None, [190, 12, 2, 96, 400]), (64, [64] * 10 + [60])]:
        eng = Engine(model, n_tokens=2048, n_slots=2, max_step_tokens=max_step)
        s, at = eng.open(), 0
        for c in cuts:
            wanted = [r - at for r in rows if at <= r < at + c]
            got = eng.step([entry(s, toks[at:at + c], wanted)])
            if wanted:
                assert_model(got, want[[at + x for x in wanted]], dtype, f"portion {at}..{at + c} of {cuts}")
            at += c
        eng.close(s)
    # decoded one by one from position 180 on, in a cache whose ring goes round; and from the very first token
    for start in (180, 0):
        eng = Engine(model, n_tokens=2048, n_slots=2, max_step_tokens=32)
        s = eng.open()
        for at in range(0, start - 20, 32):
            eng.step([entry(s, toks[at:at + 32], [])])
        if start:
            eng.step([entry(s, toks[160:180], [])])
        for i in range(start, n if start else 140):
            got = eng.step([entry(s, [toks[i]], [0])])
            if i in rows:
                assert_model(got[0], want[i], dtype, f"position {i} decoded alone")
        eng.close(s)


def test_fast_paths_agree_with_the_general_kernels():
    """The wide model in bfloat16 twice: with the tiled kernel of prompts, the decode kernels of single tokens and the tiled
    path of latent layers where its layers take them, and with the general kernels in their place."""
    name = "wide"
    model = llm(name, "bfloat16", True).model
    fast = [l.mixer for l in model.layers if l.mixer.spec.kind == "attention"]
    latent = [l.mixer for l in model.layers if l.mixer.spec.kind == "latent_attention"]
    assert all(m._exact_tiled() and m._exact_decode() for m in fast)
    assert [m._tiled() for m in latent] == [True, True, False, False, True] and all(m._fast_decode() for m in latent)
    toks = tokens_of(name, 260, 77)
    results = []
    for use_fast in (True, False):
        if not use_fast:
            for m in fast:
                m._fast_masks = lambda: False
            for m in latent:
                m._tiled = m._fast_decode = lambda: False
        try:
            eng = new_engine(name, "bfloat16", True)
            s = eng.open()
            out = [eng.step([entry(s, toks[:200], range(200))]).clone(), eng.step([entry(s, toks[200:230], range(30))]).clone()]
            out += [eng.step([entry(s, [t], [0])]).clone() for t in toks[230:]]
            results.append(torch.cat(out))
        finally:
            for m in fast + latent:
                for attr in ("_fast_masks", "_tiled", "_fast_decode"):
                    m.__dict__.pop(attr, None)
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
    """bin/trace_run on a Betirax folder: two requests together, decoded together, the rest alone."""
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
