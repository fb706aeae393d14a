"""Tukevik on the host: configuration and refusals, tensor names, caches and states of the layers, and the plain
implementation against closed forms and against itself with a mechanism left out."""
import copy
import math

import pytest
import torch

from gguf_rs_cli_b200.config import ConfigError, load_config
from gguf_rs_cli_b200.models.decoder import Decoder, tensor_requests
from tests import plain_tukevik as P
from tests.tukevik_util import CONFIGS, all_chosen, as_plain, config, tokens_of, weights


def spec_of(cfg):
    arch, typed = load_config(copy.deepcopy(cfg))
    return arch.build_spec(typed)


@pytest.mark.parametrize("name", ["small", "wide"])
def test_tensor_names_and_shapes_are_those_of_the_weights(name):
    asked = {r.name: tuple(r.shape) for r in tensor_requests(spec_of(CONFIGS[name]))}
    assert asked == {k: tuple(v.shape) for k, v in weights(name).items()}


def test_registry_picks_the_design_by_its_name():
    arch, typed = load_config(config("small"))
    assert arch.name == "Tukevik" and typed.residual_mult == 0.6
    spec = arch.build_spec(typed)
    assert [l.mixer.kind for l in spec.layers] == ["rglru", "weighted_pair"] * 3
    assert spec.layers[0].block_params == {"scale": 0.6, "unsummed": True}
    assert [l.feed_forward and l.feed_forward.kind for l in spec.layers] == ["gated_mlp", "moe", "moe", None, "moe", "gated_mlp"]
    left, right = spec.layers[1].mixer.params["left"].params, spec.layers[1].mixer.params["right"].params
    assert left["chunk"] == 13 and left["softcap"] == 4.0 and right["decay"] == [0.5, 0.96875, 0.998046875]
    assert spec.layers[1].position.params["rotary_dim"] == 8 and spec.layers[3].position is None
    assert spec.head.tensors == {"weight": "embed"}


def test_absent_keys_mean_absent_mechanisms():
    cfg = config("small")
    del cfg["residual_mult"]
    m = cfg["layers"][1]["mixer"]
    for key in ("kv_heads", "vdim", "softcap", "mask", "scale"):
        m["left"].pop(key)
    for key in ("vdim", "rot"):
        m["right"].pop(key)
    m.pop("left_scale"), m.pop("right_scale")
    cfg["layers"][1]["mlp"].pop("shared")
    spec = spec_of(cfg)
    p = spec.layers[1].mixer.params
    left = p["left"].params
    assert spec.layers[1].block_params["scale"] == 1.0 and (p["left_scale"], p["right_scale"]) == (1.0, 1.0)
    assert left["num_kv_heads"] == 6 and left["v_head_dim"] == 20 and left["softcap"] is None and left["chunk"] is None
    assert abs(left["scale"] - 20 ** -0.5) < 1e-12 and p["right"].params["vdim"] == 12 and spec.layers[1].position is None
    assert not any("l1.mlp.shared" in r.name for r in tensor_requests(spec))


def test_caches_and_states_of_the_layers():
    layout = Decoder(spec_of(config("small")), torch.float32, "meta").cache_layout()
    assert sorted(layout.kv) == [1, 3, 5]
    assert (layout.kv[1].head_dim, layout.kv[1].v_dim, layout.kv[1].window) == (20, 28, 13) and layout.kv[3].window is None
    assert layout.states["run0.S"][0] == (60,) and layout.states["run0.conv"][0] == (3, 60)
    assert layout.states["run1.right.S"][0] == (3, 12, 18) and "run4.conv" not in layout.states


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="gru"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(blocks=7), "blocks"),
    (lambda c: c["layers"][0]["mixer"].update(conv=17), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("width"), "width"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["right"]["rot"].update(dims=14), "dims"),
    (lambda c: c["layers"][1]["mixer"]["right"]["rot"].update(dims=5), "dims"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c.pop("norm"), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_refusals_name_the_key(change, text):
    cfg = config("small")
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        load_config(cfg)


def test_a_weighted_pair_refuses_branches_that_keep_their_products():
    from gguf_rs_cli_b200.config import PartSpec
    from gguf_rs_cli_b200.parts import MIXERS
    spec = spec_of(config("small")).layers[1].mixer
    gla = PartSpec("gla", dict(hidden_size=72, heads=2, dim=8, vdim=8, tau=16.0, eps=1e-5))
    with pytest.raises(ValueError, match="gla"):
        MIXERS.get("weighted_pair")(PartSpec(spec.kind, {**spec.params, "right": gla}), torch.float32, "meta")


# ------------------------------------------------------------ the plain implementation
def test_chunks_sink_and_softcap():
    assert P.visible(7, 3)[5].tolist() == [False, False, False, True, True, True, False] and P.visible(7, 3)[6].tolist() == [False] * 6 + [True]
    assert P.visible(4, None).tolist() == torch.ones(4, 4).tril().bool().tolist()
    # equal scores of 0: a token that sees n keys gives each 1 / (n + 1)
    T = 5
    z, v = torch.zeros(T, 1, 2, dtype=P.F64), torch.eye(T, dtype=P.F64)[:, None, :]
    o = P.sink_attention(z, z, v, 1.0, 2.0, P.visible(T, 3))[:, 0]
    assert torch.allclose(o[2], torch.tensor([0.25, 0.25, 0.25, 0.0, 0.0], dtype=P.F64)) and torch.allclose(o[3], torch.tensor([0, 0, 0, 0.5, 0], dtype=P.F64))
    # one key with a score far above the cap: exp(cap) / (1 + exp(cap))
    q = torch.full((1, 1, 2), 100.0, dtype=P.F64)
    o = P.sink_attention(q, q, torch.ones(1, 1, 1, dtype=P.F64), 1.0, 2.0, P.visible(1, None))
    assert abs(float(o[0, 0, 0]) - math.exp(2.0) / (1 + math.exp(2.0))) < 1e-9
    assert torch.equal(P.capped(torch.tensor([5.0]), None), torch.tensor([5.0]))


def test_retention_is_a_decayed_sum():
    g = torch.Generator().manual_seed(0)
    T, H, D, Dv = 6, 2, 3, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=P.F64) for n in (D, D, Dv))
    decay = [0.5, 1.0]
    got = P.retention(q, k, v, decay)
    for h in range(H):
        for t in range(T):
            want = sum((decay[h] ** (t - j) * float(q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1)), torch.zeros(Dv, dtype=P.F64))
            assert torch.allclose(got[t, h], want)


def test_rotation_in_halves():
    x = torch.arange(12, dtype=P.F64).view(1, 2, 6)
    y = P.rotate(x, torch.tensor([3]), {"base": 100.0, "dims": 4})
    for h in range(2):
        for i in range(2):
            u, v, a = float(x[0, h, i]), float(x[0, h, i + 2]), 3 * 100.0 ** (-2.0 * i / 4)
            assert abs(float(y[0, h, i]) - (u * math.cos(a) - v * math.sin(a))) < 1e-12
            assert abs(float(y[0, h, i + 2]) - (v * math.cos(a) + u * math.sin(a))) < 1e-12
        assert y[0, h, 4:].tolist() == x[0, h, 4:].tolist()


def test_recurrence_coefficients_and_blocks():
    W = {"ra": torch.zeros(2, 2, 2, dtype=P.F64), "ra.b": torch.zeros(2, 2, dtype=P.F64), "ri": torch.zeros(2, 2, 2, dtype=P.F64),
         "ri.b": torch.full((2, 2), 50.0, dtype=P.F64), "lam": torch.zeros(4, dtype=P.F64)}
    a, b = P.recurrence_coefficients(W, "", torch.ones(1, 4, dtype=P.F64))
    assert torch.allclose(a, torch.full((1, 4), 2.0 ** -4, dtype=P.F64))               # exp(-8 / 2 ln 2)
    assert torch.allclose(b, torch.full((1, 4), math.sqrt(1 - 2.0 ** -8), dtype=P.F64))
    u, w = torch.tensor([[1.0, 2.0, 3.0, 4.0]], dtype=P.F64), torch.tensor([[[1.0, 10.0], [0.0, 1.0]], [[2.0, 0.0], [1.0, 1.0]]], dtype=P.F64)
    assert P.block_product(u, w, torch.zeros(2, 2, dtype=P.F64)).tolist() == [[21.0, 2.0, 6.0, 7.0]]


def test_convolution_and_route():
    u = torch.tensor([[1.0], [2.0], [4.0]], dtype=P.F64)
    y = P.causal_conv(u, torch.tensor([[10.0, 1.0]], dtype=P.F64), torch.tensor([0.5], dtype=P.F64))
    assert y[:, 0].tolist() == [1.5, 12.5, 24.5]
    mlp = {"router": {"experts": 3, "top": 2}}
    W = {"m.router": torch.zeros(3, 1, dtype=P.F64), "m.router.b": torch.tensor([2.0, 1.0, 5.0], dtype=P.F64)}
    for e in range(3):          # an expert that gives silu(1) e in every entry
        W[f"m.e{e}.gate"], W[f"m.e{e}.up"], W[f"m.e{e}.down"] = (torch.full((1, 1), x, dtype=P.F64) for x in (1.0, 1.0, float(e)))
    s, w2 = 1 / (1 + math.exp(-1.0)), 1 / (1 + math.exp(-3.0))
    assert abs(float(P.moe(mlp, W, "m.", torch.ones(1, 1, dtype=P.F64))) - s * 2.0 * w2) < 1e-12


def test_every_mechanism_moves_the_logits():
    name = "small"
    cfg, w = config(name), as_plain(weights(name))
    toks = tokens_of(name, 60, 3)
    base = P.forward(cfg, w, toks)
    top = float(base.abs().max())

    def moved(change=None, w2=None):
        c = copy.deepcopy(cfg)
        if change:
            change(c)
        return float((P.forward(c, w2 or w, toks) - base).abs().max()) / top

    L = lambda c, i, side: c["layers"][i]["mixer"][side]                        # noqa: E731
    for what, change in {
            "chunk": lambda c: L(c, 1, "left")["mask"].update(size=14), "no chunks": lambda c: L(c, 1, "left").pop("mask"),
            "softcap": lambda c: L(c, 1, "left").pop("softcap"), "another softcap": lambda c: L(c, 1, "left").update(softcap=5.0),
            "score scale": lambda c: L(c, 3, "left").update(scale=0.3), "decay": lambda c: L(c, 1, "right")["decay"].__setitem__(1, 0.95),
            "rotation": lambda c: L(c, 1, "right").pop("rot"), "its base": lambda c: L(c, 1, "right")["rot"].update(base=90.0),
            "its width": lambda c: L(c, 1, "right")["rot"].update(dims=6), "residual factor": lambda c: c.update(residual_mult=0.65),
            "left factor": lambda c: c["layers"][1]["mixer"].update(left_scale=0.75),
            "right factor": lambda c: c["layers"][3]["mixer"].update(right_scale=-0.5),
            "a feed-forward left out": lambda c: c["layers"][2].update(mlp=None),
            "shared expert": lambda c: c["layers"][1]["mlp"].pop("shared")}.items():
        assert moved(change) > 0.004, what
    for key in ("l1.mix.left.q.b", "l1.mix.left.k.b", "l1.mix.left.v.b", "l1.mix.left.g", "l1.mix.right.g", "l0.mix.y.b", "l0.mix.x.b",
                "l0.mix.conv.b", "l2.mix.conv", "l0.mix.ra", "l0.mix.ra.b", "l2.mix.ri", "l2.mix.ri.b", "l0.mix.lam", "l2.norm1",
                "l1.norm2", "l1.mlp.router.b", "l1.mlp.shared.sg", "l4.mlp.router"):
        w2 = dict(w)
        w2[key] = w[key] + 2.0 * torch.linspace(-1.0, 1.0, w[key].numel(), dtype=P.F64).view(w[key].shape)
        assert moved(w2=w2) > 0.004, key
    assert float((P.forward(all_chosen(cfg), w, toks) - base).abs().max()) / top > 0.01, "the router's choice"
