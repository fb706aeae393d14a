"""Betirax on the host: configuration and refusals, tensor names, the cache that layers share, the frequency table, and the
plain implementation against closed forms and against itself with a mechanism left out."""
import copy
import math

import pytest
import torch

from gguf_rs_cli_b200.config import ConfigError, load_config
from gguf_rs_cli_b200.models.decoder import Decoder, tensor_requests
from gguf_rs_cli_b200.parts.rotary import inverse_frequencies, rotation_gain
from tests import plain_betirax as P
from tests.betirax_util import CONFIGS, all_chosen, as_plain, config, make_weights, tokens_of, weights


def spec_of(cfg):
    arch, typed = load_config(copy.deepcopy(cfg))
    return arch.build_spec(typed)


@pytest.mark.parametrize("name", ["small", "wide"])
def test_tensor_names_and_shapes_are_those_of_the_weights(name):
    asked = {r.name: tuple(r.shape) for r in tensor_requests(spec_of(CONFIGS[name]))}
    assert asked == {k: tuple(v.shape) for k, v in weights(name).items()}


def test_registry_picks_the_design_by_its_name():
    arch, typed = load_config(config("small"))
    assert arch.name == "Betirax" and typed.alpha == 1.7 and typed.embedding_scale == 1.4
    spec = arch.build_spec(typed)
    assert [l.block for l in spec.layers] == ["postnorm"] * 6 and spec.layers[0].block_params == {"alpha": 1.7}
    assert [l.feed_forward and l.feed_forward.kind for l in spec.layers] == ["mlp", "moe", "moe", None, "moe", "mlp"]
    assert [r.cache_of for r in spec.schedule] == [None, None, 0, None, None, None]
    assert spec.layers[1].mixer.params["window"] == 13 and spec.layers[3].mixer.params["window"] is None
    assert spec.head.tensors == {"weight": "embed"}


def test_absent_keys_mean_absent_mechanisms():
    cfg = config("small")
    del cfg["postln_alpha"], cfg["embedding"]
    cfg["layers"][0]["mixer"]["rot"] = {"base": 50.0, "dims": 12}
    cfg["layers"][2]["mixer"]["rot"] = {"base": 50.0, "dims": 12}
    cfg["layers"][1]["mlp"].pop("shared")
    cfg["layers"][1]["mixer"].pop("q_temp")
    spec = spec_of(cfg)
    assert spec.layers[0].block_params == {"alpha": 1.0} and spec.embedding.params["scale"] == 1.0
    assert spec.layers[0].position.params["scaling"] is None and spec.layers[1].mixer.params["q_temp"] is None
    assert not any(".l1.mlp.shared" in r.name for r in tensor_requests(spec)) and spec.layers[1].feed_forward.params["shared_ff"] is None


def test_readers_of_latent_rows_own_no_cache():
    model = Decoder(spec_of(config("wide")), torch.float32, "meta")
    layout = model.cache_layout()
    assert sorted(layout.kv) == [0, 2, 3, 5, 6]
    assert (layout.kv[0].head_dim, layout.kv[0].window) == (80, None) and layout.kv[2].window == 70
    assert model.layers[1].mixer.shares_kv and model.layers[1].mixer.kv_spec() is None
    assert model.layers[4].mixer.reads_kv_spec() == layout.kv[0] and model.layers[7].mixer.reads_kv_spec() == layout.kv[6]


@pytest.mark.parametrize("change,text", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=40), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][1]["mixer"].update(heads=5), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=23), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c.pop("norm"), "eps"),
])
def test_refusals_name_the_key(change, text):
    cfg = config("small")
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        load_config(cfg)


@pytest.mark.parametrize("rot", [CONFIGS["small"]["layers"][0]["mixer"]["rot"], CONFIGS["wide"]["layers"][0]["mixer"]["rot"],
                                 {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
                                 {"base": 10.0, "dims": 4, "scaling": {"factor": 3.0, "original": 10, "fast": 1e6, "slow": 1e-6}},
                                 {"base": 500.0, "dims": 8, "scaling": {"factor": 2.0, "original": 100, "fast": 3.0, "slow": 3.0}}])
def test_frequency_table(rot):
    sc = rot["scaling"]
    ours = {"rope_type": "yarn", "factor": sc["factor"], "original_max_position_embeddings": sc["original"], "beta_fast": sc["fast"],
            "beta_slow": sc["slow"]}
    got = torch.tensor(inverse_frequencies(rot["dims"], rot["base"], ours), dtype=P.F64)
    assert torch.allclose(got, P.rotary_frequencies(rot), rtol=1e-12)
    assert abs(rotation_gain(ours) - P.rotary_gain(rot)) < 1e-12 and rotation_gain(None) == 1.0
    assert rotation_gain({"rope_type": "linear", "factor": 2.0}) == 1.0


def test_a_factor_on_the_rotation_is_refused_where_no_kernel_applies_it():
    from gguf_rs_cli_b200.config import PartSpec
    from gguf_rs_cli_b200.parts import MIXERS, POSITIONS
    pos = POSITIONS.get("rope")(PartSpec("rope", dict(head_dim=8, rotary_dim=8, theta=10.0, pairing="half", scaling={
        "rope_type": "yarn", "factor": 2.0, "original_max_position_embeddings": 64})), torch.float32, "cpu")
    with pytest.raises(ValueError, match="factor"):
        MIXERS.get("attention")(PartSpec("attention", dict(hidden_size=8, num_heads=1, num_kv_heads=1, head_dim=8)), torch.float32, "cpu", position=pos)


# ------------------------------------------------------------ the plain implementation
def test_window_bias_and_slopes():
    assert P.visible(6, 3)[4].tolist() == [False, False, True, True, True, False] and P.visible(4, None).tolist() == torch.ones(4, 4).tril().bool().tolist()
    assert P.head_slopes(4) == [0.25, 0.0625, 0.015625, 0.00390625] and P.head_slopes(3)[0] == 2.0 ** (-8.0 / 3.0)
    # equal scores: the weights are a geometric sequence of the distance
    T, s = 5, 0.5
    q, k = torch.zeros(T, 1, 2, dtype=P.F64), torch.zeros(T, 1, 2, dtype=P.F64)
    v = torch.eye(T, dtype=P.F64)[:, None, :]
    o = P.softmax_attention(q, k, v, 1.0, P.visible(T, 3), [s])[:, 0]
    e = [math.exp(-s * d) for d in range(3)]
    assert torch.allclose(o[4], torch.tensor([0.0, 0.0, e[2], e[1], e[0]], dtype=P.F64) / sum(e))


def test_query_temperature_steps_at_its_period():
    t = P.query_temperature(torch.arange(12), {"coef": 0.5, "every": 4})
    assert t[:3].tolist() == [1.0] * 3 and torch.allclose(t[3:7], torch.full((4,), 1 + 0.5 * math.log(2.0), dtype=P.F64))
    assert abs(float(t[11]) - (1 + 0.5 * math.log(4.0))) < 1e-12


def test_rotation_carries_its_gain_and_the_ramp_its_ends():
    rot = {"base": 100.0, "dims": 4, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}}
    x = torch.arange(12, dtype=P.F64).view(1, 2, 6)
    y, f, g = P.rotate(x, torch.tensor([3]), rot), P.rotary_frequencies(rot), 0.1 * math.log(4.0) + 1.0
    for h in range(2):
        for i in range(2):
            u, v, a = float(x[0, h, i]), float(x[0, h, i + 2]), 3 * float(f[i])
            assert abs(float(y[0, h, i]) - g * (u * math.cos(a) - v * math.sin(a))) < 1e-12
            assert abs(float(y[0, h, i + 2]) - g * (v * math.cos(a) + u * math.sin(a))) < 1e-12
        assert y[0, h, 4:].tolist() == x[0, h, 4:].tolist()
    ramp = P.yarn_ramp(64, 10000.0, 4096.0, 32.0, 1.0)
    lo, hi = math.floor(64 * math.log(4096 / (64 * math.pi)) / (2 * math.log(1e4))), math.ceil(64 * math.log(4096 / (2 * math.pi)) / (2 * math.log(1e4)))
    assert ramp[lo] == 0.0 and ramp[lo + 1] > 0.0 and ramp[hi - 1] < 1.0 and ramp[hi] == 1.0


def test_layer_norm_takes_the_mean_off_and_the_route_weighs_the_chosen_only():
    x = torch.tensor([[1.0, 2.0, 3.0, 6.0]], dtype=P.F64)
    assert torch.allclose(P.layer_norm(x, torch.ones(4, dtype=P.F64), 0.5), (x - 3.0) / math.sqrt(3.5 + 0.5))
    W = {"m.router": torch.tensor([[2.0], [1.0], [5.0]], dtype=P.F64)}
    ids, w = P.route({"router": {"experts": 3, "top": 2}}, W, "m.", torch.ones(1, 1, dtype=P.F64))
    assert ids.tolist() == [[2, 0]] and abs(float(w[0, 0]) - 1 / (1 + math.exp(-3.0))) < 1e-12


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

    L = lambda c, i: c["layers"][i]["mixer"]                                    # noqa: E731
    for what, change in {
            "window": lambda c: L(c, 1)["mask"].update(size=14), "other window": lambda c: L(c, 5)["mask"].update(size=28),
            "temperature": lambda c: L(c, 1).pop("q_temp"), "temperature of every position": lambda c: L(c, 5).pop("q_temp"),
            "period of the temperature": lambda c: L(c, 1)["q_temp"].update(every=8), "alpha": lambda c: c.update(postln_alpha=1.6),
            "embedding scale": lambda c: c["embedding"].update(scale=1.3), "frequency scaling": lambda c: L(c, 0)["rot"].pop("scaling"),
            "ramp": lambda c: L(c, 0)["rot"]["scaling"].update(fast=6.0), "rotation": lambda c: L(c, 4)["rot"].update(base=20.0),
            "score scale": lambda c: L(c, 2).update(scale=0.33), "a feed-forward left out": lambda c: c["layers"][2].update(mlp=None),
            "shared expert": lambda c: c["layers"][1]["mlp"].pop("shared")}.items():
        assert moved(change) > 0.01, what
    for key in ("l1.mix.q.b", "l1.mix.k.b", "l1.mix.o.b", "l1.mix.q.norm", "l1.mix.k.norm", "l3.mix.g", "l0.mix.g", "l2.mix.dq.norm",
                "l0.mix.dkv.norm", "l2.norm1", "l2.norm2", "l4.mlp.router"):
        w2 = dict(w)
        w2[key] = w[key] + 2.0 * torch.linspace(-1.0, 1.0, w[key].numel(), dtype=P.F64).view(w[key].shape)
        assert moved(w2=w2) > 0.005, key
    assert float((P.forward(all_chosen(cfg), w, toks) - base).abs().max()) / top > 0.01, "the router's choice"
    # a reader that made latent rows of its own would give something else
    c = copy.deepcopy(cfg)
    del c["layers"][2]["mixer"]["kv_from"]
    own = as_plain(make_weights(c, seed=5))
    w2 = {**w, "l2.mix.dkv": own["l2.mix.dkv"], "l2.mix.dkv.norm": own["l2.mix.dkv.norm"]}
    assert float((P.forward(c, w2, toks) - base).abs().max()) / top > 0.01, "shared latent rows"
