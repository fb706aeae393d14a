"""Typed configuration of the Betirax design and its description as parts.

A Betirax model is a list of layers that norm the sum of what a sublayer reads and what it gives:
x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x)), all layer norms with a weight and no bias, alpha one constant
of the model.  A layer's mixer is `attention` (grouped-query attention without a rotation: q, k and output biases, an RMS
norm per head on q and k, values that are the keys as projected, a query temperature that grows with the position, a bias
that grows with the distance, a sliding window, a gate per entry) or `latent_attention` (queries through a latent of their
own, keys and values from one cached latent row per position plus one shared key part, rotated with YaRN's frequencies; a
gate per entry; a layer may read an earlier layer's latent rows instead of making its own).  The feed-forward is dense
(GELU's tanh form, no gate), a mixture of SiLU-gated experts weighed by the softmax of the chosen logits, with a shared
expert, or absent.  The embedding carries a constant factor; the logits are products with the embedding table itself.
config.json gives every size and every constant.  The reference knows one architecture only (src/model/config.rs:20-47)
and has none of these parts.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .debonex import NO_POSITION_LIMIT, _factor, _get
from .registry import ConfigError, register_architecture
from .specs import LayerSpec, ModelSpec, PartSpec, Run

MIXER_TYPES = ("attention", "latent_attention")
# head h of H loses 2^(-DISTANCE_EXPONENT (h+1) / H) times the distance from its scores
DISTANCE_EXPONENT = 8.0


@dataclass(frozen=True)
class BetiraxLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]            # None: the layer has no feed-forward


@dataclass(frozen=True)
class BetiraxConfig:
    vocab: int
    width: int
    norm_eps: float
    alpha: float                              # factor of x in every normed sum
    embedding_scale: float
    layers: List[BetiraxLayer] = field(default_factory=list)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "BetiraxConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        out = []
        for i, entry in enumerate(layers):
            where = f"layers[{i}]"
            kind = entry.get("type") if isinstance(entry, dict) else None
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not one of {list(MIXER_TYPES)}")
            read = _read_attention if kind == "attention" else _read_latent
            out.append(BetiraxLayer(kind, read(entry.get("mixer"), where + ".mixer"), _read_mlp(entry.get("mlp"), where + ".mlp")))
        for i, layer in enumerate(out):
            src = layer.mixer.get("kv_from")
            if src is None:
                continue
            where = f"layers[{i}].mixer.kv_from"
            if not 0 <= src < i or out[src].type != "latent_attention" or out[src].mixer["kv_from"] is not None:
                raise ConfigError(f"config.json: {where} = {src} must name an earlier latent_attention layer with latent rows of its own")
            if any(layer.mixer[k] != out[src].mixer[k] for k in ("kv_rank", "rot_dim", "rot")):
                raise ConfigError(f"config.json: {where}: layer {src} has another kv_rank, rot_dim or rotation than layer {i}")
        return cls(vocab=_get(raw, "vocab", "the top level"), width=_get(raw, "width", "the top level"),
                   norm_eps=_get(raw.get("norm"), "eps", "'norm'", float), alpha=_factor(raw, "postln_alpha", "the top level"),
                   embedding_scale=_factor(raw.get("embedding"), "scale", "'embedding'"), layers=out)


def _read_attention(raw, where: str) -> Dict[str, Any]:
    if not isinstance(raw, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    m = {k: _get(raw, k, where) for k in ("heads", "dim")}
    m["kv_heads"] = _get(raw, "kv_heads", where) if raw.get("kv_heads") is not None else m["heads"]
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}: heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
    if raw.get("vdim") is not None and _get(raw, "vdim", where) != m["dim"]:
        raise ConfigError(f"config.json: {where}.vdim {raw['vdim']} must equal dim {m['dim']}: the values are the keys")
    m["scale"] = _get(raw, "scale", where, float) if raw.get("scale") is not None else m["dim"] ** -0.5
    m["mask"] = None if raw.get("mask") is None else {"size": _get(raw["mask"], "size", where + ".mask")}
    m["q_temp"] = None
    if raw.get("q_temp") is not None:
        m["q_temp"] = {"coef": _get(raw["q_temp"], "coef", where + ".q_temp", float, positive=False),
                       "every": _get(raw["q_temp"], "every", where + ".q_temp")}
    return m


def _read_latent(raw, where: str) -> Dict[str, Any]:
    if not isinstance(raw, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    m = {k: _get(raw, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")}
    m["scale"] = _get(raw, "scale", where, float) if raw.get("scale") is not None else (m["dim"] + m["rot_dim"]) ** -0.5
    m["kv_from"] = None if raw.get("kv_from") is None else _get(raw, "kv_from", where, positive=False)
    if m["rot_dim"] % 2:
        raise ConfigError(f"config.json: {where}.rot_dim {m['rot_dim']} must be even")
    rot, at = raw.get("rot"), where + ".rot"
    m["rot"] = {"base": _get(rot, "base", at, float), "dims": _get(rot, "dims", at), "scaling": None}
    if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["rot_dim"]:
        raise ConfigError(f"config.json: {at}.dims {m['rot']['dims']} must be even and at most rot_dim {m['rot_dim']}")
    if rot.get("scaling") is not None:
        m["rot"]["scaling"] = {k: _get(rot["scaling"], k, at + ".scaling", float) for k in ("factor", "original", "fast", "slow")}
    return m


def _read_mlp(raw, where: str) -> Optional[Dict[str, Any]]:
    if raw is None:
        return None
    kind = raw.get("kind") if isinstance(raw, dict) else raw
    if kind == "dense":
        return {"kind": "dense", "ff": _get(raw, "ff", where)}
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not supported (dense, moe)")
    m = {"kind": "moe", "experts": _get(raw.get("router"), "experts", where + ".router"),
         "top": _get(raw.get("router"), "top", where + ".router"), "ff": _get(raw.get("expert"), "ff", where + ".expert"),
         "shared": None if raw.get("shared") is None else _get(raw["shared"], "ff", where + ".shared")}
    if m["top"] > m["experts"]:
        raise ConfigError(f"config.json: {where}.router: top {m['top']} of {m['experts']} experts")
    return m


def _rope(m) -> PartSpec:
    sc = m["rot"]["scaling"]
    scaling = None if sc is None else {"rope_type": "yarn", "factor": sc["factor"], "original_max_position_embeddings": sc["original"],
                                       "beta_fast": sc["fast"], "beta_slow": sc["slow"]}
    return PartSpec("rope", dict(head_dim=m["rot_dim"], rotary_dim=m["rot"]["dims"], theta=m["rot"]["base"], pairing="half",
                                 scaling=scaling))


def build_betirax_spec(cfg: BetiraxConfig) -> ModelSpec:
    E, layers, schedule = cfg.width, [], []

    def norm(name: str) -> PartSpec:
        return PartSpec("layernorm", dict(size=E, eps=cfg.norm_eps), {"weight": name})

    for i, layer in enumerate(cfg.layers):
        p, m, position = f"l{i}.mix.", layer.mixer, None
        if layer.type == "attention":
            mixer = PartSpec("attention", dict(hidden_size=E, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                               scale=m["scale"], window=(m["mask"] or {}).get("size"), bias=("q", "k", "o"),
                                               values="keys", head_norm_eps=cfg.norm_eps, q_temp=m["q_temp"],
                                               distance_bias=DISTANCE_EXPONENT, out_gate=True),
                             {"q": p + "q", "q_bias": p + "q.b", "k": p + "k", "k_bias": p + "k.b", "q_norm": p + "q.norm",
                              "k_norm": p + "k.norm", "g": p + "g", "o": p + "o", "o_bias": p + "o.b"})
        else:
            position = _rope(m)
            shares = m["kv_from"] is not None
            names = {"dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "uk": "uk", "uv": "uv", "g": "g", "o": "o"}
            if not shares:
                names.update(dkv="dkv", dkv_norm="dkv.norm")
            mixer = PartSpec("latent_attention", dict(hidden_size=E, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"],
                                                      vdim=m["vdim"], kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=m["scale"],
                                                      eps=cfg.norm_eps, out_gate=True, shares_kv=shares, term_f32=True),
                             {k: p + v for k, v in names.items()})
        norms, ff = {"mixer": norm(f"l{i}.norm1")}, None
        if layer.mlp is not None:
            mlp, q = layer.mlp, f"l{i}.mlp."
            norms["feed_forward"] = norm(f"l{i}.norm2")
            if mlp["kind"] == "dense":
                ff = PartSpec("mlp", dict(hidden_size=E, intermediate_size=mlp["ff"], activation="gelu_tanh"),
                              {"up": q + "up", "down": q + "down"})
            else:
                # softmax scores over the chosen experts' sum are the softmax of the chosen logits
                ff = PartSpec("moe", dict(hidden_size=E, experts=mlp["experts"], top=mlp["top"], groups=1, keep=1, scale=1.0,
                                          expert_ff=mlp["ff"], limit=None, shared_ff=mlp["shared"], shared_limit=None, score="softmax"),
                              {"router": q + "router", "experts": q + "e", "shared": q + "shared"})
        layers.append(LayerSpec(block="postnorm", mixer=mixer, feed_forward=ff, norms=norms, position=position,
                                block_params={"alpha": cfg.alpha}))
        schedule.append(Run(i, cache_of=m.get("kv_from")))
    spec = ModelSpec(
        architecture="Betirax", vocab_size=cfg.vocab, hidden_size=E,
        embedding=PartSpec("embedding", dict(vocab_size=cfg.vocab, hidden_size=E, scale=cfg.embedding_scale), {"weight": "embed"}),
        layers=layers, schedule=schedule, final_norm=norm("final.norm"),
        head=PartSpec("lm_head", dict(vocab_size=cfg.vocab, hidden_size=E, tied_to=None, tied=True), {"weight": "embed"}),
        max_position=NO_POSITION_LIMIT)
    spec.validate()
    return spec


register_architecture("Betirax", BetiraxConfig, build_betirax_spec, "betirax")
