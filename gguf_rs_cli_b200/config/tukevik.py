"""Typed configuration of the Tukevik design and its description as parts.

A Tukevik model is a list of pre-norm layers (RMS norms with plain weights) whose sublayers' results enter the residual
stream times one constant.  A layer's mixer is `rglru` (a recurrent block around a real-gated linear recurrent unit,
with a short convolution and gates from block-diagonal matrices) or `parallel` (chunked grouped-query attention without a
rotation, on heads of unit root mean square, with q/k/v biases, a softcap on the scores, a sink of score 0 and a gate per
head; beside it retention with a fixed decay per head and a rotation of q and k; a constant times each).  The feed-forward
is dense, a mixture of experts (biased router, softmax over the chosen logits, a gated shared expert), or absent; the head
is the embedding table.  config.json gives every size and every constant.  The reference knows one architecture only
(src/model/config.rs:20-47) and has none of these parts.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .debonex import NO_POSITION_LIMIT, _factor, _get
from .registry import ConfigError, register_architecture
from .specs import LayerSpec, ModelSpec, PartSpec, Run

MIXER_TYPES = ("rglru", "parallel")


@dataclass(frozen=True)
class TukevikLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]            # None: the layer has no feed-forward


@dataclass(frozen=True)
class TukevikConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float                     # what every sublayer's result is multiplied by on its way into the stream
    layers: List[TukevikLayer] = field(default_factory=list)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "TukevikConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        out = []
        for i, entry in enumerate(layers):
            where = f"layers[{i}]"
            kind = entry.get("type") if isinstance(entry, dict) else None
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not one of {list(MIXER_TYPES)}")
            read = _read_rglru if kind == "rglru" else _read_parallel
            out.append(TukevikLayer(kind, read(_object(entry, "mixer", where), where + ".mixer"),
                                    _read_mlp(entry.get("mlp"), where + ".mlp")))
        return cls(vocab=_get(raw, "vocab", "the top level"), width=_get(raw, "width", "the top level"),
                   norm_eps=_get(raw.get("norm"), "eps", "'norm'", float), residual_mult=_factor(raw, "residual_mult", "the top level"),
                   layers=out)


def _object(raw, key: str, where: str) -> Dict[str, Any]:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _read_rglru(raw, where: str) -> Dict[str, Any]:
    m = {k: _get(raw, k, where) for k in ("width", "blocks", "conv")}
    if m["width"] % m["blocks"]:
        raise ConfigError(f"config.json: {where}: width {m['width']} is not a multiple of blocks {m['blocks']}")
    if m["conv"] > 16:
        raise ConfigError(f"config.json: {where}.conv {m['conv']}: at most 16 taps are supported")
    return m


def _read_parallel(raw, where: str) -> Dict[str, Any]:
    return {"left": _read_attention(_object(raw, "left", where), where + ".left"),
            "right": _read_retention(_object(raw, "right", where), where + ".right"),
            "left_scale": _factor(raw, "left_scale", where), "right_scale": _factor(raw, "right_scale", where)}


def _read_attention(raw, where: str) -> Dict[str, Any]:
    m = {k: _get(raw, k, where) for k in ("heads", "dim")}
    m["vdim"] = _get(raw, "vdim", where) if raw.get("vdim") is not None else m["dim"]
    m["kv_heads"] = _get(raw, "kv_heads", where) if raw.get("kv_heads") is not None else m["heads"]
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"config.json: {where}: heads {m['heads']} is not a multiple of kv_heads {m['kv_heads']}")
    m["scale"] = _get(raw, "scale", where, float) if raw.get("scale") is not None else m["dim"] ** -0.5
    m["softcap"] = _get(raw, "softcap", where, float) if raw.get("softcap") is not None else None
    m["chunk"] = None if raw.get("mask") is None else _get(raw["mask"], "size", where + ".mask")
    return m


def _read_retention(raw, where: str) -> Dict[str, Any]:
    m = {k: _get(raw, k, where) for k in ("heads", "dim")}
    m["vdim"] = _get(raw, "vdim", where) if raw.get("vdim") is not None else m["dim"]
    decay = raw.get("decay")
    if not isinstance(decay, list) or len(decay) != m["heads"] or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
        raise ConfigError(f"config.json: {where}.decay must be a list of {m['heads']} numbers, one per head")
    m["decay"] = [float(d) for d in decay]
    rot, at = raw.get("rot"), where + ".rot"
    m["rot"] = None
    if rot is not None and rot.get("dims") != 0:          # no entries to rotate: no rotation
        m["rot"] = {"base": _get(rot, "base", at, float), "dims": _get(rot, "dims", at)}
        if m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["dim"]:
            raise ConfigError(f"config.json: {at}.dims {m['rot']['dims']} must be even and at most dim {m['dim']}")
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


def _attention(E: int, eps: float, m, p: str) -> PartSpec:
    tensors = {n: p + n for n in ("q", "k", "v", "g", "o")}
    tensors.update({n + "_bias": p + n + ".b" for n in ("q", "k", "v")})
    return PartSpec("attention", dict(hidden_size=E, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                      v_head_dim=m["vdim"], scale=m["scale"], chunk=m["chunk"], bias=("q", "k", "v"), qk_norm_eps=eps,
                                      softcap=m["softcap"], sink=True, out_gate="head", exact=True), tensors)


def _mixer(E: int, eps: float, layer: TukevikLayer, p: str):
    """(the mixer's description, its position encoding's or None)"""
    m = layer.mixer
    if layer.type == "rglru":
        names = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "ra": "ra",
                 "ra_bias": "ra.b", "ri": "ri", "ri_bias": "ri.b", "lam": "lam", "o": "o"}
        return PartSpec("rglru", dict(hidden_size=E, width=m["width"], blocks=m["blocks"], conv=m["conv"]),
                        {k: p + v for k, v in names.items()}), None
    r, q = m["right"], p + "right."
    right = PartSpec("retention", dict(hidden_size=E, heads=r["heads"], dim=r["dim"], vdim=r["vdim"], decay=r["decay"], eps=eps),
                     {n: q + n for n in ("q", "k", "v", "g", "o")})
    position = None if r["rot"] is None else PartSpec("rope", dict(head_dim=r["dim"], rotary_dim=r["rot"]["dims"], theta=r["rot"]["base"],
                                                                   pairing="half", scaling=None))
    return PartSpec("weighted_pair", dict(hidden_size=E, left=_attention(E, eps, m["left"], p + "left."), right=right,
                                          left_scale=m["left_scale"], right_scale=m["right_scale"], position_of="right")), position


def build_tukevik_spec(cfg: TukevikConfig) -> ModelSpec:
    E, layers = cfg.width, []

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", dict(size=E, eps=cfg.norm_eps), {"weight": name})

    for i, layer in enumerate(cfg.layers):
        mixer, position = _mixer(E, cfg.norm_eps, layer, f"l{i}.mix.")
        norms, ff = {"mixer": norm(f"l{i}.norm1")}, None
        if layer.mlp is not None:
            mlp, q = layer.mlp, f"l{i}.mlp."
            norms["feed_forward"] = norm(f"l{i}.norm2")
            if mlp["kind"] == "dense":
                ff = PartSpec("gated_mlp", dict(hidden_size=E, intermediate_size=mlp["ff"], activation="silu", term_f32=True),
                              {n: q + n for n in ("gate", "up", "down")})
            else:
                # softmax scores over the chosen experts' sum are the softmax of the chosen logits
                tensors = {"router": q + "router", "router_bias": q + "router.b", "experts": q + "e", "shared": q + "shared",
                           "shared_gate": q + "shared.sg"}
                ff = PartSpec("moe", dict(hidden_size=E, experts=mlp["experts"], top=mlp["top"], groups=1, keep=1, scale=1.0,
                                          expert_ff=mlp["ff"], limit=None, shared_ff=mlp["shared"], shared_limit=None, score="softmax",
                                          router_bias=True, shared_gate=mlp["shared"] is not None), tensors)
        layers.append(LayerSpec(block="prenorm", mixer=mixer, feed_forward=ff, norms=norms, position=position,
                                block_params={"scale": cfg.residual_mult, "unsummed": True}))
    spec = ModelSpec(
        architecture="Tukevik", vocab_size=cfg.vocab, hidden_size=E,
        embedding=PartSpec("embedding", dict(vocab_size=cfg.vocab, hidden_size=E), {"weight": "embed"}),
        layers=layers, schedule=[Run(i) for i in range(len(layers))], final_norm=norm("final.norm"),
        head=PartSpec("lm_head", dict(vocab_size=cfg.vocab, hidden_size=E, tied_to=None, tied=True), {"weight": "embed"}),
        max_position=NO_POSITION_LIMIT)
    spec.validate()
    return spec


register_architecture("Tukevik", TukevikConfig, build_tukevik_spec, "tukevik")
