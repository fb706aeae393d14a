"""Small Betirax configurations with weights of the tests' own making, as the plain implementation's dict and as an
engine of the package.

The configurations differ from each other in every size and constant and avoid coincidences that would hide a fault:
heads and key/value heads differ, layers that read another layer's latent rows have heads and sizes of their own, windows
shorter than a page and longer, a layer without a mask and without a temperature, layers without a feed-forward, mixtures
with and without a shared expert, frequency scalings whose ramp lies within the table and none at all, factors of x and of
the embedding that are not 1.  Scales are chosen so that attention is peaked.
"""
import copy
import functools

import torch


def _moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _rot(base, dims, *scaling):
    return {"base": base, "dims": dims, **({"scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))} if scaling else {})}


SMALL_ROT = _rot(50.0, 12, 4.0, 64, 4.0, 1.0)

SMALL = {
    "architecture": "Betirax", "vocab": 197, "width": 72, "norm": {"eps": 1e-5}, "postln_alpha": 1.7, "embedding": {"scale": 1.4},
    "layers": [
        {"type": "latent_attention", "mlp": _dense(50),
         "mixer": {"heads": 3, "dim": 20, "rot_dim": 12, "vdim": 28, "kv_rank": 36, "q_rank": 30, "scale": 0.25, "rot": SMALL_ROT}},
        {"type": "attention", "mlp": _moe(5, 3, 28, 20),
         "mixer": {"heads": 6, "kv_heads": 3, "dim": 24, "vdim": 24, "scale": 0.4, "mask": {"size": 13}, "q_temp": {"coef": 0.4, "every": 7}}},
        {"type": "latent_attention", "mlp": _moe(4, 2, 16),
         "mixer": {"heads": 5, "dim": 16, "rot_dim": 12, "vdim": 12, "kv_rank": 36, "q_rank": 17, "scale": 0.3, "kv_from": 0, "rot": SMALL_ROT}},
        {"type": "attention", "mlp": None, "mixer": {"heads": 2, "dim": 40, "vdim": 40, "scale": 0.3}},
        {"type": "latent_attention", "mlp": _moe(6, 1, 24, 12),
         "mixer": {"heads": 2, "dim": 10, "rot_dim": 6, "vdim": 18, "kv_rank": 44, "q_rank": 80, "scale": 0.35, "rot": _rot(1000.0, 6)}},
        {"type": "attention", "mlp": _dense(33),
         "mixer": {"heads": 3, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.5, "mask": {"size": 29}, "q_temp": {"coef": -0.1, "every": 1}}},
    ],
}

# Sizes that reach the tensor-core products (multiples of 8), the tiled attention kernel of prompts and the decode kernel
# of single tokens (keys and values of 64 and of 128 entries), the tiled path of latent attention (dim + rot_dim = vdim =
# 64 or 128; a reader on it whose rows come from a layer that is not, and the other way round), both decode kernels of
# latent attention, and the experts' tiles.
WIDE_ROT, WIDE_ROT2 = _rot(5000.0, 16, 2.5, 128, 16.0, 0.5), _rot(100.0, 16)

WIDE = {
    "architecture": "Betirax", "vocab": 520, "width": 256, "norm": {"eps": 1e-6}, "postln_alpha": 2.2, "embedding": {"scale": 0.6},
    "layers": [
        {"type": "latent_attention", "mlp": _dense(192),
         "mixer": {"heads": 4, "dim": 48, "rot_dim": 16, "vdim": 64, "kv_rank": 64, "q_rank": 96, "scale": 0.2, "rot": WIDE_ROT}},
        {"type": "latent_attention", "mlp": _moe(8, 3, 48, 80),
         "mixer": {"heads": 2, "dim": 112, "rot_dim": 16, "vdim": 128, "kv_rank": 64, "q_rank": 160, "scale": 0.12, "kv_from": 0, "rot": WIDE_ROT}},
        {"type": "attention", "mlp": _moe(6, 2, 72),
         "mixer": {"heads": 4, "kv_heads": 2, "dim": 64, "vdim": 64, "scale": 0.25, "mask": {"size": 70}, "q_temp": {"coef": 0.3, "every": 50}}},
        {"type": "attention", "mlp": _dense(136),
         "mixer": {"heads": 2, "kv_heads": 2, "dim": 128, "vdim": 128, "scale": 0.15, "mask": {"size": 96}}},
        {"type": "latent_attention", "mlp": _moe(4, 2, 56, 64),
         "mixer": {"heads": 3, "dim": 24, "rot_dim": 16, "vdim": 40, "kv_rank": 64, "q_rank": 64, "scale": 0.25, "kv_from": 0, "rot": WIDE_ROT}},
        {"type": "attention", "mlp": None, "mixer": {"heads": 4, "kv_heads": 1, "dim": 64, "vdim": 64, "scale": 0.2}},
        {"type": "latent_attention", "mlp": None,
         "mixer": {"heads": 2, "dim": 20, "rot_dim": 16, "vdim": 28, "kv_rank": 120, "q_rank": 72, "scale": 0.3, "rot": WIDE_ROT2}},
        {"type": "latent_attention", "mlp": _dense(72),
         "mixer": {"heads": 3, "dim": 48, "rot_dim": 16, "vdim": 64, "kv_rank": 120, "q_rank": 40, "scale": 0.2, "kv_from": 6, "rot": WIDE_ROT2}},
    ],
}

CONFIGS = {"small": SMALL, "wide": WIDE}


def config(name):
    return copy.deepcopy(CONFIGS[name])


def all_chosen(cfg):
    """The same model with every expert chosen for every token: no choice is left that a rounding could turn, so runs in
    bfloat16 can be compared row by row.  The weights of the original fit."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer.get("mlp") and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg


def make_weights(cfg, seed=0, gain=1.0):
    """name -> float32 tensor holding bfloat16 values.  Projections N(0, gain^2/in), so that rows stay of order one."""
    g = torch.Generator().manual_seed(seed)
    E, V, w = cfg["width"], cfg["vocab"], {}

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain / i ** 0.5

    def near_one(n):
        return 1.0 + 0.2 * torch.randn(n, generator=g)

    w["embed"] = torch.randn(V, E, generator=g) * 0.7
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        H, D = m["heads"], m["dim"]
        w[f"l{i}.norm1"] = near_one(E)
        if layer["type"] == "attention":
            G = m.get("kv_heads") or H
            w[p + "q"], w[p + "k"], w[p + "g"], w[p + "o"] = mat(H * D, E, gain), mat(G * D, E, gain), mat(H * D, E, 2.0), mat(E, H * D, 2.0)
            for n, rows in (("q.b", H * D), ("k.b", G * D), ("o.b", E)):
                w[p + n] = 0.3 * torch.randn(rows, generator=g)
            w[p + "q.norm"], w[p + "k.norm"] = near_one(D), near_one(D)
        else:
            R, Dv, C, Q = m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            w[p + "dq"], w[p + "dq.norm"], w[p + "uq"] = mat(Q, E, gain), near_one(Q), mat(H * (D + R), Q, gain)
            if m.get("kv_from") is None:
                w[p + "dkv"], w[p + "dkv.norm"] = mat(C + R, E, gain), near_one(C)
            w[p + "uk"], w[p + "uv"] = mat(H * D, C, gain), mat(H * Dv, C, gain)
            w[p + "g"], w[p + "o"] = mat(H * Dv, E, 2.0), mat(E, H * Dv, 2.0)
        mlp = layer.get("mlp")
        if not mlp:
            continue
        q = f"l{i}.mlp."
        w[f"l{i}.norm2"] = near_one(E)
        if mlp["kind"] == "dense":
            w[q + "up"], w[q + "down"] = mat(mlp["ff"], E, 1.5), mat(E, mlp["ff"], 1.5)
            continue
        for e in range(mlp["router"]["experts"]):
            F = mlp["expert"]["ff"]
            w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = mat(F, E, 1.5), mat(F, E, 1.5), mat(E, F, 1.5)
        w[q + "router"] = mat(mlp["router"]["experts"], E, 1.5)
        if mlp.get("shared"):
            Fs = mlp["shared"]["ff"]
            w[q + "shared.gate"], w[q + "shared.up"], w[q + "shared.down"] = mat(Fs, E, 1.5), mat(Fs, E, 1.5), mat(E, Fs)
    w["final.norm"] = near_one(E)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in w.items()}


@functools.lru_cache(maxsize=None)
def weights(name, seed=0):
    return make_weights(CONFIGS[name], seed)


def as_plain(w):
    """The weights as the plain implementation takes them (float64)."""
    return {k: v.double() for k, v in w.items()}


def build(cfg, w, dtype):
    from gguf_rs_cli_b200.api import _build
    from gguf_rs_cli_b200.weights import TensorSource
    return _build(copy.deepcopy(cfg), TensorSource(tensors={k: v.to(torch.bfloat16) for k, v in w.items()}, where="test weights"),
                  dtype, "cuda:0")


@functools.lru_cache(maxsize=None)
def llm(name, dtype, dense=False, seed=0):
    cfg = all_chosen(CONFIGS[name]) if dense else CONFIGS[name]
    return build(cfg, weights(name, seed), dtype)


def new_engine(name, dtype, dense=False, n_tokens=2048, n_slots=8, **kw):
    from gguf_rs_cli_b200.engine.step import Engine
    return Engine(llm(name, dtype, dense).model, n_tokens=n_tokens, n_slots=n_slots, **kw)


def tokens_of(name, n, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist()


@functools.lru_cache(maxsize=None)
def plain_logits(name, n, seed, dense=False):
    from tests import plain_betirax as P
    cfg = all_chosen(CONFIGS[name]) if dense else CONFIGS[name]
    return P.forward(cfg, as_plain(weights(name)), tokens_of(name, n, seed)).float()
