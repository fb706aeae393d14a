"""Small Tukevik configurations with weights of the tests' own making, as the plain implementation's dict and as an
engine of the package.

The configurations differ from each other in every size and constant and avoid coincidences that would hide a fault: heads
and key/value heads differ, keys and values differ in size, the two branches of a parallel layer have heads, sizes and
factors of their own, chunks shorter than a page and longer, a layer without a mask, without a softcap and without a
rotation, rotations of a part of the heads, layers without a feed-forward, mixtures with and without a shared expert, a
convolution of one tap.  Scales are chosen so that attention is peaked, softcaps bite, and decays reach from short to long
memories.
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


def _unit(width, blocks, conv, mlp):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def _pair(left, right, scales, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def _left(heads, kv_heads, dim, vdim, scale, softcap=None, chunk=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        m["softcap"] = softcap
    if chunk:
        m["mask"] = {"size": chunk}
    return m


def _right(decay, dim, vdim, base=None, dims=None):
    m = {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
    return m


SMALL = {
    "architecture": "Tukevik", "vocab": 203, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
    "layers": [
        _unit(60, 3, 4, _dense(50)),
        _pair(_left(6, 3, 20, 28, 0.3, 4.0, 13), _right([0.5, 0.96875, 0.998046875], 12, 18, 100.0, 8), (0.7, 1.3), _moe(5, 3, 28, 20)),
        _unit(88, 1, 2, _moe(4, 2, 16)),
        _pair(_left(2, 2, 24, 24, 0.25), _right([0.9], 10, 6), (1.1, -0.6), None),
        _unit(72, 6, 1, _moe(6, 1, 24, 12)),
        _pair(_left(3, 1, 18, 10, 0.4, 9.0, 100), _right([0.875, 0.75], 16, 16, 5000.0, 16), (0.9, 0.8), _dense(33)),
    ],
}

# Sizes that reach the tensor-core products (multiples of 8), the tiled attention kernel of prompts (heads of 64, 96 and 128)
# and the decode kernel of single tokens, the chunked retention (heads of 32, 64, 96 and 128), the fused recurrence with
# blocks below and above its slice of channels, and the experts' tiles.
WIDE = {
    "architecture": "Tukevik", "vocab": 520, "width": 256, "norm": {"eps": 1e-6}, "residual_mult": 0.8,
    "layers": [
        _pair(_left(4, 2, 64, 64, 0.15, 6.0, 70), _right([0.96875, 0.9990234375, 0.8], 64, 64, 10000.0, 64), (0.8, 0.9), _dense(192)),
        _unit(224, 4, 4, _moe(8, 3, 48, 80)),
        _pair(_left(4, 1, 96, 96, 0.1, 20.0, 96), _right([0.984375, 0.5], 128, 128, 500.0, 96), (1.2, 0.7), _moe(6, 2, 72)),
        _unit(288, 2, 3, _dense(136)),
        _pair(_left(2, 2, 128, 128, 0.09, 3.0), _right([0.9375, 0.998, 1.0, 0.7], 32, 32, 1000.0, 20), (0.5, 1.0), _moe(4, 2, 56, 64)),
        _unit(160, 1, 4, None),
        _pair(_left(4, 4, 32, 48, 0.2, 5.0, 33), _right([0.99], 96, 96), (0.9, 1.1), _dense(72)),
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


def make_weights(cfg, seed=0):
    """name -> float32 tensor holding bfloat16 values.  Projections N(0, gain^2/in), so that rows stay of order one."""
    g = torch.Generator().manual_seed(seed)
    E, V, w = cfg["width"], cfg["vocab"], {}

    def mat(o, i, gain=1.0):
        return torch.randn(o, i, generator=g) * gain / i ** 0.5

    def near_one(n):
        return 1.0 + 0.2 * torch.randn(n, generator=g)

    def bias(n, gain=0.3):
        return gain * torch.randn(n, generator=g)

    w["embed"] = torch.randn(V, E, generator=g) * 1.4
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        w[f"l{i}.norm1"] = near_one(E)
        if layer["type"] == "rglru":
            C, B = m["width"], m["blocks"]
            n = C // B
            w[p + "y"], w[p + "y.b"], w[p + "x"], w[p + "x.b"] = mat(C, E, 1.5), bias(C), mat(C, E, 1.5), bias(C)
            w[p + "conv"], w[p + "conv.b"] = torch.randn(C, m["conv"], generator=g) * 0.6, bias(C)
            for k in ("ra", "ri"):
                w[p + k], w[p + k + ".b"] = torch.randn(B, n, n, generator=g) * 1.5 / n ** 0.5, bias(B * n).view(B, n)
            w[p + "lam"] = -7.0 + 7.0 * torch.rand(C, generator=g)
            w[p + "o"] = mat(E, C, 1.5)
        else:
            a, r = m["left"], m["right"]
            H, G, D, Dv, q = a["heads"], a["kv_heads"], a["dim"], a["vdim"], p + "left."
            w[q + "q"], w[q + "k"], w[q + "v"], w[q + "g"], w[q + "o"] = mat(H * D, E), mat(G * D, E), mat(G * Dv, E), mat(H, E, 2.0), mat(E, H * Dv, 2.0)
            w[q + "q.b"], w[q + "k.b"], w[q + "v.b"] = bias(H * D), bias(G * D), bias(G * Dv)
            H, D, Dv, q = r["heads"], r["dim"], r["vdim"], p + "right."
            w[q + "q"], w[q + "k"], w[q + "v"], w[q + "g"], w[q + "o"] = mat(H * D, E), mat(H * D, E), mat(H * Dv, E), mat(H * Dv, E, 2.0), mat(E, H * Dv)
        mlp = layer.get("mlp")
        if not mlp:
            continue
        q = f"l{i}.mlp."
        w[f"l{i}.norm2"] = near_one(E)
        if mlp["kind"] == "dense":
            w[q + "gate"], w[q + "up"], w[q + "down"] = mat(mlp["ff"], E, 1.5), mat(mlp["ff"], E, 1.5), mat(E, mlp["ff"], 1.5)
            continue
        n = mlp["router"]["experts"]
        for e in range(n):
            F = mlp["expert"]["ff"]
            w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = mat(F, E, 1.5), mat(F, E, 1.5), mat(E, F, 1.5)
        w[q + "router"], w[q + "router.b"] = mat(n, E, 1.5), bias(n, 1.0)
        if mlp.get("shared"):
            Fs = mlp["shared"]["ff"]
            w[q + "shared.gate"], w[q + "shared.up"], w[q + "shared.down"] = mat(Fs, E, 1.5), mat(Fs, E, 1.5), mat(E, Fs, 1.5)
            w[q + "shared.sg"] = mat(1, E, 2.0)
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
    from tests import plain_tukevik as P
    cfg = all_chosen(CONFIGS[name]) if dense else CONFIGS[name]
    return P.forward(cfg, as_plain(weights(name)), tokens_of(name, n, seed)).float()
