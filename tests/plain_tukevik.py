"""A plain, slow implementation of the Tukevik design in float64, one function per mechanism, written from the
design's equations and sharing no code with the package.  It is the oracle of the tests.

A model is (cfg, W): cfg the dictionary that config.json holds, W a dictionary name -> float64 tensor.
`forward(cfg, W, tokens)` runs a whole sequence from its first token and returns the logits at every position (and,
when asked, the residual stream after every layer).  Nothing is carried between calls: a sequence that the package
runs in pieces, in a batch or token by token is compared with this one pass over all of it.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ------------------------------------------------------------------------------------------------- rotation
def rotate(x: torch.Tensor, positions: torch.Tensor, rot) -> torch.Tensor:
    """x [T, heads, n]: the first rot.dims entries of every head are turned, entry i with entry i + dims/2."""
    dims = rot["dims"]
    half = dims // 2
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


# ------------------------------------------------------------------------------------------------ attention
def visible(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] of booleans: whether position i (row) sees position j (column): earlier tokens of its own chunk."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    return ok if size is None else ok & (i // size == j // size)


def capped(s: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return s if cap is None else cap * torch.tanh(s / cap)


def sink_attention(q, k, v, scale: float, cap: Optional[float], seen: torch.Tensor) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]; the softmax's denominator counts one more key of score 0."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = capped((q[:, h] @ k[:, g].T) * scale, cap).masked_fill(~seen, -math.inf)
        m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
        e = torch.exp(s - m)
        out[:, h] = (e / (e.sum(dim=-1, keepdim=True) + torch.exp(-m))) @ v[:, g]
    return out


def attention_branch(m, eps: float, W, p: str, h: torch.Tensor) -> torch.Tensor:
    H, G, D, Dv = m["heads"], m.get("kv_heads") or m["heads"], m["dim"], m.get("vdim") or m["dim"]
    T = h.shape[0]
    q = unit_rms((h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, D), eps)
    k = unit_rms((h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, D), eps)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, Dv)
    size = m["mask"]["size"] if m.get("mask") else None
    o = sink_attention(q, k, v, float(m["scale"]), m.get("softcap"), visible(T, size))
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * Dv) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------ retention
def retention(q, k, v, decay: List[float]) -> torch.Tensor:
    """q, k [T, H, D], v [T, H, Dv] -> [T, H, Dv]: S <- decay S + k v^T from zero, read with q after the update."""
    T, H, D = q.shape
    a = torch.tensor(decay, dtype=F64)[:, None, None]
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hij,hi->hj", S, q[t])
    return o


def retention_branch(m, eps: float, W, p: str, h: torch.Tensor) -> torch.Tensor:
    H, D, Dv = m["heads"], m["dim"], m.get("vdim") or m["dim"]
    T = h.shape[0]
    pos = torch.arange(T)
    q, k = (h @ W[p + "q"].T).view(T, H, D), (h @ W[p + "k"].T).view(T, H, D)
    if m.get("rot"):
        q, k = rotate(q, pos, m["rot"]), rotate(k, pos, m["rot"])
    o = retention(q, k * D ** -0.5, (h @ W[p + "v"].T).view(T, H, Dv), m["decay"])
    return (unit_rms(o, eps).reshape(T, H * Dv) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel_mixer(m, eps: float, W, p: str, h: torch.Tensor) -> torch.Tensor:
    return float(m["left_scale"]) * attention_branch(m["left"], eps, W, p + "left.", h) \
        + float(m["right_scale"]) * retention_branch(m["right"], eps, W, p + "right.", h)


# ---------------------------------------------------------------------------------- gated linear recurrence
def causal_conv(u: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """u [T, C]; taps [C, K], the last column weighing the current row, zeros in front of the sequence."""
    T, K = u.shape[0], taps.shape[1]
    full = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=F64), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(K):
        y = y + full[j:j + T] * taps[:, j]
    return y + bias


def block_product(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, blocks*n], w [blocks, n, n] as [out, in], b [blocks, n]: every part of u by its own matrix."""
    B, n, _ = w.shape
    return (torch.einsum("tbi,boi->tbo", u.view(-1, B, n), w) + b).reshape(u.shape)


def recurrence_coefficients(W, p: str, u: torch.Tensor):
    """a [T, C] and what is added, [T, C]."""
    r = torch.sigmoid(block_product(u, W[p + "ra"], W[p + "ra.b"]))
    i = torch.sigmoid(block_product(u, W[p + "ri"], W[p + "ri.b"]))
    log_a = -8.0 * r * softplus(W[p + "lam"])
    a = torch.exp(log_a)
    return a, torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u


def rglru_mixer(m, W, p: str, h: torch.Tensor) -> torch.Tensor:
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    a, b = recurrence_coefficients(W, p, u)
    S, out = torch.zeros(u.shape[1], dtype=F64), torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return (out * y) @ W[p + "o"].T


# ---------------------------------------------------------------------------------------------- feed-forward
def expert(W, p: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def router_logits(W, p: str, h: torch.Tensor) -> torch.Tensor:
    return h @ W[p + "router"].T + W[p + "router.b"]


def moe(mlp, W, p: str, h: torch.Tensor, ids: Optional[torch.Tensor] = None) -> torch.Tensor:
    """ids [T, top]: a choice given from outside instead of the router's own; the weights follow it."""
    z = router_logits(W, p, h)
    if ids is None:
        ids = torch.topk(z, mlp["router"]["top"], dim=-1).indices
    w = torch.softmax(torch.gather(z, 1, ids), dim=-1)
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = torch.nonzero(ids == e, as_tuple=True)
        if rows.numel():
            out[rows] += w[rows, place][:, None] * expert(W, f"{p}e{e}.", h[rows])
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ W[p + "shared.sg"].T) * expert(W, p + "shared.", h)
    return out


# --------------------------------------------------------------------------------------------------- model
def forward(cfg, W: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence.  layers_out: a list that receives the stream after every layer."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)].clone()
    for i, layer in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.mix.", f"l{i}.mlp.", layer["mixer"]
        h = rms_norm(x, W[f"l{i}.norm1"], eps)
        x = x + mult * (rglru_mixer(m, W, p, h) if layer["type"] == "rglru" else parallel_mixer(m, eps, W, p, h))
        mlp = layer.get("mlp")
        if mlp:
            h = rms_norm(x, W[f"l{i}.norm2"], eps)
            x = x + mult * (expert(W, q, h) if mlp["kind"] == "dense" else moe(mlp, W, q, h))
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T
