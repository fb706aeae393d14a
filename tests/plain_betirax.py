"""A plain, slow implementation of the Betirax design in float64, one function per mechanism, written from the
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


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------- rotation
def yarn_ramp(dims: int, base: float, original: float, fast: float, slow: float) -> List[float]:
    """For every pair of entries, how much of its frequency is divided by the factor (0: none, 1: all)."""
    def entry_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(entry_of(fast)), 0), min(math.ceil(entry_of(slow)), dims - 1)
    return [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]


def rotary_frequencies(rot) -> torch.Tensor:
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc:
        ramp = yarn_ramp(dims, base, float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
        f = [x / float(sc["factor"]) * r + x * (1.0 - r) for x, r in zip(f, ramp)]
    return torch.tensor(f, dtype=F64)


def rotary_gain(rot) -> float:
    sc = rot.get("scaling")
    return 0.1 * math.log(float(sc["factor"])) + 1.0 if sc else 1.0


def rotate(x: torch.Tensor, positions: torch.Tensor, rot) -> torch.Tensor:
    """x [T, heads, n]: the first rot.dims entries of every head are turned, entry i with entry i + dims/2."""
    dims = rot["dims"]
    half, gain = dims // 2, rotary_gain(rot)
    ang = positions.to(F64)[:, None] * rotary_frequencies(rot)[None, :]          # [T, half]
    c, s = gain * torch.cos(ang)[:, None, :], gain * torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


# ------------------------------------------------------------------------------------------------- attention
def visible(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] of booleans: whether position i (row) sees position j (column); size None: every earlier one."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & (i - j < size)


def head_slopes(H: int) -> List[float]:
    return [2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]


def distance_bias(T: int, slope: float) -> torch.Tensor:
    """[T, T]: what is taken off the score of query i and key j."""
    i = torch.arange(T, dtype=F64)[:, None]
    j = torch.arange(T, dtype=F64)[None, :]
    return slope * (i - j)


def query_temperature(positions: torch.Tensor, temp) -> torch.Tensor:
    blocks = torch.div(positions + 1, int(temp["every"]), rounding_mode="floor").to(F64)
    return 1.0 + float(temp["coef"]) * torch.log(blocks + 1.0)


def softmax_attention(q, k, v, scale: float, seen: torch.Tensor, slopes: Optional[List[float]] = None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if slopes is not None:
            s = s - distance_bias(T, slopes[h])
        s = s.masked_fill(~seen, -math.inf)
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, g]
    return out


def attention_mixer(m, eps: float, W, p: str, h: torch.Tensor) -> torch.Tensor:
    H, D = m["heads"], m["dim"]
    G = m.get("kv_heads") or H
    T = h.shape[0]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, D)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, D)
    v = k                                                      # before the norm
    q, k = rms_norm(q, W[p + "q.norm"], eps), rms_norm(k, W[p + "k.norm"], eps)
    if m.get("q_temp"):
        q = q * query_temperature(torch.arange(T), m["q_temp"])[:, None, None]
    size = m["mask"]["size"] if m.get("mask") else None
    o = softmax_attention(q, k, v, float(m["scale"]), visible(T, size), head_slopes(H)).reshape(T, H * D)
    o = o * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T + W[p + "o.b"]


# ------------------------------------------------------------------------------------------ latent attention
def latent_rows(m, eps: float, W, p: str, h: torch.Tensor):
    """What a layer with a down-projection of its own keeps: c [T, kv_rank] and the rotated key part [T, 1, rot_dim]."""
    C = m["kv_rank"]
    down = h @ W[p + "dkv"].T
    c = rms_norm(down[:, :C], W[p + "dkv.norm"], eps)
    return c, rotate(down[:, None, C:], torch.arange(h.shape[0]), m["rot"])


def latent_mixer(m, eps: float, W, p: str, h: torch.Tensor, rows) -> torch.Tensor:
    """rows: (c, rotated key part) as some layer keeps them (its own or another's)."""
    H, D, R, Dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    T = h.shape[0]
    c, k_rot = rows
    cq = rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    q = (cq @ W[p + "uq"].T).view(T, H, D + R)
    q = torch.cat([q[..., :D], rotate(q[..., D:], torch.arange(T), m["rot"])], dim=-1)
    k = torch.cat([(c @ W[p + "uk"].T).view(T, H, D), k_rot.expand(T, H, R)], dim=-1)
    v = (c @ W[p + "uv"].T).view(T, H, Dv)
    o = softmax_attention(q, k, v, float(m["scale"]), visible(T, None)).reshape(T, H * Dv)
    o = o * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


# ---------------------------------------------------------------------------------------------- feed-forward
def dense(W, p: str, h: torch.Tensor) -> torch.Tensor:
    return gelu_tanh(h @ W[p + "up"].T) @ W[p + "down"].T


def expert(W, p: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(mlp, W, p: str, h: torch.Tensor, ids=None):
    """Chosen experts [T, top] and their weights.  ids: a choice given from outside; the weights follow it."""
    z = h @ W[p + "router"].T
    if ids is None:
        ids = torch.topk(z, mlp["router"]["top"], dim=-1).indices
    return ids, torch.softmax(torch.gather(z, 1, ids), dim=-1)


def moe(mlp, W, p: str, h: torch.Tensor, ids=None) -> torch.Tensor:
    ids, w = route(mlp, W, p, h, ids)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for r in range(ids.shape[1]):
            out[t] = out[t] + w[t, r] * expert(W, f"{p}e{int(ids[t, r])}.", h[t:t + 1])[0]
    if mlp.get("shared"):
        out = out + expert(W, p + "shared.", h)
    return out


# --------------------------------------------------------------------------------------------------- model
def forward(cfg, W: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None,
            choices: Optional[Dict[int, torch.Tensor]] = None, routed: Optional[dict] = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence.  layers_out: a list that receives the stream after every layer.
    choices: layer -> experts [T, top] to use instead of the router's own choice; routed: a dictionary that receives
    every layer's router logits (for tests that look for near ties)."""
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "attention":
            y = attention_mixer(m, eps, W, p, x)
        elif layer["type"] == "latent_attention":
            if m.get("kv_from") is None:
                kept[i] = latent_rows(m, eps, W, p, x)
            y = latent_mixer(m, eps, W, p, x, kept[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            raise ValueError(layer["type"])
        x = layer_norm(alpha * x + y, W[f"l{i}.norm1"], eps)
        mlp = layer.get("mlp")
        if mlp:
            q = f"l{i}.mlp."
            if mlp["kind"] == "dense":
                y = dense(W, q, x)
            else:
                if routed is not None:
                    routed[i] = x @ W[q + "router"].T
                y = moe(mlp, W, q, x, None if choices is None else choices.get(i))
            x = layer_norm(alpha * x + y, W[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W["final.norm"], eps) @ W["embed"].T
