"""A plain, slow implementation of the Tosodra decoder: whole sequences, no cache, no state carried between calls, one
function per mechanism, 64-bit floats on the CPU.  It shares no code with the package: it takes the configuration as
the dict config.json holds and the tensors by name.

The design in this file's notation (T tokens, positions 0 .. T-1, stream x):

* stream:   x = c E[token]
* layer:    x <- N1(a x + mixer(x));  x <- N2(a x + ff(x))     (a norm of the whole sum, a a constant; a layer may have
            no feed-forward, and then has no N2)
* N:        the row cut into equal parts, each part over its own root mean square, then times a weight
* mixers:   an attention whose weights are sigmoids, inside chunks of the sequence; or an attention through a latent
* ff:       experts behind a router of sigmoids, whose weight scales an expert's INPUT, and a shared expert
* output:   logits = E N_f(x)
"""

from __future__ import annotations

import math
from typing import Dict, Optional, Sequence

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------- small pieces
def unit_rms(x: torch.Tensor, eps: float, weight: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def grouped_norm(x: torch.Tensor, groups: int, eps: float, weight: torch.Tensor) -> torch.Tensor:
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return unit_rms(parts, eps).reshape(x.shape) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------- rotation
def angles(positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """[T, dims / 2]: position times base^(-2 i / dims)."""
    i = torch.arange(dims // 2, dtype=F64)
    return positions.to(F64)[:, None] * (base ** (-2.0 * i / dims))[None, :]


def turn_neighbours(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, d]: dims (2 i, 2 i + 1) below ``dims`` turned as a pair, the rest left alone."""
    a = angles(positions, dims, base)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def turn_halves(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, d]: dims (i, i + dims / 2) below ``dims`` turned as a pair, the rest left alone."""
    a = angles(positions, dims, base)[:, None, :]
    h = dims // 2
    out = x.clone()
    u, v = x[..., :h], x[..., h:dims]
    out[..., :h] = u * torch.cos(a) - v * torch.sin(a)
    out[..., h:dims] = v * torch.cos(a) + u * torch.sin(a)
    return out


# ------------------------------------------------------------------------------- attention of sigmoids in chunks
def chunk_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] True where query i sees key j: j <= i, both in the same chunk of ``size`` positions counted from 0."""
    t = torch.arange(T)
    seen = t[:, None] >= t[None, :]
    if size:
        seen = seen & (t[:, None] // size == t[None, :] // size)
    return seen


def sigmoid_attention(q, k, v, scale: float, bias: torch.Tensor, size: Optional[int]) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; a visible key's weight is sigmoid(scale q.k + bias_h)."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = chunk_mask(T, size)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        w = torch.sigmoid((q[:, h] @ k[:, g].T) * scale + bias[h])
        out[:, h] = w.masked_fill(~seen, 0.0) @ v[:, g]
    return out


def chunked_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = unit_rms(h @ w[p + "q"].T + w[p + "q.b"], eps, w[p + "q.norm"]).view(T, H, d)      # one norm over all heads' rows
    k = unit_rms(h @ w[p + "k"].T + w[p + "k.b"], eps, w[p + "k.norm"]).view(T, G, d)
    v = unit_rms((h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv), eps)                    # one per head, no weight
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    q, k = turn_neighbours(q, pos, dims, base), turn_neighbours(k, pos, dims, base)
    size = (m.get("mask") or {}).get("size")
    o = sigmoid_attention(q, k, v, float(m["scale"]), w[p + "pb"], size).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------- attention through a latent
def latent_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, dn, dr, dv, R = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    pos = torch.arange(T)
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    q = (h @ w[p + "q"].T).view(T, H, dn + dr)
    qr = turn_halves(q[..., dn:], pos, dims, base)
    down = h @ w[p + "dkv"].T
    c = unit_rms(down[:, :R], eps, w[p + "dkv.norm"])
    kr = turn_halves(down[:, None, R:], pos, dims, base)[:, 0]
    k = (c @ w[p + "uk"].T).view(T, H, dn)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    s = (torch.einsum("thd,jhd->htj", q[..., :dn], k) + torch.einsum("thd,jd->htj", qr, kr)) * float(m["scale"])
    s = s.masked_fill(~chunk_mask(T, None)[None], -math.inf)
    return torch.einsum("htj,jhd->thd", torch.softmax(s, dim=-1), v).reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------- feed-forward
def gated_ff(h, w, p) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z: torch.Tensor, top: int):
    """z [T, E] logits -> (chosen [T, top], their sigmoids): the largest, as they are."""
    s = torch.sigmoid(z)
    chosen = s.topk(top, dim=-1).indices
    return chosen, s.gather(1, chosen)


def route_margin(z: torch.Tensor, top: int) -> torch.Tensor:
    """[T]: the gap between the last chosen expert's sigmoid and the best one not chosen."""
    s = torch.sigmoid(z).sort(dim=-1, descending=True).values
    return s[:, top - 1] - s[:, top] if top < z.shape[1] else torch.full((z.shape[0],), math.inf, dtype=z.dtype)


def experts_ff(h, w, p, c, forced=None, flips=None):
    """``forced`` [T, top]: the experts every token is given instead of the router's own choice (the weights stay this
    function's own sigmoids); ``flips`` then receives (token, margin of the own choice) wherever the given experts are
    not the own ones.  For comparisons in low precision, where a choice within rounding may fall either way."""
    top = int(c["router"]["top"])
    z = h @ w[p + "router"].T
    chosen, weights = route(z, top)
    if forced is not None:
        own, margin = chosen, route_margin(z, top)
        chosen = forced.long()
        weights = torch.sigmoid(z).gather(1, chosen)
        if flips is not None:
            flips += [(t, float(margin[t])) for t in range(h.shape[0]) if sorted(own[t].tolist()) != sorted(chosen[t].tolist())]
    out = gated_ff(h, w, p + "shared.") if c.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(chosen[t].tolist(), weights[t]):
            out[t] = out[t] + gated_ff(wt * h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


# ------------------------------------------------------------------------------- the model
def load(model_dir: str):
    """(config dict, tensors by name in 64-bit; integer tensors stay integers): own reading of the folder."""
    import json
    import os
    import struct
    import numpy as np
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        head = json.loads(f.read(struct.unpack("<Q", f.read(8))[0]))
        data = f.read()
    out = {}
    for name, m in head.items():
        if name == "__metadata__":
            continue
        raw = np.frombuffer(data[m["data_offsets"][0]:m["data_offsets"][1]], dtype=np.uint8)
        if m["dtype"] == "BF16":
            t = torch.from_numpy((raw.view(np.uint16).astype(np.uint32) << 16).view(np.float32).copy()).to(F64)
        elif m["dtype"] == "F32":
            t = torch.from_numpy(raw.view(np.float32).copy()).to(F64)
        else:
            raise ValueError(m["dtype"])
        out[name] = t.reshape(m["shape"])
    return cfg, out


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[list] = None,
            routes: Optional[dict] = None, flips: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` receives the stream after every layer.  ``routes`` {layer: [T,
    top]} gives layers their experts (see ``experts_ff``); ``flips`` receives (layer, token, margin)."""
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"].get("groups") or 1)
    alpha = float(cfg["postln_alpha"])
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"attention": chunked_mixer, "latent_attention": latent_mixer}[L["type"]]
        x = grouped_norm(alpha * x + mixer(x, w, p + "mix.", L["mixer"], eps), groups, eps, w[p + "norm1"])
        if L.get("mlp"):
            mine = []
            forced = None if routes is None or i not in routes else routes[i][:len(tokens)]
            y = experts_ff(x, w, p + "mlp.", L["mlp"], forced, mine)
            if flips is not None:
                flips += [(i, t, m) for t, m in mine]
            x = grouped_norm(alpha * x + y, groups, eps, w[p + "norm2"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return grouped_norm(x, groups, eps, w["final.norm"]) @ w["embed"].T
