"""A plain, slow implementation of the Zazulix decoder: whole sequences, no cache, no state carried between calls, one
function per mechanism, 64-bit floats on the CPU.  It shares no code with the package: it takes the configuration as
the dict config.json holds and the tensors by name.

The design in this file's notation (T tokens, positions 0 .. T-1, stream x):

* stream:   x = E[token];  x += mixer(N1 x);  x += ff(N2 x)      (a layer may have no feed-forward, and then has no N2)
* N:        RMS norm times 1 + w
* mixers:   a windowed attention through a latent without positions; a differential attention (two softmax maps per
            head, one minus a multiple of the other) behind short filters; or a retention (a linear recurrence whose
            heads fade at constant rates)
* ff:       a dense one with a clamped gate and a clamped up branch of its own activation, or routed experts with a
            gated shared one
* output:   logits = E N_f(x)
"""

from __future__ import annotations

import math
from typing import Dict, Optional, Sequence

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------- small pieces
def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, eps: float, w: torch.Tensor) -> torch.Tensor:
    """The tensor is an offset from one."""
    return over_rms(x, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def turn_halves(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, d]: dims (i, i + dims / 2) below ``dims`` turned as a pair, the rest left alone."""
    h = dims // 2
    f = base ** (-2.0 * torch.arange(h, dtype=F64) / dims)
    a = (positions.to(F64)[:, None] * f[None, :])[:, None, :]
    out = x.clone()
    u, v = x[..., :h], x[..., h:dims]
    out[..., :h] = u * torch.cos(a) - v * torch.sin(a)
    out[..., h:dims] = v * torch.cos(a) + u * torch.sin(a)
    return out


def turn_if(x, pos, rot: Optional[dict]):
    return x if not rot or not rot.get("dims") else turn_halves(x, pos, int(rot["dims"]), float(rot["base"]))


def short_filter(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[:T - back]
    return y


def window_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] True where query i sees key j: 0 <= i - j (< size)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size) if size else d >= 0


def softmax_attention(q, k, v, scale: float, size: Optional[int] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; q-head h reads kv-head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    seen = window_mask(T, size)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, g]
    return out


# ------------------------------------------------------------------------------- attention through a latent
def latent_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).view(T, H, d)
    c = over_rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    o = softmax_attention(q, k, v, float(m["scale"]), (m.get("mask") or {}).get("size")).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------- differential attention
def difference_of_maps(a1: torch.Tensor, a2: torch.Tensor, lam: torch.Tensor, diff: float, eps: float) -> torch.Tensor:
    return over_rms(a1 - lam * a2, eps) * (1.0 - diff)


def map_weight(lq1, lk1, lq2, lk2, diff: float) -> torch.Tensor:
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q, k, v = (h @ w[p + n].T for n in "qkv")
    if int(m.get("conv") or 0) >= 1:
        q, k, v = (short_filter(u, w[f"{p}{n}.conv"]) for n, u in zip("qkv", (q, k, v)))
    q, k = turn_if(q.view(T, H * 2, d), pos, m.get("rot")), turn_if(k.view(T, G * 2, d), pos, m.get("rot"))
    q, k, v = q.view(T, H, 2, d), k.view(T, G, 2, d), v.view(T, G, dv)
    a1, a2 = (softmax_attention(q[:, :, i], k[:, :, i], v, float(m["scale"])) for i in (0, 1))
    lam = map_weight(*(w[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), float(m["diff"]))
    o = difference_of_maps(a1, a2, lam, float(m["diff"]), eps)
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------- retention
def retain(q, k, v, decay) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv], decay [H]: S <- decay S + k v^T;  o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdp,hd->hp", S, q[t])
    return out


def retention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    q = turn_if((h @ w[p + "q"].T).view(T, H, d), pos, m.get("rot"))
    k = turn_if((h @ w[p + "k"].T).view(T, H, d), pos, m.get("rot")) * d ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, dv)
    o = over_rms(retain(q, k, v, torch.tensor([float(x) for x in m["decay"]], dtype=F64)), eps).reshape(T, H * dv)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------- feed-forward
def clamped_ff(h, w, p, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def gated_ff(h, w, p) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choice_scores(z: torch.Tensor, correction: torch.Tensor, r: dict) -> torch.Tensor:
    """[T, E]: sigmoid + correction, closed (-inf) outside the groups that score best (a group scores what its best two add up to)."""
    c = torch.sigmoid(z) + correction
    groups = r.get("groups") or {}
    n = int(groups.get("count") or 1)
    keep = int(groups.get("keep") or n)
    T, E = c.shape
    parts = c.view(T, n, E // n)
    score = parts.topk(min(2, E // n), dim=-1).values.sum(dim=-1)
    out = torch.full_like(parts, -math.inf)
    for t in range(T):
        for g in score[t].topk(keep).indices.tolist():
            out[t, g] = parts[t, g]
    return out.view(T, E)


def weigh(z: torch.Tensor, chosen: torch.Tensor, scale: float) -> torch.Tensor:
    s = torch.sigmoid(z).gather(1, chosen)
    return s / (s.sum(dim=-1, keepdim=True) + 1e-20) * scale


def route(z: torch.Tensor, correction: torch.Tensor, r: dict):
    """z [T, E] logits -> (chosen [T, top], weights [T, top])."""
    chosen = choice_scores(z, correction, r).topk(int(r["top"]), dim=-1).indices
    return chosen, weigh(z, chosen, float(r.get("scale", 1.0)))


def route_margin(z: torch.Tensor, correction: torch.Tensor, r: dict) -> torch.Tensor:
    """[T]: how far the choice is from falling another way: the smaller of the gap between the last chosen expert and the
    best one not chosen, and the gap between the worst kept group and the best one left out."""
    top = int(r["top"])
    c = choice_scores(z, correction, r).sort(dim=-1, descending=True).values
    gap = c[:, top - 1] - c[:, top] if top < z.shape[1] else torch.full((z.shape[0],), math.inf, dtype=z.dtype)
    groups = r.get("groups") or {}
    n = int(groups.get("count") or 1)
    keep = int(groups.get("keep") or n)
    if keep < n:
        parts = (torch.sigmoid(z) + correction).view(z.shape[0], n, -1)
        s = parts.topk(min(2, parts.shape[-1]), dim=-1).values.sum(dim=-1).sort(dim=-1, descending=True).values
        gap = torch.minimum(gap, s[:, keep - 1] - s[:, keep])
    return gap


def experts_ff(h, w, p, c, forced=None, flips=None):
    """``forced`` [T, top]: the experts every token is given instead of the router's own choice (the weights stay this
    function's own); ``flips`` then receives (token, margin of the own choice) wherever the given experts are not the own
    ones.  For comparisons in low precision, where a choice within rounding may fall either way."""
    r = c["router"]
    z = h @ w[p + "router"].T
    corr = w[p + "correction"]
    chosen, weights = route(z, corr, r)
    if forced is not None:
        own, margin = chosen, route_margin(z, corr, r)
        chosen = forced.long()
        weights = weigh(z, chosen, float(r.get("scale", 1.0)))
        if flips is not None:
            flips += [(t, float(margin[t])) for t in range(h.shape[0]) if sorted(own[t].tolist()) != sorted(chosen[t].tolist())]
    out = torch.zeros_like(h)
    if c.get("shared"):
        out = gated_ff(h, w, p + "shared.") * torch.sigmoid(h @ w[p + "shared.sg"].T)
    for t in range(h.shape[0]):
        for e, wt in zip(chosen[t].tolist(), weights[t]):
            out[t] = out[t] + wt * gated_ff(h[t:t + 1], w, f"{p}e{e}.")[0]
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


MIXERS = {"latent_attention": latent_mixer, "attention": differential_mixer, "retention": retention_mixer}


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: Sequence[int], layers_out: Optional[list] = None,
            routes: Optional[dict] = None, flips: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` receives the stream after every layer.  ``routes`` {layer: [T,
    top]} gives layers their experts (see ``experts_ff``); ``flips`` receives (layer, token, margin)."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(list(tokens), dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[L["type"]](norm(x, eps, w[p + "norm1"]), w, p + "mix.", L["mixer"], eps)
        mlp = L.get("mlp")
        if mlp:
            h = norm(x, eps, w[p + "norm2"])
            if mlp["kind"] == "dense":
                x = x + clamped_ff(h, w, p + "mlp.", float(mlp["limit"]))
            else:
                mine = []
                forced = None if routes is None or i not in routes else routes[i][:len(tokens)]
                x = x + experts_ff(h, w, p + "mlp.", mlp, forced, mine)
                if flips is not None:
                    flips += [(i, t, m) for t, m in mine]
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, eps, w["final.norm"]) @ w["embed"].T
