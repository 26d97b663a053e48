"""A plain, slow statement of the Puposun decoder: one function per mechanism, whole sequences at once, on the CPU.

It shares no code with the package: it takes config.json as a dictionary and the tensors by their names, and works in
the dtype it is given (float32, or float64 to bound the float32 one).  A prompt is run whole; there is no cache and
no state that outlives a call, so it cannot have the faults that a cut prompt or a shared batch could bring.

Notation: T tokens, W width, H query heads on G key heads, D head size, E experts.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


# ---- norm ----------------------------------------------------------------------------------------------------------
def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


# ---- rotation ------------------------------------------------------------------------------------------------------
def angles(positions: torch.Tensor, base: float, dims: int):
    """cos and sin of position * base^(-2 i / dims), [T, dims / 2], in float64."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    a = positions.double()[:, None] * f[None, :]
    return torch.cos(a), torch.sin(a)


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, D]: number i of a head's first ``dims`` turns with number i + dims / 2; the others pass."""
    cos, sin = (t.to(x.dtype)[:, None, :] for t in angles(positions, base, dims))
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """The same with number 2i turning with number 2i + 1."""
    cos, sin = (t.to(x.dtype)[:, None, :] for t in angles(positions, base, dims))
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


# ---- which keys a position sees ------------------------------------------------------------------------------------
def sees_all_earlier(T: int) -> torch.Tensor:
    return torch.arange(T)[:, None] >= torch.arange(T)[None, :]


def sees_window_and_first(T: int, size: int, keep_first: int) -> torch.Tensor:
    """Position i sees j <= i where j is one of the last ``size`` positions or one of the sequence's first."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


# ---- scores and their weights --------------------------------------------------------------------------------------
def squashed(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap)


def shares(s: torch.Tensor, see: torch.Tensor) -> torch.Tensor:
    """Softmax over the visible keys of every row."""
    s = s.masked_fill(~see, float("-inf"))
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def shares_beside_a_zero_score(s: torch.Tensor, see: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) over the visible keys: the row's shares add up to less than one."""
    s = s.masked_fill(~see, float("-inf"))
    m = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


# ---- mixers --------------------------------------------------------------------------------------------------------
def capped_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    """Every earlier key, squashed scores, a zero score in the denominator, biases; the values are the keys before
    they are rotated."""
    T = h.shape[0]
    H, G, D = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    pos = torch.arange(T)
    q = (h @ w[f"{p}.q"].T + w[f"{p}.q.b"]).view(T, H, D)
    v = (h @ w[f"{p}.k"].T + w[f"{p}.k.b"]).view(T, G, D)
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    q, k = rotate_halves(q, pos, base, dims), rotate_halves(v, pos, base, dims)
    see = sees_all_earlier(T)
    heads = []
    for i in range(H):
        g = i // (H // G)
        s = squashed((q[:, i] @ k[:, g].T) * float(m["scale"]), float(m["softcap"]))
        heads.append(shares_beside_a_zero_score(s, see) @ v[:, g])
    return torch.cat(heads, dim=-1) @ w[f"{p}.o"].T + w[f"{p}.o.b"]


def window_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    """A window beside the sequence's first keys, neighbours turned together, one sigmoid gate per head."""
    T = h.shape[0]
    H, G, D = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    pos = torch.arange(T)
    q = (h @ w[f"{p}.q"].T).view(T, H, D)
    v = (h @ w[f"{p}.k"].T).view(T, G, D)
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    q, k = rotate_neighbours(q, pos, base, dims), rotate_neighbours(v, pos, base, dims)
    see = sees_window_and_first(T, int(m["mask"]["size"]), int(m["mask"]["keep_first"]))
    gate = torch.sigmoid(h @ w[f"{p}.g"].T)
    heads = []
    for i in range(H):
        g = i // (H // G)
        s = (q[:, i] @ k[:, g].T) * float(m["scale"])
        heads.append(shares(s, see) @ v[:, g] * gate[:, i:i + 1])
    return torch.cat(heads, dim=-1) @ w[f"{p}.o"].T


MIXERS = {"attention": capped_attention, "attention_2": window_attention}


# ---- routed experts ------------------------------------------------------------------------------------------------
def chosen_experts(s: torch.Tensor, correction: torch.Tensor, top: int, groups: Optional[dict]) -> List[List[int]]:
    """The experts of every row: the ``top`` largest corrected scores inside the best groups."""
    choice = s + correction
    E = s.shape[1]
    out = []
    for row in choice:
        allowed = list(range(E))
        if groups:
            n, keep = int(groups["count"]), int(groups["keep"])
            size = E // n
            score = [float(sum(sorted(row[g * size:(g + 1) * size].tolist(), reverse=True)[:2])) for g in range(n)]
            best = sorted(range(n), key=lambda g: -score[g])[:keep]
            allowed = [e for g in best for e in range(g * size, (g + 1) * size)]
        out.append(sorted(allowed, key=lambda e: -float(row[e]))[:top])
    return out


def routed_experts(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    r = mlp["router"]
    s = torch.sigmoid(h @ w[f"{p}.router"].T)
    out = torch.zeros_like(h)
    for t, chosen in enumerate(chosen_experts(s, w[f"{p}.correction"], int(r["top"]), r.get("groups"))):
        total = sum(s[t, e] for e in chosen) + 1e-20
        for e in chosen:
            z = w[f"{p}.e{e}.gate"] @ h[t]
            y = w[f"{p}.e{e}.down"] @ (z * torch.sigmoid(z) * (w[f"{p}.e{e}.up"] @ h[t]))
            out[t] += s[t, e] / total * float(r["scale"]) * y
    return out


# ---- the model -----------------------------------------------------------------------------------------------------
def layer_runs(config: dict) -> List[tuple]:
    """(layer, whether a pass after the first starts with it) in the order in which layers run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    out = [(i, False) for i in range(start)]
    for t in range(times):
        out += [(i, t > 0 and i == start) for i in range(start, stop)]
    return out + [(i, False) for i in range(stop, n)]


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float32,
            after_layers: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``after_layers``: a list that receives the stream after every layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    first = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(config["embedding"]["scale"])
    x = first
    for i, again in layer_runs(config):
        layer, L = config["layers"][i], f"l{i}"
        if again:
            x = x + first
        h = norm(x, w[f"{L}.norm1"], eps)
        y = MIXERS[layer["type"]](h, layer["mixer"], w, f"{L}.mix")
        if layer.get("mlp") is not None:
            y = y + routed_experts(h, layer["mlp"], w, f"{L}.mlp")
        x = x + y
        if after_layers is not None:
            after_layers.append(x)
    return squashed(norm(x, w["final.norm"], eps) @ w["head"].T, float(config["logit_softcap"]))


def greedy(config: dict, weights: Dict[str, torch.Tensor], prompt: List[int], n_new: int, dtype=torch.float32) -> List[int]:
    """The tokens that the largest logit picks, one after the other, the whole sequence run again for each."""
    toks, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(torch.argmax(forward(config, weights, toks, dtype)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
