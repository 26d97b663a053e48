"""A plain, slow statement of the Dasusun decoder: one function per mechanism, whole sequences at once, on the CPU.

It shares no code with the package: it takes config.json as a dictionary and the tensors by their names, and works in
the dtype it is given (float32, or float64 to bound the float32 one).  A prompt is run whole; there is no cache and
no state that outlives a call, so it cannot have the faults that a cut prompt or a shared batch could bring.

Notation: T tokens, W width, H heads, D plain key size, P rotated key size, E value size, R latent size.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def divided_by_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def plain_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return divided_by_rms(x, eps) * w


def centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """A weight of zero leaves the unit-rms row as it is."""
    return divided_by_rms(x, eps) * (1.0 + w)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x: torch.Tensor, taps_w: torch.Tensor) -> torch.Tensor:
    """y_t = sum_j w[:, j] x_(t - taps + 1 + j) per channel, zeros before the start: x [T, C], taps_w [C, taps]."""
    T, taps = x.shape[0], taps_w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += taps_w[:, j] * x[s]
    return out


def depth_average(rows: List[torch.Tensor], weights: torch.Tensor) -> torch.Tensor:
    """sum_j weights[j] rows[j] over the embedding and every layer's result so far."""
    assert len(rows) == weights.shape[0]
    total = torch.zeros_like(rows[0])
    for j, x in enumerate(rows):
        total = total + weights[j] * x
    return total


# ---- rotation ----------------------------------------------------------------------------------------------------
def frequencies(rot: dict):
    """(angle per position of every pair, factor on cos and sin), in float64."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def dim_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(dim_of(float(sc["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, P]: number i turns with number i + dims/2 (dims the first numbers of a head; the rest pass)."""
    dims = int(rot["dims"])
    f, factor = frequencies(rot)
    ang = positions.double()[:, None] * f[None, :]
    cos = (torch.cos(ang) * factor).to(x.dtype)[:, None, :]
    sin = (torch.sin(ang) * factor).to(x.dtype)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


# ---- attention over latents ----------------------------------------------------------------------------------------
def visible(T: int, window: Optional[int]) -> torch.Tensor:
    """[T, T]: position i sees j with 0 <= i - j (< window, if there is one)."""
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    see = dist >= 0
    return see & (dist < window) if window is not None else see


def softmax_over_visible(s: torch.Tensor, see: torch.Tensor) -> torch.Tensor:
    s = s.masked_fill(~see, float("-inf"))
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def latent_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    """Keys and values made per head from one latent per token, one rotated key part shared by all heads."""
    T = h.shape[0]
    H, D, P, E, R = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = torch.arange(T)
    q = (plain_norm(h @ w[f"{p}.dq"].T, w[f"{p}.dq.norm"], eps) @ w[f"{p}.uq"].T).view(T, H, D + P)
    down = h @ w[f"{p}.dkv"].T
    c = plain_norm(down[:, :R], w[f"{p}.dkv.norm"], eps)
    q_plain, q_rot = q[..., :D], rotate(q[..., D:], pos, m["rot"])
    k_rot = rotate(down[:, None, R:], pos, m["rot"])[:, 0]
    k = (c @ w[f"{p}.uk"].T).view(T, H, D)
    v = (c @ w[f"{p}.uv"].T).view(T, H, E)
    see = visible(T, int(m["mask"]["size"]) if m.get("mask") else None)
    heads = []
    for i in range(H):
        s = (q_plain[:, i] @ k[:, i].T + q_rot[:, i] @ k_rot.T) * float(m["scale"])
        heads.append(softmax_over_visible(s, see) @ v[:, i])
    return torch.cat(heads, dim=-1) @ w[f"{p}.o"].T


def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return gelu_tanh(h @ w[f"{p}.up"].T) @ w[f"{p}.down"].T


# ---- the model -----------------------------------------------------------------------------------------------------
def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float32,
            after_layers: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  ``after_layers``: a list that receives the stream after every layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    results = [x]
    for i, layer in enumerate(config["layers"]):
        L = f"l{i}"
        h = centred_norm(x, w[f"{L}.norm1"], eps)
        h = h + causal_conv(h, w[f"{L}.canon1"])
        y = latent_attention(h, layer["mixer"], w, f"{L}.mix", eps)
        x = x + centred_norm(y, w[f"{L}.norm1b"], eps) * w[f"{L}.ls1"]
        if layer.get("mlp") is not None:
            y = dense_ff(centred_norm(x, w[f"{L}.norm2"], eps), w, f"{L}.mlp")
            x = x + centred_norm(y, w[f"{L}.norm2b"], eps) * w[f"{L}.ls2"]
        results.append(x)
        x = depth_average(results, w[f"{L}.dwa"])
        if after_layers is not None:
            after_layers.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(config: dict, weights: Dict[str, torch.Tensor], prompt: List[int], n_new: int, dtype=torch.float32) -> List[int]:
    """The tokens that the largest logit picks, one after the other, the whole sequence run again for each."""
    toks, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(torch.argmax(forward(config, weights, toks, dtype)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
