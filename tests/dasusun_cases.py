"""Small Dasusun configurations and weights for the tests: sizes that differ from one another in every field, among
them values that make mechanisms degenerate (one layer, one tap, one head, a single rotated pair, a window of one
position, no window at all, no stretch of the frequencies, a layer without a feed-forward) and sizes that no vector load
or tensor-core tile takes."""
from __future__ import annotations

from typing import Dict

import torch

from inferrs_b200.engine.loading import spec_from_config
from inferrs_b200.engine.model import declared_tensors


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, window=None, scaling=None, ff=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": rot}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, eps, taps, layers, **more):
    return {"architecture": "Dasusun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "layers": layers, **more}


# latents and rotated parts that are padded (40, 72 and 12, 6), windows that are no multiples of a page, a layer that
# sees every earlier token, a layer without a feed-forward between others, stretched and plain frequencies
CASE_A = model(211, 96, 1e-5, 4, [
    latent(6, 24, 12, 20, 36, 40, 0.17, 10000.0, 23, (4.0, 64, 32.0, 1.0), 72),
    latent(4, 16, 8, 40, 64, 64, 0.2, 500.0, 50, None, None),
    latent(3, 8, 6, 12, 24, 72, 0.3, 100000.0, None, (8.0, 32, 8.0, 0.5), 50),
    latent(5, 32, 32, 16, 40, 32, 0.12, 10000.0, 31, (2.0, 4096, 32.0, 1.0), 136),
])
# everything one: one layer, one tap, one head, one rotated pair, a window that shows a token only itself
CASE_B = model(97, 64, 1e-6, 1, [latent(1, 16, 2, 24, 32, 32, 0.25, 100.0, 1, None, 40)])
# sizes of the tensor-core kernels: latents of 128 and 256, more heads than a block takes, rotated parts of 64
CASE_C = model(130, 128, 1e-5, 3, [
    latent(18, 32, 64, 32, 96, 128, 0.1, 50000.0, 70, (2.0, 512, 16.0, 1.0), 256),
    latent(16, 64, 16, 64, 128, 256, 0.11, 10000.0, None, (4.0, 128, 32.0, 1.0), 200),
    latent(2, 128, 32, 128, 64, 128, 0.08, 1000.0, 129, None, 64),
], max_positions=512)
# odd sizes everywhere; two taps; the rotation's slow end beyond the last pair, and a stretch that leaves all pairs
CASE_D = model(77, 90, 1e-5, 2, [
    latent(3, 11, 10, 7, 17, 33, 0.25, 30.0, 7, (3.0, 16, 4.0, 0.25), 33),
    latent(7, 5, 4, 9, 21, 19, 0.4, 100.0, 33, (2.0, 100000, 1.0, 0.5), None),
    latent(1, 30, 14, 50, 90, 65, 0.15, 1000.0, 16, None, 45),
])
CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D}


def make_weights(config: dict, seed: int, bare_second: bool = False) -> Dict[str, torch.Tensor]:
    """Weights of a size that keeps activations near one, so that every mechanism moves the logits: matrices N(0, 1 /
    fan-in), norm weights spread around zero (plain ones around one), scales that differ by channel, convolutions whose
    every tap counts, averages over depth that look back on every result.  Rounded to bfloat16 (returned as float32 on
    the host), so that both run dtypes and the plain statement start from the same numbers.  ``bare_second``: layers
    without a feed-forward get the norms and the scale of one all the same."""
    shapes = None
    if bare_second:
        shapes = {f"l{i}.{n}": (config["width"],) for i, l in enumerate(config["layers"]) if l.get("mlp") is None
                  for n in ("norm2", "norm2b", "ls2")}
    spec, _ = spec_from_config(config, tensor_shapes=shapes)
    g = torch.Generator().manual_seed(seed)
    out = {}
    for d in declared_tensors(spec):
        n = d.name
        r = torch.randn(d.shape, generator=g)
        if n == "embed":
            t = r
        elif ".canon" in n:
            t = r * (0.6 / d.shape[1] ** 0.5) + 0.15
        elif n.endswith(".dwa"):
            t = 0.4 * r
            t[-1] += 1.0
        elif ".mix." in n and n.endswith(".norm"):
            t = 1.0 + 0.2 * r
        elif ".ls" in n:
            t = 1.0 + 0.3 * r
        elif len(d.shape) == 1:                               # norm weights around zero
            t = 0.25 * r
        else:
            t = r * (1.0 / d.shape[1] ** 0.5)
        out[n] = t.to(torch.bfloat16).to(torch.float32)
    return out


def random_case(seed: int) -> dict:
    """A configuration drawn from a seed: every size, count, window, constant and the number of layers differ from
    draw to draw."""
    import random
    rnd = random.Random(seed)
    pick = rnd.choice

    def layer():
        rot_dim = pick([2, 4, 6, 8, 16, 20, 32, 64])
        scaling = None if rnd.random() < 0.3 else (pick([1.0, 2.0, 4.0, 10.0]), pick([16, 64, 1000, 4096]),
                                                   pick([8.0, 32.0]), pick([0.5, 1.0, 2.0]))
        return latent(pick([1, 2, 3, 5, 8, 16, 17]), pick([4, 8, 16, 24, 32, 64]), rot_dim, pick([5, 8, 16, 40, 64]),
                      pick([12, 31, 48, 64, 128]), pick([16, 24, 32, 50, 64, 96, 128, 160, 256]), pick([0.1, 0.17, 0.3]),
                      pick([50.0, 10000.0, 250000.0]), pick([None, 1, 2, 5, 17, 23, 33, 64, 65, 80]), scaling,
                      pick([None, 20, 33, 64, 200]))
    return model(pick([61, 97, 130, 256]), pick([32, 48, 64, 90, 128, 160]), pick([1e-5, 1e-6]), pick([1, 2, 3, 4, 5]),
                 [layer() for _ in range(rnd.randint(1, 6))], max_positions=512)
