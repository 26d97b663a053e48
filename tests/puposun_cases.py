"""Small Puposun configurations and weights for the tests: sizes that differ from one another in every field, among them
values that make mechanisms degenerate (one layer, one head, one expert, one group, a window of one position, no kept
tokens, no loop or a loop of one pass) and sizes that no vector load or tensor-core tile takes."""
from __future__ import annotations

import random
from typing import Dict

import torch

from inferrs_b200.engine.loading import spec_from_config
from inferrs_b200.engine.model import declared_tensors


def experts(n, top, ff, scale, groups=None):
    router = {"experts": n, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def full(heads, kv_heads, dim, rot, base, scale, cap, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": cap,
         "rot": {"base": base, "dims": rot}}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def windowed(heads, kv_heads, dim, rot, base, scale, size, keep, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
         "mask": {"size": size, "keep_first": keep}, "rot": {"base": base, "dims": rot}}
    return {"type": "attention_2", "mixer": m, "mlp": mlp}


def model(vocab, width, eps, scale, cap, layers, loop=None, **more):
    out = {"architecture": "Puposun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "logit_softcap": cap, "layers": layers, **more}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


# windows that are no multiples of a page beside kept tokens that are none, a layer without a feed-forward, a loop over
# the middle layers that runs three times and ends on a layer with an output bias
CASE_A = model(211, 96, 1e-5, 3.0, 9.0, [
    windowed(6, 2, 24, 16, 10000.0, 0.25, 23, 5, experts(6, 2, 40, 1.5, (3, 2))),
    windowed(4, 4, 16, 8, 500.0, 0.3, 17, 19, None),
    full(6, 3, 32, 32, 100000.0, 0.2, 7.0, experts(9, 3, 24, 0.7, (3, 1))),
    full(5, 1, 16, 4, 3000.0, 0.3, 30.0, experts(4, 1, 72, 2.0)),
    windowed(8, 2, 40, 24, 250000.0, 0.17, 40, 3, experts(8, 4, 16, 1.0, (4, 3))),
], loop=(1, 4, 3))
# everything one: one layer, one head, one expert in one group, a window that shows a token itself beside the first
CASE_B = model(97, 64, 1e-6, 1.0, 4.0, [windowed(1, 1, 16, 2, 100.0, 0.4, 1, 1, experts(1, 1, 40, 1.0, (1, 1)))], loop=(0, 1, 1))
# sizes of the tensor-core kernels, more kept tokens than a tile of keys, the whole model looped
CASE_C = model(130, 128, 1e-5, 2.0, 12.0, [
    full(8, 2, 64, 64, 50000.0, 0.15, 11.0, experts(12, 2, 64, 1.2, (4, 2))),
    windowed(4, 2, 128, 32, 10000.0, 0.1, 70, 77, experts(8, 2, 32, 1.0, (2, 1))),
    full(6, 2, 128, 128, 1000000.0, 0.09, 25.0, experts(8, 3, 40, 2.5)),
    windowed(8, 4, 96, 48, 5000.0, 0.12, 33, 20, experts(4, 2, 128, 1.0, (2, 2))),
], loop=(0, 4, 2), max_positions=512)
# odd sizes everywhere; no kept tokens; groups of one expert
CASE_D = model(77, 90, 1e-5, 5.0, 6.0, [
    full(3, 3, 11, 6, 30.0, 0.4, 3.0, experts(5, 2, 33, 1.1, (5, 3))),
    windowed(7, 7, 9, 4, 100.0, 0.5, 7, 0, experts(7, 3, 21, 0.9)),
    windowed(3, 1, 30, 14, 1000.0, 0.2, 16, 16, experts(6, 2, 45, 1.3, (2, 1))),
], loop=(1, 3, 2))
CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D}


def make_weights(config: dict, seed: int) -> Dict[str, torch.Tensor]:
    """Weights of a size that keeps activations near one, so that every mechanism moves the logits: matrices N(0, 1 /
    fan-in), biases and gates that count, corrections that change which experts are chosen (some choice scores are
    negative).  Rounded to bfloat16 (returned as float32 on the host), so that both run dtypes and the plain statement
    start from the same numbers."""
    spec, _ = spec_from_config(config)
    g = torch.Generator().manual_seed(seed)
    out = {}
    for d in declared_tensors(spec):
        n = d.name
        r = torch.randn(d.shape, generator=g)
        if n == "embed":
            t = r / config["embedding"]["scale"]
        elif n.endswith(".b"):
            t = 0.5 * r
        elif n.endswith(".correction"):
            t = 0.7 * r - 0.3
        elif len(d.shape) == 1:                               # norm weights around one
            t = 1.0 + 0.2 * r
        else:
            size = 1.3 if n.endswith((".q", ".k")) else 2.0 if n.endswith((".router", ".g")) else \
                0.6 if n.endswith((".o", ".down")) else 1.0
            t = r * (size / d.shape[1] ** 0.5)
        out[n] = t.to(torch.bfloat16).to(torch.float32)
    return out


def random_case(seed: int) -> dict:
    """A configuration drawn from a seed: every size, count, window, constant, the order of layers and the loop differ
    from draw to draw."""
    rnd = random.Random(seed)
    pick = rnd.choice

    def ff():
        if rnd.random() < 0.25:
            return None
        count, size = pick([1, 2, 3, 4]), pick([1, 2, 3, 5])
        keep = rnd.randint(1, count)
        top = rnd.randint(1, min(keep * size, 4))
        return experts(count * size, top, pick([8, 20, 33, 64]), pick([0.5, 1.0, 2.5]), None if rnd.random() < 0.2 else (count, keep))

    def layer():
        kv, group, dim = pick([1, 2, 3]), pick([1, 2, 3, 4]), pick([8, 16, 24, 32, 48, 64, 80, 96, 128])
        rot = pick([r for r in (2, 4, 8, 16, 24, 32, 48, 64, 128) if r <= dim])
        base, scale = pick([50.0, 10000.0, 1000000.0]), pick([0.1, 0.2, 0.35])
        if rnd.random() < 0.4:
            return full(kv * group, kv, dim, rot, base, scale, pick([2.0, 10.0, 30.0]), ff())
        return windowed(kv * group, kv, dim, rot, base, scale, pick([1, 2, 5, 17, 23, 33, 64, 65]), pick([0, 1, 4, 15, 16, 17, 40, 65]),
                        ff())

    n = rnd.randint(1, 5)
    loop = None
    if rnd.random() < 0.8:
        start = rnd.randint(0, n - 1)
        loop = (start, rnd.randint(start + 1, n), pick([1, 2, 3]))
    return model(pick([61, 97, 130, 256]), pick([32, 48, 64, 90, 128, 160]), pick([1e-5, 1e-6]), pick([1.0, 4.0, 12.0]),
                 pick([3.0, 15.0]), [layer() for _ in range(n)], loop=loop, max_positions=512)
