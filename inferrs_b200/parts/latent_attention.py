"""Attention over a paged cache of latents: one vector per token from which every head makes its key and value.

The cache holds only the latent c (one plane of pages, ``kv_rank`` numbers per token).  The heads' key and value
matrices are not applied to the cached tokens but to the query and to the result:

    score_h(i, j) = q_h(i) . (K_h c_j) = (K_h^T q_h(i)) . c_j          out_h(i) = V_h sum_j p_h(i, j) c_j

so a step costs two batched products per layer (one per head with the step's rows) and the attention kernel reads
each cached latent once for all heads, as key and as value.  Positions, where a description has them, ride in a short key
part behind the latent that all heads share: it is rotated before it is cached, the heads' query parts are rotated inside the
attention kernel as it fetches them.  The cached vector's two parts are padded with zeros to whole tensor-core steps (the
latent to 32 numbers, the rotated part to 16).  A layer may read the latents that another layer
writes (``own_kv=False``) with key and value matrices of its own.

Every size is a field of the description; the part does not know which model or which layer it is in.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch
import torch.nn.functional as F

from .. import kernels
from ..cache.storage import KVNeed
from ..runtime import Runtime
from .basic import Linear, build_position, fuse_rows
from .registry import register_mixer
from .spec import LatentAttentionSpec, TensorDecl


def _up(n: int, step: int) -> int:
    return (n + step - 1) // step * step


def cached_parts(spec: LatentAttentionSpec):
    """(places of the latent, places of the rotated part) in a cached vector."""
    return (spec.kv_rank, 0) if not spec.rot_dim else (_up(spec.kv_rank, 32), _up(spec.rot_dim, 16))


class LatentAttention:
    graph_safe = True  # launches depend only on shapes, never on the step's host-side values

    @staticmethod
    def declare(spec: LatentAttentionSpec) -> List[TensorDecl]:
        hd, he = spec.n_heads * (spec.key_dim + spec.rot_dim), spec.n_heads * spec.value_dim
        d = [TensorDecl(spec.dq_proj, (spec.q_rank, spec.width)),
             TensorDecl(spec.dq_norm, (spec.q_rank,), init="norm"),
             TensorDecl(spec.uq_proj, (hd, spec.q_rank)),
             TensorDecl(spec.uk_proj, (spec.n_heads * spec.key_dim, spec.kv_rank)),
             TensorDecl(spec.uv_proj, (he, spec.kv_rank)),
             TensorDecl(spec.o_proj, (spec.width, he))]
        if spec.gate_proj is not None:
            d.append(TensorDecl(spec.gate_proj, (he, spec.width)))
        if spec.own_kv:
            d += [TensorDecl(spec.dkv_proj, (spec.kv_rank + spec.rot_dim, spec.width)),
                  TensorDecl(spec.dkv_norm, (spec.kv_rank,), init="norm")]
        return d

    @staticmethod
    def cache_need(spec: LatentAttentionSpec) -> Optional[KVNeed]:
        # one plane: the latent is key and value at once
        return KVNeed(n_kv_heads=1, head_dim=sum(cached_parts(spec)), window=spec.window, planes=1)

    @staticmethod
    def state_need(spec: LatentAttentionSpec):
        return None

    @staticmethod
    def writes_cache(spec: LatentAttentionSpec) -> bool:
        return spec.own_kv

    def __init__(self, spec: LatentAttentionSpec, weights: Dict[str, torch.Tensor], rt: Runtime):
        if spec.own_kv and (spec.dkv_proj is None or spec.dkv_norm is None):
            raise ValueError("a latent-attention layer with latents of its own needs dkv_proj and dkv_norm")
        if spec.rot_dim and spec.position is None:
            raise ValueError("a latent-attention layer with a rotated part needs its position description")
        self.spec, self.rt = spec, rt
        h, d, e, r, p = spec.n_heads, spec.key_dim, spec.value_dim, spec.kv_rank, spec.rot_dim
        self.rank, rot_width = cached_parts(spec)
        # query latent, key/value latent with the rotated part behind it, gate: one product
        mats = [weights[spec.dq_proj]] + ([weights[spec.dkv_proj]] if spec.own_kv else []) \
            + ([weights[spec.gate_proj]] if spec.gate_proj is not None else [])
        self.down = Linear(fuse_rows(mats), rt)
        self.kv_col = spec.q_rank
        self.gate_col = spec.q_rank + (r + p if spec.own_kv else 0)
        self.q_norm = weights[spec.dq_norm]
        self.kv_norm = weights[spec.dkv_norm] if spec.own_kv else None
        if self.kv_norm is not None and self.kv_norm.dtype != self.q_norm.dtype:
            self.q_norm, self.kv_norm = self.q_norm.float(), self.kv_norm.float()
        self.uq = Linear(weights[spec.uq_proj], rt)
        # per head: K_h^T as the matrix of a product "query times weight transposed" [H, R, D], V_h as it is [H, E, R]
        pad = self.rank - r
        self.uk_t = F.pad(weights[spec.uk_proj].reshape(h, d, r).transpose(1, 2), (0, 0, 0, pad)).contiguous()
        self.uv = F.pad(weights[spec.uv_proj].reshape(h, e, r), (0, pad)).contiguous()
        self.o = Linear(weights[spec.o_proj], rt)
        self.rot = None
        if p:
            cos, sin, dims = build_position(spec.position, rt).tables()
            if dims > p:
                raise ValueError(f"a rotation of {dims} numbers does not fit the rotated part of {p}")
            self.rot = kernels.LatentRotation(at=self.rank, src=p, width=rot_width, half=dims // 2, cos=cos, sin=sin)

    def forward(self, ctx, cache_id: int, x):
        s = self.spec
        n, h, d, p = x.shape[0], s.n_heads, s.key_dim, s.rot_dim
        dev, act = x.device, self.rt.dtype
        proj = self.down(x)
        k_pages, _v, group = ctx.storage.pages(cache_id)
        plane = k_pages.view(k_pages.shape[0], k_pages.shape[2], k_pages.shape[3])     # [pages, page_size, cached vector]
        table = ctx.block_tables[group]
        cq = torch.empty((n, s.q_rank), dtype=act, device=dev)
        kernels.latent_norm_store(proj, 0, self.q_norm, cq, self.kv_col, self.kv_norm, plane if s.own_kv else None,
                                  table, ctx.row_request, ctx.positions, s.eps, rot=self.rot)
        q = self.uq(cq).view(n, h, d + p)
        q_lat = torch.empty((h, n, self.rank), dtype=act, device=dev)     # the queries in the latents' space
        kernels.batched_linear(q[:, :, :d].transpose(0, 1), self.uk_t, q_lat, act)
        mixed = torch.empty_like(q_lat)
        rows_for_dispatch = ctx.extra.get("dispatch_rows", ctx.n_rows)
        # a window bounds the keys that a row can see (and one key tile more, where it begins inside one)
        most_keys = ctx.max_kv_len if s.window is None else min(ctx.max_kv_len, s.window + kernels.LATENT_TILE_KEYS)
        n_slices = kernels.latent_slices(rows_for_dispatch, h, most_keys)
        tiles = None
        if not ctx.decode_only and n_slices == 1 and act == torch.bfloat16 and self.rank % 32 == 0:
            # prompt portions: two tokens of a request per block (the kernel's tensor-core form)
            tile_req, tile_row0, n_tiles = ctx.attention_tiles(kernels.LATENT_TILE_TOKENS)
            tiles = (tile_req, tile_row0, n_tiles, ctx.q_start)
        kernels.latent_attention(q_lat, plane, table, ctx.row_request, ctx.positions, s.scale, s.window, mixed, n_slices,
                                 tiles, q_rot=q[:, :, d:] if p else None, rot=self.rot)
        if s.gate_proj is None:
            out = torch.empty((n, h * s.value_dim), dtype=act, device=dev)
            kernels.batched_linear(mixed, self.uv, out.view(n, h, s.value_dim).transpose(0, 1), act)
            return self.o(out)
        heads = torch.empty((h, n, s.value_dim), dtype=act, device=dev)
        kernels.batched_linear(mixed, self.uv, heads, act)
        gated = torch.empty((n, h * s.value_dim), dtype=act, device=dev)
        kernels.head_norm_gate(heads.transpose(0, 1), proj[:, self.gate_col:], None, False, kernels.GATE_SIGMOID, s.eps,
                               gated)
        return self.o(gated)


register_mixer("latent_attention", LatentAttention)
