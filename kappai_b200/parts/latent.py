"""Attention over cached latents (kind ``latent_cache_attention``).

    c = norm(h Wdkv^T) * w            one low-rank latent a token (``kv_rank``), beside
    r = rot(h Wkr^T)                  a key part of ``rot_dim`` that all heads share, rotated by position
    q = h Wq^T                        a head [head_dim unrotated | rot_dim rotated]
    k_h = Wuk_h c ,  v_h = Wuv_h c    the heads' unrotated keys and their values
    s_h(t) = (q_h . k_h(t) + qr_h . r(t)) scale ,  causal softmax,  o_h = sum_t softmax(s_h)_t v_h(t)

and the concatenated heads, times ``sigmoid(h Wg^T)`` (``gate`` = ``"sigmoid"``), go through the output matrix.  Only c and
r are cached: one row a token in a page group of one plane, padded to a multiple of 64.  (:class:`~.attention.LatentAttention`
is the kind that expands the latents before it caches them.)

Decoded tokens, short portions and every row of the 32-bit mode run *absorbed*: the expanding matrices are applied to the
query and to the weighted sum of latents, and all heads read the cached rows as they are.  Longer portions (16-bit mode)
run *expanded*: the latents of the request's whole context are gathered from its pages, one product makes the heads'
keys and values of them, and a tiled kernel reads those (on the tcgen05 tensor cores for value heads of up to 128 columns).
csrc/latent.cu has the kernels and how they sum.

The query, the latent, the key part and the gate read the layer's input in one product; one kernel norms and rotates
what comes out of it and writes the cache row.  The gate of absorbed rows runs in the epilogue of their last product, that
of expanded rows in the attention kernel's last store.

Params: hidden_size, num_heads, head_dim, rot_dim, value_dim, kv_rank, scale, norm_eps, gate (None | "sigmoid"), position (None
| a rope PartSpec over at most rot_dim dimensions).
"""
from __future__ import annotations

from typing import Dict

import numpy as np
import torch

from ..cache.spec import PagedKVSpec
from ..config.schema import ConfigError, PartSpec
from ..ops import kernels as K
from ..ops.linear import linear
from .attention import PagedAttentionKernels, attention_tiles
from .base import Part, WeightSpec, make_part, register_part


def _up16(n: int) -> int:
    return -(-n // 16) * 16


def latent_tiles(segs):
    """Step tables of the expanded pass: the row tiles of :func:`~.attention.attention_tiles` and, for the segments that it
    takes, where their contexts' rows begin among the gathered ones (``ctx_base`` [n_seg + 1]; the leading short segments
    have none).  None for a step of short segments only."""
    tables = attention_tiles(segs)
    if tables is None:
        return None
    lead = tables.scalars["n_short_tiles"]
    ctx = [0 if i < lead else int(segs.seg_pos[i]) + segs.seg_len[i] for i in range(segs.n_seg)]
    base = np.concatenate([[0], np.cumsum(ctx)]).astype(np.int32)
    tables.arrays["ctx_base"] = base
    tables.scalars["n_ctx"] = int(base[-1])
    return tables


class LatentCacheAttention(PagedAttentionKernels, Part):
    category = "mixer"
    graph_safe = True

    def __init__(self, params, env):
        super().__init__(params, env)
        self.d = int(self._p("hidden_size"))
        self.H = int(self._p("num_heads"))
        self.dim = int(self._p("head_dim"))
        self.rdim = int(self._p("rot_dim"))
        self.vdim = int(self._p("value_dim", self.dim))
        self.rank = int(self._p("kv_rank"))
        self.scale = float(self._p("scale"))
        self.eps = float(self._p("norm_eps"))
        gate = self._p("gate", None)
        if gate not in (None, "sigmoid"):
            raise ConfigError(f"latent_cache_attention: gate='{gate}' (expected 'sigmoid' or none)")
        self.gated = gate is not None
        if min(self.H, self.dim, self.rdim, self.vdim, self.rank) < 1:
            raise ConfigError("latent_cache_attention: heads, head sizes and the rank must be positive")
        # the sizes as the kernels see them: zero rows and columns behind every part up to a multiple of 16
        self.dimp, self.rotp, self.vdimp, self.rankp = _up16(self.dim), _up16(self.rdim), _up16(self.vdim), _up16(self.rank)
        self.row = -(-(self.rankp + self.rotp) // 64) * 64                             # elements of a cache row and an absorbed query
        pos = self._p("position", None)
        pos = PartSpec("none") if pos is None else (PartSpec(**pos) if isinstance(pos, dict) else pos)
        self.position = make_part("position", pos, env)
        if not hasattr(self.position, "fused_rotary"):
            raise ConfigError("latent_cache_attention: the position encoding must be one that the kernels apply themselves")
        self.rotary = self.position.fused_rotary()
        if self.rotary[2] > self.rdim:
            raise ConfigError(f"latent_cache_attention: rotary_dim={self.rotary[2]} exceeds rot_dim={self.rdim}")
        self.expands = (env.dtype == torch.bfloat16 and self.dimp + self.rotp <= K.LATENT_PREFILL_MAX[0]
                        and self.vdimp <= K.LATENT_PREFILL_MAX[1])
        if self.expands:
            self.step_tables_key = ("latent_tiles",)

    def step_tables(self, segs):
        return latent_tiles(segs)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        d, H = self.d, self.H
        s = {"q_proj.weight": WeightSpec((H * (self.dim + self.rdim), d)), "kv_down.weight": WeightSpec((self.rank + self.rdim, d)),
             "kv_norm.weight": WeightSpec((self.rank,), "norm"), "k_up.weight": WeightSpec((H * self.dim, self.rank)),
             "v_up.weight": WeightSpec((H * self.vdim, self.rank)), "out_proj.weight": WeightSpec((d, H * self.vdim))}
        if self.gated:
            s["gate_proj.weight"] = WeightSpec((H * self.vdim, d))
        return s

    def bind(self, w):
        d, H = self.d, self.H

        def padded(x, *sizes):
            """x with zeros behind its own entries up to ``sizes``, axis by axis."""
            if tuple(x.shape) == sizes:
                return x.contiguous()
            out = torch.zeros(sizes, dtype=x.dtype, device=x.device)
            out[tuple(slice(0, n) for n in x.shape)] = x
            return out

        q = w["q_proj.weight"].reshape(H, self.dim + self.rdim, d)
        q = torch.cat([padded(q[:, :self.dim], H, self.dimp, d), padded(q[:, self.dim:], H, self.rotp, d)], 1).reshape(-1, d)
        kv = w["kv_down.weight"]
        rows = [q, padded(kv[:self.rank], self.rankp, d), padded(kv[self.rank:], self.rotp, d)]
        self.c_col = q.shape[0]
        self.g_col = self.c_col + self.rankp + self.rotp
        if self.gated:
            rows.append(padded(w["gate_proj.weight"].reshape(H, self.vdim, d), H, self.vdimp, d).reshape(-1, d))
        self.w_in = torch.cat(rows, 0).contiguous()                                    # (a multiple of 16 rows)
        self.norm_w = w["kv_norm.weight"].float().contiguous()
        uk = padded(w["k_up.weight"].reshape(H, self.dim, self.rank), H, self.dimp, self.rankp)
        uv = padded(w["v_up.weight"].reshape(H, self.vdim, self.rank), H, self.vdimp, self.rankp)
        self.w_uk_t = uk.transpose(1, 2).contiguous()                                  # [H, rank, dim]: onto the query
        self.w_uv = uv                                                                 # [H, vdim, rank]: onto the weighted latent
        self.w_ex = torch.cat([uk.reshape(-1, self.rankp), uv.reshape(-1, self.rankp)], 0).contiguous() if self.expands else None
        self.w_o = padded(w["out_proj.weight"].reshape(d, H, self.vdim), d, H, self.vdimp).reshape(d, -1)

    def cache_spec(self):
        return PagedKVSpec(1, self.row, planes=1)

    # (a mixer whose first product can be run together with others': see parallel.py)
    def input_product(self):
        return self.w_in, None

    def drop_input_product(self):
        self.w_in = None

    def forward(self, h, residual, ctx, cache):
        """``cache``: a :class:`~kappai_b200.cache.storage.KVLayerView` of one plane."""
        self.forward_projected(linear(h, self.w_in), residual, ctx, cache)

    def forward_projected(self, p, residual, ctx, cache):
        """``p``: the rows of the input product, [q | latent | key part | gate], possibly columns of a wider one."""
        H, n = self.H, ctx.n_rows
        view = ctx.paged[cache.group]
        tiles = ctx.tables.get(self.step_tables_key) if self.expands else None
        na = n if tiles is None else tiles.n_short_rows                                # rows that run absorbed: the first na
        qa = torch.empty((na, H, self.row), dtype=p.dtype, device=p.device) if na else None
        K.latent_prep(p, 0, self.c_col, H, self.dimp, self.rotp, self.rank, self.rankp, self.row, self.norm_w, self.eps, self.rotary,
                      ctx.positions, view.slot_map, cache.tensor if cache.writes else None, view.page_size, qa, na)
        o = torch.empty((n, H * self.vdimp), dtype=p.dtype, device=p.device)
        gate = p[:, self.g_col:self.g_col + H * self.vdimp] if self.gated else None
        if na:
            self._absorbed(p[:na], qa, o[:na], gate[:na] if self.gated else None, ctx, view, cache)
        if na < n:
            self._expanded(p, o, gate, ctx, view, cache, tiles)
        linear(o, self.w_o, out=residual, accumulate=True)

    def _absorbed(self, p, qa, o, gate, ctx, view, cache):
        H, n = self.H, p.shape[0]
        heads = lambda x, width: x.unflatten(1, (H, width))
        K.head_gemm(heads(p[:, :H * (self.dimp + self.rotp)], self.dimp + self.rotp)[:, :, :self.dimp], self.w_uk_t, qa[:, :, :self.rankp])
        ws = self._scratch(K.latent_split_scratch(n, H, self.rankp, self.row, ctx.max_context, view.page_size, p.dtype), p.device)
        u = torch.empty((n, H, self.rankp), dtype=p.dtype, device=p.device)
        K.latent_split(qa, cache.tensor, view.block_table, ctx.row_seg[:n], ctx.positions[:n], ws, ctx.max_context, u, self.scale, view.page_size)
        K.head_gemm(u, self.w_uv, heads(o, self.vdimp), None if gate is None else heads(gate, self.vdimp))

    def _expanded(self, p, o, gate, ctx, view, cache, tiles):
        H, t0, na = self.H, tiles.n_short_tiles, tiles.n_short_rows
        rows = K.latent_gather(cache.tensor, view.block_table, tiles.ctx_base, tiles.n_ctx, view.page_size)
        ex = linear(rows[:, :self.rankp], self.w_ex)
        q, sizes = p[:, :H * (self.dimp + self.rotp)], (self.rankp, self.dimp, self.rotp, self.vdimp)
        if K.latent_prefill_tc_ok(q, ex, self.dimp, self.rotp, self.vdimp):
            K.latent_prefill_tc(q, ex, rows, *sizes, ctx.cu_rows, ctx.seg_pos, tiles.big_tile_seg, tiles.big_tile_row0, tiles.ctx_base, o,
                                self.scale, H, gate)
            return
        K.latent_prefill(q, ex, rows, *sizes, ctx.cu_rows, ctx.seg_pos, tiles.tile_seg[t0:], tiles.tile_row0[t0:], tiles.ctx_base, o,
                         self.scale, H)
        if gate is not None:
            K.sigmoid_gate(o[na:], gate[na:])


register_part("mixer", "latent_cache_attention", LatentCacheAttention)
