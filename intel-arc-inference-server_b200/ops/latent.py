"""Bindings of the latent-attention kernels (``csrc/latent.cu``), the norms on fp32 residual rows (``csrc/norm_rows.cu``)
and the linears over unquantised weights (``csrc/gemv_bf16.cu``).

The element type of a call (bf16, or fp32 for models served in 32-bit) is that of its tensors."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from . import lib as K

GEMV_ROWS = 16                       # most rows of the weight-streaming form
EPI_PART, EPI_BF16, EPI_SILU, EPI_RELU2 = 0, 1, 2, 4
ACT_NONE, ACT_SILU, ACT_RELU2 = 0, 1, 2


def _f32(t: torch.Tensor) -> int:
    if t.dtype not in (torch.float32, torch.bfloat16):
        raise TypeError(f"element type {t.dtype}")
    return int(t.dtype == torch.float32)


def gemv_splits(n: int, k: int) -> int:
    return K.lib().b2_gemv_bf16_splits(n, k)


def gemv_bf16(w, x, out, m: int, n: int, k: int, splits: int = 1, epi: int = EPI_PART):
    """``x @ w.T`` for ``m`` <= 16 rows: fp32 slices ``[splits][m][n]``, bf16, relu(x)^2 as bf16, or SiLU(gate) * up of
    interleave16 rows."""
    K._check(K.lib().b2_gemv_bf16(K._p(w), None, 1, K._p(x), x.stride(0), 1, K._p(out), m, n, k, splits, epi, K._stream()),
             "gemv_bf16")


def gemv_bf16_planes(w, x, plane_rows: int, out, m: int, n: int, k: int, splits: int = 1):
    """fp32 slices ``[splits][m][n]`` where rows ``n`` of the weight read plane ``min(n // plane_rows, planes - 1)`` of the
    activations ``x`` ``[planes][m][k]``."""
    K._check(K.lib().b2_gemv_bf16_planes(K._p(w), K._p(x), x.stride(1), plane_rows, x.shape[0], ctypes.c_longlong(x.stride(0)), K._p(out),
                                         m, n, k, splits, K._stream()), "gemv_bf16_planes")


def gemv_bf16_glu(w, x, out, m: int, n: int, k: int, limit: float, alpha: float, shift: float, gelu: bool = False, bias=None):
    """The gated product of ``gemm.gemm_glu`` for ``m`` <= 16 rows."""
    K._check(K.lib().b2_gemv_bf16_glu(K._p(w), K._p(x), x.stride(0), K._p(out), m, n, k, ctypes.c_float(limit), ctypes.c_float(alpha),
                                      ctypes.c_float(shift), int(gelu), K._p(bias), K._stream()), "gemv_bf16_glu")


def glu_rows_f32(x, out, m: int, n: int, limit: float, alpha: float, shift: float, gelu: bool = False, bias=None):
    K._check(K.lib().b2_glu_rows_f32(K._p(x), K._p(out), m, n, ctypes.c_float(limit), ctypes.c_float(alpha), ctypes.c_float(shift),
                                     int(gelu), K._p(bias), K._stream()), "glu_rows_f32")


def gemv_bf16_experts(w, ids, batches: int, x, x_div: int, out, n: int, k: int, splits: int = 1, epi: int = EPI_PART):
    """Batch ``b``: row ``b // x_div`` of ``x`` against expert ``ids[b]`` of ``w`` ``[E][n][k]``."""
    K._check(K.lib().b2_gemv_bf16(K._p(w), K._p(ids), batches, K._p(x), x.stride(0), x_div, K._p(out), 1, n, k, splits, epi,
                                  K._stream()), "gemv_bf16_experts")


def linear_f32(a, w, c, m: int, squared: bool = False):
    """``c[:m] = a[:m] @ w.T`` in fp32 (``c``: rows of any stride); ``squared``: relu of it, squared."""
    n, k = w.shape
    K._check(K.lib().b2_linear_f32(K._p(a), K._p(w), K._p(c), m, n, k, c.stride(0), int(squared), K._stream()), "linear_f32")


def linear_f32_experts(w, ids, batches: int, x, x_div: int, out, act: int):
    """Batch ``b``: row ``b // x_div`` of ``x`` against expert ``ids[b]``; ``act``: ``ACT_SILU`` (of interleave16 rows), ``ACT_RELU2``."""
    e, n, k = w.shape
    for b0 in range(0, batches, 65520 // x_div * x_div):      # grid rows of one launch
        nb = min(batches - b0, 65520 // x_div * x_div)
        outs = n // 2 if act == ACT_SILU else n
        K._check(K.lib().b2_linear_f32_rows(K._p(w), K._p(ids[b0:]), nb, K._p(x[b0 // x_div:]), x.stride(0), x_div,
                                            K._p(out.view(-1)[b0 * outs:]), n, k, act, K._stream()), "linear_f32_rows")


# ----------------------------------------------------------------------------- norms and residual rows
def embed_rows(embed, tokens, m: int, x, h, flag=None):
    K._check(K.lib().b2_embed_rows(K._p(embed), K._p(tokens), embed.shape[0], m, embed.shape[1], K._p(x), K._p(h), _f32(embed),
                                   K._p(flag), K._stream()), "embed_rows")


def sublayer_norm(y, m: int, width: int, w, eps: float, x, h, *, slices: int = 1, slice_elems: int = 0, row_elems: int = 0,
                  slots: int = 1, slot_w=None, row_of=None, add: bool = True):
    """``x[:m] += LN(y) * w`` and ``h`` = the new rows in its element type.  ``y`` row (or slot) ``r`` starts at
    ``r * row_elems`` and has ``slices`` slices ``slice_elems`` apart; with ``slots`` > 1 a row is the sum of its slots
    weighted by ``slot_w`` (slot ``s`` of row ``i``: value row ``row_of[i * slots + s]``, or ``i * slots + s``)."""
    K._check(K.lib().b2_sublayer_norm(K._p(y), int(y.dtype == torch.bfloat16), K._p(row_of), K._p(slot_w),
                                      ctypes.c_longlong(slice_elems), ctypes.c_longlong(row_elems), slots, slices, m, width,
                                      x.shape[-1], K._p(w), ctypes.c_float(eps), K._p(x), K._p(h), _f32(h), int(add),
                                      K._stream()), "sublayer_norm")


def layer_norm_rows(x, rows, w, eps: float, m: int, width: int, h):
    """``h[i] = LN(x[rows[i]]) * w`` (``rows`` None: row ``i``)."""
    K._check(K.lib().b2_layer_norm_rows(K._p(x), K._p(rows), K._p(w), ctypes.c_float(eps), m, width, x.shape[-1], K._p(h),
                                        _f32(h), K._stream()), "layer_norm_rows")


def row_argmax(logits, m: int, n: int, val, idx):
    K._check(K.lib().b2_row_argmax(K._p(logits), m, n, K._p(val), K._p(idx), K._stream()), "row_argmax")


# ----------------------------------------------------------------------------- latent attention
def prep(part, s: int, m: int, g, q_norm, kv_norm, eps: float, req, pos, block_table, rope, cq, cache):
    """``g``: ``models.latent.LatentGeometry``; ``rope``: (cos, sin) tables of ``g.rope_dims / 2`` columns."""
    K._check(K.lib().b2_latent_prep(K._p(part), s, m, g.q_rank, g.qp, g.kv_rank, g.kvp, g.rot, g.rp, K._p(q_norm),
                                    K._p(kv_norm), ctypes.c_float(eps), K._p(req), K._p(pos), K._p(block_table),
                                    block_table.shape[1], K._p(rope[0]), K._p(rope[1]), g.rope_dims, K._p(cq), K._p(cache),
                                    _f32(cache), K._stream()), "latent_prep")


def absorb(q, s: int, m: int, g, w_uk, pos, rope, out):
    K._check(K.lib().b2_latent_absorb(K._p(q), s, m, g.heads, g.dn, g.rp, g.rot, g.kvp, K._p(w_uk), K._p(pos), K._p(rope[0]),
                                      K._p(rope[1]), g.rope_dims, K._p(out), _f32(out), K._stream()), "latent_absorb")


def rows_ok(g) -> bool:
    return bool(K.lib().b2_latent_rows_ok(g.heads, g.kvp, g.rp))


def rows(q, cache, m: int, g, req, pos, block_table, o_part, ml_part, nsplit: int, window: int, scale: float):
    K._check(K.lib().b2_latent_rows(K._p(q), K._p(cache), cache.shape[0], m, g.heads, g.kvp, g.rp, K._p(req), K._p(pos),
                                    K._p(block_table), block_table.shape[1], K._p(o_part), K._p(ml_part), nsplit, window,
                                    ctypes.c_float(scale), K._stream()), "latent_rows")


def simple(q, cache, m: int, g, req, pos, block_table, o_part, ml_part, window: int, scale: float):
    K._check(K.lib().b2_latent_simple(K._p(q), K._p(cache), m, g.heads, g.kvp, g.rp, K._p(req), K._p(pos), K._p(block_table),
                                      block_table.shape[1], K._p(o_part), K._p(ml_part), window, ctypes.c_float(scale),
                                      _f32(cache), K._stream()), "latent_simple")


def merge(o_part, ml_part, m: int, g, nsplit: int, w_uv, out):
    K._check(K.lib().b2_latent_merge(K._p(o_part), K._p(ml_part), m, g.heads, nsplit, g.kvp, g.dv, K._p(w_uv), K._p(out),
                                     out.stride(0), _f32(out), K._stream()), "latent_merge")


def gather(cache, kreq, kpos, n: int, block_table, g, c, kr):
    K._check(K.lib().b2_latent_gather(K._p(cache), K._p(kreq), K._p(kpos), n, K._p(block_table), block_table.shape[1], g.kvp,
                                      g.rp, K._p(c), K._p(kr), K._stream()), "latent_gather")


def rope_q(q, pos, m: int, g, rope):
    K._check(K.lib().b2_latent_rope_q(K._p(q), K._p(pos), m, g.heads, g.dn, g.rp, K._p(rope[0]), K._p(rope[1]), g.rope_dims,
                                      K._stream()), "latent_rope_q")


def prefill_rows_per_tile(g) -> int:
    """Query rows one CTA column of the expanded prompt attention serves (0: the sizes are outside its forms)."""
    return K.lib().b2_attn_rows_per_tile(g.dn + g.rp, g.dv)


def attn_prefill_rows(q, k, kr, v, out, tiles, n_tiles: int, q_rows: int, k_rows: int, g, scale: float, window: int):
    K._check(K.lib().b2_attn_prefill_rows(K._p(q), K._p(k), K._p(kr), K._p(v), K._p(out), K._p(tiles), n_tiles, q_rows, k_rows,
                                          g.heads, g.dn, g.dn + g.rp, g.dv, ctypes.c_float(scale), window, K._stream()),
             "attn_prefill_rows")
