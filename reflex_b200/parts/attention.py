"""Grouped-query attention over the paged cache.

q = x Wq^T, k = x Wk^T, v = x Wv^T (no bias); per-head RMSNorm of q and k when
the spec has one; rotary encoding of q and k; k and v written to the cache at
the row's position; then for the query at position p, head h (kv head
h / group): keys j with 0 <= p - j < window (all j <= p without a window),
softmax((q . k_j) * scale) in 32-bit, weighted sum of v_j; out = attn Wo^T
(src/model/dense.rs:1337-1431; src/kernels_cuda/attention_online.cuh:64-102).
The q, k, v weights are stacked into one matrix at load; the reference fuses
the three products by kernel instead (src/kernels_cuda/gemv_fused.cu:16-87).

Values may have another size than keys (`v_head_dim`): both are then stored `pad`
wide (the larger of the two in steps of 16, zeros beyond), q and Wo's columns are
padded alike.

Options, by the spec's parameters: `values_are_keys` (there is no Wv; a value
head is its key head as projected, before the norm and the rotation),
`output_gate` (a further matrix Wg; the concatenated heads are multiplied by
sigmoid(x Wg^T) before Wo), `head_gate` (Wg has a row a head, and the one number
sigmoid(x Wg^T)_h scales all that head h gives), `reads_cache` (the layer has no keys
and values of its own, and so no Wk, Wv and key norm: its runs read the entry of
another layer of the same head sizes) and `keep_first` (with a window: the first so many
positions of a sequence stay visible to every later query, i - j < window or
j < keep_first, and keep their own positions).

The part knows sizes only from its spec.  What it needs from the step is in
`ctx`: row positions, row slots, and the cache entry's pages and page table.
"""

from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from ..cache.specs import KVSpec
from ..config.spec import MixerSpec
from ..errors import InvalidInput
from .registry import NORMS, POSITIONS, TensorInfo, register_mixer


def any_reader(spec: MixerSpec) -> bool:
    """Whether a run of this mixer may read another run's keys and values (it then
    needs its query and gate rows apart from the key and value rows)."""
    return bool(spec.param("shares_cache", False))


@register_mixer("gqa_attention")
class GQAttention:
    def __init__(self, spec: MixerSpec, dtype: torch.dtype, device):
        if spec.num_heads % spec.num_kv_heads:
            raise InvalidInput("num_heads must be a multiple of num_kv_heads")
        self.spec = spec
        self.dtype = dtype
        self.device = device
        self.position = (
            POSITIONS.get(spec.position.kind)(spec.position, dtype, device)
            if spec.position is not None
            else None
        )
        self.values_are_keys = bool(spec.param("values_are_keys", False))
        self.output_gate = bool(spec.param("output_gate", False))
        self.head_gate = bool(spec.param("head_gate", False))
        self.reads_cache = bool(spec.param("reads_cache", False))
        self.keep_first = int(spec.param("keep_first", 0) or 0) if spec.window else 0
        d, dv = spec.head_dim, spec.value_dim
        plain = d == dv and not (self.head_gate or self.reads_cache)
        self.pad = d if plain else (max(d, dv) + 15) // 16 * 16
        if d != dv and (self.values_are_keys or self.output_gate) or self.output_gate and self.head_gate:
            raise InvalidInput("gqa_attention: values of another size go with neither option, and one gate is enough")
        self.general = (self.values_are_keys or self.output_gate or self.head_gate or self.reads_cache
                        or self.keep_first > 0 or d != dv)
        self.qkv = None
        self.q_only = None
        self.o = None
        self.q_norm = None
        self.k_norm = None

    @classmethod
    def tensor_specs(cls, spec: MixerSpec) -> Dict[str, TensorInfo]:
        H, d, dv = spec.hidden_size, spec.head_dim, spec.value_dim
        out = {
            "q_proj": TensorInfo((spec.num_heads * d, H), "matrix"),
            "k_proj": TensorInfo((spec.num_kv_heads * d, H), "matrix"),
            "v_proj": TensorInfo((spec.num_kv_heads * dv, H), "matrix"),
            "o_proj": TensorInfo((H, spec.num_heads * dv), "matrix"),
        }
        if spec.param("values_are_keys", False):
            del out["v_proj"]
        if spec.param("output_gate", False):
            out["g_proj"] = TensorInfo((spec.num_heads * dv, H), "matrix")
        elif spec.param("head_gate", False):
            out["g_proj"] = TensorInfo((spec.num_heads, H), "matrix")
        if spec.qk_norm is not None:
            out["q_norm"] = TensorInfo((d,), "norm")
            out["k_norm"] = TensorInfo((d,), "norm")
        if spec.param("reads_cache", False):
            for role in ("k_proj", "v_proj", "k_norm"):
                out.pop(role, None)
        return out

    def cache_spec(self) -> KVSpec:
        return KVSpec(self.spec.num_kv_heads, self.pad, self.spec.window, keep_first=self.keep_first)

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        def dev(t):
            return t.to(device=self.device, dtype=self.dtype)

        q = dev(tensors["q_proj"])
        stack = [q]
        if not self.reads_cache:
            stack.append(dev(tensors["k_proj"]))
            if not self.values_are_keys:
                stack.append(dev(tensors["v_proj"]))
        self.kv_cols = sum(t.shape[0] for t in stack)  # the q | k | v columns of the stacked product
        self.gate_col = self.kv_cols
        if self.head_gate:
            # zero rows so that the gate's columns, and the product's rows, start on 16 bytes
            stack.append(torch.zeros((-self.kv_cols % 8, q.shape[1]), dtype=self.dtype, device=self.device))
            self.gate_col += -self.kv_cols % 8
            stack.append(dev(tensors["g_proj"]))
            stack.append(torch.zeros((-self.spec.num_heads % 8, q.shape[1]), dtype=self.dtype, device=self.device))
        elif self.output_gate:
            stack.append(dev(tensors["g_proj"]))  # the gate's columns ride in the same product
        self.qkv = torch.cat(stack, dim=0).contiguous()
        # rows [0, nq*d) of the stacked matrix: the query part, for runs that
        # read another run's keys and values
        self.q_only = self.qkv[: q.shape[0]]
        self.q_gate = (torch.cat([q, dev(tensors["g_proj"])], dim=0).contiguous()
                       if self.output_gate and any_reader(self.spec) else None)
        o, dv = dev(tensors["o_proj"]), self.spec.value_dim
        if self.pad != dv:  # the attention's heads come out `pad` wide: zero columns for what lies beyond the values
            wide = torch.zeros((o.shape[0], self.spec.num_heads, self.pad), dtype=o.dtype, device=o.device)
            wide[:, :, :dv] = o.view(o.shape[0], self.spec.num_heads, dv)
            o = wide.view(o.shape[0], self.spec.num_heads * self.pad)
        self.o = o.contiguous()
        if self.spec.qk_norm is not None:
            self.q_norm = tensors["q_norm"].to(device=self.device, dtype=torch.float32).contiguous()
            if not self.reads_cache:
                self.k_norm = tensors["k_norm"].to(device=self.device, dtype=torch.float32).contiguous()

    supports_fused_residual = True
    accepts_normed_input = True  # its first product finishes a norm that the product before began

    @property
    def capturable(self) -> bool:
        """Positions, slots and the page table are read from device memory, so a
        decode step's launches may be captured, if the position part's may."""
        return self.position is None or bool(getattr(self.position, "capturable", False))

    def forward(self, x, ctx, residual=None):
        """x: normed rows (or rows awaiting their norm factor, `ops.NormedInput`).
        With `residual` = (hidden, next norm) the output projection may add
        itself to `hidden`; it then returns the rows for the product after that
        norm (an `ops.NormedInput`) or None (added, the norm not begun).
        Otherwise the delta [rows, hidden] is returned."""
        s = self.spec
        kv = ctx.kv  # the cache entry's view
        batch = ctx.batch
        w = self.qkv if ctx.writes_cache else self.q_only
        rotation = None if self.position is None else self.position.rotation()
        norm = s.qk_norm
        if self.general:
            return self._forward_general(x, ctx, rotation)
        if ops.qkv_fused_takes(x, s.head_dim, rotation, w):
            # a few rows: norms, rotation and the cache write are the product's epilogue
            q = ops.qkv_fused(
                x, w, self.q_norm, self.k_norm, norm.eps if norm else 0.0,
                norm.weight_offset if norm else 0.0, rotation, batch.row_pos, batch.row_slot,
                kv.k_pages, kv.v_pages, kv.page_table, kv.page_size, s.num_heads, s.num_kv_heads,
                s.head_dim, ctx.writes_cache)
            ops.prof_mark("qkv_gemm")
        else:
            qkv = ops.linear(x, w, out_dtype=torch.float32 if x.shape[0] <= ops.GEMV_MAX_ROWS else None)
            ops.prof_mark("qkv_gemm")
            q = ops.qkv_post(
                qkv, self.q_norm, self.k_norm, norm.eps if norm else 0.0,
                norm.weight_offset if norm else 0.0, rotation, batch.row_pos, batch.row_slot,
                kv.k_pages, kv.v_pages, kv.page_table, kv.page_size, s.num_heads, s.num_kv_heads,
                s.head_dim, ctx.writes_cache, self.dtype)
            ops.prof_mark("norm_rope")
        attn = ops.attention(q, kv.k_pages, kv.v_pages, kv.page_table, kv.page_size, batch,
                             s.num_heads, s.num_kv_heads, s.head_dim, s.window, s.scale)
        ops.prof_mark("attn")
        if residual is not None:
            fused = ops.linear_residual(attn, self.o, residual[0], residual[1])
            if fused is not None:
                ops.prof_mark("o_proj")
                return None if fused is ops.ADDED else fused  # None: nothing left to add
        out = ops.linear(attn, self.o, out_dtype=torch.float32)
        ops.prof_mark("o_proj")
        return out

    def _forward_general(self, x, ctx, rotation):
        """The form with any of the options: one stacked product [q | k | (v) | (gate)],
        `qkv_post` on its first columns, the attention, the gate, the output
        projection; the delta [rows, hidden] comes back 32-bit."""
        s, kv, batch, norm = self.spec, ctx.kv, ctx.batch, self.spec.qk_norm
        if isinstance(x, ops.NormedInput):
            raise InvalidInput("gqa_attention: this form takes plain normed rows")
        nq_cols = s.num_heads * s.head_dim
        if self.reads_cache and ctx.writes_cache:
            raise InvalidInput("gqa_attention: a layer without keys and values reads another's cache entry")
        if self.head_gate and not ctx.writes_cache and not self.reads_cache:
            raise InvalidInput("gqa_attention: with a gate per head a layer writes its own entry, or has none")
        if ctx.writes_cache or self.reads_cache:
            w, cols, gate_col = self.qkv, self.kv_cols, self.gate_col
        elif self.output_gate:
            if self.q_gate is None:
                raise InvalidInput("gqa_attention: a run that reads another's cache needs `shares_cache` in its spec")
            w, cols, gate_col = self.q_gate, nq_cols, nq_cols
        else:
            w, cols, gate_col = self.q_only, nq_cols, nq_cols
        proj = ops.linear(x, w, out_dtype=torch.float32 if x.shape[0] <= ops.GEMV_MAX_ROWS else None)
        ops.prof_mark("qkv_gemm")
        if self.pad != s.head_dim or self.pad != s.value_dim:
            q, _ = ops.rot_qkv_post(
                proj, None, rotation, None, None, None, False, batch.row_pos, batch.row_slot, kv.k_pages, kv.v_pages,
                kv.page_table, kv.page_size, s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim, self.pad,
                ctx.writes_cache, self.dtype,
                norms=(self.q_norm, self.k_norm, norm.eps, norm.weight_offset) if norm else None)
        else:
            q = ops.qkv_post(
                proj, self.q_norm, self.k_norm, norm.eps if norm else 0.0, norm.weight_offset if norm else 0.0,
                rotation, batch.row_pos, batch.row_slot, kv.k_pages, kv.v_pages, kv.page_table, kv.page_size,
                s.num_heads, s.num_kv_heads, s.head_dim, ctx.writes_cache, self.dtype,
                values_are_keys=self.values_are_keys, ld=cols)
        ops.prof_mark("norm_rope")
        attn = ops.attention(q, kv.k_pages, kv.v_pages, kv.page_table, kv.page_size, batch, s.num_heads,
                             s.num_kv_heads, self.pad, s.window, s.scale, keep_first=self.keep_first,
                             gate=(proj, gate_col) if self.head_gate else None)
        if self.output_gate:
            ops.sigmoid_gate_mul_(attn, proj, gate_col)
        ops.prof_mark("attn")
        out = ops.linear(attn, self.o, out_dtype=torch.float32)
        ops.prof_mark("o_proj")
        return out
