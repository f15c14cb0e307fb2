"""Latent attention: queries and keys/values through low-rank latents, only
the key/value latent cached.

With h the mixer's input [rows, hidden]:
  c_q = RMSNorm(W_dq h),  q = W_uq c_q             per head `head_dim` elements
  c   = RMSNorm(W_dkv h)                           `kv_rank` elements, cached
  k_j = W_uk c_j,  v_j = W_uv c_j                  per head, never materialised
  s_ij = (q_i . k_j) * scale  for 0 <= i - j < window
  p = exp(s) / (sum_j exp(s_ij) + exp(sink_h))     the sink has no key and no value
  out = W_o concat_h( sigmoid(W_g h)_h * sum_j p_ij v_j )
There is no position encoding.

With `rot_dim` (the rotated form; without `q_rank` it takes q = W_q h) q has per head
`head_dim` unrotated and `rot_dim` rotated elements, [unrotated | rotated], and
W_dkv h has `rot_dim` more rows: one rotated key part r_j all heads share, not normed:
  s_ij = (q_i . k_j + rot(q_i') . rot(r_j)) * scale
`gate` "element" (of this form): out = W_o (sigmoid(W_g h) * concat_h(...)), element by
element.  A rotation of neighbouring elements (`pairing` "consecutive") becomes one of
halves by the order of the rotated rows of W_uq and W_dkv, the same for both, which
changes no score.
The cached row is then [c | rot(r) | zeros], and the folded query is followed by
its rotated part.  For a prompt's many rows the other order of the same products is
cheaper: every head's keys [W_uk c | rot(r)] and values W_uv c of the step's
sequences are made once from the cached rows, one product, and an ordinary
attention runs over them.

Since k_j = W_uk c_j, the score is
(W_uk,h^T q_i) . c_j and the weighted values are W_uv,h (sum_j p_ij c_j): the
attention runs over the cached latents themselves as one shared key/value head
of `kv_rank` elements (keys and values are the same rows of the cache), with
the query folded through W_uk before it and W_uv applied after it, head by
head.  Norms, scores, the softmax and the gates are 32-bit.
"""

from __future__ import annotations

import dataclasses
from typing import Dict

import torch

from .. import ops
from ..cache.specs import KVSpec
from ..config.spec import MixerSpec
from ..errors import InvalidInput
from .registry import POSITIONS, TensorInfo, register_mixer


@register_mixer("latent_attention")
class LatentAttention:
    capturable = True  # positions, slots and the page table are read from device memory

    @property
    def supports_fused_residual(self) -> bool:
        return not self.rotated

    def __init__(self, spec: MixerSpec, dtype: torch.dtype, device):
        self.spec = spec
        self.dtype = dtype
        self.device = device
        self.q_rank = int(spec.param("q_rank", 0) or 0)  # 0: queries straight from the input
        self.rot_dim = int(spec.param("rot_dim", 0) or 0)
        self.position = (POSITIONS.get(spec.position.kind)(spec.position, dtype, device)
                         if spec.position is not None else None)
        self.kv_rank = int(spec.param("kv_rank"))
        self.eps = float(spec.param("eps"))
        self.has_sink = bool(spec.param("sink", False))
        self.rotated = self.rot_dim > 0 or not self.q_rank  # cached rows with room beside the latent
        self.has_gate = spec.param("gate") == "head"
        self.element_gate = spec.param("gate") == "element"
        if not self.rotated and self.position is not None:
            raise InvalidInput("latent_attention: a rotation needs a rotated part")
        if self.has_gate if self.rotated else self.element_gate:
            raise InvalidInput("latent_attention: a gate per head goes with no rotated part, one per element with one")
        # elements of a cached row: the latent and the rotated part, in steps the tensor-core kernels take
        step = ops.LATENT_WIDTH_STEP if dtype == torch.bfloat16 else 16
        self.width = (self.kv_rank + self.rot_dim + step - 1) // step * step if self.rotated else self.kv_rank
        # the form that makes every head's keys and values (prompts): padded key and value sizes
        d, dv = spec.head_dim + self.rot_dim, spec.value_dim
        self.dk, self.dvp = (d + 63) // 64 * 64, (dv + 63) // 64 * 64
        self.expands = (self.rotated and dtype == torch.bfloat16 and self.dk <= 192 and self.dvp <= 128
                        and self.dvp <= self.dk and dv % 16 == 0 and spec.scale > 0)
        self.kv_up = None
        self.down = self.q_up = self.k_absorb = self.v_up = self.o = None
        self.q_norm = self.kv_norm = self.sink = None

    @classmethod
    def tensor_specs(cls, spec: MixerSpec) -> Dict[str, TensorInfo]:
        W, H, d, dv = spec.hidden_size, spec.num_heads, spec.head_dim, spec.value_dim
        qr, kr = int(spec.param("q_rank", 0) or 0), int(spec.param("kv_rank"))
        rot = int(spec.param("rot_dim", 0) or 0)
        if qr:
            out = {"q_down": TensorInfo((qr, W), "matrix"), "q_norm": TensorInfo((qr,), "norm"),
                   "q_up": TensorInfo((H * (d + rot), qr), "matrix")}
        else:
            out = {"q_proj": TensorInfo((H * (d + rot), W), "matrix")}
        out.update({
            "kv_down": TensorInfo((kr + rot, W), "matrix"), "kv_norm": TensorInfo((kr,), "norm"),
            "k_up": TensorInfo((H * d, kr), "matrix"), "v_up": TensorInfo((H * dv, kr), "matrix"),
            "o_proj": TensorInfo((W, H * dv), "matrix"),
        })
        if spec.param("sink", False):
            out["sink"] = TensorInfo((H,), "bias")
        if spec.param("gate") == "head":
            out["gate"] = TensorInfo((H, W), "matrix")
        elif spec.param("gate") == "element":
            out["gate"] = TensorInfo((H * dv, W), "matrix")
        return out

    def cache_spec(self) -> KVSpec:
        # one latent a position serves as key and as value
        return KVSpec(1, self.width, self.spec.window, shared_kv=True)

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        H, d, dv = s.num_heads, s.head_dim, s.value_dim

        def dev(t):
            return t.to(device=self.device, dtype=self.dtype)

        def f32(t):
            return t.to(device=self.device, dtype=torch.float32).contiguous()

        q_rows, kv_down = dev(tensors["q_up" if self.q_rank else "q_proj"]), dev(tensors["kv_down"])
        order = self._pair_order()
        if order is not None:  # rotated rows: all pairs' first elements, then all second ones
            q_rows = q_rows.view(H, d + self.rot_dim, -1)[:, order["query"]].reshape(q_rows.shape)
            kv_down = kv_down[order["key"]]
        parts = [dev(tensors["q_down"]) if self.q_rank else q_rows, kv_down]
        if self.has_gate:
            parts.append(dev(tensors["gate"]))

        def padded():
            # zero rows up to a multiple of 8: the product's rows stay 16-byte aligned
            rows = sum(p.shape[0] for p in parts)
            parts.append(torch.zeros((-rows % 8, s.hidden_size), dtype=self.dtype, device=self.device))

        if self.rotated:
            padded()
        if self.element_gate:
            self.gate_col = sum(p.shape[0] for p in parts)
            parts.append(dev(tensors["gate"]))
            padded()
        self.down = torch.cat(parts, dim=0).contiguous()  # one product for both latents and the gates
        if self.q_rank:
            self.q_up = q_rows.contiguous()
            self.q_norm = f32(tensors["q_norm"])
        # W_uk per head, transposed: [H, kv_rank, dim], so that q_h -> W_uk,h^T q_h is a per-head product
        self.k_absorb = dev(tensors["k_up"]).view(H, d, self.kv_rank).transpose(1, 2).contiguous()
        self.v_up = dev(tensors["v_up"]).view(H, dv, self.kv_rank).contiguous()
        self.o = dev(tensors["o_proj"]).contiguous()
        self.kv_norm = f32(tensors["kv_norm"])
        if self.expands:
            # one matrix from a cached row to every head's key [W_uk c | rotated part | zeros] (the
            # rotated part passes through) and value
            rank, rot = self.kv_rank, self.rot_dim
            up = torch.zeros((H * (self.dk + self.dvp), self.width), dtype=self.dtype, device=self.device)
            keys = up[: H * self.dk].view(H, self.dk, self.width)
            keys[:, :d, :rank] = dev(tensors["k_up"]).view(H, d, rank)
            for j in range(rot):
                keys[:, d + j, rank + j] = 1.0
            up[H * self.dk:].view(H, self.dvp, self.width)[:, :dv, :rank] = dev(tensors["v_up"]).view(H, dv, rank)
            self.kv_up = up
        self.sink = f32(tensors["sink"]) if self.has_sink else None

    def forward(self, x, ctx, residual=None):
        s = self.spec
        kv, batch = ctx.kv, ctx.batch
        H = s.num_heads
        if self.rotated:
            return self._forward_rotated(x, ctx)
        proj = ops.linear(x, self.down, out_dtype=torch.float32)
        ops.prof_mark("qkv_gemm")
        cq, gate = ops.latent_post(proj, self.q_norm, self.kv_norm, self.eps, batch.row_pos, batch.row_slot,
                                   kv.k_pages, kv.page_table, kv.page_size, self.q_rank, self.kv_rank,
                                   H if self.has_gate else 0, ctx.writes_cache, self.dtype)
        ops.prof_mark("latent_post")
        q = ops.linear(cq, self.q_up)
        ops.prof_mark("q_up")
        qa = ops.heads_linear(q, self.k_absorb)  # [rows, H * kv_rank]
        ops.prof_mark("q_absorb")
        attn = ops.attention(qa, kv.k_pages, kv.k_pages, kv.page_table, kv.page_size, batch, H, 1,
                             self.kv_rank, s.window, s.scale, sink=self.sink)
        ops.prof_mark("attn")
        vals = ops.heads_linear(attn, self.v_up, scale=gate if self.has_gate else None)
        ops.prof_mark("v_up")
        if residual is not None:
            fused = ops.linear_residual(vals, self.o, residual[0], residual[1])
            if fused is not None:
                ops.prof_mark("o_proj")
                return None if fused is ops.ADDED else fused
        out = ops.linear(vals, self.o, out_dtype=torch.float32)
        ops.prof_mark("o_proj")
        return out

    def _pair_order(self):
        """The order that turns pairs of neighbours into pairs of halves, for a head's query
        rows and for the rows of W_dkv; None where the pairs are halves already."""
        if self.position is None or self.position.rotation().pairing == "half":
            return None
        pairs = torch.arange(self.rot_dim, device=self.device)
        halves = torch.cat([pairs[0::2], pairs[1::2]])
        return {"query": torch.cat([torch.arange(self.spec.head_dim, device=self.device), self.spec.head_dim + halves]),
                "key": torch.cat([torch.arange(self.kv_rank, device=self.device), self.kv_rank + halves])}

    def _rotation(self):
        if self.position is None:
            return None
        return dataclasses.replace(self.position.rotation(), pairing="half")  # `_pair_order` made it so

    def _forward_rotated(self, x, ctx):
        """The form with a rotated part; the delta [rows, hidden] comes back 32-bit."""
        s, kv, batch = self.spec, ctx.kv, ctx.batch
        H, d = s.num_heads, s.head_dim
        proj = ops.linear(x, self.down, out_dtype=torch.float32)
        ops.prof_mark("qkv_gemm")
        rotation = self._rotation()
        expand = self._expand(batch)
        gate = (proj, self.gate_col) if self.element_gate else None
        rows, writes = proj, ctx.writes_cache
        if self.q_rank:
            cq = ops.latent_low_post(proj, self.q_norm, self.kv_norm, self.eps, rotation, batch.row_pos, batch.row_slot,
                                     kv.k_pages, kv.page_table, kv.page_size, self.q_rank, self.kv_rank, self.rot_dim,
                                     self.width, writes, self.dtype)
            ops.prof_mark("latent_post")
            rows = ops.linear(cq, self.q_up, out_dtype=torch.float32 if x.shape[0] <= ops.GEMV_MAX_ROWS else None)
            ops.prof_mark("q_up")
            writes = False  # the latents are cached already: only queries are left
        post = (rows, self.kv_norm, self.eps, rotation, batch.row_pos, batch.row_slot, kv.k_pages, kv.page_table,
                kv.page_size, H, d, self.rot_dim, self.kv_rank, self.width, writes, self.dtype)
        if expand:
            if self.q_rank and rows.dtype == self.dtype and d + self.rot_dim == self.dk and self.rot_dim % 4 == 0 \
                    and rotation is not None:
                q = ops.rotate_tails_(rows, H, self.rot_dim, rotation, batch.row_pos)  # as wide as they are to be
            else:
                q = ops.latent_rot_post(*post, query_width=self.dk)
            ops.prof_mark("latent_post")
            rows, base = ops.latent_gather(kv.k_pages, kv.page_table, kv.page_size, batch, self.width)
            both = ops.linear(rows, self.kv_up)
            ops.prof_mark("kv_up")
            vals = ops.attention_prefill_tc_rows(q, both, base, batch, H, self.dk, self.dvp, s.value_dim, s.window,
                                                 s.scale, sink=self.sink, gate=gate)
            ops.prof_mark("attn")
        else:
            flat, qa = ops.latent_rot_post(*post)
            ops.prof_mark("latent_post")
            ops.heads_linear(flat, self.k_absorb, out=qa)
            ops.prof_mark("q_absorb")
            attn = ops.latent_attention(qa, kv.k_pages, kv.page_table, kv.page_size, batch, H, self.width,
                                        self.kv_rank, s.window, s.scale, sink=self.sink)
            ops.prof_mark("attn")
            # of each head the latent's elements; the rest is dropped
            vals = ops.heads_linear(attn, self.v_up, gate=gate)
            ops.prof_mark("v_up")
        out = ops.linear(vals, self.o, out_dtype=torch.float32)
        ops.prof_mark("o_proj")
        return out

    def _expand(self, batch) -> bool:
        """Whether this step makes every head's keys and values: a prompt's rows share them."""
        if not self.expands or batch.max_new < ops.LATENT_EXPAND_MIN_ROWS:
            return False
        rows = sum(a + b for a, b in zip(batch.starts, batch.new_counts))
        return 2 * rows * self.spec.num_heads * (self.dk + self.dvp) <= ops.LATENT_EXPAND_MAX_BYTES
