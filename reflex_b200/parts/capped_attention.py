"""Grouped-query attention with capped scores, queries and keys of unit root mean
square, and values mixed across layers.

With h the mixer's input [rows, hidden]:
  q = W_q h + b_q, k = W_k h + b_k, v = W_v h + b_v
  q, k <- rotated; then, with `unit_eps`, x / sqrt(mean(x^2) + unit_eps) per head
  v <- (1 - m) v + m v_first      where `value_mix` is "mix": m one stored number, v_first
                                  the values of the same tokens in the run that says "first"
  s_ij = (q_i . k_j) * scale, then softcap * tanh(s / softcap)    for 0 <= i - j < window
  out = W_o concat_h(sum_j softmax(s)_ij v_j)
The options are the spec's parameters: `bias`, `unit_eps` (None: no norm),
`softcap` (0: none), `value_mix` (None, "first", "mix").  The mixed v is what is
cached; a step's first values live as long as the step (`ctx.shared`), since a
token's values only ever meet those of the same token.  Key and value heads may
differ in size: both are stored `pad` wide (the larger of the two, rounded up to
16, zeros beyond), q and the output projection's columns are padded alike, and
one attention kernel serves both.  Rotation, norms, the mix, scores and softmax
are 32-bit.
"""

from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..cache.specs import KVSpec
from ..config.spec import MixerSpec
from ..errors import InvalidInput
from .registry import POSITIONS, TensorInfo, register_mixer


@register_mixer("capped_attention")
class CappedAttention:
    FIRST = "first_values"  # where a step's first values lie in `ctx.shared`

    def __init__(self, spec: MixerSpec, dtype: torch.dtype, device):
        if spec.num_heads % spec.num_kv_heads:
            raise InvalidInput("num_heads must be a multiple of num_kv_heads")
        self.spec = spec
        self.dtype = dtype
        self.device = device
        self.has_bias = bool(spec.param("bias", False))
        self.unit_eps = spec.param("unit_eps")
        self.softcap = float(spec.param("softcap", 0.0) or 0.0)
        self.value_mix = spec.param("value_mix")
        if self.value_mix not in (None, "first", "mix"):
            raise InvalidInput(f"capped_attention: value_mix must be None, 'first' or 'mix', got {self.value_mix!r}")
        self.position = (POSITIONS.get(spec.position.kind)(spec.position, dtype, device)
                         if spec.position is not None else None)
        self.pad = (max(spec.head_dim, spec.value_dim) + 15) // 16 * 16
        # a normed query or key is sqrt(dim) long at most (its rounding to 16 bits adds less than
        # a hundredth): no scaled score is larger than this
        self.score_bound = abs(spec.scale) * spec.head_dim * 1.02 if self.unit_eps is not None else 0.0
        self.qkv = self.bias = self.mix = self.o = None

    @property
    def capturable(self) -> bool:
        return self.position is None or bool(getattr(self.position, "capturable", False))

    @classmethod
    def tensor_specs(cls, spec: MixerSpec) -> Dict[str, TensorInfo]:
        W, H, G, d, dv = spec.hidden_size, spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim
        out = {
            "q_proj": TensorInfo((H * d, W), "matrix"), "k_proj": TensorInfo((G * d, W), "matrix"),
            "v_proj": TensorInfo((G * dv, W), "matrix"), "o_proj": TensorInfo((W, H * dv), "matrix"),
        }
        if spec.param("bias", False):
            out.update({"q_bias": TensorInfo((H * d,), "bias"), "k_bias": TensorInfo((G * d,), "bias"),
                        "v_bias": TensorInfo((G * dv,), "bias")})
        if spec.param("value_mix") is not None:
            out["value_mix"] = TensorInfo((), "bias")  # the first such layer stores one too and leaves it alone
        return out

    def cache_spec(self) -> KVSpec:
        return KVSpec(self.spec.num_kv_heads, self.pad, self.spec.window)

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        H, dv, pad = s.num_heads, s.value_dim, self.pad

        def dev(t):
            return t.to(device=self.device, dtype=self.dtype)

        def f32(t):
            return t.to(device=self.device, dtype=torch.float32).contiguous()

        mats = [dev(tensors[k]) for k in ("q_proj", "k_proj", "v_proj")]
        rows = sum(m.shape[0] for m in mats)
        # zero rows up to a multiple of 8: the product's rows stay 16-byte aligned
        zeros = torch.zeros((-rows % 8, s.hidden_size), dtype=self.dtype, device=self.device)
        self.qkv = torch.cat(mats + [zeros], dim=0).contiguous()
        if self.has_bias:
            self.bias = torch.cat([f32(tensors[k]) for k in ("q_bias", "k_bias", "v_bias")]).contiguous()
        if self.value_mix == "mix":
            self.mix = f32(tensors["value_mix"]).reshape(1)
        o = dev(tensors["o_proj"])
        if pad != dv:  # the attention's heads come out `pad` wide: zero columns for what lies beyond the values
            wide = torch.zeros((o.shape[0], H, pad), dtype=o.dtype, device=o.device)
            wide[:, :, :dv] = o.view(o.shape[0], H, dv)
            o = wide.view(o.shape[0], H * pad)
        self.o = o.contiguous()

    def forward(self, x, ctx):
        s, kv, batch = self.spec, ctx.kv, ctx.batch
        if not ctx.writes_cache:
            raise InvalidInput("capped_attention: a run of it writes its own cache entry")
        v_first = None
        if self.value_mix == "mix":
            v_first = ctx.shared.get(self.FIRST)
            if v_first is None:
                raise InvalidInput("capped_attention: no earlier run of this step kept its values")
        proj = ops.linear(x, self.qkv, out_dtype=torch.float32 if x.shape[0] <= ops.GEMV_MAX_ROWS else None)
        ops.prof_mark("qkv_gemm")
        q, kept = ops.rot_qkv_post(
            proj, self.bias, None if self.position is None else self.position.rotation(), self.unit_eps, self.mix,
            v_first, self.value_mix == "first", batch.row_pos, batch.row_slot, kv.k_pages, kv.v_pages, kv.page_table,
            kv.page_size, s.num_heads, s.num_kv_heads, s.head_dim, s.value_dim, self.pad, True, self.dtype)
        if kept is not None:
            ctx.shared[self.FIRST] = kept
        ops.prof_mark("norm_rope")
        attn = ops.attention(q, kv.k_pages, kv.v_pages, kv.page_table, kv.page_size, batch, s.num_heads,
                             s.num_kv_heads, self.pad, s.window, s.scale, softcap=self.softcap,
                             score_bound=self.score_bound)
        ops.prof_mark("attn")
        out = ops.linear(attn, self.o, out_dtype=torch.float32)
        ops.prof_mark("o_proj")
        return out
