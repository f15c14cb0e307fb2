"""The gated delta rule: a matrix memory per head with one decay and one write rate.

With h the mixer's input, `num_heads` value heads of `v_head_dim` channels and
`num_kv_heads` query/key heads of `head_dim` (head i reads query/key head
i // (num_heads / num_kv_heads)):
  q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))
      one filter a channel over the last `taps` tokens, zeros before the start
  q, k <- x / sqrt(sum(x^2) + unit_eps) per head, q also times `scale`
  beta = sigmoid(W_b h),  g = exp(-exp(A_log) softplus(W_a h + dt_bias))     one a head
  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
  o = o / rms(o) per head (eps), times a weight the heads share, times silu(W_g h)
  out = W_o o
Per sequence the state is the last taps - 1 rows of the convolutions' inputs and S
of every head, 32-bit, one vector of the cache's state group, zero at a
sequence's start.  The projections are one product in the compute type with
32-bit results; everything between it and the output product is 32-bit.
"""

from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..cache.specs import StateSpec
from ..config.spec import MixerSpec
from ..errors import InvalidInput
from .registry import TensorInfo, register_mixer


@register_mixer("gated_delta")
class GatedDelta:
    capturable = True  # sequences' slots and rows are read from device memory
    STACK = ("q_proj", "k_proj", "v_proj", "g_proj", "b_proj", "a_proj")

    def __init__(self, spec: MixerSpec, dtype: torch.dtype, device):
        if spec.num_heads % spec.num_kv_heads:
            raise InvalidInput("num_heads must be a multiple of num_kv_heads")
        self.spec = spec
        self.dtype = dtype
        self.device = device
        self.heads, self.kv_heads = int(spec.num_heads), int(spec.num_kv_heads)
        self.dim, self.vdim = int(spec.head_dim), int(spec.value_dim)
        self.taps = int(spec.param("taps", 1))
        self.unit_eps = float(spec.param("unit_eps"))
        self.eps = float(spec.param("eps"))
        self.channels = 2 * self.kv_heads * self.dim + self.heads * self.vdim
        # where S begins in a slot's vector, and its floats: key channels and both parts in fours
        self.state_off = ((self.taps - 1) * self.channels + 3) // 4 * 4
        self.state_floats = self.heads * self.vdim * ((self.dim + 3) // 4 * 4)
        self.stacked = self.filters = self.dt_bias = self.A = self.norm = self.o = None

    @classmethod
    def tensor_specs(cls, spec: MixerSpec) -> Dict[str, TensorInfo]:
        W, H, G, d, dv = spec.hidden_size, spec.num_heads, spec.num_kv_heads, spec.head_dim, spec.value_dim
        taps = int(spec.param("taps", 1))
        return {
            "q_proj": TensorInfo((G * d, W), "matrix"), "k_proj": TensorInfo((G * d, W), "matrix"),
            "v_proj": TensorInfo((H * dv, W), "matrix"), "g_proj": TensorInfo((H * dv, W), "matrix"),
            "b_proj": TensorInfo((H, W), "matrix"), "a_proj": TensorInfo((H, W), "matrix"),
            "q_conv": TensorInfo((G * d, taps), "filter"), "k_conv": TensorInfo((G * d, taps), "filter"),
            "v_conv": TensorInfo((H * dv, taps), "filter"),
            "A_log": TensorInfo((H,), "bias"), "dt_bias": TensorInfo((H,), "bias"),
            "norm": TensorInfo((dv,), "norm"), "o_proj": TensorInfo((W, H * dv), "matrix"),
        }

    def cache_spec(self) -> StateSpec:
        return StateSpec((self.state_off + self.state_floats,), "float32")

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        def dev(t):
            return t.to(device=self.device, dtype=self.dtype)

        def f32(t):
            return t.to(device=self.device, dtype=torch.float32).contiguous()

        mats = [dev(tensors[r]) for r in self.STACK]
        rows = sum(m.shape[0] for m in mats)
        # zero rows up to a multiple of 8: the product's rows stay 16-byte aligned
        pad = torch.zeros((-rows % 8, self.spec.hidden_size), dtype=self.dtype, device=self.device)
        self.stacked = torch.cat(mats + [pad], dim=0).contiguous()
        self.gate_col = self.channels
        self.b_col = self.gate_col + self.heads * self.vdim
        self.a_col = self.b_col + self.heads
        # transposed, [taps, channels]: neighbouring channels' taps side by side
        self.filters = torch.cat([f32(tensors[k]) for k in ("q_conv", "k_conv", "v_conv")], dim=0).t().contiguous()
        self.dt_bias = f32(tensors["dt_bias"])
        self.A = (-torch.exp(f32(tensors["A_log"]))).contiguous()  # made once: the weights do not change
        self.norm = f32(tensors["norm"])
        self.o = dev(tensors["o_proj"]).contiguous()

    def forward(self, x, ctx):
        batch, state = ctx.batch, ctx.state
        proj = ops.linear(x, self.stacked, out_dtype=torch.float32)  # [q | k | v | g | b | a | zeros]
        ops.prof_mark("qkv_gemm")
        single = proj.shape[0] == batch.seq_slot.numel()  # a row a sequence: the filters' launch moves their state on
        qkv, gates = ops.gated_delta_prep(
            proj, self.b_col, self.a_col, self.filters, state, batch, self.dt_bias, self.A, self.unit_eps,
            self.spec.scale, self.heads, self.kv_heads, self.dim, self.vdim, update_state=single,
            exact=self.dtype == torch.float32)
        if not single:
            ops.conv_state_update(proj, 0, self.channels, None, self.taps, state, batch)
        ops.prof_mark("conv_post")
        o = ops.gated_delta_scan(qkv, gates, state, self.state_off, batch, self.heads, self.kv_heads, self.dim, self.vdim,
                                 exact=self.dtype == torch.float32)
        ops.prof_mark("scan")
        o = ops.group_norm_gate(o, self.norm, self.eps, self.heads, self.dtype, gate=proj, gate_col=self.gate_col,
                                activation="silu")
        ops.prof_mark("scan_norm")
        out = ops.linear(o, self.o, out_dtype=torch.float32)
        ops.prof_mark("o_proj")
        return out
