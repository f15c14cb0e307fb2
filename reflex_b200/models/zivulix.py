"""Zivulix as data: its typed config turned into a `ModelSpec`.

The design: a normed token embedding; layers that norm only what a sublayer
gives, x <- x + norm1(mixer(x)), x <- x + norm2(ff(x)), with norm weights stored
around zero; the mixer is a latent attention (one cached latent a position for
all heads' keys and values, beside it one rotated key part all heads share), a
grouped attention (biases, a half-split rotation of a head's first dimensions
with divided frequencies, queries and keys over their root mean square after
it, capped scores, a sliding window, values mixed with those of the first such
layer) or a gated delta rule (short filters and silu, unit queries and keys, a
matrix memory per head with one decay and one write rate, a per-head norm and a
silu gate); the feed-forward is gated with the tanh form of gelu, or absent;
the model's norm, then an untied head.  Tensor names are the checkpoint's; the
right columns of `*_NAMES` are the only place they occur.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.spec import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec
from ..config.zivulix import ZivulixConfig

LATENT_NAMES = (("q_proj", "mix.q"), ("kv_down", "mix.dkv"), ("kv_norm", "mix.dkv.norm"), ("k_up", "mix.uk"),
                ("v_up", "mix.uv"), ("o_proj", "mix.o"))
ATTENTION_NAMES = (("q_proj", "mix.q"), ("k_proj", "mix.k"), ("v_proj", "mix.v"), ("q_bias", "mix.q.b"),
                   ("k_bias", "mix.k.b"), ("v_bias", "mix.v.b"), ("value_mix", "mix.vmix"), ("o_proj", "mix.o"))
DELTA_NAMES = (("q_proj", "mix.q"), ("k_proj", "mix.k"), ("v_proj", "mix.v"), ("q_conv", "mix.q.conv"),
               ("k_conv", "mix.k.conv"), ("v_conv", "mix.v.conv"), ("b_proj", "mix.b"), ("a_proj", "mix.a"),
               ("A_log", "mix.A_log"), ("dt_bias", "mix.dt_bias"), ("g_proj", "mix.g"), ("norm", "mix.norm"),
               ("o_proj", "mix.o"))
DENSE_NAMES = (("gate_proj", "mlp.gate"), ("up_proj", "mlp.up"), ("down_proj", "mlp.down"))
BLOCK_NAMES = (("mixer_norm", "norm1"), ("feed_forward_norm", "norm2"))

UNIT_EPS = 1e-6  # fixed by the design: under the root of the delta rule's unit queries and keys


def rotation(rot: dict, head_dim: int):
    if not int(rot["dims"]):
        return None
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    return PositionSpec("rope_linear", head_dim=head_dim, rotary_dim=int(rot["dims"]), theta=float(rot["base"]),
                        params=(("factor", factor),))


def build_zivulix_spec(cfg: ZivulixConfig) -> ModelSpec:
    eps, W = cfg.norm_eps, cfg.width
    norm = NormSpec("rmsnorm", W, eps, weight_offset=1.0)
    layers = []
    mixes = False  # whether a layer before this one already mixes values
    for i, l in enumerate(cfg.layers):
        m = l.mixer
        if l.type == "latent_attention":
            mixer = MixerSpec(
                "latent_attention", hidden_size=W, num_heads=int(m["heads"]), num_kv_heads=1, head_dim=int(m["dim"]),
                v_head_dim=int(m["vdim"]), scale=float(m["scale"]), names=LATENT_NAMES,
                position=rotation(m["rot"], int(m["rot_dim"])),
                params=(("kv_rank", int(m["kv_rank"])), ("rot_dim", int(m["rot_dim"])), ("eps", eps)))
        elif l.type == "attention":
            mix = None
            if m.get("v_mix"):
                mix, mixes = ("mix" if mixes else "first"), True
            mixer = MixerSpec(
                "capped_attention", hidden_size=W, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]),
                head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]), scale=float(m["scale"]),
                window=int(m["mask"]["size"]) if m.get("mask") else None,
                position=rotation(m["rot"], int(m["dim"])), names=ATTENTION_NAMES,
                params=(("bias", True), ("unit_eps", eps), ("softcap", float(m.get("softcap") or 0.0)),
                        ("value_mix", mix)))
        else:
            mixer = MixerSpec(
                "gated_delta", hidden_size=W, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]),
                head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]), scale=float(m["dim"]) ** -0.5, names=DELTA_NAMES,
                params=(("taps", int(m["conv"])), ("unit_eps", UNIT_EPS), ("eps", eps)))
        ffn = None
        if l.mlp is not None:
            ffn = FeedForwardSpec("geglu", hidden_size=W, intermediate_size=int(l.mlp["ff"]), names=DENSE_NAMES)
        layers.append(LayerSpec(
            block="postnorm", prefix=f"l{i}.", mixer=mixer, feed_forward=ffn, mixer_norm=norm,
            feed_forward_norm=norm if ffn is not None else None, names=BLOCK_NAMES))
    return ModelSpec(
        architecture="zivulix", vocab_size=cfg.vocab, hidden_size=W, layers=layers, final_norm=norm,
        tie_word_embeddings=False, max_positions=cfg.max_positions, embedding_name="embed",
        embedding_norm=norm, embedding_norm_name="embed.norm", final_norm_name="final.norm", head_name="head")


ZIVULIX = register_architecture(("Zivulix", "zivulix"), ZivulixConfig.from_dict, build_zivulix_spec)
