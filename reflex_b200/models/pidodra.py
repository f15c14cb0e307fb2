"""Pidodra as data: its typed config turned into a `ModelSpec`.

The design: a token embedding times a scale; layers that norm the sum of a
multiple of the stream and what a sublayer makes of it, h = norm1(a h +
mixer(h)), h = norm2(a h + ff(h)); the mixer is a latent attention (queries
through a normed latent, one cached latent a position for all heads' keys and
values, beside it one rotated key part all heads share with neighbouring elements
as pairs, a sink in the softmax's denominator, a sigmoid gate on every element) or
a grouped attention (per-head RMS norm of queries and keys, a half-split rotation
with YaRN-scaled frequencies and magnitude, a sigmoid gate per head), which may use
the keys and values of an earlier layer in place of its own; the feed-forward is a
mixture of gated silu experts, chosen among the best groups and weighted by their
softmax scores as they are, or absent; the model's norm, then an untied head.
Tensor names are the checkpoint's; the right columns of `*_NAMES` are the only
place they occur.
"""

from __future__ import annotations

from ..config.pidodra import PidodraConfig
from ..config.registry import register_architecture
from ..config.spec import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, RunEntry

LATENT_NAMES = (("q_down", "mix.dq"), ("q_norm", "mix.dq.norm"), ("q_up", "mix.uq"), ("kv_down", "mix.dkv"),
                ("kv_norm", "mix.dkv.norm"), ("k_up", "mix.uk"), ("v_up", "mix.uv"), ("sink", "mix.sink"),
                ("gate", "mix.g"), ("o_proj", "mix.o"))
ATTENTION_NAMES = (("q_proj", "mix.q"), ("k_proj", "mix.k"), ("v_proj", "mix.v"), ("q_norm", "mix.q.norm"),
                   ("k_norm", "mix.k.norm"), ("g_proj", "mix.g"), ("o_proj", "mix.o"))
MOE_NAMES = (("router", "mlp.router"), ("expert_gate", "mlp.e{expert}.gate"), ("expert_up", "mlp.e{expert}.up"),
             ("expert_down", "mlp.e{expert}.down"))
BLOCK_NAMES = (("mixer_norm", "norm1"), ("feed_forward_norm", "norm2"))


def attention_position(rot: dict, head_dim: int):
    if not int(rot["dims"]):
        return None
    sc = rot.get("scaling")
    return PositionSpec("rope_yarn" if sc else "rope_neox", head_dim=head_dim, rotary_dim=int(rot["dims"]),
                        theta=float(rot["base"]),
                        params=tuple((k, float(sc[k])) for k in ("factor", "original", "fast", "slow")) if sc else ())


def build_pidodra_spec(cfg: PidodraConfig) -> ModelSpec:
    eps, W = cfg.norm_eps, cfg.width
    norm = NormSpec("rmsnorm", W, eps)
    layers, order = [], []
    for i, l in enumerate(cfg.layers):
        m = l.mixer
        source = m.get("kv_from") if l.type == "attention" else None
        if l.type == "latent_attention":
            rd = int(m["rot_dim"])
            mixer = MixerSpec(
                "latent_attention", hidden_size=W, num_heads=int(m["heads"]), num_kv_heads=1, head_dim=int(m["dim"]),
                v_head_dim=int(m["vdim"]), scale=float(m["scale"]), names=LATENT_NAMES,
                position=PositionSpec("rope_neox", head_dim=rd, rotary_dim=rd, theta=float(m["rot"]["base"]),
                                      params=(("pairing", "consecutive"),)),
                params=(("q_rank", int(m["q_rank"])), ("kv_rank", int(m["kv_rank"])), ("rot_dim", rd), ("eps", eps),
                        ("sink", True), ("gate", "element")))
        else:
            d = int(m["dim"])
            mixer = MixerSpec(
                "gqa_attention", hidden_size=W, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), head_dim=d,
                v_head_dim=int(m["vdim"]), scale=float(m["scale"]), qk_norm=NormSpec("rmsnorm", d, eps),
                position=attention_position(m["rot"], d), names=ATTENTION_NAMES,
                params=(("head_gate", True), ("reads_cache", source is not None)))
        ffn = None
        if l.mlp is not None:
            r = l.mlp["router"]
            g = r.get("groups")
            ffn = FeedForwardSpec(
                "moe", hidden_size=W, intermediate_size=int(l.mlp["expert"]["ff"]), names=MOE_NAMES,
                params=(("experts", int(r["experts"])), ("top", int(r["top"])), ("activation", "swiglu"),
                        ("scores", "softmax"), ("score_scale", float(1.0 if r.get("scale") is None else r["scale"])),
                        ("groups", (int(g["count"]), int(g["keep"])) if g else None)))
        layers.append(LayerSpec(
            block="sum_norm", prefix=f"l{i}.", mixer=mixer, feed_forward=ffn, mixer_norm=norm,
            feed_forward_norm=norm if ffn is not None else None, names=BLOCK_NAMES, params=(("alpha", cfg.alpha),)))
        # a layer that uses another's keys and values reads that layer's cache entry
        order.append(RunEntry(i, i if source is None else int(source), writes_cache=source is None))
    return ModelSpec(
        architecture="pidodra", vocab_size=cfg.vocab, hidden_size=W, layers=layers, final_norm=norm,
        tie_word_embeddings=False, max_positions=cfg.max_positions, embedding_name="embed",
        final_norm_name="final.norm", head_name="head", run_order=order, embedding_scale=cfg.embedding_scale)


PIDODRA = register_architecture(("Pidodra", "pidodra"), PidodraConfig.from_dict, build_pidodra_spec)
