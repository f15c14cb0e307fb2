"""Typed configuration of the Pidodra design, read from config.json.

config.json keys: `architecture` ("Pidodra"), `vocab`, `width`, `norm.eps`,
`embedding.scale`, `postln_alpha` (the stream's factor in every norm's sum), and
`layers`, a list whose entries give `type` (the mixer: "latent_attention" or
"attention"), `mixer` (its sizes and constants) and `mlp` (`kind` "moe" with
`expert.ff` and `router`: `experts`, `top`, optional `scale` and `groups` {`count`,
`keep`}; null for a layer without a feed-forward).

A "latent_attention" mixer: `heads`, `dim` (unrotated query/key dimensions a
head), `rot_dim` (rotated ones), `vdim`, `q_rank`, `kv_rank`, `scale`, `rot`
{`base`, `dims` = `rot_dim`}.  An "attention" mixer: `heads`, `kv_heads`, `dim`,
`vdim`, `scale`, `rot` {`base`, `dims`, optional `scaling` {`factor`, `original`,
`fast`, `slow`}}, optional `kv_from` (the layer whose keys and values it uses).
Every size and every constant that differs between models comes from here.
Missing or ill-typed keys are reported together, by name.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from ..errors import CheckpointError

NUM = (int, float)

SIZES = {
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"),
    "attention": ("heads", "kv_heads", "dim", "vdim"),
}
SCALING = ("factor", "original", "fast", "slow")


@dataclass
class PidodraLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclass
class PidodraConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    alpha: float
    layers: List[PidodraLayer] = field(default_factory=list)
    torch_dtype: str = "bfloat16"
    # the design fixes no longest context; the cache bounds it
    max_positions: int = 1 << 20
    raw: Dict[str, Any] = field(default_factory=dict)

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any]) -> "PidodraConfig":
        problems: List[str] = []

        def need(d, key, types, where):
            v = d.get(key) if isinstance(d, dict) else None
            if v is None or isinstance(v, bool) or not isinstance(v, types):
                problems.append(f"{where}{key}")
                return None
            return v

        vocab = need(cfg, "vocab", int, "")
        width = need(cfg, "width", int, "")
        eps = need(cfg.get("norm"), "eps", NUM, "norm.")
        emb = need(cfg.get("embedding"), "scale", NUM, "embedding.")
        alpha = need(cfg, "postln_alpha", NUM, "")
        layers_in = cfg.get("layers")
        layers: List[PidodraLayer] = []
        if not isinstance(layers_in, list) or not layers_in:
            problems.append("layers")
            layers_in = []
        for i, l in enumerate(layers_in):
            where = f"layers[{i}]."
            kind = need(l, "type", str, where)
            if kind is not None and kind not in SIZES:
                problems.append(f"{where}type={kind!r} (known: {', '.join(sorted(SIZES))})")
                continue
            mixer = l.get("mixer") if isinstance(l, dict) and isinstance(l.get("mixer"), dict) else None
            if mixer is None:
                problems.append(where + "mixer")
                continue
            for k in SIZES.get(kind, ()):
                need(mixer, k, int, where + "mixer.")
            need(mixer, "scale", NUM, where + "mixer.")
            rot = mixer.get("rot")
            need(rot, "base", NUM, where + "mixer.rot.")
            need(rot, "dims", int, where + "mixer.rot.")
            if kind == "attention":
                if isinstance(rot, dict) and rot.get("scaling") is not None:
                    for k in SCALING:
                        need(rot["scaling"], k, NUM, where + "mixer.rot.scaling.")
                if mixer.get("kv_from") is not None:
                    need(mixer, "kv_from", int, where + "mixer.")
            mlp = l.get("mlp")
            if mlp is not None:
                mk = need(mlp, "kind", str, where + "mlp.")
                if mk == "moe":
                    need(mlp.get("expert"), "ff", int, where + "mlp.expert.")
                    router = mlp.get("router")
                    for k in ("experts", "top"):
                        need(router, k, int, where + "mlp.router.")
                    if isinstance(router, dict):
                        if router.get("scale") is not None:
                            need(router, "scale", NUM, where + "mlp.router.")
                        if router.get("groups") is not None:
                            for k in ("count", "keep"):
                                need(router["groups"], k, int, where + "mlp.router.groups.")
                elif mk is not None:
                    problems.append(f"{where}mlp.kind={mk!r} (known: moe)")
            layers.append(PidodraLayer(kind, dict(mixer), None if mlp is None else dict(mlp)))
        if problems:
            raise CheckpointError("config.json: missing or ill-typed keys: " + ", ".join(problems))
        out = cls(vocab=vocab, width=width, norm_eps=float(eps), embedding_scale=float(emb), alpha=float(alpha),
                  layers=layers, torch_dtype=str(cfg.get("torch_dtype", "bfloat16")),
                  max_positions=int(cfg.get("max_positions", 1 << 20)), raw=dict(cfg))
        out.validate()
        return out

    def validate(self) -> None:
        def bad(msg: str) -> None:
            raise CheckpointError(f"config.json: {msg}")

        if self.vocab <= 0 or self.width <= 0:
            bad("vocab and width must be positive")
        if not (self.norm_eps > 0):
            bad("norm.eps must be positive")
        for i, l in enumerate(self.layers):
            m, where = l.mixer, f"layers[{i}].mixer"
            for k in SIZES[l.type]:
                if m[k] <= 0:
                    bad(f"{where}.{k} must be positive")
            dims, room = m["rot"]["dims"], m["rot_dim"] if l.type == "latent_attention" else m["dim"]
            if dims % 2 or not (0 <= dims <= room):
                bad(f"{where}.rot.dims must be even and at most the head's size")
            if l.type == "latent_attention" and dims != room:
                bad(f"{where}.rot.dims must be rot_dim")
            if not (m["rot"]["base"] > 0):
                bad(f"{where}.rot.base must be positive")
            if l.type == "attention":
                if m["heads"] % m["kv_heads"]:
                    bad(f"{where}: heads must be a multiple of kv_heads")
                sc = m["rot"].get("scaling")
                if sc:
                    if not all(sc[k] > 0 for k in SCALING):
                        bad(f"{where}.rot.scaling: {', '.join(SCALING)} must be positive")
                    if m["rot"]["base"] == 1:
                        bad(f"{where}.rot.base must not be 1 with a scaling")
                j = m.get("kv_from")
                if j is not None:
                    if not (0 <= j < i) or self.layers[j].type != "attention" or \
                            self.layers[j].mixer.get("kv_from") is not None:
                        bad(f"{where}.kv_from must name an earlier attention layer with keys and values of its own")
                    if any(self.layers[j].mixer[k] != m[k] for k in ("kv_heads", "dim", "vdim")):
                        bad(f"{where}: kv_heads, dim and vdim must be those of layer {j}")
            if l.mlp is not None:
                r = l.mlp["router"]
                if l.mlp["expert"]["ff"] <= 0 or not (0 < r["top"] <= r["experts"]):
                    bad(f"layers[{i}].mlp: expert.ff must be positive and 0 < router.top <= router.experts")
                g = r.get("groups")
                if g is not None:
                    if g["count"] <= 0 or r["experts"] % g["count"] or not (0 < g["keep"] <= g["count"]):
                        bad(f"layers[{i}].mlp.router.groups: count must divide experts and 0 < keep <= count")
                    if r["top"] > g["keep"] * (r["experts"] // g["count"]):
                        bad(f"layers[{i}].mlp.router: top is more than the kept groups hold")

    def to_dict(self) -> Dict[str, Any]:
        out = dict(self.raw)
        out.update({
            "architecture": "Pidodra", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
            "embedding": {"scale": self.embedding_scale}, "postln_alpha": self.alpha,
            "layers": [{"type": l.type, "mixer": l.mixer, "mlp": l.mlp} for l in self.layers],
        })
        return out
