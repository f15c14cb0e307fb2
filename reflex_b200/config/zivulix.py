"""Typed configuration of the Zivulix design, read from config.json.

config.json keys: `architecture` ("Zivulix"), `vocab`, `width`, `norm.eps`, and
`layers`, a list whose entries give `type` (the mixer: "latent_attention",
"attention" or "delta"), `mixer` (its sizes and constants) and `mlp` (`kind`
"dense" with `ff`; null for a layer without a feed-forward).

A "latent_attention" mixer: `heads`, `dim` (unrotated query/key dimensions a
head), `rot_dim` (rotated ones), `vdim`, `kv_rank`, `scale`, `rot` {`base`,
`dims` = `rot_dim`}.  An "attention" mixer: `heads`, `kv_heads`, `dim`, `vdim`,
`scale`, `softcap`, `rot` {`base`, `dims`, optional `scaling` {`factor`}},
optional `mask` {`size`} and `v_mix`.  A "delta" mixer: `heads`, `kv_heads`,
`dim`, `vdim`, `conv` (taps).  Every size and every constant that differs
between models comes from here.  Missing or ill-typed keys are reported
together, by name.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from ..errors import CheckpointError

NUM = (int, float)

SIZES = {
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank"),
    "attention": ("heads", "kv_heads", "dim", "vdim"),
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}


@dataclass
class ZivulixLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclass
class ZivulixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[ZivulixLayer] = field(default_factory=list)
    torch_dtype: str = "bfloat16"
    # the design fixes no longest context; the cache bounds it
    max_positions: int = 1 << 20
    raw: Dict[str, Any] = field(default_factory=dict)

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any]) -> "ZivulixConfig":
        problems: List[str] = []

        def need(d, key, types, where):
            v = d.get(key) if isinstance(d, dict) else None
            if v is None or isinstance(v, bool) or not isinstance(v, types):
                problems.append(f"{where}{key}")
                return None
            return v

        vocab = need(cfg, "vocab", int, "")
        width = need(cfg, "width", int, "")
        norm = cfg.get("norm") if isinstance(cfg.get("norm"), dict) else {}
        eps = need(norm, "eps", NUM, "norm.")
        layers_in = cfg.get("layers")
        layers: List[ZivulixLayer] = []
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
            if kind in ("attention", "latent_attention"):
                need(mixer, "scale", NUM, where + "mixer.")
                rot = mixer.get("rot")
                need(rot, "base", NUM, where + "mixer.rot.")
                need(rot, "dims", int, where + "mixer.rot.")
                if isinstance(rot, dict) and rot.get("scaling") is not None:
                    need(rot["scaling"], "factor", NUM, where + "mixer.rot.scaling.")
            if kind == "attention":
                if mixer.get("softcap") is not None:
                    need(mixer, "softcap", NUM, where + "mixer.")
                if mixer.get("mask") is not None:
                    need(mixer["mask"], "size", int, where + "mixer.mask.")
                if mixer.get("v_mix") is not None and not isinstance(mixer["v_mix"], bool):
                    problems.append(where + "mixer.v_mix")
            mlp = l.get("mlp")
            if mlp is not None:
                mk = need(mlp, "kind", str, where + "mlp.")
                if mk == "dense":
                    need(mlp, "ff", int, where + "mlp.")
                elif mk is not None:
                    problems.append(f"{where}mlp.kind={mk!r} (known: dense)")
            layers.append(ZivulixLayer(kind, dict(mixer), None if mlp is None else dict(mlp)))
        if problems:
            raise CheckpointError("config.json: missing or ill-typed keys: " + ", ".join(problems))
        out = cls(vocab=vocab, width=width, norm_eps=float(eps), layers=layers,
                  torch_dtype=str(cfg.get("torch_dtype", "bfloat16")),
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
        mixed = None  # kv_heads * vdim of the layers whose values are mixed
        for i, l in enumerate(self.layers):
            m, where = l.mixer, f"layers[{i}].mixer"
            for k in SIZES[l.type]:
                if m[k] <= 0:
                    bad(f"{where}.{k} must be positive")
            if l.type != "latent_attention" and m["heads"] % m["kv_heads"]:
                bad(f"{where}: heads must be a multiple of kv_heads")
            if l.type != "delta":
                dims, room = m["rot"]["dims"], m["rot_dim"] if l.type == "latent_attention" else m["dim"]
                if dims % 2 or not (0 <= dims <= room):
                    bad(f"{where}.rot.dims must be even and at most the head's size")
                if l.type == "latent_attention" and dims != room:
                    bad(f"{where}.rot.dims must be rot_dim")
                if not (m["rot"]["base"] > 0):
                    bad(f"{where}.rot.base must be positive")
                if m["rot"].get("scaling") and not (m["rot"]["scaling"]["factor"] > 0):
                    bad(f"{where}.rot.scaling.factor must be positive")
            if l.type == "attention":
                if m.get("softcap") is not None and not (m["softcap"] > 0):
                    bad(f"{where}.softcap must be positive")
                if m.get("mask") is not None and m["mask"]["size"] <= 0:
                    bad(f"{where}.mask.size must be positive")
                if m.get("v_mix"):
                    size = m["kv_heads"] * m["vdim"]
                    if mixed not in (None, size):
                        bad(f"{where}: layers whose values are mixed need the same kv_heads * vdim")
                    mixed = size
            if l.mlp is not None and l.mlp["ff"] <= 0:
                bad(f"layers[{i}].mlp.ff must be positive")

    def to_dict(self) -> Dict[str, Any]:
        out = dict(self.raw)
        out.update({
            "architecture": "Zivulix", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
            "layers": [{"type": l.type, "mixer": l.mixer, "mlp": l.mlp} for l in self.layers],
        })
        return out
