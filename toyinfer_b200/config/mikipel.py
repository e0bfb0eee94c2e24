"""Configuration of the Mikipel decoder.

config.json names the design in ``architecture`` and gives: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``,
``residual_mult`` (what a layer's output is multiplied by before it is added), ``logit_softcap`` (absent or null: none), and
``layers``: per layer its ``type`` with the mixer's sizes and constants under ``mixer`` (``attention``: heads, kv_heads, dim,
vdim, scale, optionally ``rot`` {dims, base, optionally ``scaling`` {factor}}; ``latent_attention``: heads, dim, rot_dim, vdim,
kv_rank, scale, and ``rot`` with dims = rot_dim unless that is 0; ``delta``: heads, kv_heads, dim, vdim, conv) and its
feed-forward under ``mlp`` (null; ``kind`` dense with ``ff``; or ``kind`` moe with ``expert`` {ff} and ``router`` {experts, top}).
Every size and constant comes from there; nothing is assumed equal between layers.
"""
from __future__ import annotations

from typing import List

from .base import Key, ModelConfig
from .kadodra import _check_fields, _number

MIXER_KEYS = {
    "attention": {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float},
    "latent_attention": {"heads": int, "dim": int, "rot_dim": int, "vdim": int, "kv_rank": int, "scale": float},
    "delta": {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "conv": int},
}


class MikipelConfig(ModelConfig):
    KEYS = {
        "architecture": Key("str"),
        "vocab": Key("int"),
        "width": Key("int"),
        "norm": Key("any"),
        "embedding": Key("any", required=False, default=None, nullable=True),
        "residual_mult": Key("float", required=False, default=1.0),
        "logit_softcap": Key("float", required=False, default=None, nullable=True),
        "layers": Key("any"),
        "max_positions": Key("int", required=False, default=131072),
        "stop_tokens": Key("int_or_list", required=False, default=()),
    }

    def _check_mixer(self, w: str, kind: str, m, p: List[str]) -> None:
        if not _check_fields(w, m, MIXER_KEYS[kind], p):
            return
        sizes = [k for k, t in MIXER_KEYS[kind].items() if t is int and not (kind == "latent_attention" and k in ("dim", "rot_dim"))]
        if min(m[k] for k in sizes) < 1:
            p.append(f"{w}: {', '.join(sizes)} must be positive")
            return
        if "kv_heads" in m and m["heads"] % m["kv_heads"]:
            p.append(f"{w}: {m['heads']} heads over {m['kv_heads']} kv heads")
        if kind == "delta":
            if m["conv"] > 8:
                p.append(f"{w}.conv: expected 1 to 8 taps, got {m['conv']}")
            return
        if kind == "latent_attention":
            if m["dim"] < 0 or m["rot_dim"] < 0 or m["rot_dim"] % 2 or m["dim"] + m["rot_dim"] == 0:
                p.append(f"{w}: {m['dim']} unrotated and {m['rot_dim']} rotated elements per head")
            if m["rot_dim"] == 0:
                return
        r = m.get("rot")
        if r is None:
            if kind == "latent_attention":
                p.append(f"{w}.rot: missing, with {m['rot_dim']} rotated elements")
            return
        if _check_fields(w + ".rot", r, {"dims": int, "base": float}, p):
            if kind == "latent_attention" and r["dims"] != m["rot_dim"]:
                p.append(f"{w}.rot.dims: expected rot_dim = {m['rot_dim']}, got {r['dims']}")
            if r["dims"] < 2 or r["dims"] % 2 or (kind == "attention" and r["dims"] > m["dim"]):
                p.append(f"{w}.rot.dims: expected an even number from 2 to the head's size, got {r['dims']}")
            if not r["base"] > 0:
                p.append(f"{w}.rot.base: expected a positive number")
            if r.get("scaling") is not None:
                if _check_fields(w + ".rot.scaling", r["scaling"], {"factor": float}, p) and not r["scaling"]["factor"] > 0:
                    p.append(f"{w}.rot.scaling.factor: expected a positive number")

    def _check_mlp(self, w: str, f, p: List[str]) -> None:
        if not isinstance(f, dict) or f.get("kind") not in ("dense", "moe"):
            p.append(f"{w}.kind: expected dense or moe")
        elif f["kind"] == "dense":
            if _check_fields(w, f, {"ff": int}, p) and f["ff"] < 1:
                p.append(f"{w}.ff: expected a positive number")
        elif _check_fields(w + ".expert", f.get("expert"), {"ff": int}, p) and \
                _check_fields(w + ".router", f.get("router"), {"experts": int, "top": int}, p):
            if not 1 <= f["router"]["top"] <= f["router"]["experts"]:
                p.append(f"{w}.router: top must lie in 1 .. experts")

    def validate(self) -> List[str]:
        p: List[str] = []
        if self.vocab <= 0 or self.width <= 0:
            p.append("vocab and width must be positive")
        if not isinstance(self.norm, dict) or not _number(self.norm.get("eps")) or not self.norm["eps"] > 0:
            p.append("norm.eps: missing or not a positive number")
        if self.embedding is not None and (not isinstance(self.embedding, dict) or not _number(self.embedding.get("scale", 1.0))):
            p.append("embedding.scale: not a number")
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            p.append("logit_softcap: expected a positive number")
        if not isinstance(self.layers, list) or not self.layers:
            p.append("layers: expected a non-empty list")
            return p
        for i, L in enumerate(self.layers):
            w = f"layers[{i}]"
            if not isinstance(L, dict) or L.get("type") not in MIXER_KEYS:
                p.append(f"{w}.type: expected one of {sorted(MIXER_KEYS)}")
                continue
            self._check_mixer(w + ".mixer", L["type"], L.get("mixer"), p)
            if L.get("mlp") is not None:
                self._check_mlp(w + ".mlp", L["mlp"], p)
        return p

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def embedding_scale(self) -> float:
        return float((self.embedding or {}).get("scale", 1.0))

    @property
    def stop_token_ids(self) -> tuple:
        return tuple(self.stop_tokens)
