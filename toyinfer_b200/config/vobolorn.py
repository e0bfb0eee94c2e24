"""Configuration of the Vobolorn decoder.

config.json names the design in ``architecture`` and gives: ``vocab``, ``width``, ``norm.eps``, ``logit_softcap`` (absent or
null: none), and ``layers``: per layer its ``type`` with the mixer's sizes and constants under ``mixer`` (``attention``: heads,
kv_heads, dim, vdim, scale, v_mix; ``attention_2``: the same and optionally ``q_temp`` {coef, every}; ``latent_attention``:
heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, and ``rot`` {dims, base} with dims = rot_dim unless that is 0) and its
feed-forward under ``mlp`` (null, or ``kind`` dense with ``ff``).  Every size and constant comes from there; nothing is assumed
equal between layers, except that layers with ``v_mix`` share kv_heads and vdim, since they blend their values.
"""
from __future__ import annotations

from typing import List

from .base import Key, ModelConfig
from .kadodra import _check_fields, _number

MIXER_KEYS = {
    "attention": {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float},
    "attention_2": {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "scale": float},
    "latent_attention": {"heads": int, "dim": int, "rot_dim": int, "vdim": int, "kv_rank": int, "q_rank": int, "scale": float},
}


class VobolornConfig(ModelConfig):
    KEYS = {
        "architecture": Key("str"),
        "vocab": Key("int"),
        "width": Key("int"),
        "norm": Key("any"),
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
        if kind == "latent_attention":
            if m["dim"] < 0 or m["rot_dim"] < 0 or m["rot_dim"] % 2 or m["dim"] + m["rot_dim"] == 0:
                p.append(f"{w}: {m['dim']} unrotated and {m['rot_dim']} rotated elements per head")
            elif m["rot_dim"] > 0 and _check_fields(w + ".rot", m.get("rot"), {"dims": int, "base": float}, p):
                if m["rot"]["dims"] != m["rot_dim"]:
                    p.append(f"{w}.rot.dims: expected rot_dim = {m['rot_dim']}, got {m['rot']['dims']}")
                if not m["rot"]["base"] > 0:
                    p.append(f"{w}.rot.base: expected a positive number")
            return
        if m["heads"] % m["kv_heads"]:
            p.append(f"{w}: {m['heads']} heads over {m['kv_heads']} kv heads")
        if not isinstance(m.get("v_mix", False), bool):
            p.append(f"{w}.v_mix: expected true or false")
        t = m.get("q_temp")
        if kind == "attention_2" and t is not None and _check_fields(w + ".q_temp", t, {"coef": float, "every": float}, p):
            if not (t["every"] >= 1 and float(t["every"]).is_integer()):
                p.append(f"{w}.q_temp.every: expected a positive integer, got {t['every']}")

    def validate(self) -> List[str]:
        p: List[str] = []
        if self.vocab <= 0 or self.width <= 0:
            p.append("vocab and width must be positive")
        if not isinstance(self.norm, dict) or not _number(self.norm.get("eps")) or not self.norm["eps"] > 0:
            p.append("norm.eps: missing or not a positive number")
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
            f = L.get("mlp")
            if f is not None:
                if not isinstance(f, dict) or f.get("kind") != "dense":
                    p.append(f"{w}.mlp.kind: expected dense")
                elif _check_fields(w + ".mlp", f, {"ff": int}, p) and f["ff"] < 1:
                    p.append(f"{w}.mlp.ff: expected a positive number")
        if not p:
            mixing = self.mixing_layers()
            for i in mixing[1:]:
                a, b = self.layers[mixing[0]]["mixer"], self.layers[i]["mixer"]
                if (a["kv_heads"], a["vdim"]) != (b["kv_heads"], b["vdim"]):
                    p.append(f"layers[{i}].mixer: {b['kv_heads']} kv heads of {b['vdim']} value elements cannot be blended with "
                             f"layers[{mixing[0]}]'s {a['kv_heads']} of {a['vdim']}")
        return p

    def mixing_layers(self) -> List[int]:
        """The layers whose values are blended, in order; the first of them gives the values that the others blend in."""
        return [i for i, L in enumerate(self.layers) if L["type"] != "latent_attention" and L["mixer"].get("v_mix")]

    @property
    def eps(self) -> float:
        return float(self.norm["eps"])

    @property
    def stop_token_ids(self) -> tuple:
        return tuple(self.stop_tokens)
