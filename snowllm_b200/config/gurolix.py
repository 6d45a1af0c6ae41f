"""Typed configuration of the Gurolix design, read from its config.json.

    {"architecture": "Gurolix", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": T, "mixer": {...}, "mlp": {...} | null}, ...]}

``type`` names the layer's mixer; ``mixer`` holds that mixer's sizes and constants:

* ``mamba2``:      heads, vdim, state, groups, norm_groups, conv (taps)
* ``attention``:   heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor, low, high, original}},
                   softcap, v_mix; q and k are normalised per head
* ``attention_2``: the same keys; q and k are not normalised

``mlp``: ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "identity", "groups": {"count",
"keep"}}}``, or null.  What a file leaves out is off: no ``rot`` (no rotation), no ``rot.scaling``, no
``softcap``, no ``v_mix``, ``identity`` 0, no ``groups`` (one group of all experts), no ``mlp``; ``norm_groups``
and ``groups`` of the state-space mixer are 1.  Every size and constant comes from the file; what is missing
or unusable is reported in one ConfigError that lists every key."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any

from ..errors import ConfigError
from .beledra import _Reader

ARCHITECTURE = "Gurolix"
ATTENTION_TYPES = ("attention", "attention_2")
LAYER_TYPES = ("mamba2",) + ATTENTION_TYPES
MAX_CONV_TAPS = 16
MAX_STATE = 256


@dataclass(frozen=True)
class GurolixLayer:
    type: str
    mixer: dict
    mlp: dict | None     # {"ff", "experts", "top", "identity", "groups": (count, keep)}


@dataclass(frozen=True)
class GurolixConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: tuple

    def to_json_dict(self) -> dict[str, Any]:
        """config.json content that reads back to this configuration."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps},
                "layers": [{"type": l.type, "mixer": _mixer_json(l.mixer), "mlp": _mlp_json(l.mlp)}
                           for l in self.layers]}


def _mixer_json(mixer: dict) -> dict:
    m = copy.deepcopy(mixer)
    if m.get("rot") is not None and m["rot"].get("scaling") is None:
        m["rot"].pop("scaling", None)
    return {k: v for k, v in m.items() if v is not None and v is not False}


def _mlp_json(mlp):
    if mlp is None:
        return None
    router = {"experts": mlp["experts"], "top": mlp["top"]}
    if mlp["identity"]:
        router["identity"] = mlp["identity"]
    if mlp["groups"] != (1, 1):
        router["groups"] = {"count": mlp["groups"][0], "keep": mlp["groups"][1]}
    return {"kind": "moe", "expert": {"ff": mlp["ff"]}, "router": router}


def _optional_count(r: _Reader, d, key: str, where: str, default: int, least: int) -> int:
    v = d.get(key) if isinstance(d, dict) else None
    if v is None:
        return default
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        r.bad.append(f"{where}{key}={v!r} (want an integer of at least {least})")
        return default
    return v


def _divides(r: _Reader, where: str, whole: str, n: int, part: str, d: int) -> None:
    if n and d and n % d:
        r.bad.append(f"{where}{whole}={n} is no multiple of {part}={d}")


def _read_state_space(r: _Reader, m: dict, w: str) -> dict:
    out = dict(heads=r.positive_int(m, "heads", w), vdim=r.positive_int(m, "vdim", w),
               state=r.positive_int(m, "state", w), groups=_optional_count(r, m, "groups", w, 1, 1),
               norm_groups=_optional_count(r, m, "norm_groups", w, 1, 1), conv=r.positive_int(m, "conv", w))
    _divides(r, w, "heads", out["heads"], "groups", out["groups"])
    _divides(r, w, "heads * vdim", out["heads"] * out["vdim"], "norm_groups", out["norm_groups"])
    if out["conv"] > MAX_CONV_TAPS:
        r.bad.append(f"{w}conv={out['conv']} (at most {MAX_CONV_TAPS} taps)")
    if out["state"] > MAX_STATE:
        r.bad.append(f"{w}state={out['state']} (at most {MAX_STATE})")
    return out


def _read_rot(r: _Reader, rot, dim: int, w: str):
    if rot is None:
        return None
    out = dict(dims=r.positive_int(rot, "dims", w), base=r.positive(rot, "base", w), scaling=None)
    if out["dims"] and (out["dims"] % 2 or (dim and out["dims"] > dim)):
        r.bad.append(f"{w}dims={out['dims']} (want an even number, at most dim={dim})")
    scaling = rot.get("scaling") if isinstance(rot, dict) else None
    if scaling is not None:
        s = out["scaling"] = {k: r.positive(scaling, k, w + "scaling.") for k in ("factor", "low", "high", "original")}
        if s["low"] and s["high"] and not s["high"] > s["low"]:
            r.bad.append(f"{w}scaling.high={s['high']} (want more than low={s['low']})")
    return out


def _read_attention(r: _Reader, m: dict, w: str) -> dict:
    out = dict(heads=r.positive_int(m, "heads", w), kv_heads=r.positive_int(m, "kv_heads", w),
               dim=r.positive_int(m, "dim", w), vdim=r.positive_int(m, "vdim", w), scale=r.positive(m, "scale", w),
               rot=None, softcap=None, v_mix=False)
    _divides(r, w, "heads", out["heads"], "kv_heads", out["kv_heads"])
    out["rot"] = _read_rot(r, m.get("rot"), out["dim"], w + "rot.")
    if m.get("softcap") is not None:
        out["softcap"] = r.positive(m, "softcap", w)
    if m.get("v_mix") is not None:
        if not isinstance(m["v_mix"], bool):
            r.bad.append(f"{w}v_mix={m['v_mix']!r} (want true or false)")
        out["v_mix"] = m["v_mix"] is True
    return out


def _read_mlp(r: _Reader, mlp, where: str):
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    w = where + "mlp."
    if kind != "moe":
        r.bad.append(f"{w}kind={kind!r} (want 'moe')")
        return None
    ro, wr = mlp.get("router"), w + "router."
    out = dict(ff=r.positive_int(mlp.get("expert"), "ff", w + "expert."), experts=r.positive_int(ro, "experts", wr),
               top=r.positive_int(ro, "top", wr), identity=_optional_count(r, ro, "identity", wr, 0, 0), groups=(1, 1))
    total = out["experts"] + out["identity"]
    groups = ro.get("groups") if isinstance(ro, dict) else None
    if groups is not None:
        count, keep = (r.positive_int(groups, k, wr + "groups.") for k in ("count", "keep"))
        if count and keep:
            out["groups"] = (count, keep)
            if total % count:
                r.bad.append(f"{wr}groups.count={count} does not divide the {total} router outputs")
            if keep > count:
                r.bad.append(f"{wr}groups.keep={keep} exceeds count={count}")
    reach = total // out["groups"][0] * out["groups"][1]
    if out["experts"] and out["top"] > reach:
        r.bad.append(f"{wr}top={out['top']} exceeds the {reach} experts that can be chosen")
    return out


def read_gurolix_config(cfg: dict) -> GurolixConfig:
    r = _Reader()
    vocab, width = r.positive_int(cfg, "vocab", ""), r.positive_int(cfg, "width", "")
    eps = r.positive(cfg.get("norm"), "eps", "norm.")
    raw_layers = cfg.get("layers")
    layers = []
    if not isinstance(raw_layers, list) or not raw_layers:
        r.missing.append("layers")
        raw_layers = []
    mixed = None                                  # (layer, kv_heads, vdim) of the first layer whose values mix
    for i, layer in enumerate(raw_layers):
        where = f"layers[{i}]."
        kind = layer.get("type") if isinstance(layer, dict) else None
        if kind not in LAYER_TYPES:
            r.bad.append(f"{where}type={kind!r} (want one of {LAYER_TYPES})")
            continue
        m = layer.get("mixer")
        if not isinstance(m, dict):
            r.missing.append(where + "mixer")
            continue
        read = _read_state_space if kind == "mamba2" else _read_attention
        mixer = read(r, m, where + "mixer.")
        if mixer.get("v_mix"):
            shape = (mixer["kv_heads"], mixer["vdim"])
            if mixed is None:
                mixed = (i, shape)
            elif mixed[1] != shape:
                r.bad.append(f"{where}mixer: values of {shape[0]} x {shape[1]} cannot mix with layer {mixed[0]}'s "
                             f"{mixed[1][0]} x {mixed[1][1]}")
        layers.append(GurolixLayer(kind, mixer, _read_mlp(r, layer.get("mlp"), where)))
    if r.missing or r.bad:
        parts = []
        if r.missing:
            parts.append("missing keys: " + ", ".join(r.missing))
        if r.bad:
            parts.append("unusable values: " + "; ".join(r.bad))
        raise ConfigError(f"unsupported {ARCHITECTURE} configuration: " + " | ".join(parts))
    return GurolixConfig(ARCHITECTURE, vocab, width, eps, tuple(layers))
