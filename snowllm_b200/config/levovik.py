"""Typed configuration of the Levovik design, read from its config.json.

    {"architecture": "Levovik", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "logit_scale": c, "token_side": {"dim": d},
     "layers": [{"type": T, "mixer": {"left": {...}, "right": {...}, "left_scale": a, "right_scale": b},
                 "mlp": {...} | null}, ...]}

``type`` names the pair of mixers that a layer runs side by side:

* ``parallel``:   left: heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor, low, high, original}};
                  right: heads, kv_heads, dim, vdim, conv (taps): the gated delta rule
* ``parallel_2``: left: the same keys, the values being the keys (vdim, where given, equals dim);
                  right: heads, dim, vdim, tau: gated linear attention

``mlp``: ``{"kind": "dense", "ff"}``, ``{"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top", "scale",
"groups": {"count", "keep"}}}``, or null.  What a file leaves out is off: no ``rot`` (no rotation), no ``rot.scaling``,
no ``groups`` (one group of all experts), no ``token_side``, no ``mlp``; ``kv_heads`` of a delta rule is then ``heads``,
and the scales are 1.  The ranks of the low-rank products are the tensors' to say; ``decay_rank`` and ``gate_rank`` of a
right mixer are optional keys for weights that are drawn, not read.  Every size and constant comes from the file; what is
missing or unusable is reported in one ConfigError that lists every key."""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any

from ..errors import ConfigError
from .beledra import _Reader
from .gurolix import _divides, _read_rot

ARCHITECTURE = "Levovik"
DELTA, LINEAR = "parallel", "parallel_2"        # a layer's type by the recurrence on its right
LAYER_TYPES = (DELTA, LINEAR)
MAX_CONV_TAPS = 16
MAX_HEAD_DIM = 256                              # rows of a matrix memory


@dataclass(frozen=True)
class LevovikLayer:
    type: str
    mixer: dict          # {"left", "right", "left_scale", "right_scale"}
    mlp: dict | None     # {"kind": "dense", "ff"} or {"kind": "moe", "ff", "limit", "experts", "top", "scale", "groups"}


@dataclass(frozen=True)
class LevovikConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    token_side: int | None      # width of one layer's share of the tokens' side rows
    layers: tuple

    def to_json_dict(self) -> dict[str, Any]:
        """config.json content that reads back to this configuration."""
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
               "logit_scale": self.logit_scale,
               "layers": [{"type": l.type, "mixer": _mixer_json(l.mixer), "mlp": _mlp_json(l.mlp)}
                          for l in self.layers]}
        if self.token_side is not None:
            out["token_side"] = {"dim": self.token_side}
        return out


def _mixer_json(mixer: dict) -> dict:
    m = copy.deepcopy(mixer)
    rot = m["left"].get("rot")
    if rot is not None and rot.get("scaling") is None:
        rot.pop("scaling", None)
    for side in ("left", "right"):
        m[side] = {k: v for k, v in m[side].items() if v is not None}
    return m


def _mlp_json(mlp):
    if mlp is None or mlp["kind"] == "dense":
        return copy.deepcopy(mlp)
    router = {"experts": mlp["experts"], "top": mlp["top"], "scale": mlp["scale"]}
    if mlp["groups"] != (1, 1):
        router["groups"] = {"count": mlp["groups"][0], "keep": mlp["groups"][1]}
    return {"kind": "moe", "expert": {"ff": mlp["ff"], "limit": mlp["limit"]}, "router": router}


def _optional_int(r: _Reader, d: dict, key: str, where: str):
    return r.positive_int(d, key, where) or None if d.get(key) is not None else None


def _optional_number(r: _Reader, d, key: str, where: str, default: float) -> float:
    return r.number(d, key, where) if isinstance(d, dict) and d.get(key) is not None else default


def _side(r: _Reader, m: dict, key: str, where: str) -> dict:
    if not isinstance(m.get(key), dict):
        r.missing.append(where + key)
        return {}
    return m[key]


def _read_left(r: _Reader, m: dict, w: str, shared: bool) -> dict:
    out = dict(heads=r.positive_int(m, "heads", w), kv_heads=r.positive_int(m, "kv_heads", w),
               dim=r.positive_int(m, "dim", w), scale=r.positive(m, "scale", w))
    if shared:
        out["vdim"] = _optional_int(r, m, "vdim", w) or out["dim"]
        if out["vdim"] != out["dim"]:
            r.bad.append(f"{w}vdim={out['vdim']} (the keys are the values: want dim={out['dim']})")
    else:
        out["vdim"] = r.positive_int(m, "vdim", w)
    _divides(r, w, "heads", out["heads"], "kv_heads", out["kv_heads"])
    out["rot"] = _read_rot(r, m.get("rot"), out["dim"], w + "rot.")
    return out


def _read_right(r: _Reader, m: dict, w: str, kind: str) -> dict:
    out = dict(heads=r.positive_int(m, "heads", w), dim=r.positive_int(m, "dim", w),
               vdim=r.positive_int(m, "vdim", w), decay_rank=_optional_int(r, m, "decay_rank", w))
    if kind == DELTA:
        out.update(kv_heads=_optional_int(r, m, "kv_heads", w) or out["heads"], conv=r.positive_int(m, "conv", w),
                   gate_rank=_optional_int(r, m, "gate_rank", w))
        _divides(r, w, "heads", out["heads"], "kv_heads", out["kv_heads"])
        if out["conv"] > MAX_CONV_TAPS:
            r.bad.append(f"{w}conv={out['conv']} (at most {MAX_CONV_TAPS} taps)")
    else:
        out["tau"] = r.positive(m, "tau", w)
    if out["dim"] > MAX_HEAD_DIM:
        r.bad.append(f"{w}dim={out['dim']} (at most {MAX_HEAD_DIM})")
    return out


def _read_mlp(r: _Reader, mlp, where: str):
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    w = where + "mlp."
    if kind == "dense":
        return dict(kind="dense", ff=r.positive_int(mlp, "ff", w))
    if kind != "moe":
        r.bad.append(f"{w}kind={kind!r} (want 'dense' or 'moe')")
        return None
    ro, wr, we = mlp.get("router"), w + "router.", w + "expert."
    out = dict(kind="moe", ff=r.positive_int(mlp.get("expert"), "ff", we), limit=r.positive(mlp.get("expert"), "limit", we),
               experts=r.positive_int(ro, "experts", wr), top=r.positive_int(ro, "top", wr),
               scale=_optional_number(r, ro, "scale", wr, 1.0), groups=(1, 1))
    groups = ro.get("groups") if isinstance(ro, dict) else None
    if groups is not None:
        count, keep = (r.positive_int(groups, k, wr + "groups.") for k in ("count", "keep"))
        if count and keep:
            out["groups"] = (count, keep)
            if out["experts"] % count:
                r.bad.append(f"{wr}groups.count={count} does not divide the {out['experts']} experts")
            if keep > count:
                r.bad.append(f"{wr}groups.keep={keep} exceeds count={count}")
    reach = out["experts"] // out["groups"][0] * out["groups"][1]
    if out["experts"] and out["top"] > reach:
        r.bad.append(f"{wr}top={out['top']} exceeds the {reach} experts that can be chosen")
    return out


def read_levovik_config(cfg: dict) -> LevovikConfig:
    r = _Reader()
    vocab, width = r.positive_int(cfg, "vocab", ""), r.positive_int(cfg, "width", "")
    eps = r.positive(cfg.get("norm"), "eps", "norm.")
    embedding_scale = _optional_number(r, cfg.get("embedding"), "scale", "embedding.", 1.0)
    logit_scale = _optional_number(r, cfg, "logit_scale", "", 1.0)
    side = None
    if cfg.get("token_side") is not None:
        side = r.positive_int(cfg["token_side"], "dim", "token_side.") or None
    raw_layers = cfg.get("layers")
    layers = []
    if not isinstance(raw_layers, list) or not raw_layers:
        r.missing.append("layers")
        raw_layers = []
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
        w = where + "mixer."
        mixer = dict(left=_read_left(r, _side(r, m, "left", w), w + "left.", shared=kind == LINEAR),
                     right=_read_right(r, _side(r, m, "right", w), w + "right.", kind),
                     left_scale=_optional_number(r, m, "left_scale", w, 1.0),
                     right_scale=_optional_number(r, m, "right_scale", w, 1.0))
        layers.append(LevovikLayer(kind, mixer, _read_mlp(r, layer.get("mlp"), where)))
    if r.missing or r.bad:
        parts = []
        if r.missing:
            parts.append("missing keys: " + ", ".join(r.missing))
        if r.bad:
            parts.append("unusable values: " + "; ".join(r.bad))
        raise ConfigError(f"unsupported {ARCHITECTURE} configuration: " + " | ".join(parts))
    return LevovikConfig(ARCHITECTURE, vocab, width, eps, embedding_scale, logit_scale, side, tuple(layers))
