"""Small Levovik configurations, weights that make faults show, and helpers to run a request through the engine's step
function (any cut into steps) and through the plain implementation."""
from __future__ import annotations

import copy

import torch

import plain_levovik as plain
from beledra_cases import cuts_of, relative_error, run_cuts, tokens_for, worst_row_error  # noqa: F401

SCALING = {"factor": 5.0, "low": 1.5, "high": 6.0, "original": 70}


def moe(ff=24, experts=6, top=2, groups=(3, 2), limit=0.8, scale=1.7):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def _rot(dims, base, scaling):
    if not dims:
        return None
    rot = {"dims": dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(scaling)
    return rot


def _left(heads, kv_heads, dim, vdim, scale, rot):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        left["rot"] = rot
    return left


def delta_layer(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.3, rot_dims=8, base=900.0, scaling=SCALING, r_heads=4,
                r_kv_heads=2, r_dim=10, r_vdim=14, conv=3, ranks=(5, 7), scales=(0.7, 1.3), mlp="moe"):
    """parallel: attention with sinks beside the gated delta rule."""
    right = {"heads": r_heads, "kv_heads": r_kv_heads, "dim": r_dim, "vdim": r_vdim, "conv": conv, "decay_rank": ranks[0],
             "gate_rank": ranks[1]}
    return {"type": "parallel", "mixer": {"left": _left(heads, kv_heads, dim, vdim, scale, _rot(rot_dims, base, scaling)),
                                          "right": right, "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": moe() if mlp == "moe" else mlp}


def linear_layer(heads=6, kv_heads=2, dim=10, scale=0.5, rot_dims=6, base=50.0, scaling=SCALING, r_heads=3, r_dim=9,
                 r_vdim=12, tau=4.0, rank=6, scales=(1.1, 0.6), mlp="moe"):
    """parallel_2: attention whose values are its keys beside gated linear attention."""
    right = {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "tau": tau, "decay_rank": rank}
    return {"type": "parallel_2", "mixer": {"left": _left(heads, kv_heads, dim, dim, scale, _rot(rot_dims, base, scaling)),
                                            "right": right, "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": moe() if mlp == "moe" else mlp}


def config(layers, vocab=90, width=44, eps=1e-5, side=8, embedding_scale=1.5, logit_scale=0.7):
    cfg = {"architecture": "Levovik", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": embedding_scale}, "logit_scale": logit_scale, "layers": copy.deepcopy(layers)}
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


# both pairs, layers of one kind with different sizes, with each feed-forward and none, one kv head per head, q and k heads
# of the delta rule shared and not, one tap, whole and partial rotation, no scaling
MIXED = config([delta_layer(mlp=dense()),
                linear_layer(),
                delta_layer(heads=2, kv_heads=2, dim=16, vdim=6, rot_dims=16, scaling=None, r_heads=3, r_kv_heads=3, r_dim=20,
                            r_vdim=8, conv=1, mlp=None),
                linear_layer(heads=3, kv_heads=1, dim=20, rot_dims=20, scaling=None, r_heads=2, r_dim=32, r_vdim=10, tau=1.0,
                             mlp=moe(16, 4, 3, None, 3.0, 0.4)),
                delta_layer(heads=6, kv_heads=2, r_heads=6, r_kv_heads=1, r_dim=16, r_vdim=16, conv=5,
                            mlp=moe(8, 8, 4, (2, 1), 1.5, 1.0))])

# heads of 64 for keys and values, memories of tensor-core sizes: the sizes the fast kernels take
HEADS_OF_64 = config([linear_layer(heads=6, kv_heads=3, dim=64, scale=0.16, rot_dims=32, r_heads=2, r_dim=64, r_vdim=32,
                                   tau=8.0, rank=16, mlp=moe(32, 6, 2, (2, 1))),
                      delta_layer(heads=6, kv_heads=3, dim=64, vdim=64, scale=0.2, rot_dims=64, r_heads=4, r_kv_heads=2,
                                  r_dim=32, r_vdim=64, conv=4, ranks=(16, 8), mlp=dense(48)),
                      delta_layer(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.15, rot_dims=16, r_heads=1, r_kv_heads=1,
                                  r_dim=128, r_vdim=128, conv=4, ranks=(8, 16), mlp=None)], width=64, side=16)


def draw_weights(cfg: dict, seed: int = 0, dtype=torch.bfloat16) -> dict:
    """name -> tensor (as stored: ``dtype``) from the framework's seeded generator, with the small tensors redrawn so that
    each mechanism carries weight: sinks that take a share, decays from nearly none to a few tokens, write strengths and
    routers that are spread out, norm weights away from one."""
    from snowllm_b200.loader import build_model
    from snowllm_b200.weights import random_tensors
    model = build_model(cfg, "float32")
    tensors = random_tensors(model, seed, torch.float32, fan_in_scaled=True, norm_jitter=0.2)
    gen = torch.Generator().manual_seed(seed + 1)
    for name, t in tensors.items():
        def randn(scale=1.0):
            return torch.randn(t.shape, generator=gen) * scale
        leaf = name.split(".")[-1]
        if name in ("embed", "side.embed"):
            tensors[name] = randn()
        elif leaf == "sink":
            tensors[name] = 1.0 + randn()
        elif leaf in ("router", "b") and t.dim() == 2:
            tensors[name] = t * 2.0
        elif leaf == "A_log":
            tensors[name] = torch.rand(t.shape, generator=gen) * 3.0 - 2.5
        elif leaf == "dt_bias":
            tensors[name] = torch.rand(t.shape, generator=gen) * 3.0 - 3.0
        elif leaf == "b":                                  # the bias of the linear attention's decays
            tensors[name] = 1.0 + randn(1.5)
        elif leaf in ("a1", "a2", "g1", "g2"):
            tensors[name] = t * 1.3
        elif leaf == "conv":
            tensors[name] = randn(0.7)
    return {k: v.to(dtype) for k, v in tensors.items()}


def write_folder(path, cfg: dict, tensors: dict):
    from snowllm_b200.loader import build_model
    from snowllm_b200.weights import write_model_folder
    return write_model_folder(path, build_model(cfg, "float32").config.to_json_dict(), tensors)


def plain_logits(cfg, tensors, tokens, layers_out=None, **kw):
    return plain.forward({"config": cfg, "tensors": tensors}, list(tokens), torch.float64, layers_out, **kw)
