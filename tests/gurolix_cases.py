"""Small Gurolix configurations, weights that make faults show, and helpers to run a request through the
engine's step function (any cut into steps) and through the plain implementation."""
from __future__ import annotations

import copy

import torch

import plain_gurolix as plain
from beledra_cases import cuts_of, relative_error, run_cuts, tokens_for, worst_row_error  # noqa: F401


def moe(ff=24, experts=5, top=2, identity=1, groups=(3, 2)):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


SCALING = {"factor": 5.0, "low": 1.5, "high": 6.0, "original": 70}


def _attention(kind, heads, kv_heads, dim, vdim, scale, rot_dims, base, scaling, softcap, v_mix, mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
        if scaling is not None:
            m["rot"]["scaling"] = dict(scaling)
    if softcap is not None:
        m["softcap"] = softcap
    if v_mix is not None:
        m["v_mix"] = v_mix
    return {"type": kind, "mixer": m, "mlp": moe() if mlp == "moe" else mlp}


def normed_layer(heads=4, kv_heads=2, dim=12, vdim=8, scale=0.4, rot_dims=8, base=900.0, scaling=None, softcap=None,
                 v_mix=True, mlp="moe"):
    """attention: q and k normalised per head."""
    return _attention("attention", heads, kv_heads, dim, vdim, scale, rot_dims, base, scaling, softcap, v_mix, mlp)


def capped_layer(heads=6, kv_heads=2, dim=10, vdim=8, scale=0.5, rot_dims=10, base=50.0, scaling=SCALING, softcap=3.0,
                 v_mix=True, mlp="moe"):
    """attention_2: no norms, rescaled frequencies, a cap on the scores."""
    return _attention("attention_2", heads, kv_heads, dim, vdim, scale, rot_dims, base, scaling, softcap, v_mix, mlp)


def state_layer(heads=6, vdim=10, state=12, groups=2, norm_groups=3, conv=3, mlp="moe"):
    """mamba2."""
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                        "norm_groups": norm_groups, "conv": conv},
            "mlp": moe() if mlp == "moe" else mlp}


def config(layers, vocab=90, width=44, eps=1e-5):
    return {"architecture": "Gurolix", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": copy.deepcopy(layers)}


# every mixer, layers of one kind with different sizes, with and without a feed-forward, values that mix beside ones
# that do not, one kv head per head, one group and one norm group, all experts of a group picked, no identity experts
MIXED = config([state_layer(),
                normed_layer(v_mix=None, vdim=20, mlp=None),
                capped_layer(),
                state_layer(heads=3, vdim=24, state=40, groups=3, norm_groups=1, conv=4, mlp=moe(16, 6, 3, 0, (2, 1))),
                normed_layer(heads=2, kv_heads=2, dim=16, rot_dims=16, base=5e4, scaling=SCALING, mlp=moe(8, 3, 1, 5, None)),
                state_layer(heads=2, vdim=6, state=7, groups=1, norm_groups=2, conv=2, mlp=None),
                capped_layer(heads=4, kv_heads=2, dim=20, rot_dims=6, scaling=None, softcap=1.5)])

# heads of 64 for keys and values and a state-space mixer of tensor-core sizes: the sizes the fast kernels take
HEADS_OF_64 = config([capped_layer(heads=6, kv_heads=3, dim=64, vdim=64, scale=0.16, rot_dims=32, softcap=4.0),
                      state_layer(heads=4, vdim=64, state=64, groups=2, norm_groups=2, conv=4, mlp=moe(32, 6, 2, 2, (2, 1))),
                      normed_layer(heads=6, kv_heads=3, dim=64, vdim=64, scale=0.2, rot_dims=64, mlp=None),
                      state_layer(heads=2, vdim=128, state=128, groups=1, norm_groups=1, conv=4, mlp=moe(16, 3, 2, 1, None)),
                      normed_layer(heads=6, kv_heads=3, dim=64, vdim=64, scale=0.15, rot_dims=16, softcap=9.0)], width=64)


def draw_weights(cfg: dict, seed: int = 0, dtype=torch.bfloat16) -> dict:
    """name -> tensor (as stored: ``dtype``) from the framework's seeded generator, with the small tensors redrawn so
    that each mechanism carries weight: norm weights away from zero, gates and routers whose logits are spread out, a
    depth average of comparable shares, decays from nearly none to a few tokens, corrections that change the choice
    and keep every choice score negative."""
    from snowllm_b200.loader import build_model
    from snowllm_b200.weights import random_tensors
    model = build_model(cfg, "float32")
    tensors = random_tensors(model, seed, torch.float32, fan_in_scaled=True, norm_jitter=0.2)
    gen = torch.Generator().manual_seed(seed + 1)
    for name, t in tensors.items():
        def randn(scale=1.0):
            return torch.randn(t.shape, generator=gen) * scale
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm1b", "norm2", "norm2b") or name in ("embed.norm", "final.norm"):
            tensors[name] = randn(0.3)
        elif leaf == "dwa":
            tensors[name] = randn(0.4)
            tensors[name][-1] += 0.6
        elif leaf in ("rg1", "rg2"):
            tensors[name] = t * 2.0
        elif leaf == "router":
            tensors[name] = t * 2.0
        elif leaf == "correction":
            tensors[name] = randn(0.3) - 2.0
        elif leaf == "A_log":
            tensors[name] = torch.rand(t.shape, generator=gen) * 4.5 - 3.5
        elif leaf == "dt_bias":
            tensors[name] = torch.rand(t.shape, generator=gen) * 3.0 - 3.0
        elif leaf == "D":
            tensors[name] = randn(1.0)
        elif leaf == "conv":
            tensors[name] = randn(0.7)
        elif leaf == "vmix":
            tensors[name] = 0.2 + 0.6 * torch.rand(t.shape, generator=gen)
        elif leaf == "b":
            tensors[name] = randn(0.7)
    return {k: v.to(dtype) for k, v in tensors.items()}


def write_folder(path, cfg: dict, tensors: dict):
    from snowllm_b200.loader import build_model
    from snowllm_b200.weights import write_model_folder
    return write_model_folder(path, build_model(cfg, "float32").config.to_json_dict(), tensors)


def plain_logits(cfg, tensors, tokens, layers_out=None, **kw):
    return plain.forward({"config": cfg, "tensors": tensors}, list(tokens), torch.float64, layers_out, **kw)
