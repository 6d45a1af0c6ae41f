"""Gurolix without a GPU: the configuration reader, the model spec, the rescaled rotary table, and the plain
implementation's own mechanisms on cases worked by hand."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import gurolix_cases as cases
import plain_gurolix as plain
from snowllm_b200.cache import CacheManager
from snowllm_b200.config.registry import resolve
from snowllm_b200.errors import ConfigError, KernelError
from snowllm_b200.loader import build_model
from snowllm_b200.parts.position import BandedRotaryPosition
from snowllm_b200.parts.spec import PagedKVSpec, SlotStateSpec
from snowllm_b200.weights.loader import load_tensors


def test_config_reads_back_and_builds_the_parts():
    model = build_model(cases.MIXED, "float32")
    cfg = model.config
    assert resolve(["Gurolix"]).read_config(cfg.to_json_dict()) == cfg
    kinds = [(type(b.mixer).__name__, b.ffn is not None) for b in model.blocks]
    assert kinds == [("Mamba2", True), ("RotaryAttention", False), ("RotaryAttention", True), ("Mamba2", True),
                     ("RotaryAttention", True), ("Mamba2", False), ("RotaryAttention", True)]
    assert [getattr(b.mixer, "value_role", None) for b in model.blocks] == [None, None, "first", None, "mix", None, "mix"]
    assert [getattr(b.mixer, "softcap", None) for b in model.blocks] == [None, None, 3.0, None, None, None, 1.5]
    assert model.blocks[0].ffn.groups == (3, 2) and model.blocks[0].ffn.identity == 1 and model.blocks[4].ffn.groups == (1, 1)
    specs = model.cache_specs()
    assert specs[0] == SlotStateSpec(((6, 12, 10), (2, 60 + 2 * 2 * 12)), ("f32", "compute"))
    assert specs[1] == PagedKVSpec(2, 12, None, 20, separate=True) and specs[2] == PagedKVSpec(2, 10, None, 8, separate=True)
    shapes = {spec.name: spec.shape for _, spec in model.declare(lambda n: False)}
    assert shapes["l0.mix.in"] == (60 + 60 + 2 * 24 + 6, 44) and shapes["l0.mix.conv"] == (108, 3)
    assert shapes["l0.mlp.router"] == (6, 44) and shapes["l0.mlp.correction"] == (6,)
    assert shapes["l4.mlp.router"] == (8, 44) and shapes["l6.dwa"] == (8,) and shapes["l0.dwa"] == (2,)
    assert shapes["l1.rg1"] == (44, 44) and shapes["embed.norm"] == (44,) and shapes["l2.mix.vmix"] == ()
    assert "l4.mlp.e2.down" in shapes and "l4.mlp.e3.down" not in shapes      # identity experts have no tensors
    assert "l1.mix.q.norm" in shapes and "l2.mix.q.norm" not in shapes
    assert "l1.norm2" not in shapes and "l1.rg2" not in shapes and "l1.norm2b" not in shapes and "l1.mix.vmix" not in shapes
    assert "sandwich" in model.libraries() and "state_space" in model.libraries()


def test_what_a_file_leaves_out_is_off():
    layer = cases.capped_layer(rot_dims=0, softcap=None, v_mix=None, mlp=cases.moe(8, 4, 2, 0, None))
    state = cases.state_layer(mlp=None)
    del state["mixer"]["groups"], state["mixer"]["norm_groups"]
    model = build_model(cases.config([layer, state]), "float32")
    mixer, ffn, other = model.blocks[0].mixer, model.blocks[0].ffn, model.blocks[1].mixer
    assert mixer.softcap is None and mixer.value_role is None and mixer.position.rotary("cpu") == (None, 0)
    assert ffn.identity == 0 and ffn.groups == (1, 1)
    assert other.num_groups == 1 and other.norm_groups == 1 and model.blocks[1].ffn is None


def test_config_errors_name_every_key():
    cfg = copy.deepcopy(cases.MIXED)
    del cfg["vocab"]
    cfg["layers"][0]["mixer"]["groups"] = 4
    cfg["layers"][0]["mlp"]["router"]["groups"]["count"] = 4
    cfg["layers"][1]["mixer"]["rot"]["dims"] = 7
    cfg["layers"][2]["mixer"]["rot"]["scaling"].pop("low")
    cfg["layers"][3]["mlp"]["router"]["top"] = 4                    # one group of three can be chosen from
    cfg["layers"][4]["mixer"]["kv_heads"] = 1                       # its values cannot mix with layer 2's
    cfg["layers"][5]["type"] = "mamba3"
    cfg["layers"][6]["mixer"]["softcap"] = -1
    with pytest.raises(ConfigError) as e:
        build_model(cfg, "float32")
    for part in ("vocab", "heads=6 is no multiple of groups=4", "groups.count=4", "rot.dims=7", "rot.scaling.low",
                 "top=4 exceeds the 3", "cannot mix with layer 2", "mamba3", "softcap=-1"):
        assert part in str(e.value), part


def test_weights_load_and_norms_are_kept_around_one():
    tensors = cases.draw_weights(cases.MIXED, 4)
    model = build_model(cases.MIXED, "bfloat16")
    load_tensors(model, tensors, "cpu")
    w = model.blocks[0].mixer_norm.weight
    assert w.dtype == torch.float32 and torch.equal(w, tensors["l0.norm1"].float() + 1.0)
    assert torch.equal(model.embedding.norm.weight, tensors["embed.norm"].float() + 1.0)
    assert torch.equal(model.blocks[3].average.weight, tensors["l3.dwa"].float())
    assert model.blocks[4].mixer.value_lambda == float(tensors["l4.mix.vmix"])
    m = model.blocks[0].mixer                                       # the convolved columns come first
    assert torch.equal(m.w_in[:108], tensors["l0.mix.in"][60:168]) and torch.equal(m.w_in[108:168], tensors["l0.mix.in"][:60])
    assert torch.equal(m.w_in[168:174], tensors["l0.mix.in"][168:])
    assert torch.allclose(m.rate, -torch.exp(tensors["l0.mix.A_log"].float()))


def test_cache_manager_keeps_state_slots_and_pages():
    model = build_model(cases.MIXED, "float32")
    cache = CacheManager(model.cache_specs(), 4, 12, 2, torch.float32, device=None)
    assert set(cache.groups) == {("paged", None)}
    rc = cache.admit()
    assert cache.ensure(rc, 30) and cache.groups[("paged", None)].held() == 8
    cache.commit(rc, 30)
    cache.free(rc)
    assert cache.groups[("paged", None)].held() == 0 and cache.slots.free_count == 2


def test_rescaled_frequencies_keep_the_fast_ones_and_stretch_the_slow_ones():
    s = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}
    pos = BandedRotaryPosition(head_dim=16, theta=100.0, rot_dim=12, scaling=s)
    plain_f = [100.0 ** (-2.0 * i / 12) for i in range(6)]
    got = pos.frequencies()
    waves = [2 * math.pi / f for f in plain_f]
    assert waves[0] < 64 / 4 < waves[3] < 64 < waves[-1]
    for f, g, wave in zip(plain_f, got, waves):
        if wave < 16:
            assert g == f
        elif wave > 64:
            assert g == f / 4
        else:
            share = (64 / wave - 1.0) / 3.0
            assert abs(g - ((1 - share) * f / 4 + share * f)) < 1e-15 and f / 4 < g < f
    assert got == pytest.approx(plain.frequencies(100.0, 12, s), rel=1e-14)
    table, dims = pos.rotary("cpu")
    assert dims == 12 and table.dtype == torch.float32 and table.tolist() == [float(torch.tensor(f, dtype=torch.float32)) for f in got]
    assert BandedRotaryPosition(head_dim=16, theta=100.0).frequencies() == [100.0 ** (-2.0 * i / 16) for i in range(8)]


# --- the plain implementation on cases worked by hand ---------------------------------------------------

def test_plain_state_space_by_hand():
    x = torch.tensor([[[2.0]], [[3.0]]], dtype=torch.float64)
    B = torch.tensor([[[1.0, -1.0]], [[0.5, 2.0]]], dtype=torch.float64)
    C = torch.tensor([[[1.0, 1.0]], [[4.0, 1.0]]], dtype=torch.float64)
    step = torch.tensor([[0.5], [2.0]], dtype=torch.float64)
    decay = torch.tensor([[0.9], [0.25]], dtype=torch.float64)
    y = plain.state_space(x, B, C, step, decay, torch.tensor([10.0], dtype=torch.float64))
    # S_1 = 0.5 * 2 * (1, -1); S_2 = 0.25 S_1 + 2 * 3 * (0.5, 2) = (3.25, 11.75)
    assert y[0, 0, 0] == pytest.approx(0.0 + 20.0) and y[1, 0, 0] == pytest.approx(4 * 3.25 + 11.75 + 30.0)
    assert float(plain.softplus(torch.tensor(0.0))) == pytest.approx(math.log(2)) and float(plain.softplus(torch.tensor(50.0))) == 50.0


def test_plain_choice_within_the_best_groups_with_negative_scores():
    choice = torch.tensor([[-1.0, -5.0, -2.0, -2.5, -9.0, -1.5]], dtype=torch.float64)
    assert plain.choose(choice, 2, 3, 1).tolist() == [[0, 1]]        # group 0 holds the best score; its second is taken
    assert plain.choose(choice, 2, 3, 2).tolist() == [[0, 5]]
    assert plain.choose(choice, 3, 1, 1).tolist() == [[0, 2, 5]]


def test_plain_experts_weigh_by_the_uncorrected_softmax_and_identity_returns_its_input():
    h = torch.tensor([[1.0, 2.0]], dtype=torch.float64)
    t = {"router": torch.zeros(3, 2, dtype=torch.float64), "correction": torch.tensor([-3.0, -1.0, -2.0], dtype=torch.float64),
         "e0.up": torch.ones(1, 2, dtype=torch.float64), "e0.down": torch.ones(2, 1, dtype=torch.float64),
         "e1.up": torch.tensor([[1.0, 0.0], [-1.0, 0.0]], dtype=torch.float64), "e1.down": torch.eye(2, dtype=torch.float64) * 6}
    out, picks = plain.experts(h, t, {"router": {"experts": 2, "top": 2, "identity": 1}}, "")
    # relu(1)^2 = 1 and relu(-1)^2 = 0 through the second expert; the third output is h itself; thirds each
    assert picks.tolist() == [[1, 2]] and out[0].tolist() == pytest.approx([(6 + 1) / 3, 2 / 3])


def test_plain_values_mix_before_they_are_read():
    g = torch.Generator().manual_seed(1)
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0}
    t = {n: torch.zeros(2, 3, dtype=torch.float64) for n in ("q", "k")}
    t["v"] = torch.randn(2, 3, generator=g).double()
    t.update({n + ".b": torch.zeros(2, dtype=torch.float64) for n in ("q", "k")})
    t["v.b"] = torch.tensor([1.0, -1.0], dtype=torch.float64)
    t["o"], t["vmix"] = torch.eye(2, dtype=torch.float64), torch.tensor(0.25, dtype=torch.float64)
    h = torch.randn(2, 3, generator=g).double()
    first = torch.randn(2, 1, 2, generator=g).double()
    out, own = plain.attention(h, t, m, 1e-6, "", torch.arange(2), first, normed=False)
    v = 0.75 * (h @ t["v"].T + t["v.b"]) + 0.25 * first[:, 0]
    assert torch.allclose(out, torch.stack((v[0], v.mean(0)))) and torch.allclose(own[:, 0], h @ t["v"].T + t["v.b"])


def test_a_pending_update_does_not_pretend_to_be_a_delta():
    from snowllm_b200.ops import kernels
    delta = kernels.NormedDelta(torch.ones(2, 4), weight=torch.ones(4), eps=1e-6)
    assert torch.allclose(delta.total(torch.zeros(2, 4)), torch.ones(2, 4), atol=1e-5)
    with pytest.raises(KernelError):
        delta.dense()


def test_bench_design_option_builds_both_models_at_equal_size():
    import bench
    name, ours_of, (other, theirs_of), _ = bench.DESIGNS["gurolix"]
    assert name == "Gurolix" and other == "lfm2_moe_alternating"
    for width, layers, ff in bench.DESIGN_SIZES.values():
        ours, theirs = build_model(ours_of(width, layers, ff), "bfloat16"), build_model(theirs_of(width, layers, ff), "bfloat16")
        assert len(ours.run) == len(theirs.run) == layers and ours.spec.hidden_size == theirs.spec.hidden_size == width
        for mine, theirs_block in zip(ours.blocks, theirs.blocks):
            attends = type(mine.mixer).__name__ == "RotaryAttention"
            assert attends == (type(theirs_block.mixer).__name__ == "Attention")
            if attends:
                assert (mine.mixer.num_heads, mine.mixer.num_kv_heads, mine.mixer.head_dim) == \
                       (theirs_block.mixer.num_heads, theirs_block.mixer.num_kv_heads, theirs_block.mixer.head_dim)
        routed, theirs_routed = ours.blocks[1].ffn, theirs.blocks[1].ffn
        assert routed.num_experts + routed.identity == theirs_routed.num_experts and routed.top_k == theirs_routed.top_k
        assert routed.intermediate_size == theirs_routed.intermediate_size


def test_an_output_gate_rides_in_its_mixers_projection():
    tensors = cases.draw_weights(cases.MIXED, 4)
    model = build_model(cases.MIXED, "bfloat16")
    load_tensors(model, tensors, "cpu")
    for i, block in enumerate(model.blocks):
        gate, col = block.gates[0], block.gates[0]._rides[1]
        assert gate.weight is None and col % 16 == 0
        assert torch.equal(block.mixer.w_in[col:col + 44], tensors[f"l{i}.rg1"])
        if getattr(block.mixer, "proj_bias", None) is not None:
            assert block.mixer.proj_bias.shape[0] == block.mixer.w_in.shape[0] and not block.mixer.proj_bias[col:].any()
        if block.ffn is not None:
            assert torch.equal(block.gates[1].weight, tensors[f"l{i}.rg2"])
