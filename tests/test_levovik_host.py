"""Levovik without a GPU: the configuration reader, the model spec, the layout of rotated heads, what rides in what, and
the plain implementation's own mechanisms on cases worked by hand."""
from __future__ import annotations

import copy
import importlib.util
import math
import pathlib

import pytest
import torch

import levovik_cases as cases
import plain_levovik as plain
from snowllm_b200.cache import CacheManager
from snowllm_b200.config.registry import resolve
from snowllm_b200.errors import ConfigError
from snowllm_b200.loader import build_model
from snowllm_b200.ops import kernels
from snowllm_b200.parts.channel_memory import LowRank
from snowllm_b200.parts.position import halves_order
from snowllm_b200.parts.spec import PagedKVSpec, SlotStateSpec
from snowllm_b200.weights.loader import load_tensors


def test_config_reads_back_and_builds_the_parts():
    model = build_model(cases.MIXED, "float32")
    cfg = model.config
    assert resolve(["Levovik"]).read_config(cfg.to_json_dict()) == cfg
    kinds = [(type(b.mixer.left).__name__, type(b.mixer.right).__name__, type(b.ffn).__name__) for b in model.blocks]
    assert kinds == [("RotaryAttention", "DeltaRule", "GatedFFN"), ("RotaryAttention", "GatedLinear", "SigmoidMoE"),
                     ("RotaryAttention", "DeltaRule", "NoneType"), ("RotaryAttention", "GatedLinear", "SigmoidMoE"),
                     ("RotaryAttention", "DeltaRule", "SigmoidMoE")]
    assert [b.mixer.mix for b in model.blocks[:2]] == [(0.7, 1.3), (1.1, 0.6)]
    left, right = model.blocks[0].mixer.left, model.blocks[0].mixer.right
    assert left.with_sink and not left.norm_weights and not left.keys_are_values and not left.biased
    other = model.blocks[1].mixer.left
    assert other.keys_are_values and other.norm_weights and not other.with_sink and other.position.layout == "pairs"
    assert right.num_kv_heads == 2 and right.conv_taps == 3 and model.blocks[1].mixer.right.tau == 4.0
    assert model.blocks[1].ffn.choice == {"group_score": "top2", "renorm_eps": 1e-20}
    assert model.blocks[0].ffn.activation == "relu" and model.final_norm.gain == 0.7 and model.embedding.scale == 1.5
    assert [b.side.index for b in model.blocks] == list(range(5)) and model.embedding.side_size == 40
    specs = model.cache_specs()
    assert specs[0] == (PagedKVSpec(2, 12, None, 20, separate=True),
                        SlotStateSpec(((4, 10, 14), (2, 2 * 2 * 10 + 4 * 14)), ("f32", "compute")))
    assert specs[1] == (PagedKVSpec(2, 10, None, 10, separate=True), SlotStateSpec(((3, 9, 12),), ("f32",)))
    assert specs[2][1] == SlotStateSpec(((3, 20, 8),), ("f32",))                    # one tap keeps no rows
    shapes = {spec.name: spec.shape for _, spec in model.declare(lambda n: False)}
    assert shapes["side.embed"] == (90, 40) and shapes["l3.side.gate"] == (8, 44) and shapes["l3.side.proj"] == (44, 8)
    assert shapes["l0.mix.right.a2"] == (40, 5) and shapes["l0.mix.right.g2"] == (56, 7)
    assert "l1.mix.left.v" not in shapes and "l0.mix.left.q.norm" not in shapes and shapes["l1.mix.left.q.norm"] == (10,)
    assert shapes["l0.mix.left.sink"] == (4,) and "l1.mix.left.sink" not in shapes and "l2.norm2" not in shapes
    assert {"layer_norm", "channel_memory"} <= set(model.libraries()) and "streams" not in model.libraries()


def test_ranks_come_from_the_tensors():
    cfg = copy.deepcopy(cases.MIXED)
    tensors = cases.draw_weights(cfg, 1)
    for layer in cfg["layers"]:
        for key in ("decay_rank", "gate_rank"):
            layer["mixer"]["right"].pop(key, None)
    model = build_model(cfg, "float32")
    load_tensors(model, tensors, "cpu")
    low = model.blocks[0].mixer.right.low
    assert low.a.shape == (16, 44) and low.b.shape == (96, 16)           # ranks 5 + 7, rounded up to 16
    tensors["l1.mix.right.a2"] = tensors["l1.mix.right.a2"][:, :-1].contiguous()
    with pytest.raises(ConfigError, match="ranks 6 and 5"):
        load_tensors(build_model(cfg, "float32"), tensors, "cpu")


def test_what_a_file_leaves_out_is_off():
    delta, linear = cases.delta_layer(rot_dims=0), cases.linear_layer(rot_dims=0, mlp=cases.moe(8, 4, 2, None))
    for layer in (delta, linear):
        layer["mixer"].pop("left_scale"), layer["mixer"].pop("right_scale")
    delta["mixer"]["right"].pop("kv_heads")
    linear["mixer"]["left"].pop("vdim")
    linear["mlp"]["router"].pop("scale")
    cfg = cases.config([delta, linear], side=0)
    cfg.pop("embedding"), cfg.pop("logit_scale")
    model = build_model(cfg, "float32")
    a, b = model.blocks
    assert a.mixer.mix == (1.0, 1.0) and a.mixer.right.num_kv_heads == 4 and a.side is None and model.embedding.side is None
    assert a.mixer.left.position.rotary("cpu") == (None, 0) and b.mixer.left.position.rotary("cpu") == (None, 0)
    assert b.ffn.groups == (1, 1) and b.ffn.routed_scaling_factor == 1.0
    assert model.embedding.scale == 1.0 and model.final_norm.gain == 1.0


def test_config_errors_name_every_key():
    cfg = copy.deepcopy(cases.MIXED)
    del cfg["vocab"]
    cfg["token_side"]["dim"] = 0
    cfg["layers"][0]["mixer"]["right"]["kv_heads"] = 3
    cfg["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("low")
    cfg["layers"][1]["mixer"]["left"]["vdim"] = 12
    cfg["layers"][1]["mlp"]["router"]["groups"]["count"] = 4
    cfg["layers"][2]["mixer"].pop("right")
    cfg["layers"][3]["mixer"]["right"]["tau"] = -1
    cfg["layers"][3]["mlp"]["kind"] = "wide"
    cfg["layers"][4]["mlp"]["router"]["top"] = 5                    # one group of four can be chosen from
    with pytest.raises(ConfigError) as e:
        build_model(cfg, "float32")
    for part in ("vocab", "token_side.dim=0", "heads=4 is no multiple of kv_heads=3", "rot.scaling.low", "vdim=12",
                 "groups.count=4", "layers[2].mixer.right", "tau=-1", "kind='wide'", "top=5 exceeds the 4"):
        assert part in str(e.value), part


def test_projections_are_laid_out_for_the_kernels():
    tensors = cases.draw_weights(cases.MIXED, 4)
    model = build_model(cases.MIXED, "bfloat16")
    load_tensors(model, tensors, "cpu")
    assert halves_order(8, 6) == [0, 2, 4, 1, 3, 5, 6, 7]
    left, p = model.blocks[1].mixer.left, "l1.mix.left."            # heads of 10, the first 6 turn
    order = halves_order(10, 6)
    q = tensors[p + "q"].view(6, 10, 44)[:, order].reshape(60, 44)
    k = tensors[p + "k"].view(2, 10, 44)[:, order].reshape(20, 44)
    assert torch.equal(left.w_in[:60], q) and torch.equal(left.w_in[60:80], k) and left._columns()[:3] == (0, 60, 60)
    assert torch.equal(left.wo, tensors[p + "o"].view(44, 6, 10)[:, :, order].reshape(44, 60))     # values go along
    assert torch.equal(left.q_norm, tensors[p + "q.norm"][order])
    right, col = model.blocks[1].mixer.right, 80                    # its projection is the rest of the left one's
    assert right._rides[1] == col and right.w_in is None
    assert torch.equal(left.w_in[col:col + 27], tensors["l1.mix.right.q"])
    plain_left = model.blocks[0].mixer.left                         # halves as they are
    assert torch.equal(plain_left.w_in[:48], tensors["l0.mix.left.q"])


def test_reordered_heads_give_the_same_scores():
    g = torch.Generator().manual_seed(0)
    T, d, n = 9, 10, 6
    x = torch.randn(2, T, 1, d, generator=g, dtype=torch.float64)
    freqs, pos = plain.frequencies(30.0, n), torch.arange(T) * 7
    order = halves_order(d, n)
    pairs = [plain.rotate(a, pos, freqs, True) for a in x]
    halves = [plain.rotate(a[..., order], pos, freqs, False) for a in x]
    assert torch.allclose(pairs[0][..., order], halves[0])
    assert torch.allclose((pairs[0] * pairs[1]).sum(-1), (halves[0] * halves[1]).sum(-1))
    # a rotation keeps a head's length: its root mean square may be taken before or after
    assert torch.allclose(plain.over_rms(pairs[0], 1e-5), plain.rotate(plain.over_rms(x[0], 1e-5), pos, freqs, True))


def test_low_rank_pairs_share_two_products():
    g = torch.Generator().manual_seed(1)
    a1, b1, a2, b2 = (torch.randn(*s, generator=g) for s in ((3, 20), (11, 3), (6, 20), (5, 6)))
    low = LowRank([(a1, b1), (a2, b2)], "test")
    x = torch.randn(4, 20, generator=g)
    assert low.a.shape == (16, 20)
    want = torch.cat((x @ a1.T @ b1.T, x @ a2.T @ b2.T), 1)
    assert torch.allclose(x @ low.a.T @ low.b.T, want, atol=1e-5)


def test_cache_manager_keeps_state_slots_and_pages():
    model = build_model(cases.MIXED, "float32")
    cache = CacheManager(model.cache_specs(), 4, 12, 2, torch.float32, device=None)
    assert set(cache.groups) == {("paged", None)}
    rc = cache.admit()
    assert cache.ensure(rc, 30) and cache.groups[("paged", None)].held() == 8
    cache.commit(rc, 30)
    cache.free(rc)
    assert cache.groups[("paged", None)].held() == 0 and cache.slots.free_count == 2


def test_sums_that_norms_take_apart():
    a, b = torch.randn(3, 4), torch.randn(3, 4)
    s = kernels.WeightedSum(a, b, 0.25, -2.0)
    assert torch.allclose(s.dense(), 0.25 * a - 2.0 * b) and s.shape == (3, 4)
    assert torch.allclose(kernels.DeltaSum(s, a).a, s.dense())
    assert kernels._route_flags(True, "sigmoid", None, (4, 2)) == 1 | 4 << 8 | 2 << 20
    assert kernels._route_flags(True, "sigmoid", None, (4, 2), group_score="top2", renorm_eps=1e-20) == 49 | 4 << 8 | 2 << 20


# --- the plain implementation on cases worked by hand -----------------------------------------------

def test_plain_delta_rule_replaces_what_a_key_answers():
    k = torch.tensor([[1.0, 0.0], [1.0, 0.0], [0.0, 1.0]], dtype=torch.float64).view(3, 1, 2)
    v = torch.tensor([[5.0], [7.0], [2.0]], dtype=torch.float64).view(3, 1, 1)
    one, q = torch.ones(3, 1, 2, dtype=torch.float64), torch.ones(3, 1, 2, dtype=torch.float64)
    out = plain.delta_rule(q, k, v, one, torch.ones(3, 1, dtype=torch.float64)).flatten()
    assert out.tolist() == [5.0, 7.0, 9.0]                 # the second write to a key takes the first one off
    half = plain.delta_rule(q, k, v, one, torch.full((3, 1), 0.5, dtype=torch.float64)).flatten()
    assert half.tolist() == [2.5, 4.75, 5.75]
    fades = plain.delta_rule(q, k, v, one * torch.tensor([0.5, 1.0]), torch.ones(3, 1, dtype=torch.float64)).flatten()
    assert fades.tolist() == [5.0, 7.0, 5.5]               # a decay acts on the rows of its key channel, before the write
    assert plain.linear_memory(q, k, v, one * torch.tensor([0.5, 1.0])).flatten().tolist() == [5.0, 9.5, 6.75]


def test_plain_choice_takes_a_groups_two_best():
    s = torch.tensor([[0.9, 0.0, 0.1, 0.6, 0.5, 0.2], [0.3, 0.2, 0.9, 0.1, 0.0, 0.8]], dtype=torch.float64)
    assert plain.choose(s, 2, 2, 1).tolist() == [[3, 4], [2, 0]] or plain.choose(s, 2, 2, 1).tolist() == [[3, 4], [0, 2]]
    assert plain.choose(s, 2, 1, 1).tolist() == [[0, 3], [2, 5]]
    assert plain.choose(s, 1, 6, 2).tolist() == [[0], [2]]          # groups of one: their only score


def test_plain_sink_takes_its_share_and_counts_once():
    q = torch.zeros(2, 1, 3, dtype=torch.float64)
    v = torch.tensor([[3.0], [6.0]], dtype=torch.float64).view(2, 1, 1)
    out = plain.attend(q, q, v, 0.5, torch.tensor([math.log(2.0)], dtype=torch.float64)).flatten()
    assert torch.allclose(out, torch.tensor([1.0, 9.0 / 4], dtype=torch.float64))


def test_bench_option_builds_the_design_and_its_neighbour():
    spec = importlib.util.spec_from_file_location("bench_levovik", pathlib.Path(__file__).resolve().parent.parent / "bench.py")
    bench = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(bench)
    name, ours, (other, theirs), _ = bench.DESIGNS["levovik"]
    for width, layers, ff in bench.DESIGN_SIZES.values():
        a, b = build_model(ours(width, layers, ff)), build_model(theirs(width, layers, ff))
        assert a.config.architecture == name and len(a.blocks) == len(b.blocks) == layers
        assert a.blocks[0].mixer.left.num_heads == b.blocks[0].mixer.left.num_heads
        assert a.blocks[1].mixer.right.num_heads == b.blocks[1].mixer.right.num_heads
