"""Levovik on the GPU against the plain implementation (tests/plain_levovik.py): every mechanism alone, the kernels on
inputs that make a wrong key, a lost state, a wrong group or a missing sink show, and one model with everything fed whole,
token by token, in portions and in mixed batches over pools and slots that are used again."""
from __future__ import annotations

import pytest
import torch

import levovik_cases as cases
import plain_levovik as plain

pytestmark = pytest.mark.gpu

F32_TOL = 5e-5          # float32 engine against the float64 plain implementation
BF16_TOL = 0.06         # bfloat16 engine against the plain implementation on the same (rounded) weights


def load(cfg, tensors, dtype):
    from snowllm_b200.loader import build_model
    from snowllm_b200.weights.loader import load_tensors
    model = build_model(cfg, dtype)
    load_tensors(model, tensors, "cuda")
    return model


def replay(model, max_tokens=512, requests=4, page_size=16):
    from snowllm_b200.engine.replay import Replay
    return Replay(model, None, max_tokens, requests, page_size=page_size)


def reference(cfg, tensors, tokens, layers_out=None, **kw):
    return cases.plain_logits(cfg, {k: v.double() for k, v in tensors.items()}, tokens, layers_out, **kw)


def tolerance(dtype):
    return F32_TOL if dtype == "float32" else BF16_TOL


def engine_picks(rp):
    return [t.cpu() for n, t in rp.runner.taps if n == "moe_route"]


def routed_layers(cfg):
    return [i for i, l in enumerate(cfg["layers"]) if l["mlp"] is not None and l["mlp"]["kind"] == "moe"]


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


# --- each mechanism alone -------------------------------------------------------------------------

ALONE = {
    "delta": dict(layers=[cases.delta_layer()]),
    "delta_no_ff_no_side": dict(layers=[cases.delta_layer(mlp=None)], side=0),
    "delta_dense": dict(layers=[cases.delta_layer(mlp=cases.dense(36))]),
    "delta_one_tap_own_keys": dict(layers=[cases.delta_layer(r_heads=3, r_kv_heads=3, conv=1, mlp=None)]),
    "delta_heads_share_keys": dict(layers=[cases.delta_layer(r_heads=6, r_kv_heads=1, r_dim=16, r_vdim=8, conv=7)]),
    "delta_wide_memory": dict(layers=[cases.delta_layer(r_heads=1, r_kv_heads=1, r_dim=136, r_vdim=72, mlp=None)]),
    "delta_tensor_core_sizes": dict(layers=[cases.delta_layer(heads=4, kv_heads=2, dim=80, vdim=40, rot_dims=48, r_heads=2,
                                                              r_kv_heads=1, r_dim=64, r_vdim=64, ranks=(16, 16))]),
    "delta_no_rotation_one_scale": dict(layers=[cases.delta_layer(rot_dims=0, scales=(1.0, 1.0))]),
    "linear": dict(layers=[cases.linear_layer()]),
    "linear_no_ff": dict(layers=[cases.linear_layer(mlp=None)]),
    "linear_plain_rotation": dict(layers=[cases.linear_layer(scaling=None, rot_dims=10, tau=1.0)]),
    "linear_one_head": dict(layers=[cases.linear_layer(heads=5, kv_heads=1, dim=16, rot_dims=4, r_heads=1, r_dim=20, r_vdim=33)]),
    "linear_tensor_core_sizes": dict(layers=[cases.linear_layer(heads=4, kv_heads=2, dim=96, rot_dims=96, r_heads=2, r_dim=128,
                                                                r_vdim=32, tau=16.0, rank=16)]),
    "experts_no_groups": dict(layers=[cases.linear_layer(mlp=cases.moe(16, 5, 3, None, 2.0, 1.0))]),
    "experts_groups_of_one": dict(layers=[cases.delta_layer(mlp=cases.moe(16, 5, 2, (5, 3), 0.5, 2.0))]),
    "experts_all_picked": dict(layers=[cases.linear_layer(mlp=cases.moe(24, 4, 4, (2, 2), 1.0, 0.5))]),
    "heads_of_128": dict(layers=[cases.delta_layer(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09, rot_dims=128),
                                 cases.linear_layer(heads=2, kv_heads=1, dim=128, scale=0.09, rot_dims=64)], width=48),
    "heads_of_64": dict(layers=cases.HEADS_OF_64["layers"], width=64, side=24),
    # sizes that are multiples of nothing: the products leave the tensor cores
    "odd_sizes": dict(layers=[cases.delta_layer(heads=3, kv_heads=1, dim=10, vdim=6, rot_dims=6, r_heads=5, r_kv_heads=5, r_dim=7,
                                                r_vdim=9, conv=4, ranks=(3, 2), mlp=cases.moe(22, 9, 3, (3, 2))),
                              cases.linear_layer(heads=34, kv_heads=2, dim=6, rot_dims=2, r_heads=5, r_dim=11, r_vdim=7, rank=1,
                                                 mlp=cases.dense(10))], width=37, vocab=50, side=5),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALONE))
def test_each_mechanism_alone(name, dtype):
    kw = dict(ALONE[name])
    cfg = cases.config(kw.pop("layers"), **kw)
    tensors = cases.draw_weights(cfg, seed=len(name))
    tokens = cases.tokens_for(cfg, 70)
    model = load(cfg, tensors, dtype)
    rp = replay(model)
    rp.runner.taps = []
    got = cases.run_cuts(rp, "a", tokens, [len(tokens)])
    # the plain experts are put on the engine's picks: a near tie may fall either way, the rest must agree
    routed = routed_layers(cfg)
    force = dict(zip(routed, [t.long().sort(-1).values for t in engine_picks(rp)]))
    assert len(force) == len(routed)
    want_layers, free = [], {}
    want = reference(cfg, tensors, tokens, want_layers, picks=force)
    reference(cfg, tensors, tokens, picks_out=free)
    for i in routed:
        differ = (free[i] != force[i]).any(-1).float().mean()
        assert float(differ) <= (0.0 if dtype == "float32" else 0.15), (i, float(differ))
    layers = [t for n, t in rp.runner.taps if n == "layer_out"]
    assert len(layers) == len(want_layers)
    for x, w in zip(layers, want_layers):
        assert cases.relative_error(x.cpu(), w) < tolerance(dtype)
    assert cases.worst_row_error(got, want) < tolerance(dtype) * 2
    # token by token through the cache and the state gives the same
    rp.runner.taps = None
    again = cases.run_cuts(rp, "b", tokens, [1] * len(tokens))
    assert cases.worst_row_error(again, want) < tolerance(dtype) * 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("pair", ["delta", "linear"])
def test_a_key_far_back_owns_a_row(pair, dtype):
    """Attention alone (the memory's share is off): one early token's key answers a late token's query, in a prompt and in
    decoding, in heads of 64 (prompt and decode kernels of their own) and of another size."""
    for dim in (64, 24):
        layer = (cases.delta_layer(heads=2, kv_heads=1, dim=dim, vdim=dim, scale=8.0 / dim, rot_dims=0, scales=(1.0, 0.0), mlp=None)
                 if pair == "delta" else
                 cases.linear_layer(heads=2, kv_heads=1, dim=dim, scale=8.0 / dim, rot_dims=0, scales=(1.0, 0.0), mlp=None))
        cfg = cases.config([layer], vocab=40, width=32, side=0, embedding_scale=0.4)
        tensors = cases.draw_weights(cfg, 3)
        tokens = [t % 38 for t in cases.tokens_for(cfg, 300)]
        tokens[4], tokens[-1], tokens[-40] = 39, 38, 38             # the pair that must meet: 39 far back, 38 late
        p = "l0.mix.left."
        e = tensors["embed"].double()
        h = plain.centred_norm(e[[39, 38]] * 0.4, tensors["l0.norm1"].double(), 1e-5)
        # the query of 38 looks along the key of 39: a rank-one addition to W_q
        key = h[0] @ tensors[p + "k"].double().T
        add = torch.outer(torch.cat([key, key]), h[1]) / (h[1] @ h[1]) * 20
        tensors[p + "q"] = (tensors[p + "q"].double() + add).to(torch.bfloat16)
        want = reference(cfg, tensors, tokens)
        other = list(tokens)
        other[4] = 1
        moved = reference(cfg, tensors, other)
        assert cases.worst_row_error(moved[-1:], want[-1:]) > 0.3   # without that key the row is another
        rp = replay(load(cfg, tensors, dtype))
        for cuts in ([300], [259] + [1] * 41, [128, 128, 3] + [1] * 41):
            got = cases.run_cuts(rp, "a", tokens, cuts)
            assert cases.worst_row_error(got[-1:], want[-1:]) < tolerance(dtype) * 2, (dim, cuts)
            assert cases.worst_row_error(got[-40:-39], want[-40:-39]) < tolerance(dtype) * 2, (dim, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_large_sink_empties_the_heads(dtype):
    cfg = cases.config([cases.delta_layer(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.1, rot_dims=64, scales=(1.0, 0.0), mlp=None)],
                       width=64, side=0, embedding_scale=0.3)
    tensors = cases.draw_weights(cfg, 8)
    tensors["l0.mix.left.sink"] = torch.tensor([30.0, 2.0, -30.0, 5.0]).to(torch.bfloat16)
    tokens = cases.tokens_for(cfg, 150)
    want = reference(cfg, tensors, tokens)
    left_out = reference(cfg, dict(tensors, **{"l0.mix.left.sink": torch.full((4,), -60.0)}), tokens)
    assert cases.worst_row_error(left_out, want) > 0.3
    rp = replay(load(cfg, tensors, dtype))
    for cuts in ([150], [100] + [1] * 50):
        assert cases.worst_row_error(cases.run_cuts(rp, "a", tokens, cuts), want) < tolerance(dtype) * 2


# --- the memories --------------------------------------------------------------------------------

def memory_case(delta, H, G, dk, dv, T, seed, strong=False, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return dict(u=torch.randn(T, 2 * G * dk + H * dv, generator=g).to(dtype),
                z=torch.randn(T, H * dk, generator=g) * (6.0 if strong else 1.5), bias=torch.randn(H * dk, generator=g) * 0.5,
                rate=-torch.exp(torch.rand(H, generator=g) * 3 - 1.5) if delta else None,
                beta=(torch.randn(T, H, generator=g) * 2).to(dtype) if delta else None, sharp=0.3)


def plain_memory(c, H, G, dk, dv):
    T = c["u"].shape[0]
    q, k, v = torch.split(c["u"].double(), [G * dk, G * dk, H * dv], -1)
    q, k = (a.view(T, G, dk).repeat_interleave(H // G, 1) for a in (q, k))
    v, z = v.view(T, H, dv), (c["z"].double() + c["bias"].double()).view(T, H, dk)
    if c["rate"] is None:
        return plain.linear_memory(q * dk ** -0.5, k, v, torch.exp(-c["sharp"] * plain.softplus(-z))).view(T, -1)
    decay = torch.exp(c["rate"].double()[None, :, None] * plain.softplus(z))
    return plain.delta_rule(plain.over_length(q) * dk ** -0.5, plain.over_length(k), v, decay,
                            plain.sigmoid(c["beta"].double())).view(T, -1)


def run_memory(parts, state, G, rows_before=3, col=8):
    """One step over several segments: ``parts`` = [(case, first row, rows, slot)]; the rows lie behind ``col`` other
    columns, as in a product that two mixers share."""
    from types import SimpleNamespace
    from snowllm_b200.ops import kernels
    from snowllm_b200.parts.decay_memory import memory_pieces
    H, dk, dv = state.shape[1:]
    first = parts[0][0]

    def rows(name):
        return torch.cat([c[name][at:at + n] for c, at, n, _ in parts])
    u = rows("u")
    u = torch.cat((torch.full((u.shape[0], col), float("nan"), dtype=u.dtype), u), 1).contiguous().cuda()
    lens = [n for _, _, n, _ in parts]
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    pieces = memory_pieces(SimpleNamespace(capture_max_len=None, host_seg_len=lens, memo={}, device="cuda"), kernels.MEMORY_CHUNK)
    kw = {}
    if first["rate"] is not None:
        kw = dict(rate=first["rate"].cuda(), beta=rows("beta").contiguous().cuda())
    return kernels.channel_memory(u, col, col + G * dk, col + 2 * G * dk, rows("z").contiguous().cuda(), 0, first["bias"].cuda(),
                                  i32(cu), i32([at for _, at, _, _ in parts]), i32([s for _, _, _, s in parts]), state, G, max(lens),
                                  sharp=first["sharp"], q_scale=dk ** -0.5, unit_eps=1e-6, pieces=pieces, **kw).cpu()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,G,dk,dv", [(2, 1, 128, 128), (4, 4, 48, 32), (3, 1, 20, 9), (1, 1, 200, 40), (2, 2, 64, 132), (1, 1, 32, 256)])
@pytest.mark.parametrize("delta", [True, False])
def test_memory_kernels(delta, H, G, dk, dv, strong, dtype):
    """Whole, in portions on both sides of every path's limit and of every chunk's edge, and token by token: the rows and
    the state that is handed on are float sums in every case, also where a decay all but ends a channel."""
    if not delta:
        G = H
    T = 130
    c = memory_case(delta, H, G, dk, dv, T, H * dk + dv, strong, dtype)
    want = plain_memory(c, H, G, dk, dv)
    size = float(want.abs().max())
    for cuts in ([T], [15, 33, 16, 17, 2, 47], cases.cuts_of(T, [2]), [1] * T, [100] + [1] * 30, [34, 32, 31, 33]):
        state = torch.randn(3, H, dk, dv).cuda()                    # what a slot held before must not matter
        kept, out, at = state.clone(), [], 0
        for n in cuts:
            out.append(run_memory([(c, at, n, 1)], state, G))
            at += n
        assert float((torch.cat(out).double() - want).abs().max()) < 1.5e-6 * size, cuts
        assert torch.equal(state[[0, 2]], kept[[0, 2]])


@pytest.mark.parametrize("delta", [True, False])
@pytest.mark.parametrize("lens", [[40, 1, 17, 1], [1, 1, 1, 1], [3, 2, 20, 1], [100, 64, 33, 32]])
def test_memory_kernels_keep_requests_apart(delta, lens):
    H, G, dk, dv = 2, 2, 32, 24
    runs = [memory_case(delta, H, G, dk, dv, 150, 50 + i) for i in range(4)]
    for other in runs[1:]:                                           # one layer's constants
        other.update(bias=runs[0]["bias"], rate=runs[0]["rate"])
    want = [plain_memory(c, H, G, dk, dv) for c in runs]
    state = torch.full((5, H, dk, dv), float("nan")).cuda()
    starts = [0, 21, 0, 40]
    for i, s in enumerate(starts):
        if s:
            run_memory([(runs[i], 0, s, 4 - i)], state, G)
    got = run_memory([(runs[i], starts[i], n, 4 - i) for i, n in enumerate(lens)], state, G)
    at = 0
    for i, n in enumerate(lens):
        w = want[i][starts[i]:starts[i] + n]
        assert float((got[at:at + n].double() - w).abs().max()) < 5e-6, i
        at += n


def test_memory_keeps_what_barely_decays():
    """A channel that forgets nothing beside channels that forget at once: a write far back is read, in every path."""
    H, dk, dv, T = 1, 32, 16, 200
    for delta in (True, False):
        u = torch.zeros(T, 2 * dk + H * dv)
        u[3, dk] = 1.0                                               # k of the one token that writes: channel 0
        u[3, 2 * dk:] = torch.arange(1.0, dv + 1)
        u[-1, 0] = 1.0
        z = torch.full((T, H * dk), 25.0 if delta else -40.0)        # gone within a token
        z[:, 0] = -25.0 if delta else 25.0
        c = dict(u=u, z=z, bias=torch.zeros(dk), rate=torch.tensor([-4.0]) if delta else None,
                 beta=torch.full((T, 1), 30.0) if delta else None, sharp=1.0)
        for dtype in (torch.float32, torch.bfloat16):
            c["u"], c["beta"] = c["u"].to(dtype), c["beta"].to(dtype) if delta else None
            for cuts in ([T], [70, 70, 60], [1] * T, cases.cuts_of(T, [2, 37])):
                state, out, at = torch.zeros(1, H, dk, dv).cuda(), [], 0
                for n in cuts:
                    out.append(run_memory([(c, at, n, 0)], state, 1))
                    at += n
                assert torch.allclose(torch.cat(out)[-1], torch.arange(1.0, dv + 1) * dk ** -0.5, rtol=1e-4), (delta, cuts)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,L,col", [(24, 4, 16), (7, 2, 3), (64, 3, 32)])
def test_conv_kernel_on_columns_further_in(dtype, C, L, col):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(C * L)
    T = 60
    rows, w = torch.randn(T, col + C + 4, generator=g).to(dtype), torch.randn(C, L, generator=g)
    want = plain.silu(plain.causal_taps(rows[:, col:col + C].double(), w.double()))
    for cuts in ([T], cases.cuts_of(T, [2, 9, 1, 3]), [1] * T):
        state = torch.randn(2, L - 1, C, generator=g).to(dtype).cuda()
        out, at = [], 0
        for n in cuts:
            out.append(kernels.causal_conv(rows[at:at + n].contiguous().cuda(), C, w.cuda(), state, i32([0, n]), i32([at]),
                                           i32([1]), torch.zeros(n, dtype=torch.int32, device="cuda"), silu=True, col=col).cpu())
            at += n
        assert float((torch.cat(out).double() - want).abs().max()) < (1e-5 if dtype == torch.float32 else 0.05), cuts


# --- router and experts -------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,E,k,groups", [(5, 8, 3, (4, 2)), (40, 18, 4, (2, 1)), (70, 6, 6, (3, 3)), (300, 16, 3, (1, 1)),
                                          (33, 120, 5, (40, 3)), (200, 256, 8, (8, 3)), (7, 9, 1, (9, 1))])
def test_router_scores_groups_by_their_two_best(dtype, M, E, k, groups):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(M + E)
    x = torch.randn(M, 64, generator=g).to(dtype)
    w = (torch.randn(E, 64, generator=g) * 0.3).to(dtype)
    s = plain.sigmoid(x.double() @ w.double().T)
    ids, wts = (t.cpu() for t in kernels.moe_route_sort(x.cuda(), w.cuda(), None, k, True, 1.7, "sigmoid", groups,
                                                        group_score="top2", renorm_eps=1e-20)[:2])
    want = plain.choose(s, k, *groups)
    agree = (ids.long().sort(-1).values == want).all(-1)
    assert float(agree.float().mean()) > 0.97, float(agree.float().mean())           # the rest: near ties
    picked = torch.gather(s, 1, ids.long())
    assert float((wts.double() - picked / picked.sum(-1, keepdim=True) * 1.7).abs().max()) < 1e-5
    if 1 < groups[0] and E // groups[0] > 2 and groups[1] < groups[0]:               # a group's one best would choose others
        best = s.view(M, groups[0], -1).max(-1).values.argsort(-1, descending=True)[:, :groups[1]].sort(-1).values
        two = s.view(M, groups[0], -1).sort(-1, descending=True).values[..., :2].sum(-1).argsort(-1, descending=True)
        assert not torch.equal(best, two[:, :groups[1]].sort(-1).values)


def test_weights_of_tiny_scores_are_renormalised_to_the_scale():
    """Scores of 1e-9: what joins the sum must not swallow them."""
    from snowllm_b200.ops import kernels
    x, w = torch.ones(3, 8), torch.full((4, 8), -2.6)
    for M in (3, 100):
        wts = kernels.moe_route_sort(x.repeat(-(-M // 3), 1)[:M].contiguous().cuda(), w.cuda(), None, 2, True, 3.0, "sigmoid",
                                     group_score="top2", renorm_eps=1e-20)[1]
        assert torch.allclose(wts.cpu(), torch.full((M, 2), 1.5), rtol=1e-5)


# --- the seams ----------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,W", [(7, 44), (200, 64), (5, 37), (3, 1030), (9, 2048), (200, 2048), (2, 4096), (2, 6000), (3, 9000)])
def test_layer_norm_with_the_sums_before_it(dtype, M, W):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(M * W)

    def randn(*shape):
        return torch.randn(*shape, generator=g)
    res, a, b = randn(M, W) + 30.0, randn(M, W), randn(M, W)         # a mean far from zero: the centring must be exact
    w, w1, k = 1 + 0.3 * randn(W), 1 + 0.3 * randn(W), 3
    rows, pw = randn(M * k, W), torch.rand(M, k, generator=g)
    pos = torch.randperm(M * k, generator=g).int()
    routed = (pw.double()[..., None] * rows.double()[pos.long()].view(M, k, W)).sum(1)
    experts = kernels.ExpertSum(rows.cuda(), pos.cuda(), pw.cuda())
    A, B = a.cuda(), b.cuda()
    da, db = a.double(), b.double()
    forms = [(None, 0 * da), (A, da), (kernels.WeightedSum(A, B, 0.3, -1.7), 0.3 * da - 1.7 * db), (experts, routed),
             (kernels.DeltaSum(A, experts), da + routed), (kernels.DeltaSum(A, B), da + db),
             (kernels.ScaledDelta(A, 0.2), 0.2 * da), (kernels.ScaledDelta(experts, 0.2), 0.2 * routed),
             (kernels.NormedDelta(A, weight=w1.cuda(), eps=1e-2), plain.over_rms(da, 1e-2) * w1.double()),
             (kernels.NormedDelta(experts, weight=w1.cuda(), eps=1e-2), plain.over_rms(routed, 1e-2) * w1.double())]
    tol = 3e-5 if dtype == torch.float32 else 0.04
    for delta, add in forms:
        x = res.double() + add
        want = plain.centred_norm(x, w.double(), 1e-2) * 1.3
        r = res.clone().cuda()
        out = kernels.layer_norm(r, delta, w.cuda(), 1e-2, dtype, gain=1.3)
        assert float((out.cpu().double() - want).abs().max()) < tol
        assert float((r.cpu().double() - x).abs().max()) < 2e-5
        r = res.clone().cuda()
        out = kernels.layer_norm(r, delta, w.cuda(), 1e-2, dtype, gain=1.3, rows=i32([M - 1, 0]))
        assert float((out.cpu().double() - want[[M - 1, 0]]).abs().max()) < tol and torch.equal(r.cpu(), res)
        r = res.clone().cuda()
        out = kernels.layer_norm(r, delta, None, 0.0, dtype)         # the sum itself
        assert torch.equal(out, r.to(dtype)) and float((r.cpu().double() - x).abs().max()) < 2e-5


def test_other_norms_take_a_weighted_sum():
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(0)
    res, a, b = (torch.randn(5, 64, generator=g) for _ in range(3))
    x = res.double() + 0.3 * a.double() - 1.7 * b.double()
    for wrap in (lambda s: s, lambda s: kernels.ScaledDelta(s, 1.0), lambda s: kernels.DeltaSum(s, torch.zeros(5, 64).cuda())):
        r = res.clone().cuda()
        out = kernels.add_rmsnorm(r, wrap(kernels.WeightedSum(a.cuda(), b.cuda(), 0.3, -1.7)), torch.ones(64).cuda(), 1e-3, torch.float32)
        assert float((out.cpu().double() - plain.over_rms(x, 1e-3)).abs().max()) < 1e-5
    y = kernels.NormedDelta(kernels.WeightedSum(a.cuda(), b.cuda(), 0.3, -1.7), weight=torch.ones(64).cuda(), eps=1e-3)
    r = res.clone().cuda()
    out = kernels.add_rmsnorm(r, y, torch.ones(64).cuda(), 1e-3, torch.float32)
    x = res.double() + plain.over_rms(0.3 * a.double() - 1.7 * b.double(), 1e-3)
    assert float((out.cpu().double() - plain.over_rms(x, 1e-3)).abs().max()) < 1e-5
    with pytest.raises(kernels.KernelError):
        kernels.layer_norm(r, kernels.NormedDelta(a.cuda()), torch.ones(64).cuda(), 1e-3, torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_side_gate_reads_each_tokens_own_columns(dtype):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(1)
    z, table = torch.randn(6, 10, generator=g) * 2, torch.randn(30, 34, generator=g).to(dtype)
    ids = [3, 29, 0, 3, -1, -3]                                      # the last two: tokens the device still holds
    pending = i32([17, 5, 8])
    got = kernels.side_gate(z.cuda(), table.cuda(), i32(ids), 20, dtype, pending=pending).cpu().double()
    want = plain.gelu_tanh(z.double()) * table.double()[[3, 29, 0, 3, 17, 8]][:, 20:30]
    assert float((got - want).abs().max()) < (1e-5 if dtype == torch.float32 else 0.05)


# --- one model with everything ----------------------------------------------------------------------

@pytest.fixture(scope="module", params=["mixed", "heads_of_64"])
def mixed(request):
    cfg = cases.MIXED if request.param == "mixed" else cases.HEADS_OF_64
    tensors = cases.draw_weights(cfg, seed=3)
    return cfg, tensors


def forced_reference(cfg, tensors, tokens, model):
    """Plain logits with the experts on the picks the engine made for the whole prompt."""
    rp = replay(model, max_tokens=1024)
    rp.runner.taps = []
    cases.run_cuts(rp, "picks", tokens, [len(tokens)])
    force = dict(zip(routed_layers(cfg), [t.long().sort(-1).values for t in engine_picks(rp)]))
    return reference(cfg, tensors, tokens, picks=force)


def close_rows(got, want, dtype, tol):
    """Every row within ``tol``; in bfloat16 a row whose router met a near tie on another cut, or whose side
    input normalises a small output, may leave (few do)."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    rows = torch.sqrt((d * d).mean(-1)) / torch.sqrt((w * w).mean())
    return float((rows > tol).float().mean()) <= (0.0 if dtype == "float32" else 0.03)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_token_by_token_and_portions_agree(mixed, dtype):
    cfg, tensors = mixed
    model = load(cfg, tensors, dtype)
    tokens = cases.tokens_for(cfg, 150, seed=1)
    want = forced_reference(cfg, tensors, tokens, model)
    tol = tolerance(dtype) * 2
    rp = replay(model)
    whole = cases.run_cuts(rp, "w", tokens, [len(tokens)])
    # (in bfloat16 a row whose side input's raw output is small, and then normalised, may leave)
    assert close_rows(whole, want, dtype, tol)
    for cuts in ([1] * len(tokens), cases.cuts_of(len(tokens), [2]), cases.cuts_of(len(tokens), [3, 16, 2, 31, 1, 17]),
                 [100] + [1] * 50, [64, 64, 22]):
        got = cases.run_cuts(rp, "c", tokens, cuts)
        assert close_rows(got, want, dtype, tol), cuts
        if dtype == "float32":
            assert cases.worst_row_error(got, whole) < 2e-5, cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page_size", [8, 64])
def test_mixed_batches_over_pages_and_slots_that_are_used_again(mixed, dtype, page_size):
    """Requests of unequal lengths in waves over a pool that holds only the live ones and four slots; prompt
    portions sit beside single tokens; every request equals its run alone."""
    cfg, tensors = mixed
    model = load(cfg, tensors, dtype)
    lengths = [70, 3, 41, 1, 97, 26, 64, 2, 55]
    prompts = [cases.tokens_for(cfg, n, seed=10 + i) for i, n in enumerate(lengths)]
    alone = replay(model, page_size=page_size)
    want = [cases.run_cuts(alone, "x", p, [len(p)]) for p in prompts]
    rp = replay(model, max_tokens=4 * 128, requests=4, page_size=page_size)
    from helpers import poison_free
    portions = [7, 2, 16, 1, 33]
    state = {}                                        # request index -> tokens fed
    got = {i: [] for i in range(len(prompts))}
    waiting = list(range(len(prompts)))
    turn = 0
    while waiting or state:
        while waiting and len(state) < 4:
            state[waiting.pop(0)] = 0
        poison_free(rp)                               # whatever is free holds NaN before every step
        entries, end = [], []
        for j, (i, fed) in enumerate(sorted(state.items())):
            left = len(prompts[i]) - fed
            # the last ten tokens of a request one by one; before that portions of changing size
            n = 1 if left <= 10 else min(portions[(turn + j) % len(portions)], left - 10)
            entries.append({"id": f"r{i}", "tokens": prompts[i][fed:fed + n], "want": list(range(n))})
            state[i] = fed + n
            if state[i] == len(prompts[i]):
                end.append(f"r{i}")
        out = rp.step(entries, end).double()
        at = 0
        for e in entries:
            got[int(e["id"][1:])].append(out[at:at + len(e["tokens"])])
            at += len(e["tokens"])
        for name in end:
            del state[int(name[1:])]
        turn += 1
    for i in range(len(prompts)):
        rows = torch.cat(got[i])
        if dtype == "float32":
            assert cases.worst_row_error(rows, want[i]) < 2e-5, i
        elif len(prompts[i]) > 20:
            assert close_rows(rows, want[i], dtype, tolerance(dtype) * 2), i
    assert all(p.held() == 0 for p in rp.cache.groups.values()) and rp.cache.slots.free_count == 4


def test_long_decoding(mixed):
    cfg, tensors = mixed
    model = load(cfg, tensors, "float32")
    tokens = cases.tokens_for(cfg, 400, seed=7)
    want = forced_reference(cfg, tensors, tokens, model)
    rp = replay(model, max_tokens=448, requests=1)
    got = cases.run_cuts(rp, "d", tokens, [5] + [1] * 395, end=False)
    assert cases.worst_row_error(got, want) < F32_TOL * 2
    rp.step([], ["d"])
    assert all(pool.held() == 0 for pool in rp.cache.groups.values())


def test_greedy_generation_through_the_engine(mixed, tmp_path):
    """The framework's own entry point: a model folder, the scheduler with portions of 16 tokens, captured
    decode steps; the tokens are the plain implementation's greedy ones."""
    import snowllm_b200
    from snowllm_b200.engine import Engine, SamplingParams
    cfg, tensors = mixed
    cases.write_folder(tmp_path, cfg, tensors)
    for eager in (True, False):
        engine = Engine(snowllm_b200.load(tmp_path, "float32", "cuda"), max_num_seqs=3, max_model_len=256,
                        prefill_chunk=16, enforce_eager=eager, page_size=16)
        prompts = [cases.tokens_for(cfg, n, seed=20 + n) for n in (37, 5, 60)]
        outs = engine.generate(prompts, SamplingParams(temperature=0, max_new_tokens=24))
        for p, o in zip(prompts, outs):
            assert len(o) == 24
            logits = reference(cfg, tensors, p + o)
            for i, tok in enumerate(o):
                row = logits[len(p) - 1 + i]
                assert float(row.max() - row[tok]) < 1e-3, (eager, i)
