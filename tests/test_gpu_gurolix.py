"""Gurolix on the GPU against the plain implementation (tests/plain_gurolix.py): every mechanism alone, the kernels
on inputs that make a wrong key, a lost state, a wrong group or a missing gate show, and one model with everything
fed whole, token by token, in portions and in mixed batches over pools and slots that are used again."""
from __future__ import annotations

import pytest
import torch

import gurolix_cases as cases
import plain_gurolix as plain

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
    return [i for i, l in enumerate(cfg["layers"]) if l["mlp"] is not None]


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


# --- each mechanism alone -------------------------------------------------------------------------

ALONE = {
    "state_moe": dict(layers=[cases.state_layer()]),
    "state_no_ff_one_group_one_tap": dict(layers=[cases.state_layer(heads=4, vdim=8, state=16, groups=1, norm_groups=1, conv=1,
                                                                    mlp=None)]),
    "state_a_group_per_head": dict(layers=[cases.state_layer(heads=3, vdim=16, state=24, groups=3, norm_groups=6, conv=7)]),
    "state_tensor_core_sizes": dict(layers=[cases.state_layer(heads=4, vdim=32, state=32, groups=2, norm_groups=2, conv=4)]),
    "state_wide": dict(layers=[cases.state_layer(heads=1, vdim=136, state=200, groups=1, norm_groups=4, conv=4, mlp=None)]),
    "normed": dict(layers=[cases.normed_layer(v_mix=None)]),
    "normed_part_of_the_head_turns": dict(layers=[cases.normed_layer(heads=5, kv_heads=1, dim=20, vdim=6, rot_dims=4, v_mix=None,
                                                                     mlp=None)]),
    "normed_no_rotation": dict(layers=[cases.normed_layer(rot_dims=0)]),
    "capped": dict(layers=[cases.capped_layer()]),
    "capped_tensor_core_sizes": dict(layers=[cases.capped_layer(heads=6, kv_heads=2, dim=80, vdim=40, rot_dims=48, softcap=2.0)]),
    "capped_normed": dict(layers=[cases.normed_layer(softcap=1.0, scaling=cases.SCALING)]),
    "uncapped_unscaled": dict(layers=[cases.capped_layer(softcap=None, scaling=None)]),
    "values_mix_over_layers": dict(layers=[cases.capped_layer(), cases.normed_layer(v_mix=None, vdim=12),
                                           cases.normed_layer(kv_heads=2, vdim=8), cases.capped_layer(heads=2)]),
    "experts_no_groups_no_identity": dict(layers=[cases.state_layer(mlp=cases.moe(16, 4, 3, 0, None))]),
    "experts_all_picked": dict(layers=[cases.state_layer(mlp=cases.moe(16, 3, 4, 1, (2, 2)))]),
    "experts_mostly_identity": dict(layers=[cases.normed_layer(mlp=cases.moe(12, 1, 2, 7, (4, 1)))]),
    "heads_of_128": dict(layers=[cases.capped_layer(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09, rot_dims=128, softcap=3.0),
                                 cases.normed_layer(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.09, rot_dims=64)], width=48),
    "heads_of_64": dict(layers=cases.HEADS_OF_64["layers"], width=64),
    # sizes that are multiples of nothing: the products leave the tensor cores
    "odd_sizes": dict(layers=[cases.state_layer(heads=5, vdim=7, state=9, groups=5, norm_groups=7, conv=5,
                                                mlp=cases.moe(22, 7, 3, 2, (3, 2))),
                              cases.normed_layer(heads=3, kv_heads=1, dim=10, vdim=6, rot_dims=6, mlp=cases.moe(10, 3, 2, 0, None)),
                              cases.capped_layer(heads=34, kv_heads=2, dim=6, vdim=10, rot_dims=6, v_mix=None)], width=37, vocab=50),
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


# --- the attention kernels on keys that stand out ---------------------------------------------------

def plain_attention(q, k, v, scale, cap=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv], float64: out [T, H, dv] through a plain mask and softmax."""
    T, H = q.shape[:2]
    G = k.shape[1]
    mask = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        out.append(torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ v[:, h // (H // G)])
    return torch.stack(out, 1)


def paged(k, v, P, dtype, gen, spare=3):
    """Keys and values in pages of P in a scrambled order: (key pool, value pool, block table [1, pages])."""
    T, G = k.shape[:2]
    pages = -(-T // P)
    order = torch.randperm(pages + spare, generator=gen)[:pages].int()
    kpool = torch.zeros(pages + spare, G, P, k.shape[2], dtype=dtype, device="cuda")
    vpool = torch.zeros(pages + spare, G, P, v.shape[2], dtype=dtype, device="cuda")
    for t in range(T):
        kpool[order[t // P], :, t % P] = k[t].to(dtype)
        vpool[order[t // P], :, t % P] = v[t].to(dtype)
    return kpool, vpool, order.view(1, -1).cuda().contiguous()


FAR, OWN = 250, 3       # a far row and the early key that is made to stand out for it


def standing_out(T, H, G, dk, dv, dtype, gen, size=2.0):
    """Rows, keys and values with one far key that owns a row, and one key at each page and tile border that owns the
    row after the next."""
    q = torch.randn(T, H, dk, generator=gen).to(dtype)
    k = (torch.randn(T, G, dk, generator=gen) * 0.1).to(dtype)
    v = torch.randn(T, G, dv, generator=gen).to(dtype)
    size = max(size, 100.0 / dk)
    k[OWN, 0] = (q[FAR, 1].float() * size).to(dtype)
    for edge in (15, 16, 31, 32, 127, 128):
        k[edge, 1] = (q[edge + 2, H - 1].float() * size).to(dtype)
    return q, k, v


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("mode", ["rows", "tiles", "chunks"])
@pytest.mark.parametrize("dk,dv", [(10, 20), (80, 40), (64, 64)])
@pytest.mark.parametrize("cap", [None, 2.5, 30.0])
def test_attention_kernel_caps_its_scores(dtype, mode, dk, dv, cap):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(5)
    T, H, G, P = 300, 4, 2, 16
    q, k, v = standing_out(T, H, G, dk, dv, dtype, g)
    kpool, vpool, table = paged(k, v, P, dtype, g)
    positions = torch.arange(T, dtype=torch.int32, device="cuda")
    kw = dict(softcap=cap, tile_rows=kernels.split_attention_tile_rows(H, G, 1, dk, dv, dtype, mode != "tiles"))
    if mode == "tiles":
        n = kw["tile_rows"]
        kw["tiles"] = i32([[s, min(n, T - s)] for s in range(0, T, n)])
    if mode == "chunks":
        chunk = kernels.split_attention_decode_chunk(H, G, 1, dk, dv, dtype)
        kw.update(num_chunks=-(-T // chunk), chunk=chunk)
    got = kernels.split_attention(q.cuda(), kpool, vpool, table, P, positions, torch.zeros_like(positions), 0.25, **kw)
    want = plain_attention(q.double(), k.double(), v.double(), 0.25, cap)
    assert float((got.cpu().double() - want).abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2)
    free = plain_attention(q.double(), k.double(), v.double(), 0.25)
    if cap == 2.5:                       # the far key owns its row without the cap, and no longer with it
        assert float((free[FAR, 1] - v[OWN, 0].double()).abs().max()) < 0.05
        assert float((want[FAR, 1] - free[FAR, 1]).abs().max()) > 0.2


@pytest.mark.parametrize("P", [16, 64])
@pytest.mark.parametrize("cap", [2.5, 30.0])
@pytest.mark.parametrize("T", [700, 129])
def test_prompt_kernel_on_tensor_memory_caps_its_scores(P, cap, T):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(7)
    H, G, d, dtype = 4, 2, 64, torch.bfloat16
    q, k, v = standing_out(max(T, 300), H, G, d, d, dtype, g, 1.5)
    q, k, v = q[:T], k[:T], v[:T]
    kpool, vpool, table = paged(k, v, P, dtype, g)
    tiles = i32([[0, s, min(128, T - s), s] for s in range(0, T, 128)])
    out = torch.empty(T, H, d, dtype=dtype, device="cuda")
    kernels.attention_prefill_tc_split(q.cuda(), kpool, vpool, table, P, tiles, 0.25, out, softcap=cap)
    assert kernels.attention_tc_status() == 0
    want = plain_attention(q.double(), k.double(), v.double(), 0.25, cap)
    assert float((out.cpu().double() - want).abs().max()) < 3e-2
    free = plain_attention(q.double(), k.double(), v.double(), 0.25)
    assert float((want - free).abs().max()) > (0.3 if cap == 2.5 else 1e-4)


@pytest.mark.parametrize("P", [16, 64])
@pytest.mark.parametrize("d", [64, 128])
@pytest.mark.parametrize("cap", [2.5, 30.0])
def test_decode_kernel_by_tma_caps_its_scores(P, d, cap):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(8)
    T, H, G, dtype = 700, 4, 2, torch.bfloat16
    q, k, v = standing_out(T, H, G, d, d, dtype, g, 96.0 / d)
    kpool, vpool, table = paged(k, v, P, dtype, g)
    positions = torch.arange(T, dtype=torch.int32, device="cuda")
    out = torch.empty(T, H, d, dtype=dtype, device="cuda")
    kernels.attention_decode_tma_split(q.cuda(), kpool, vpool, table, P, positions, torch.zeros_like(positions), 0.25,
                                       -(-T // 256), out, softcap=cap)
    assert kernels.attention_decode_status() == 0
    want = plain_attention(q.double(), k.double(), v.double(), 0.25, cap)
    assert float((out.cpu().double() - want).abs().max()) < 3e-2


# (dk, dv): sizes the scalar kernel takes, and rows of 16-byte vectors (the vector kernel)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,rot", [(5, 2, 10, 6, 6), (6, 3, 64, 96, 64), (6, 2, 16, 8, 16)])
@pytest.mark.parametrize("normed", [True, False])
def test_prepare_adds_biases_turns_and_mixes_values(dtype, H, G, dk, dv, rot, normed):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(9)
    M, P, lam = 9, 4, 0.3
    width = H * dk + G * dk + G * dv
    width += -width % 16
    k_off, v_off = H * dk, H * dk + G * dk
    proj = torch.randn(M, width, generator=g).to(dtype)
    bias = torch.randn(width, generator=g)
    lead = 16
    other = torch.randn(M, lead + G * dv + (-(lead + G * dv) % 16), generator=g).to(dtype)
    other_bias = torch.randn(other.shape[1], generator=g)
    wq, wk = (1 + 0.3 * torch.randn(dk, generator=g)).to(dtype), (1 + 0.3 * torch.randn(dk, generator=g)).to(dtype)
    freqs = plain.frequencies(50.0, rot, cases.SCALING)
    positions = torch.arange(3, 3 + M)
    table = i32([[3, 1, 0]])
    kpool = torch.zeros(4, G, P, dk, dtype=dtype, device="cuda")
    vpool = torch.zeros(4, G, P, dv, dtype=dtype, device="cuda")
    q = kernels.split_prepare(proj.cuda(), 0, k_off, v_off, wq.cuda() if normed else None, wk.cuda() if normed else None, 1e-3,
                              torch.tensor(freqs, dtype=torch.float32, device="cuda"), rot, 1.0, positions.int().cuda(),
                              torch.zeros(M, dtype=torch.int32, device="cuda"), table, P, kpool, vpool, H, G, 1, dk, dv,
                              proj_bias=bias.cuda(), value_mix=(other.cuda(), lead, other_bias.cuda(), lam))
    full = proj.double() + bias.double()
    qk = [full[:, :k_off].view(M, H, dk), full[:, k_off:v_off].view(M, G, dk)]
    if normed:
        qk = [plain.over_rms(x, 1e-3) * w.double() for x, w in zip(qk, (wq, wk))]
    want_q, want_k = (plain.rotate_halves(x, positions, freqs) for x in qk)
    first = (other.double() + other_bias.double())[:, lead:lead + G * dv].view(M, G, dv)
    want_v = (1 - lam) * full[:, v_off:v_off + G * dv].view(M, G, dv) + lam * first
    tol = 2e-5 if dtype == torch.float32 else 0.05
    assert float((q.cpu().double() - want_q).abs().max()) < tol
    for m in range(M):
        page, at = int(table[0, (3 + m) // P]), (3 + m) % P
        assert float((kpool[page, :, at].cpu().double() - want_k[m]).abs().max()) < tol
        assert float((vpool[page, :, at].cpu().double() - want_v[m]).abs().max()) < tol


# --- the state-space recurrence -----------------------------------------------------------------------

def draw_recurrence(T, H, P, N, G, dtype, g):
    """(rows [T, x | B | C | dt], step bias, rate, skip): decays from nearly none to a few tokens."""
    rows = torch.randn(T, H * P + 2 * G * N + H + 3, generator=g).to(dtype)
    return rows, torch.rand(H, generator=g) * 3 - 3, -torch.exp(torch.rand(H, generator=g) * 5 - 4), torch.randn(H, generator=g)


def plain_recurrence(rows, bias, rate, skip, H, P, N, G):
    T = rows.shape[0]
    x, B, C, dt = torch.split(rows.double()[:, :H * P + 2 * G * N + H], [H * P, G * N, G * N, H], -1)
    B, C = (a.view(T, G, N).repeat_interleave(H // G, 1) for a in (B, C))
    step = plain.softplus(dt + bias.double())
    return plain.state_space(x.view(T, H, P), B, C, step, torch.exp(rate.double() * step), skip.double()).view(T, H * P)


def run_recurrence(parts, bias, rate, skip, state, H, P, N, G):
    """One step: parts [(rows, start, slot)]."""
    from snowllm_b200.ops import kernels
    flat = torch.cat([r for r, _, _ in parts]).cuda()
    lens = [len(r) for r, _, _ in parts]
    cu = i32([sum(lens[:i]) for i in range(len(lens) + 1)])
    b_off = H * P
    return kernels.state_space(flat, 0, b_off, b_off + G * N, flat, b_off + 2 * G * N, bias.cuda(), rate.cuda(), skip.cuda(), cu,
                               i32([s for _, s, _ in parts]), i32([s for _, _, s in parts]), state, G, max(lens)).cpu()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,P,N,G", [(4, 10, 12, 2), (2, 64, 64, 1), (3, 24, 40, 3), (2, 64, 128, 2), (1, 132, 200, 1), (2, 5, 7, 1),
                                     (2, 128, 16, 1), (4, 16, 16, 2), (2, 40, 48, 2), (2, 128, 256, 1)])
def test_state_space_kernel_carries_its_state_and_starts_fresh_in_a_used_slot(dtype, H, P, N, G):
    """Fed whole, in portions down to two tokens, and token by token; the slot holds another request's state."""
    g = torch.Generator().manual_seed(P * N)
    T = 333
    rows, *small = draw_recurrence(T, H, P, N, G, dtype, g)
    want = plain_recurrence(rows, *small, H, P, N, G)
    scale = float(want.abs().max())
    for cuts in ([T], cases.cuts_of(T, [2, 70, 1, 129, 64, 3]), [T - 20] + [1] * 20, [63, 64, 65, 141], [1] * T):
        state = torch.randn(3, H, N, P, generator=g).cuda() * 5
        before = state.clone()
        out, at = [], 0
        for n in cuts:
            out.append(run_recurrence([(rows[at:at + n], at, 1)], *small, state, H, P, N, G))
            at += n
        assert float((torch.cat(out).double() - want).abs().max()) < 3e-6 * scale, cuts[:6]
        assert torch.equal(state[0], before[0]) and torch.equal(state[2], before[2])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_state_space_kernel_serves_unequal_segments_side_by_side(dtype):
    g = torch.Generator().manual_seed(3)
    H, P, N, G = 4, 64, 64, 2
    lens, starts, slots = [90, 300, 1, 2, 1, 200], [14, 0, 45, 1, 0, 130], [2, 0, 3, 1, 5, 4]
    _, *small = draw_recurrence(1, H, P, N, G, dtype, g)
    seqs = [draw_recurrence(s + n, H, P, N, G, dtype, g)[0] for s, n in zip(starts, lens)]
    want = [plain_recurrence(r, *small, H, P, N, G) for r in seqs]
    state = torch.randn(7, H, N, P, generator=g).cuda()
    for r, s, slot in zip(seqs, starts, slots):
        if s:
            run_recurrence([(r[:s], 0, slot)], *small, state, H, P, N, G)
    got = run_recurrence([(r[s:], s, slot) for r, s, slot in zip(seqs, starts, slots)], *small, state, H, P, N, G)
    at = 0
    for w, s, n in zip(want, starts, lens):
        assert float((got[at:at + n].double() - w[s:]).abs().max()) < 3e-6 * float(w.abs().max())
        at += n
    # and one more token each from the state they left (the same token for all)
    more = draw_recurrence(1, H, P, N, G, dtype, g)[0]
    got = run_recurrence([(more, s + n, slot) for s, n, slot in zip(starts, lens, slots)], *small, state, H, P, N, G)
    for i, r in enumerate(seqs):
        w = plain_recurrence(torch.cat((r, more)), *small, H, P, N, G)
        assert float((got[i].double() - w[-1]).abs().max()) < 3e-6 * float(w.abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_state_space_kernel_keeps_what_barely_decays(dtype):
    """A head that forgets nothing (rate -1e-6) beside one that forgets at once: a token far back is read."""
    g = torch.Generator().manual_seed(4)
    H, P, N, G, T = 2, 64, 64, 1, 600
    rows = torch.zeros(T, H * P + 2 * N + H).to(dtype)
    rows[5, :H * P] = torch.randn(H * P, generator=g).to(dtype)
    rows[5, H * P:H * P + N] = 1.0                                  # B of the one token that writes
    rows[-1, H * P + N:H * P + 2 * N] = 1.0                         # C of the last one
    bias, rate = torch.tensor([0.5, 0.5]), torch.tensor([-1e-6, -20.0])
    small = (bias, rate, torch.zeros(2))
    for cuts in ([T], [200] * 3, cases.cuts_of(T, [2, 131])):
        state, out, at = torch.zeros(1, H, N, P, device="cuda"), [], 0
        for n in cuts:
            out.append(run_recurrence([(rows[at:at + n], at, 0)], *small, state, H, P, N, G))
            at += n
        last = torch.cat(out)[-1].double().view(H, P)
        step = float(plain.softplus(torch.tensor(0.5, dtype=torch.float64)))
        assert torch.allclose(last[0], N * step * rows[5, :P].double(), rtol=1e-3) and float(last[1].abs().max()) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,parts,col", [(60, 3, 5), (512, 2, 8), (512, 1, 0), (35, 7, 1), (2048, 8, 4), (4100, 1, 4)])
def test_gate_before_the_norm_in_parts(dtype, n, parts, col):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(n)
    M = 9
    y, z = torch.randn(M, n, generator=g) * 2, torch.randn(M, col + n + 3, generator=g).to(dtype)
    y[:, :n // parts] *= 50                                          # one part far larger than the others
    w = (1 + 0.3 * torch.randn(n, generator=g)).to(dtype)
    got = kernels.gate_group_norm(y.cuda(), z.cuda(), col, w.cuda(), parts, 1e-3).cpu().double()
    v = y.double() * plain.silu(z[:, col:col + n].double())
    want = plain.over_rms(v.view(M, parts, -1), 1e-3).view(M, n) * w.double()
    assert float((got - want).abs().max()) < (2e-5 if dtype == torch.float32 else 0.05)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,L", [(24, 4), (7, 2), (64, 3), (16, 1), (40, 6)])
def test_conv_kernel_adds_its_bias_and_activation(dtype, C, L):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(C * L)
    T = 60
    rows, w, b = torch.randn(T, C + 4, generator=g).to(dtype), torch.randn(C, L, generator=g), torch.randn(C, generator=g)
    want = plain.silu(plain.causal_taps(rows[:, :C].double(), w.double(), b.double()))
    for cuts in ([T], cases.cuts_of(T, [2, 9, 1, 3]), [1] * T, [40] + [1] * 20):
        state = torch.randn(2, max(L - 1, 0), C, generator=g).to(dtype).cuda()
        out, at = [], 0
        for n in cuts:
            out.append(kernels.causal_conv(rows[at:at + n].contiguous().cuda(), C, w.cuda(), state, i32([0, n]), i32([at]),
                                           i32([1]), torch.zeros(n, dtype=torch.int32, device="cuda"), bias=b.cuda(),
                                           silu=True).cpu())
            at += n
        assert float((torch.cat(out).double() - want).abs().max()) < (1e-5 if dtype == torch.float32 else 0.05), cuts


# --- router and experts -------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,E,k,groups", [(5, 8, 3, (4, 2)), (40, 18, 4, (2, 1)), (70, 6, 6, (3, 3)), (300, 16, 3, (1, 1)),
                                          (33, 120, 5, (40, 3)), (200, 128, 8, (8, 3)), (7, 9, 1, (9, 1))])
def test_router_chooses_within_groups_by_corrected_scores(dtype, M, E, k, groups):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(M + E)
    H, same = 64, 2
    x = torch.randn(M, H, generator=g).to(dtype)
    w = (torch.randn(E, H, generator=g) * 0.4).to(dtype)
    b = torch.randn(E, generator=g) * 0.3 - 2.0                      # every choice score is negative
    s = torch.softmax(x.double() @ w.double().T, -1)
    choice = s + b.double()
    ids, wts, offsets, pair_pos, sorted_pair = (t.cpu() for t in kernels.moe_route_sort(
        x.cuda(), w.cuda(), b.float().cuda(), k, False, 1.0, "softmax", groups, same))
    want = plain.choose(choice, k, *groups)
    agree = (ids.long().sort(-1).values == want).all(-1)
    assert float(agree.float().mean()) > 0.97, float(agree.float().mean())           # the rest: near ties
    assert float((wts.double() - torch.gather(s, 1, ids.long())).abs().max()) < 1e-5     # the uncorrected scores
    if groups[1] < min(k, groups[0]):    # without the groups the choice is another
        assert not torch.equal(plain.choose(choice, k, 1, 1), want)
    assert torch.all(choice < 0)
    flat = ids.view(-1).long()
    counts = torch.bincount(flat, minlength=E)
    assert torch.equal(offsets.long(), torch.cat((torch.zeros(1, dtype=torch.long), counts.cumsum(0))))
    assert torch.equal(flat[sorted_pair.long()], flat.sort().values)
    for p in range(M * k):
        assert int(pair_pos[p]) == -1 if flat[p] >= E - same else int(sorted_pair[pair_pos[p]]) == p


def test_combine_takes_the_input_for_pairs_without_a_row():
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(2)
    M, k, H = 6, 3, 20
    y, x, w = torch.randn(M * k, H, generator=g), torch.randn(M, H, generator=g), torch.rand(M, k, generator=g)
    y[10:] = float("nan")                                            # rows no product wrote
    pos = torch.randperm(10, generator=g).repeat(2)[:M * k].view(M, k).int()
    pos[:, 1] = -1
    got = kernels.ExpertSum(y.cuda(), pos.view(-1).cuda().contiguous(), w.cuda(), x=x.cuda()).dense().cpu()
    rows = torch.where((pos >= 0)[..., None], y[pos.clamp(min=0).long()], x[:, None, :])
    assert torch.allclose(got, (w[..., None] * rows).sum(1), atol=1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M", [3, 40, 300])
@pytest.mark.parametrize("ff", [24, 22])
def test_experts_against_the_plain_ones(dtype, M, ff):
    cfg = cases.config([cases.state_layer(mlp=cases.moe(ff, 9, 3, 3, (4, 2)))], width=48)
    tensors = cases.draw_weights(cfg, 5)
    ffn = load(cfg, tensors, dtype).blocks[0].ffn
    x = torch.randn(M, 48, generator=torch.Generator().manual_seed(M)).to(ffn.dtype)
    delta = ffn.forward(None, x.cuda())
    ids = ffn.route(x.cuda())[0].cpu().long().sort(-1).values
    t = {k[len("l0.mlp."):]: v.double() for k, v in tensors.items() if k.startswith("l0.mlp.")}
    want, _ = plain.experts(x.double(), t, cfg["layers"][0]["mlp"], "", picks=ids)
    assert cases.relative_error(delta.dense().cpu(), want) < (1e-5 if dtype == "float32" else 0.01)
    assert (ids >= 9).any() and (ids < 9).any()


# --- norms on both sides, gates, the depth average ----------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,W", [(7, 44), (200, 64), (5, 37), (3, 1030), (9, 2048), (2, 4096), (2, 6000), (3, 9000)])
@pytest.mark.parametrize("pieces", [False, True])
def test_seam_applies_gate_norm_average_and_the_next_norm(dtype, M, W, pieces):
    from snowllm_b200.ops import kernels
    g = torch.Generator().manual_seed(M * W)
    layers, at, col = 5, 3, 8

    def randn(*shape):
        return torch.randn(*shape, generator=g)
    res, y, hist = randn(M, W), randn(M, W), randn(layers, M, W)
    logits, bias = randn(M, col + W + (-W) % 4).to(dtype), randn(W)
    w1, w2, avg = 1 + 0.3 * randn(W), 1 + 0.3 * randn(W), randn(at + 1)
    delta_y = y.cuda()
    if pieces:
        k, rows = 3, randn(3 * M, W)
        x, pw = randn(M, W).to(dtype), torch.rand(M, k, generator=g)
        pos = torch.randint(0, 3 * M, (M, k), generator=g).int()
        pos[:, 1] = -1
        pos[0] = -1
        y = (pw.double()[..., None] * torch.where((pos >= 0)[..., None], rows.double()[pos.clamp(min=0).long()],
                                                  x.double()[:, None])).sum(1)
        delta_y = kernels.ExpertSum(rows.cuda(), pos.view(-1).cuda().contiguous(), pw.cuda(), x=x.cuda())
    tol = 2e-5 if dtype == torch.float32 else 0.04

    def check(want_x, want_out, r, out, rows=None):
        pick = slice(None) if rows is None else rows.cpu().long()
        assert float((out.cpu().double() - want_out[pick]).abs().max()) < tol
        if rows is None:
            assert float((r.cpu().double() - want_x).abs().max()) < 2e-5
        else:
            assert torch.equal(r.cpu(), res)

    gated = y.double() * torch.sigmoid(logits.double()[:, col:col + W] + bias.double())
    mid = res.double() + plain.over_rms(gated, 1e-3) * w1.double()
    gate = (logits.cuda(), col, bias.cuda())
    # in the middle of a layer
    r = res.clone().cuda()
    out = kernels.add_rmsnorm(r, kernels.NormedDelta(delta_y, gate=gate, weight=w1.cuda(), eps=1e-3), w2.cuda(), 1e-2, dtype)
    check(mid, plain.over_rms(mid, 1e-2) * w2.double(), r, out)
    # at its end: recorded, averaged
    mixed = avg.double()[at] * mid + (avg.double()[:at, None, None] * hist.double()[:at]).sum(0)
    want = plain.over_rms(mixed, 1e-2) * w2.double()
    for rows in (None, i32([M - 1, 0])):
        r, h = res.clone().cuda(), hist.clone().cuda()
        delta = kernels.NormedDelta(delta_y, gate=gate, weight=w1.cuda(), eps=1e-3, history=h, index=at, average=avg.cuda())
        assert float((delta.total(r).cpu().double() - mixed).abs().max()) < 1e-4
        out = kernels.add_rmsnorm(r, delta, w2.cuda(), 1e-2, dtype, rows=rows)
        check(mixed, want, r, out, rows)
        kept = hist.clone().double()
        if rows is None:
            kept[at] = mid
        assert float((h.cpu().double() - kept).abs().max()) < 2e-5
    # the first seam: nothing pending, the embedding output is recorded
    r, h = res.clone().cuda(), hist.clone().cuda()
    out = kernels.add_rmsnorm(r, kernels.NormedDelta(None, history=h, index=0), w2.cuda(), 1e-2, dtype)
    check(res.double(), plain.over_rms(res.double(), 1e-2) * w2.double(), r, out)
    assert torch.equal(h[0].cpu(), res) and torch.equal(h[1:].cpu(), hist[1:])


def test_embedding_rows_are_normed_in_float():
    cfg = cases.config([cases.state_layer(mlp=None)])
    tensors = cases.draw_weights(cfg, 6)
    emb = load(cfg, tensors, "bfloat16").embedding

    class Ctx:
        token_ids, pending_tokens = i32([3, 0, 89, 3]), None
    got = emb.forward(Ctx())
    t = {k: v.double() for k, v in tensors.items()}
    want = plain.one_plus_norm(t["embed"][[3, 0, 89, 3]], t["embed.norm"], 1e-5)
    assert got.dtype == torch.float32 and float((got.cpu().double() - want).abs().max()) < 1e-5


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
    """Every row within ``tol``; in bfloat16 a row whose router met a near tie on another cut may leave (few do)."""
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
    assert cases.worst_row_error(whole, want) < tol
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
