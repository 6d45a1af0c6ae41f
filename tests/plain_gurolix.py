"""A plain, slow implementation of the Gurolix design on the CPU: one function per mechanism, written from the
design's equations, whole sequences at a time, no cache.  It shares nothing with the engine: the softmax is a
plain one over an explicit mask, the state-space recurrence a loop over tokens, the experts are looped over.

Notation: W x means ``x @ W.T`` for a weight stored [out, in]; a sequence is [T, width] from position 0.
Everything runs in ``dtype`` (float64 by default).  A model is a dict: ``config`` (the parsed config.json) and
``tensors`` (name -> tensor)."""
from __future__ import annotations

import math

import torch


def over_rms(x, eps):
    """x over the root of its mean square along the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_plus_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return over_rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# --- positions ------------------------------------------------------------------------------------

def frequencies(base: float, dims: int, scaling=None) -> list:
    """f_i = base^(-2i/dims); with ``scaling`` (factor, low, high, original) a frequency whose wavelength is
    shorter than original/high stays, one longer than original/low is divided by the factor, and between the two
    the result goes over linearly in original/wavelength."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            factor, low, high, original = (scaling[k] for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave < original / high:
                pass
            elif wave > original / low:
                f = f / factor
            else:
                s = (original / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_halves(x, positions, freqs):
    """x [T, heads, d]: element i < n turns with element i + n by positions * freqs[i], n = len(freqs);
    elements from 2n on pass."""
    out = x.clone()
    n = len(freqs)
    for i, f in enumerate(freqs):
        a = positions.to(x.dtype) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + n]
        out[..., i] = u * c - v * s
        out[..., i + n] = v * c + u * s
    return out


# --- attention ------------------------------------------------------------------------------------

def attention(h, t, m: dict, eps: float, p: str, positions, v_first=None, normed: bool = True):
    """Causal grouped-query attention: biased projections; with ``normed`` q and k RMS-normed per head (one
    plain weight of ``dim`` for all heads) before the rotation; scores capped when the mixer has ``softcap``;
    v goes over to (1 - vmix) v + vmix v_first where ``v_first`` is given.  Returns (output, v before mixing)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ t[p + "q"].T + t[p + "q.b"]).view(T, H, d)
    k = (h @ t[p + "k"].T + t[p + "k.b"]).view(T, G, d)
    own = (h @ t[p + "v"].T + t[p + "v.b"]).view(T, G, dv)
    if normed:
        q, k = over_rms(q, eps) * t[p + "q.norm"], over_rms(k, eps) * t[p + "k.norm"]
    rot = m.get("rot")
    freqs = [] if rot is None else frequencies(rot["base"], rot["dims"], rot.get("scaling"))
    q, k = rotate_halves(q, positions, freqs), rotate_halves(k, positions, freqs)
    v = own
    if v_first is not None:
        lam = t[p + "vmix"]
        v = (1.0 - lam) * own + lam * v_first
    mask = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for head in range(H):
        g = head // (H // G)
        s = q[:, head] @ k[:, g].T * m["scale"]
        if m.get("softcap") is not None:
            s = m["softcap"] * torch.tanh(s / m["softcap"])
        s = s.masked_fill(~mask, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append(e / e.sum(-1, keepdim=True) @ v[:, g])
    return torch.cat(out, -1) @ t[p + "o"].T, own


# --- the state-space mixer ------------------------------------------------------------------------

def causal_taps(u, w, b):
    """Depthwise causal convolution over time with a bias: u [T, C], w [C, taps];
    y[t] = b + sum_j w[:, j] * u[t - taps + 1 + j], zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat((torch.zeros(taps - 1, C, dtype=u.dtype), u), 0)
    y = b.expand(T, C).clone()
    for j in range(taps):
        y = y + w[:, j] * padded[j:j + T]
    return y


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def state_space(x, B, C, step, decay, skip):
    """x [T, H, P], B and C [T, H, N] (each head's own copy), step and decay [T, H], skip [H]:
    S_t = decay_t S_(t-1) + step_t B_t x_t^T, y_t = S_t^T C_t + skip x_t; S starts at zero."""
    T, H, P = x.shape
    S = torch.zeros(H, B.shape[-1], P, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        S = decay[t][:, None, None] * S + step[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t][:, :, None]).sum(1) + skip[:, None] * x[t]
    return y


def mamba2(h, t, m: dict, eps: float, p: str):
    """Projection [z | x | B | C | dt]; x, B, C through a short convolution and silu; the recurrence; the gate
    silu(z) BEFORE an RMS norm in ``norm_groups`` equal parts; output product."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m.get("groups", 1)
    inner = H * P
    z, x, B, C, dt = torch.split(h @ t[p + "in"].T, [inner, inner, G * N, G * N, H], -1)
    u = silu(causal_taps(torch.cat((x, B, C), -1), t[p + "conv"], t[p + "conv.b"]))
    x, B, C = torch.split(u, [inner, G * N, G * N], -1)
    B, C = (a.view(T, G, N).repeat_interleave(H // G, 1) for a in (B, C))
    step = softplus(dt + t[p + "dt_bias"])
    decay = torch.exp(-torch.exp(t[p + "A_log"]) * step)
    y = state_space(x.view(T, H, P), B, C, step, decay, t[p + "D"]).reshape(T, inner)
    y = y * silu(z)
    parts = m.get("norm_groups", 1)
    y = over_rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * t[p + "norm"]
    return y @ t[p + "o"].T


# --- routed experts -------------------------------------------------------------------------------

def choose(choice, top: int, count: int, keep: int):
    """The ``top`` largest choice scores [T, E] among the experts of the ``keep`` best of ``count`` equal groups
    of neighbours (a group's score is its largest choice score); ties to the lower index."""
    T, E = choice.shape
    best = choice.view(T, count, E // count).max(-1).values
    groups = torch.argsort(-best, dim=-1, stable=True)[:, :keep]
    allowed = torch.zeros(T, count, dtype=torch.bool).scatter_(1, groups, True)
    allowed = allowed.repeat_interleave(E // count, 1)
    masked = choice.masked_fill(~allowed, -math.inf)
    return torch.sort(torch.argsort(-masked, dim=-1, stable=True)[:, :top], -1).values


def experts(h, t, mlp: dict, p: str, picks=None, router_input=None):
    """Scores s: the softmax over all router outputs.  s + correction chooses, s weighs (not renormalised).  An
    expert is down(relu(up h)^2); the last ``identity`` router outputs stand for the input itself.
    ``picks`` [T, top] forces the choice.  Returns (output, the choice)."""
    r = mlp["router"]
    E, same, g = r["experts"], r.get("identity") or 0, r.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax((h if router_input is None else router_input) @ t[p + "router"].T, -1)
    if picks is None:
        picks = choose(s + t[p + "correction"], r["top"], g["count"], g["keep"])
    out = torch.zeros_like(h)
    for e in range(E + same):
        hit = (picks == e).any(-1)
        if not bool(hit.any()):
            continue
        rows = h[hit]
        if e < E:
            y = torch.clamp(rows @ t[p + f"e{e}.up"].T, min=0.0) ** 2 @ t[p + f"e{e}.down"].T
        else:
            y = rows
        out[hit] = out[hit] + s[hit, e:e + 1] * y
    return out, picks


# --- the model ------------------------------------------------------------------------------------

def forward(model: dict, tokens, dtype=torch.float64, layers_out=None, picks=None, picks_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` (a list) receives the stream as each layer hands
    it on; ``picks`` {layer: [T, top]} forces the experts, ``picks_out`` (a dict) receives {layer: the choice made}."""
    cfg = model["config"]
    t = {k: v.to(dtype) for k, v in model["tensors"].items()}
    eps = cfg["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x = one_plus_norm(t["embed"][torch.tensor(tokens)], t["embed.norm"], eps)
    history = [x]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{i}."
        m = layer["mixer"]
        h = one_plus_norm(x, t[n + "norm1"], eps)
        if layer["type"] == "mamba2":
            y = mamba2(h, t, m, eps, n + "mix.")
        else:
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, t, m, eps, n + "mix.", positions, v_first if mixes else None,
                               normed=layer["type"] == "attention")
            if mixes and v_first is None:
                v_first = own
        y = y * sigmoid(h @ t[n + "rg1"].T + t[n + "rg1.b"])
        x = x + one_plus_norm(y, t[n + "norm1b"], eps)
        if layer.get("mlp") is not None:
            h = one_plus_norm(x, t[n + "norm2"], eps)
            y, chosen = experts(h, t, layer["mlp"], n + "mlp.", picks=None if picks is None else picks.get(i))
            if picks_out is not None:
                picks_out[i] = chosen
            y = y * sigmoid(h @ t[n + "rg2"].T + t[n + "rg2.b"])
            x = x + one_plus_norm(y, t[n + "norm2b"], eps)
        history.append(x)
        x = sum(t[n + "dwa"][j] * history[j] for j in range(i + 2))
        if layers_out is not None:
            layers_out.append(x)
    return one_plus_norm(x, t["final.norm"], eps) @ t["head"].T
