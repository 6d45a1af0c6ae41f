"""A plain, slow implementation of the Levovik design on the CPU: one function per mechanism, written from the
design's equations, whole sequences at a time, no cache.  It shares nothing with the engine: the softmax is a plain
one over an explicit mask, both recurrences are loops over tokens, the experts are looped over.

Notation: W x means ``x @ W.T`` for a weight stored [out, in]; a sequence is [T, width] from position 0.
Everything runs in ``dtype`` (float64 by default).  A model is a dict: ``config`` (the parsed config.json) and
``tensors`` (name -> tensor)."""
from __future__ import annotations

import math

import torch


def centred_norm(x, w, eps):
    """Layer norm with a weight and no bias."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def over_rms(x, eps):
    """x over the root of its mean square along the last axis (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def over_length(x):
    """x as a unit vector along the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


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


def rotate(x, positions, freqs, interleaved: bool):
    """x [T, heads, d]: pair i = elements (2i, 2i + 1) if ``interleaved``, else (i, i + n) with n = len(freqs), turns by
    positions * freqs[i]; elements from 2n on pass."""
    out = x.clone()
    n = len(freqs)
    for i, f in enumerate(freqs):
        a = positions.to(x.dtype) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        j, l = (2 * i, 2 * i + 1) if interleaved else (i, i + n)
        u, v = x[..., j], x[..., l]
        out[..., j] = u * c - v * s
        out[..., l] = v * c + u * s
    return out


# --- softmax attention ----------------------------------------------------------------------------

def attend(q, k, v, scale: float, sink=None):
    """Causal attention: q [T, H, d], k [T, G, d], v [T, G, dv]; head h reads group h // (H / G).  ``sink`` [H]: one
    more term exp(sink) in the sum under the weights, without a key, a value or the scale."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    mask = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T * scale).masked_fill(~mask, -math.inf)
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[h].expand_as(top))
        e = torch.exp(s - top)
        total = e.sum(-1, keepdim=True)
        if sink is not None:
            total = total + torch.exp(sink[h] - top)
        out.append(e / total @ v[:, h // per])
    return torch.stack(out, 1)


def sink_side(h, t, m: dict, eps: float, p: str, positions):
    """Keys and values of their own, halves rotated, q and k over their root mean square after it, a sink per head."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (h @ t[p + "q"].T).view(T, H, d), (h @ t[p + "k"].T).view(T, G, d)
    v = (h @ t[p + "v"].T).view(T, G, dv)
    rot = m.get("rot")
    freqs = [] if rot is None else frequencies(rot["base"], rot["dims"], rot.get("scaling"))
    q, k = (over_rms(rotate(a, positions, freqs, False), eps) for a in (q, k))
    return attend(q, k, v, m["scale"], t[p + "sink"]).reshape(T, -1) @ t[p + "o"].T


def shared_side(h, t, m: dict, eps: float, p: str, positions):
    """The projected keys are the values; q and k weighted norms per head, then neighbours rotated."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q, raw = (h @ t[p + "q"].T).view(T, H, d), (h @ t[p + "k"].T).view(T, G, d)
    rot = m.get("rot")
    freqs = [] if rot is None else frequencies(rot["base"], rot["dims"], rot.get("scaling"))
    q = rotate(over_rms(q, eps) * t[p + "q.norm"], positions, freqs, True)
    k = rotate(over_rms(raw, eps) * t[p + "k.norm"], positions, freqs, True)
    return attend(q, k, raw, m["scale"]).reshape(T, -1) @ t[p + "o"].T


# --- recurrences ----------------------------------------------------------------------------------

def causal_taps(u, w):
    """Depthwise causal convolution over time: u [T, C], w [C, taps]; y[t] = sum_j w[:, j] * u[t - taps + 1 + j]."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat((torch.zeros(taps - 1, C, dtype=u.dtype), u), 0)
    return sum(w[:, j] * padded[j:j + T] for j in range(taps))


def delta_rule(q, k, v, decay, beta):
    """q, k, decay [T, H, d], v [T, H, dv], beta [T, H]: S is decayed by rows, then what it already answers to k is
    taken off v before it is written; o_t reads S after the write.  S starts at zero."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = decay[t][:, :, None] * S
        known = (S * k[t][:, :, None]).sum(1)
        u = beta[t][:, None] * (v[t] - known)
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def linear_memory(q, k, v, decay):
    """The same without the correction: S_t = diag(decay_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def delta_side(h, t, m: dict, eps: float, p: str):
    """Gated delta rule: convolved projections, unit q and k, a write strength per head, a decay per key channel."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_taps(h @ t[p + n].T, t[p + n + ".conv"])) for n in "qkv")
    q, k = (over_length(a.view(T, G, d)).repeat_interleave(H // G, 1) for a in (q, k))
    z = (h @ t[p + "a1"].T) @ t[p + "a2"].T + t[p + "dt_bias"]
    rate = torch.exp(t[p + "A_log"])[None, :, None]
    decay = torch.exp(-rate * softplus(z).view(T, H, d))
    o = delta_rule(q * d ** -0.5, k, v.view(T, H, dv), decay, sigmoid(h @ t[p + "b"].T))
    gate = sigmoid((h @ t[p + "g1"].T) @ t[p + "g2"].T)
    return ((over_rms(o, eps) * t[p + "norm"]).reshape(T, -1) * gate) @ t[p + "o"].T


def gla_side(h, t, m: dict, eps: float, p: str):
    """Gated linear attention: a decay per key channel, sigmoid(z)^(1/tau)."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k = (h @ t[p + "q"].T).view(T, H, d) * d ** -0.5, (h @ t[p + "k"].T).view(T, H, d)
    z = (h @ t[p + "a1"].T) @ t[p + "a2"].T + t[p + "a2.b"]
    decay = torch.exp(-softplus(-z) / m["tau"]).view(T, H, d)
    o = linear_memory(q, k, (h @ t[p + "v"].T).view(T, H, dv), decay)
    return ((over_rms(o, eps) * t[p + "norm"]).reshape(T, -1) * silu(h @ t[p + "g"].T)) @ t[p + "o"].T


def mixer(h, t, layer: dict, eps: float, p: str, positions):
    m = layer["mixer"]
    if layer["type"] == "parallel":
        left = sink_side(h, t, m["left"], eps, p + "left.", positions)
        right = delta_side(h, t, m["right"], eps, p + "right.")
    else:
        left = shared_side(h, t, m["left"], eps, p + "left.", positions)
        right = gla_side(h, t, m["right"], eps, p + "right.")
    return m["left_scale"] * left + m["right_scale"] * right


# --- feed-forwards --------------------------------------------------------------------------------

def dense(h, t, p: str):
    return (torch.clamp(h @ t[p + "gate"].T, min=0.0) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def clamped_expert(h, t, p: str, limit: float):
    g = torch.clamp(h @ t[p + "gate"].T, max=limit)
    u = torch.clamp(h @ t[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ t[p + "down"].T


def choose(s, top: int, count: int, keep: int):
    """The ``top`` largest scores [T, E] among the experts of the ``keep`` best of ``count`` equal groups of neighbours;
    a group's score is the sum of its two largest scores; ties to the lower index."""
    T, E = s.shape
    size = E // count
    best = torch.sort(s.view(T, count, size), dim=-1, descending=True).values[..., :2].sum(-1)
    groups = torch.argsort(-best, dim=-1, stable=True)[:, :keep]
    allowed = torch.zeros(T, count, dtype=torch.bool).scatter_(1, groups, True).repeat_interleave(size, 1)
    masked = s.masked_fill(~allowed, -math.inf)
    return torch.sort(torch.argsort(-masked, dim=-1, stable=True)[:, :top], -1).values


def experts(h, t, mlp: dict, p: str, picks=None):
    """``picks`` [T, top] forces the choice.  Returns (output, the choice)."""
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    s = sigmoid(h @ t[p + "router"].T)
    if picks is None:
        picks = choose(s, r["top"], g["count"], g["keep"])
    w = torch.gather(s, 1, picks)
    w = w / (w.sum(-1, keepdim=True) + 1e-20) * r["scale"]
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        for j in range(picks.shape[1]):
            hit = picks[:, j] == e
            if bool(hit.any()):
                out[hit] = out[hit] + w[hit, j:j + 1] * clamped_expert(h[hit], t, p + f"e{e}.", mlp["expert"]["limit"])
    return out, picks


# --- the model ------------------------------------------------------------------------------------

def token_side(x, e, t, eps: float, p: str):
    """What a layer adds for its share ``e`` [T, dim] of the tokens' side rows."""
    y = (gelu_tanh(x @ t[p + "gate"].T) * e) @ t[p + "proj"].T
    return over_rms(y, eps) * t[p + "norm"]


def forward(model: dict, tokens, dtype=torch.float64, layers_out=None, picks=None, picks_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out`` (a list) receives the stream after each layer;
    ``picks`` {layer: [T, top]} forces the experts, ``picks_out`` (a dict) receives {layer: the choice made}."""
    cfg = model["config"]
    t = {k: v.to(dtype) for k, v in model["tensors"].items()}
    eps = cfg["norm"]["eps"]
    ids, positions = torch.tensor(tokens), torch.arange(len(tokens))
    x = t["embed"][ids] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{i}."
        x = x + mixer(centred_norm(x, t[n + "norm1"], eps), t, layer, eps, n + "mix.", positions)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = centred_norm(x, t[n + "norm2"], eps)
            if mlp["kind"] == "dense":
                y = dense(h, t, n + "mlp.")
            else:
                y, chosen = experts(h, t, mlp, n + "mlp.", picks=None if picks is None else picks.get(i))
                if picks_out is not None:
                    picks_out[i] = chosen
            x = x + y
        if cfg.get("token_side") is not None:
            d = cfg["token_side"]["dim"]
            x = x + token_side(x, t["side.embed"][ids][:, i * d:(i + 1) * d], t, eps, n + "side.")
        if layers_out is not None:
            layers_out.append(x)
    return centred_norm(x, t["final.norm"], eps) @ t["head"].T * cfg["logit_scale"]
