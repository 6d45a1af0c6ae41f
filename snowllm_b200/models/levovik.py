"""Levovik as data: configuration -> ModelSpec.

A stack of pre-norm layers (block ``prenorm``, norm ``layernorm``: centred, a weight, no bias), each with two mixers side
by side on the same input (``side_by_side`` without output norms: a constant times each output) and, after its
feed-forward, an input of its own from a second table of token rows (``side_rows`` in the embedding, ``token_side`` in
the block).  ``parallel``: softmax attention with a sink per head, q and k over their root mean square, halves rotated
(``rotary_attention``), beside the gated delta rule (``delta_rule``).  ``parallel_2``: softmax attention whose values are
its projected keys, neighbours rotated (``rotary_attention``), beside gated linear attention (``gated_linear``).  The
feed-forward is dense with relu (``gated``) or routed experts with sigmoid scores chosen within the best groups
(``routed_experts``), or none.  Tensor names: ``embed``, ``side.embed``, ``l<i>.norm{1,2}``,
``l<i>.mix.{left,right}.<what>``, ``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{router, e<j>.{gate,up,down}}``,
``l<i>.side.{gate,proj,norm}``, ``final.norm``, ``head``.  This file only names parts and passes them their constants."""
from __future__ import annotations

from ..config.levovik import ARCHITECTURE, DELTA, LevovikConfig, read_levovik_config
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry

UNIT_EPS = 1e-6          # added to a squared length before its root where q and k become unit vectors
RENORM_EPS = 1e-20       # added to the sum of the picked experts' scores


def _left(m: dict, width: int, eps: float, p: str, delta: bool) -> PartSpec:
    rot = m["rot"]
    position = {"kind": "none"}
    if rot is not None:
        position = dict(kind="rope_bands", head_dim=m["dim"], theta=rot["base"], rot_dim=rot["dims"],
                        scaling=rot["scaling"], layout="halves" if delta else "pairs")
    return PartSpec("rotary_attention",
                    dict(hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                         v_head_dim=m["vdim"], scale=m["scale"], qk_norm_eps=eps, position=position, biased=False,
                         qk_norm_weights=not delta, with_sink=delta, keys_are_values=not delta),
                    dict(q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", out_proj=p + "o", q_norm=p + "q.norm",
                         k_norm=p + "k.norm", sink=p + "sink"))


def _right(m: dict, width: int, eps: float, p: str, delta: bool) -> PartSpec:
    common = dict(hidden_size=width, num_heads=m["heads"], head_dim=m["dim"], v_head_dim=m["vdim"], head_norm_eps=eps,
                  decay_rank=m["decay_rank"])
    names = dict(q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", decay_a=p + "a1", decay_b=p + "a2", norm=p + "norm",
                 out_proj=p + "o")
    if delta:
        return PartSpec("delta_rule", dict(common, num_kv_heads=m["kv_heads"], conv_taps=m["conv"], unit_eps=UNIT_EPS,
                                           gate_rank=m["gate_rank"]),
                        dict(names, q_conv=p + "q.conv", k_conv=p + "k.conv", v_conv=p + "v.conv", beta_proj=p + "b",
                             a_log=p + "A_log", dt_bias=p + "dt_bias", gate_a=p + "g1", gate_b=p + "g2"))
    return PartSpec("gated_linear", dict(common, tau=m["tau"]), dict(names, decay_bias=p + "a2.b", gate_proj=p + "g"))


def _ffn(mlp: dict, width: int, f: str) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("gated", dict(hidden_size=width, intermediate_size=mlp["ff"], activation="relu"),
                        dict(gate=f + "gate", up=f + "up", down=f + "down"))
    return PartSpec("routed_experts",
                    dict(hidden_size=width, intermediate_size=mlp["ff"], num_experts=mlp["experts"], top_k=mlp["top"],
                         norm_topk_prob=True, renorm_eps=RENORM_EPS, use_expert_bias=False,
                         routed_scaling_factor=mlp["scale"], scoring="sigmoid", activation="swish_clamp",
                         limit=mlp["limit"], groups=mlp["groups"], group_score="top2"),
                    dict(router=f + "router", experts=f + "e", expert_gate="gate", expert_up="up", expert_down="down",
                         fused_gate_up=f + "gate_up", fused_down=f + "down_all"))


def levovik_model_spec(c: LevovikConfig) -> ModelSpec:
    W, eps = c.width, c.norm_eps

    def norm(name, gain=1.0):
        return PartSpec("layernorm", dict(size=W, eps=eps, gain=gain), dict(weight=name))
    layers, run = [], []
    for i, layer in enumerate(c.layers):
        n, m = f"l{i}.", layer.mixer
        delta = layer.type == DELTA
        mixer = PartSpec("side_by_side",
                         dict(hidden_size=W, left=_left(m["left"], W, eps, n + "mix.left.", delta),
                              right=_right(m["right"], W, eps, n + "mix.right.", delta), eps=None,
                              weights=(m["left_scale"], m["right_scale"])))
        ffn = ffn_norm = None
        if layer.mlp is not None:
            ffn, ffn_norm = _ffn(layer.mlp, W, n + "mlp."), norm(n + "norm2")
        block = {}
        if c.token_side is not None:
            block = dict(side=PartSpec("token_side", dict(hidden_size=W, dim=c.token_side, index=i, eps=eps),
                                       dict(gate=n + "side.gate", proj=n + "side.proj", norm=n + "side.norm")))
        layers.append(LayerSpec("prenorm", mixer, ffn, norm(n + "norm1"), ffn_norm, block))
        run.append(RunEntry(i))
    params, names = dict(vocab_size=c.vocab, hidden_size=W, scale=c.embedding_scale), dict(weight="embed")
    if c.token_side is not None:
        params["side_size"] = c.token_side * len(c.layers)
        names["side"] = "side.embed"
    # logits = head(x) * logit_scale: the factor rides in the norm before the head
    return ModelSpec(architecture=c.architecture, vocab_size=c.vocab, hidden_size=W,
                     embedding=PartSpec("embedding", params, names), layers=layers, run=run,
                     final_norm=norm("final.norm", c.logit_scale),
                     head=PartSpec("linear_head", dict(vocab_size=c.vocab, hidden_size=W, tied=False),
                                   dict(weight="head")))


register_architecture(ARCHITECTURE, read_levovik_config, levovik_model_spec)
