"""Gurolix as data: configuration -> ModelSpec.

A stack of layers with a norm before and after each sublayer, a gate per element on each sublayer's output and,
after each layer, a learned average over the embedding output and all layers so far (block ``sandwich``; the
norms' weights are stored around zero; the embedding is normed as well).  The mixers are ``mamba2`` and
``rotary_attention`` (biased projections, optionally per-head norms of q and k, rescaled rotary frequencies, a
score cap, values mixed with the first such layer's).  The feed-forward is ``routed_experts``: softmax scores, a
correction that only chooses, experts chosen within the best groups, ungated experts with the square of relu,
identity experts; or none.  Tensor names: ``embed``, ``embed.norm``, ``l<i>.norm{1,1b,2,2b}``,
``l<i>.rg{1,2}``, ``l<i>.rg{1,2}.b``, ``l<i>.dwa``, ``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}`` or
``l<i>.mix.{q,k,v}``, ``.{q,k,v}.b``, ``.{q,k}.norm``, ``.vmix``, ``.o``, ``l<i>.mlp.{router,correction,
e<j>.up,e<j>.down}``, ``final.norm``, ``head``.  This file only names parts and passes them their constants."""
from __future__ import annotations

from ..config.gurolix import ARCHITECTURE, GurolixConfig, read_gurolix_config
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def _mixer(layer, width: int, eps: float, p: str, value_mix) -> PartSpec:
    m = layer.mixer
    if layer.type == "mamba2":
        return PartSpec("mamba2",
                        dict(hidden_size=width, num_heads=m["heads"], head_dim=m["vdim"], state_size=m["state"],
                             num_groups=m["groups"], norm_groups=m["norm_groups"], conv_taps=m["conv"], norm_eps=eps),
                        dict(in_proj=p + "in", conv=p + "conv", conv_bias=p + "conv.b", dt_bias=p + "dt_bias",
                             a_log=p + "A_log", skip=p + "D", norm=p + "norm", out_proj=p + "o"))
    rot = m["rot"]
    position = {"kind": "none"}
    if rot is not None:
        position = dict(kind="rope_bands", head_dim=m["dim"], theta=rot["base"], rot_dim=rot["dims"],
                        scaling=rot["scaling"])
    return PartSpec("rotary_attention",
                    dict(hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                         v_head_dim=m["vdim"], scale=m["scale"], qk_norm_eps=eps if layer.type == "attention" else None,
                         softcap=m["softcap"], position=position, value_mix=value_mix),
                    dict(q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", out_proj=p + "o", q_bias=p + "q.b",
                         k_bias=p + "k.b", v_bias=p + "v.b", q_norm=p + "q.norm", k_norm=p + "k.norm",
                         value_mix=p + "vmix"))


def gurolix_model_spec(c: GurolixConfig) -> ModelSpec:
    W, eps = c.width, c.norm_eps

    def norm(name):
        return PartSpec("rmsnorm", dict(size=W, eps=eps, offset=1.0), dict(weight=name))
    layers, run = [], []
    mixing = False                                # whether an earlier layer's values are there to mix with
    for i, layer in enumerate(c.layers):
        n = f"l{i}."
        role = ("mix" if mixing else "first") if layer.mixer.get("v_mix") else None
        mixing = mixing or role is not None
        mixer = _mixer(layer, W, eps, n + "mix.", role)
        ffn = ffn_norm = None
        posts, gates = [norm(n + "norm1b")], [dict(weight=n + "rg1", bias=n + "rg1.b")]
        if layer.mlp is not None:
            f, mlp = n + "mlp.", layer.mlp
            ffn = PartSpec("routed_experts",
                           dict(hidden_size=W, intermediate_size=mlp["ff"], num_experts=mlp["experts"],
                                top_k=mlp["top"], norm_topk_prob=False, use_expert_bias=True,
                                routed_scaling_factor=1.0, scoring="softmax", activation="relu2", gated=False,
                                groups=mlp["groups"], identity=mlp["identity"]),
                           dict(router=f + "router", expert_bias=f + "correction", experts=f + "e", expert_up="up",
                                expert_down="down"))
            ffn_norm = norm(n + "norm2")
            posts.append(norm(n + "norm2b"))
            gates.append(dict(weight=n + "rg2", bias=n + "rg2.b"))
        layers.append(LayerSpec("sandwich", mixer, ffn, norm(n + "norm1"), ffn_norm,
                                dict(hidden_size=W, post_norms=tuple(posts), gates=tuple(gates),
                                     average=dict(index=i, layers=len(c.layers), name=n + "dwa"))))
        run.append(RunEntry(i))
    embedding = PartSpec("embedding", dict(vocab_size=c.vocab, hidden_size=W, norm=norm("embed.norm")),
                         dict(weight="embed"))
    head = PartSpec("linear_head", dict(vocab_size=c.vocab, hidden_size=W, tied=False), dict(weight="head"))
    return ModelSpec(architecture=c.architecture, vocab_size=c.vocab, hidden_size=W, embedding=embedding,
                     layers=layers, run=run, final_norm=norm("final.norm"), head=head)


register_architecture(ARCHITECTURE, read_gurolix_config, gurolix_model_spec)
