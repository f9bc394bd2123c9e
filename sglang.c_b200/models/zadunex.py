"""Zadunex as a plan of parts: a token table whose rows start several residual streams; pre-norm layers
whose sublayers read the norm of one combination of the streams and write into all of them; the mixer is
a selective state space (Mamba-2) or softmax attention with biases on queries, keys and values, a norm
over the whole query and key projections, half-split partial rotation and a constant 1 in the softmax's
denominator; the feed-forward is a gated MLP with bounded gates, a mixture of experts with softmax
routing whose weights are not renormalised, or absent; a run of layers may repeat with the same weights,
each pass with a cache and state of its own; a final norm over the sum of the streams, whose gain
takes the logits' multiplier, and a head of its own.

Tensor names: `embed`, `final.norm`, `head`, and for layer i `l<i>.norm1|norm2`, `l<i>.hc1|hc2.in|out|mix`,
`l<i>.mix.*` (mamba2: in, conv, conv.b, dt_bias, A_log, D, norm, o; attention: q, k, v with `.b` each,
q.norm, k.norm, o) and `l<i>.mlp.*` (dense: gate, up, down; experts: router, e<j>.gate|up|down).
"""
from ..config.registry import register_architecture
from ..config.zadunex import ZadunexConfig
from ..parts.plan import LayerPlan, ModelPlan, PartSpec, looped_order

GATE_SLOPE = 1.702      # of the bounded gate's sigmoid


def _mixer(cfg, lc, p):
    m, E = lc.mixer, cfg.width
    if lc.type == "mamba2":
        return PartSpec("mamba2", {"size": E, "n_heads": m.heads, "v_dim": m.vdim, "dim": m.state, "n_groups": m.groups,
                                   "conv": m.conv, "norm_groups": m.norm_groups, "eps": cfg.norm_eps},
                        {"in_weight": p + "in", "conv": p + "conv", "conv_bias": p + "conv.b", "dt_bias": p + "dt_bias",
                         "A_log": p + "A_log", "D": p + "D", "norm": p + "norm", "out_weight": p + "o"})
    rotary = {"dims": m.rot_dims, "base": m.rot_base, "scaling": None, "pairing": "halves"}
    return PartSpec("rotary_attention",
                    {"size": E, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim,
                     "scale": m.scale, "rotary": rotary if m.rot_dims else None, "qk_norm": "row_gain",
                     "eps": cfg.norm_eps, "chunk": None, "window": None, "sink": "one", "bias": True, "out_bias": False},
                    {"q_weight": p + "q", "q_bias": p + "q.b", "k_weight": p + "k", "k_bias": p + "k.b",
                     "v_weight": p + "v", "v_bias": p + "v.b", "q_norm": p + "q.norm", "k_norm": p + "k.norm",
                     "out_weight": p + "o"})


def _mlp(cfg, mlp, p):
    if mlp is None:
        return None
    if mlp.kind == "dense":
        return PartSpec("gated_mlp", {"size": cfg.width, "inner_size": mlp.ff, "bias": False, "activation": "clamped",
                                      "slope": GATE_SLOPE, "limit": mlp.limit},
                        {"gate_weight": p + "gate", "up_weight": p + "up", "down_weight": p + "down"})
    w = {"router": p + "router"}
    for e in range(mlp.experts):
        w.update({f"gate_{e}": f"{p}e{e}.gate", f"up_{e}": f"{p}e{e}.up", f"down_{e}": f"{p}e{e}.down"})
    return PartSpec("routed_experts", {"size": cfg.width, "inner_size": mlp.ff, "n_experts": mlp.experts, "top": mlp.top,
                                       "score": "softmax", "renorm": False, "correction": False}, w)


def build_plan(cfg: ZadunexConfig) -> ModelPlan:
    E, S = cfg.width, cfg.streams
    norm = lambda name, mult=1.0: PartSpec("rms_norm", {"size": E, "eps": cfg.norm_eps, "out_mult": mult}, {"weight": name})
    layers = []
    for i, lc in enumerate(cfg.layers):
        p = f"l{i}."
        hc = lambda q: ("stream_mix", PartSpec("stream_connection", {"streams": S},
                                               {k: f"{p}hc{q}.{k}" for k in ("in", "out", "mix")}))
        ffn = _mlp(cfg, lc.mlp, p + "mlp.")
        parts = {"hc1": hc(1)}
        if ffn is not None:
            parts["hc2"] = hc(2)
        layers.append(LayerPlan(name=f"l{i}", block=PartSpec("stream_pre_norm"), norm1=norm(p + "norm1"),
                                mixer=_mixer(cfg, lc, p + "mix."), norm2=norm(p + "norm2") if ffn is not None else None,
                                ffn=ffn, parts=parts))
    return ModelPlan(
        hidden_size=E, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("token_table", {"vocab_size": cfg.vocab, "size": E}, {"table": "embed"}),
        position=PartSpec("none", {}, {}), layers=layers, order=looped_order(len(cfg.layers), cfg.loop),
        final_norm=norm("final.norm", cfg.logit_scale),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "size": E}, {"weight": "head"}),
        eos_token_id=cfg.eos_token_id, entries=[PartSpec("residual_streams", {"size": E, "streams": S})])


register_architecture("Zadunex", ZadunexConfig, build_plan, model_types=("zadunex",))
