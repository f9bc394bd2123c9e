"""Fupapel as a plan of parts: a token table; layers x += m (mixer(norm1(x)) + ff(norm2(x))) whose norms
have gains stored around zero and whose mixer reads its normed rows moved towards the token before; a
final norm and a head.  The mixer is chunked softmax attention with a constant 1 in the denominator and
results gated entry by entry; chunked attention behind short convolutions over q, k and v, with a
factor and a sink per head (a layer may read the keys and values an earlier layer cached, and then
still convolves its own queries); or latent attention with a turned part, a sink and a gate per head.
The feed-forward is a mixture of experts with softmax scores, a choice correction and groups that
count as their best member, some of whose experts are the identity.

The multiplier m costs nothing: the plan keeps the stream as x / m.  Every sublayer reads the stream
through an RMS norm, and x / sqrt(mean(x^2) + eps) = y / sqrt(mean(y^2) + eps / m^2) for y = x / m; so
the token rows are scaled by 1 / m once, the norms take eps / m^2, and the sublayers' products add to
the stream as they are.

Tensor names: `embed`, `final.norm`, `head`, and for layer i `l<i>.norm1`, `l<i>.norm2`, `l<i>.shift`,
`l<i>.mix.*` (attention: q, k, v, g, o, q.norm, k.norm; attention_2: q, k, v, o, q.norm, k.norm, q.conv,
k.conv, v.conv, temp, sink, without those of k and v under kv_from; latent_attention: dq, dq.norm, uq,
dkv, dkv.norm, uk, uv, sink, g, o) and `l<i>.mlp.*` (router, correction, e<j>.gate|up|down).
"""
import math

from ..config.fupapel import FupapelConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerCall, LayerPlan, ModelPlan, PartSpec


def _rotary(rot):
    if rot is None:
        return None
    return {"dims": rot.dims, "base": rot.base, "pairing": "halves",
            "scaling": None if rot.scaling is None else rot.scaling.to_dict()}


def _attention(cfg, m, p, kept_chunk):
    """Both softmax mixers; the second has convolutions, factors and learned sinks, the first a gate."""
    second, own = m.conv is not None, m.kv_from is None
    params = {"size": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim,
              "scale": m.scale, "rotary": _rotary(m.rot), "qk_norm": "row_gain", "eps": cfg.norm_eps, "chunk": m.chunk,
              "window": None, "bias": False, "own_kv": own, "sink": True if second else "one",
              "gate": None if second else "entry", "temp": second, "conv": m.conv, "cache_chunk": kept_chunk}
    w = {"q_weight": p + "q", "q_norm": p + "q.norm", "out_weight": p + "o"}
    if own:
        w.update({"k_weight": p + "k", "v_weight": p + "v", "k_norm": p + "k.norm"})
    if second:
        w.update({"q_conv": p + "q.conv", "temp": p + "temp", "sink": p + "sink"})
        if own:
            w.update({"k_conv": p + "k.conv", "v_conv": p + "v.conv"})
    else:
        w["gate_weight"] = p + "g"
    return PartSpec("rotary_attention", params, w)


def _latent(cfg, m, p):
    return PartSpec("latent_attention",
                    {"size": cfg.width, "n_heads": m.heads, "qk_dim": m.dim, "v_dim": m.vdim, "kv_rank": m.kv_rank,
                     "q_rank": m.q_rank, "scale": m.scale, "eps": cfg.norm_eps, "own_latent": True, "window": None,
                     "rot_dim": m.rot_dim, "rotary": _rotary(m.rot), "sink": True, "gate": "head"},
                    {"q_down": p + "dq", "q_norm": p + "dq.norm", "q_up": p + "uq", "kv_down": p + "dkv",
                     "kv_norm": p + "dkv.norm", "k_up": p + "uk", "v_up": p + "uv", "sink": p + "sink",
                     "gate_weight": p + "g", "out_weight": p + "o"})


def _mlp(cfg, mlp, p):
    if mlp is None:
        return None
    w = {"router": p + "router", "correction": p + "correction"}
    for e in range(mlp.experts):
        w.update({f"gate_{e}": f"{p}e{e}.gate", f"up_{e}": f"{p}e{e}.up", f"down_{e}": f"{p}e{e}.down"})
    return PartSpec("routed_experts", {"size": cfg.width, "inner_size": mlp.ff, "n_experts": mlp.experts, "top": mlp.top,
                                       "score": "softmax", "correction": True, "n_groups": mlp.groups, "keep": mlp.keep,
                                       "group_score": "max", "n_identity": mlp.identity}, w)


def _kept_chunk(layers, i):
    """The chunk by which layer i's pages may go back: a multiple of its own and of every reader's."""
    chunks = [layers[i].mixer.chunk] + [lc.mixer.chunk for lc in layers
                                        if lc.type == "attention_2" and lc.mixer.kv_from == i]
    return None if any(c is None for c in chunks) else math.lcm(*chunks)


def build_plan(cfg: FupapelConfig) -> ModelPlan:
    E, m = cfg.width, cfg.residual_mult
    norm = lambda name: PartSpec("rms_norm", {"size": E, "eps": cfg.norm_eps / (m * m), "one_plus": True}, {"weight": name})
    layers, order, unread = [], [], []
    for i, lc in enumerate(cfg.layers):
        p = f"l{i}."
        kv_from = None
        if lc.type == "latent_attention":
            mixer = _latent(cfg, lc.mixer, p + "mix.")
        else:
            kv_from = lc.mixer.kv_from
            mixer = _attention(cfg, lc.mixer, p + "mix.", _kept_chunk(cfg.layers, i if kv_from is None else kv_from))
        ffn = _mlp(cfg, lc.mlp, p + "mlp.")
        if ffn is None:
            unread.append(p + "norm2")        # (a file may still hold the norm ahead of a feed-forward that is not there)
        layers.append(LayerPlan(name=f"l{i}", block=PartSpec("parallel_two_norms", {}), mixer=mixer,
                                norm1=norm(p + "norm1"), ffn=ffn, norm2=norm(p + "norm2") if ffn is not None else None,
                                parts={"shift": ("token_mix", PartSpec("token_shift", {"size": E}, {"mix": p + "shift"}))}))
        order.append(LayerCall(i, cache_of=kv_from))
    return ModelPlan(
        hidden_size=E, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding=PartSpec("token_table", {"vocab_size": cfg.vocab, "size": E, "scale": 1.0 / m}, {"table": "embed"}),
        position=PartSpec("none", {}, {}),
        layers=layers, order=order, final_norm=norm("final.norm"),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "size": E}, {"weight": "head"}),
        eos_token_id=cfg.eos_token_id, ignorable=tuple(unread))


register_architecture("Fupapel", FupapelConfig, build_plan, model_types=("fupapel",))
