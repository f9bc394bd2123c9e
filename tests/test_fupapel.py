"""Fupapel without a device: configuration, plan, tensors, cache groups (a layer that reads another
layer's keys and values and keeps states of its own beside them), and the plain implementation's own
consistency."""
import copy
import math

import numpy as np
import pytest

import plain_fupapel as P
from fupapel_models import FUP, make_dir, make_sharp_dir


def _cfg(name):
    from sglang_c_b200.config import resolve_architecture
    arch = resolve_architecture(FUP[name])
    return arch, arch.config_class.from_dict(FUP[name])


class HostOnly:                     # parts are built without a device: only their needs are asked
    dtype, device = "float32", None


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_config_round_trip_and_plan(name):
    from sglang_c_b200.weights.loader import required_tensors
    arch, cfg = _cfg(name)
    assert arch.name == "Fupapel"
    assert arch.config_class.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict()["layers"] == FUP[name]["layers"]
    plan = arch.build_plan(cfg)
    need = required_tensors(plan)
    E, mult = FUP[name]["width"], FUP[name]["residual_mult"]
    assert len(plan.order) == len(plan.layers) == len(FUP[name]["layers"])
    for i, layer in enumerate(FUP[name]["layers"]):
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}.mix."
        assert plan.order[i].layer == i and plan.order[i].cache_of == m.get("kv_from")
        assert need[f"l{i}.norm1"].shape == need[f"l{i}.shift"].shape == (E,)
        assert (f"l{i}.norm2" in need) == (mlp is not None)
        if layer["type"] == "latent_attention":
            H = m["heads"]
            assert need[p + "dkv"].shape == (m["kv_rank"] + m["rot_dim"], E) and need[p + "dq"].shape == (m["q_rank"], E)
            assert need[p + "uq"].shape == (H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            assert need[p + "uk"].shape == (H * m["dim"], m["kv_rank"]) and need[p + "uv"].shape == (H * m["vdim"], m["kv_rank"])
            assert need[p + "g"].shape == (H, E) and need[p + "sink"].shape == (H,)
        else:
            H, G = m["heads"], m["kv_heads"]
            assert need[p + "q.norm"].shape == (H * m["dim"],) and need[p + "o"].shape == (E, H * m["vdim"])
            own, second = "kv_from" not in m, layer["type"] == "attention_2"
            for t in ("k", "v", "k.norm"):
                assert (p + t in need) == own
            for t in ("k.conv", "v.conv"):
                assert (p + t in need) == (own and second)
            assert (p + "q.conv" in need) == (p + "temp" in need) == (p + "sink" in need) == second
            assert (p + "g" in need) == (not second)
            if second:
                assert need[p + "q.conv"].shape == (H * m["dim"], m["conv"])
            else:
                assert need[p + "g"].shape == (H * m["vdim"], E)
        if mlp is not None:
            r = mlp["router"]
            n = r["experts"]
            assert need[f"l{i}.mlp.router"].shape == (n + r.get("identity", 0), E)
            assert need[f"l{i}.mlp.correction"].shape == (n + r.get("identity", 0),)
            assert need[f"l{i}.mlp.e{n - 1}.down"].shape == (E, mlp["expert"]["ff"]) and f"l{i}.mlp.e{n}.up" not in need
    assert plan.head.weights["weight"] == "head" and plan.embedding.weights["table"] == "embed"
    # the stream is kept divided by the multiplier
    assert plan.embedding.params["scale"] == 1.0 / mult
    assert math.isclose(plan.final_norm.params["eps"], FUP[name]["norm"]["eps"] / mult ** 2)


def test_config_errors_name_the_key():
    from sglang_c_b200.config import ConfigError, resolve_architecture
    arch = resolve_architecture(FUP["A"])

    def broken(change):
        d = copy.deepcopy(FUP["A"])
        change(d)
        with pytest.raises(ConfigError) as e:
            arch.config_class.from_dict(d)
        return str(e.value)

    mix = lambda d, i: d["layers"][i]["mixer"]
    assert "type" in broken(lambda d: d["layers"][0].update(type="mlstm"))
    assert "conv" in broken(lambda d: mix(d, 0).pop("conv"))
    assert "kv_heads" in broken(lambda d: mix(d, 0).update(kv_heads=3))
    assert "q_rank" in broken(lambda d: mix(d, 1).pop("q_rank"))
    assert "dims" in broken(lambda d: mix(d, 1)["rot"].update(dims=18))
    assert "dims" in broken(lambda d: mix(d, 2)["rot"].update(dims=13))
    assert "original" in broken(lambda d: mix(d, 0)["rot"]["scaling"].pop("original"))
    assert "high" in broken(lambda d: mix(d, 0)["rot"]["scaling"].update(high=0.5))
    assert "kv_from" in broken(lambda d: mix(d, 3).update(kv_from=4))            # not earlier
    assert "kv_from" in broken(lambda d: mix(d, 3).update(kv_from=2))            # another kind of layer
    assert "layer 0" in broken(lambda d: mix(d, 3).update(dim=16, rot=mix(d, 0)["rot"]))
    assert "groups" in broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=2))
    assert "keep" in broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4))
    assert "top" in broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=7))
    assert "residual_mult" in broken(lambda d: d.pop("residual_mult"))
    assert "residual_mult" in broken(lambda d: d.update(residual_mult=0.0))
    assert "eps" in broken(lambda d: d["norm"].pop("eps"))


def test_cache_of_a_layer_that_reads_anothers_pages_and_keeps_states_of_its_own():
    from sglang_c_b200.cache import CacheManager
    from sglang_c_b200.engine.model import Model
    arch, cfg = _cfg("A")
    model = Model(arch.build_plan(cfg), HostOnly())
    needs, cache_of = model.cache_needs()
    assert cache_of == [None, None, None, 0, None]
    assert [[n.kind for n in need] for need in needs] == [["paged_kv", "state", "state"], ["paged_kv", "state"],
                                                          ["paged_kv", "state"], ["paged_kv", "state", "state"],
                                                          ["paged_kv", "state"]]
    # pages of the shared keys stay for as long as either chunk needs them; the reader's convolution is over
    # its queries alone
    assert needs[0][0] == needs[3][0] and needs[0][0].chunk == math.lcm(24, 36) and needs[2][0].chunk == 20
    assert needs[0][1].state_shape == (2, 4 * 32 + 2 * (32 + 16)) and needs[3][1].state_shape == (2, 4 * 32)
    assert all(need[-1].state_shape == (64,) and need[-1].private for need in needs)
    made = []
    cm = CacheManager(needs, cache_of, page_size=8, n_pages=20, max_requests=2,
                      make_tensor=lambda shape, dt: made.append(np.zeros(shape)) or made[-1])
    b0, b3 = cm.binding(0), cm.binding(3)
    assert b0[0].group == b3[0].group and b0[0].write and not b3[0].write and b3[0].tensor is not None
    assert b3[1].write and b3[2].write
    bases = [(b.tensor.__array_interface__["data"][0]) for i in range(5) for b in cm.binding(i) if b.kind == "state"]
    assert len(set(bases)) == len(bases) == 7                    # every state has a place of its own
    kept = model.layers[3].bindings(b3)
    assert kept["mixer"][0] is b3[0] and kept["mixer"][1] is b3[1] and kept["shift"] is b3[2]
    assert model.layers[2].bindings(cm.binding(2))["mixer"] is cm.binding(2)[0]


def test_private_needs_do_not_follow_another_calls_cache():
    from sglang_c_b200.cache import CacheError, CacheManager, CacheNeed
    kv, tail, wide = CacheNeed.paged_kv(2, 8), CacheNeed.state((3,), private=True), CacheNeed.state((5,), private=True)
    cm = CacheManager([(kv, tail), (wide, kv), tail], [None, 0, None], 4, 6, 2)
    assert cm.binding(1)[1].group == cm.binding(0)[0].group and not cm.binding(1)[1].write and cm.binding(1)[0].write
    assert cm.binding(2).group == cm.binding(0)[1].group
    with pytest.raises(CacheError):                              # a state that is not private is the owner's or nobody's
        CacheManager([(kv, tail), (kv, CacheNeed.state((3,)))], [None, 0], 4, 6, 2)
    with pytest.raises(CacheError):
        CacheManager([tail, (kv, tail)], [None, 0], 4, 6, 2)


def test_scaled_frequencies_of_the_position_part():
    from sglang_c_b200.parts.registry import get_part
    for dims, base, sc in ((64, 10000.0, (8.0, 1.0, 4.0, 512)), (32, 500.0, (3.0, 0.5, 6.0, 40)), (16, 20.0, (2.0, 2.0, 2.0, 30)),
                           (8, 1e6, None)):
        d = None if sc is None else dict(zip(("factor", "low", "high", "original"), sc))
        part = get_part("position", "rotary")({"dims": dims, "base": base, "scaling": d}, None)
        part.load({}, None)
        want = P.frequencies(dims, base, d)
        assert np.allclose(part.frequencies.numpy(), want, rtol=1e-13) and part.multiplier == 1.0
        if sc is not None and sc[1] != sc[2]:       # all three kinds of pairs occur
            ratio = want / P.frequencies(dims, base)
            assert (ratio == 1).any() and np.isclose(ratio, 1 / sc[0]).any()
            assert ((ratio < 0.999) & (ratio > 1.001 / sc[0])).any()


def test_plain_mechanisms_agree_with_themselves(tmp_path):
    """The oracle's own consistency, and what the mechanisms do in it: a position's logits do not depend on
    what follows; a lost row ahead of the shift, a lost tail of the convolution, a chunk one longer, a
    missing sink, a dropped identity expert, a group counted by another rule: each moves the result."""
    d = make_sharp_dir(tmp_path, "A")
    cfg, w = P.read_model_dir(d)
    rng = np.random.default_rng(3)
    toks = [int(t) for t in rng.integers(0, cfg["vocab"], 80)]
    full, streams = P.forward(cfg, w, toks, True)
    assert np.abs(P.forward(cfg, w, toks[:31]) - full[:31]).max() < 1e-9
    size = full.std()
    moves = {}

    def planted(name, **patch):
        old = {k: getattr(P, k) for k in patch}
        try:
            for k, v in patch.items():
                setattr(P, k, v)
            moves[name] = np.abs(P.forward(cfg, w, toks) - full)[41:].max() / size
        finally:
            for k, v in old.items():
                setattr(P, k, v)
    shift, conv, attend, route = P.token_shift, P.short_convolution, P.softmax_attention, P.route

    def lost_row(h, mu):
        y = shift(h, mu)
        y[40] = h[40] - h[40] * mu                  # token 40 finds no row before it
        return y

    def lost_tail(u, taps):
        return np.concatenate([conv(u[:40], taps), conv(u[40:], taps)], 0)
    planted("row", token_shift=lost_row)
    planted("tail", short_convolution=lost_tail)
    planted("chunk", softmax_attention=lambda q, k, v, s, chunk=None, sinks=None: attend(q, k, v, s, chunk + 1 if chunk else None, sinks))
    planted("sink", softmax_attention=lambda q, k, v, s, chunk=None, sinks=None: attend(q, k, v, s, chunk, None))
    planted("far", softmax_attention=lambda q, k, v, s, chunk=None, sinks=None: attend(q, k, v, s, chunk or 40, sinks))
    planted("identity", moe_ff=lambda w_, p, mlp, h: _moe_without_identity(w_, p, mlp, h))
    planted("groups", route=lambda z, c, top, n, keep: route(z, c, top, 1, 1))
    assert all(v > 0.02 for v in moves.values()), moves
    # routing by hand: negative choice scores, a kept group that is best by its best member
    z = np.log(np.array([[0.05, 0.2, 0.3, 0.1, 0.25, 0.1]]))
    c = np.array([-1.0, -0.5, -0.9, -0.9, -0.4, -2.0])
    got = P.route(z, c, 2, 3, 1)
    assert np.allclose(got, [[0, 0, 0, 0, 0.25, 0.1]])           # group 2 has the best member, and -1.9 is still in it
    # the frequencies' blend meets both ends
    f = P.frequencies(64, 1e4, dict(factor=8.0, low=1.0, high=4.0, original=512))
    assert f[0] == 1.0 and math.isclose(f[-1], 1e4 ** (-62 / 64) / 8.0) and (np.diff(f) < 0).all()
    # a sink of score zero is a one in the denominator
    q, k, v = (rng.standard_normal((5, 1, 4)) for _ in range(3))
    o = P.softmax_attention(q, k, v, 0.5, sinks=np.zeros(1))
    e = np.exp(0.5 * (q[4, 0] @ k[:, 0].T))
    assert np.allclose(o[4, 0], (e[:, None] * v[:, 0]).sum(0) / (1 + e.sum()))


def _moe_without_identity(w, p, mlp, h):
    r = mlp["router"]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    dense = P.route(h @ w[p + "router"].T, w[p + "correction"], r["top"], gr["count"], gr["keep"])
    return sum(dense[:, e:e + 1] * P.gated_expert(w, f"{p}e{e}.", h) for e in range(r["experts"]))


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_routing_choices_of_the_test_models_are_not_all_close_calls(tmp_path, name):
    """The whole-model tests compare logits: their models' choices must be decided by more than rounding."""
    cfg, w = P.read_model_dir(make_dir(tmp_path, name))
    rng = np.random.default_rng(5)
    margins = []
    route = P.route

    def watch(z, c, top, n_groups=1, keep=1):
        s = np.exp(z - z.max(-1, keepdims=True))
        s = np.sort(s / s.sum(-1, keepdims=True) + c, -1)
        if 0 < top < z.shape[1]:
            margins.extend(s[:, -top] - s[:, -top - 1])
        return route(z, c, top, n_groups, keep)
    try:
        P.route = watch
        P.forward(cfg, w, rng.integers(0, cfg["vocab"], 120))
    finally:
        P.route = route
    assert np.median(margins) > 0.03
