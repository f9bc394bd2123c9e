"""Zadunex without a device: configuration, plan, tensors, caches and states of repeated layers, and the plain
implementation's own consistency."""
import copy

import numpy as np
import pytest

import plain_zadunex as P
from zadunex_models import ZAD, make_dir, make_sharp_dir


def _cfg(name):
    from sglang_c_b200.config import resolve_architecture
    arch = resolve_architecture(ZAD[name])
    return arch, arch.config_class.from_dict(ZAD[name])


class HostOnly:                     # parts are built without a device: only their needs are asked
    dtype, device = "float32", None


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_config_round_trip_and_plan(name):
    from sglang_c_b200.weights.loader import required_tensors
    arch, cfg = _cfg(name)
    d = ZAD[name]
    assert arch.name == "Zadunex"
    assert arch.config_class.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict() == d
    plan = arch.build_plan(cfg)
    need = required_tensors(plan)
    E, S = d["width"], d["streams"]
    assert [c.layer for c in plan.order] == P.running_order(d)
    assert all(c.cache_of is None and c.enter is None for c in plan.order)
    for i, layer in enumerate(d["layers"]):
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}.mix."
        for q in (1, 2):
            there = q == 1 or mlp is not None
            assert (f"l{i}.norm{q}" in need) == (f"l{i}.hc{q}.in" in need) == (f"l{i}.hc{q}.mix" in need) == there
            if there:
                assert need[f"l{i}.hc{q}.in"].shape == need[f"l{i}.hc{q}.out"].shape == (S,)
                assert need[f"l{i}.hc{q}.mix"].shape == (S, S)
        H, V = m["heads"], m["vdim"]
        assert need[p + "o"].shape == (E, H * V) and p + "o.b" not in need
        if layer["type"] == "mamba2":
            C = H * V + 2 * m["groups"] * m["state"]
            assert need[p + "in"].shape == (H * V + C + H, E) and need[p + "conv"].shape == (C, m["conv"])
            assert need[p + "conv.b"].shape == (C,) and need[p + "norm"].shape == (H * V,)
            assert need[p + "A_log"].shape == need[p + "dt_bias"].shape == need[p + "D"].shape == (H,)
        else:
            G, D = m["kv_heads"], m["dim"]
            assert need[p + "q"].shape == (H * D, E) and need[p + "q.b"].shape == need[p + "q.norm"].shape == (H * D,)
            assert need[p + "k.norm"].shape == need[p + "k.b"].shape == (G * D,) and need[p + "v.b"].shape == (G * V,)
            assert p + "sink" not in need
        if mlp is not None and mlp["kind"] == "moe":
            n = mlp["router"]["experts"]
            assert need[f"l{i}.mlp.router"].shape == (n, E) and f"l{i}.mlp.e{n}.up" not in need
            assert need[f"l{i}.mlp.e{n - 1}.down"].shape == (E, mlp["expert"]["ff"])
        elif mlp is not None:
            assert need[f"l{i}.mlp.gate"].shape == need[f"l{i}.mlp.up"].shape == (mlp["ff"], E)
            assert plan.layers[i].ffn.params["limit"] == mlp["limit"] and f"l{i}.mlp.gate.b" not in need
    assert plan.head.weights["weight"] == "head" and plan.embedding.weights["table"] == "embed"
    assert plan.final_norm.params["out_mult"] == d["logit_scale"]


def test_config_errors_name_the_key():
    from sglang_c_b200.config import ConfigError, resolve_architecture
    arch = resolve_architecture(ZAD["A"])

    def broken(change):
        d = copy.deepcopy(ZAD["A"])
        change(d)
        with pytest.raises(ConfigError) as e:
            arch.config_class.from_dict(d)
        return str(e.value)

    mix = lambda d, i: d["layers"][i]["mixer"]
    assert "type" in broken(lambda d: d["layers"][0].update(type="mlstm"))
    for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
        assert k in broken(lambda d: mix(d, 0).pop(k))
    assert "groups" in broken(lambda d: mix(d, 0).update(groups=4))
    assert "norm_groups" in broken(lambda d: mix(d, 0).update(norm_groups=7))
    assert "kv_heads" in broken(lambda d: mix(d, 1).update(kv_heads=4))
    assert "scale" in broken(lambda d: mix(d, 1).pop("scale"))
    assert "dims" in broken(lambda d: mix(d, 1)["rot"].update(dims=34))
    assert "dims" in broken(lambda d: mix(d, 1)["rot"].update(dims=5))
    assert "base" in broken(lambda d: mix(d, 1)["rot"].pop("base"))
    assert "limit" in broken(lambda d: d["layers"][1]["mlp"].pop("limit"))
    assert "top" in broken(lambda d: d["layers"][0]["mlp"]["router"].update(top=7))
    assert "kind" in broken(lambda d: d["layers"][0]["mlp"].update(kind="sparse"))
    assert "streams" in broken(lambda d: d.pop("streams"))
    assert "loop" in broken(lambda d: d["loop"].update(stop=6))
    assert "times" in broken(lambda d: d["loop"].update(times=0))
    assert "eps" in broken(lambda d: d["norm"].pop("eps"))


def test_every_pass_of_a_repeated_layer_has_a_cache_and_a_state_of_its_own():
    from sglang_c_b200.cache import CacheManager
    from sglang_c_b200.engine.model import Model
    arch, cfg = _cfg("A")
    model = Model(arch.build_plan(cfg), HostOnly())
    needs, cache_of = model.cache_needs()
    assert [c.layer for c in model.plan.order] == [0, 1, 2, 1, 2, 3, 4] and cache_of == [None] * 7
    kinds = [n.kind if not isinstance(n, tuple) else [x.kind for x in n] for n in needs]
    assert kinds == [["state", "state"], "paged_kv", ["state", "state"], "paged_kv", ["state", "state"], "paged_kv",
                     ["state", "state"]]
    assert needs[0][0].state_shape == (6, 24, 20) and needs[0][1].state_shape == (3, 6 * 20 + 2 * 3 * 24)
    assert needs[2][1].state_shape == (1, 4 * 16 + 2 * 40) and needs[2] == needs[4]
    made = []
    cm = CacheManager(needs, cache_of, page_size=8, n_pages=20, max_requests=2,
                      make_tensor=lambda shape, dt: made.append(np.zeros(shape)) or made[-1])
    where = []
    for i in range(7):
        b = cm.binding(i)
        where += [x.tensor.__array_interface__["data"][0] for x in (b if isinstance(b, (tuple, list)) else (b,))]
    assert len(set(where)) == len(where) == 11


def test_orders_of_repeated_layers():
    from sglang_c_b200.config.base import LayerLoop
    from sglang_c_b200.parts.plan import looped_order
    run = lambda n, lp, e=None: [(c.layer, c.enter) for c in looped_order(n, lp, e)]
    assert run(3, None) == [(0, None), (1, None), (2, None)]
    assert run(3, LayerLoop(1, 2, 3)) == [(0, None), (1, None), (1, None), (1, None), (2, None)]
    assert run(3, LayerLoop(0, 2, 2), 0) == [(0, (0, 0)), (1, None), (0, (0, 1)), (1, None), (2, None)]
    assert run(2, LayerLoop(0, 2, 1)) == [(0, None), (1, None)]


def test_plain_mechanisms_agree_with_themselves(tmp_path):
    """The oracle's own consistency, and what the mechanisms do in it: a position's logits do not depend on
    what follows; a state or a convolution's tail lost on the way, a far key, the constant in the softmax,
    an order of the streams, a bound, an order of gate and norm: each moves the result."""
    d = make_sharp_dir(tmp_path, "A")
    cfg, w = P.read_model_dir(d)
    rng = np.random.default_rng(3)
    toks = [int(t) for t in rng.integers(0, cfg["vocab"], 80)]
    full, sums = P.forward(cfg, w, toks, True)
    assert len(sums) == 7
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
    space, conv, attend, route = P.state_space, P.short_convolution, P.softmax_attention, P.route
    halves = lambda f, n_rows: lambda *a: np.concatenate([f(*[x[:40] for x in a[:n_rows]], *a[n_rows:]),
                                                          f(*[x[40:] for x in a[:n_rows]], *a[n_rows:])], 0)
    planted("state", state_space=lambda *a: (halves(lambda *b: space(*b)[0], 4)(*a), None))
    planted("tail", short_convolution=halves(conv, 1))
    planted("far", softmax_attention=lambda q, k, v, s: np.concatenate(
        [attend(q, k, v, s)[:40], attend(q[40:], k[40:], v[40:], s)], 0))
    planted("one", softmax_attention=lambda q, k, v, s: attend(q, k, v, s) * 1.02)
    planted("skip", state_space=lambda x, B, C, dt, A, D: space(x, B, C, dt, A, 0 * D))
    planted("write", streams_write=lambda X, y, o, m: np.stack(
        [sum(m[t, s] * X[s] for s in range(len(X))) + o[t] * y for t in range(len(X))]))
    planted("read", streams_read=lambda X, i: X.mean(0))
    planted("bound", clamped_gate=lambda g, u, limit: g * P.sigmoid(1.702 * g) * (u + 1.0))
    planted("groups", group_rms_norm=lambda x, g, eps, n: P.rms_norm(x, g, eps))
    planted("weights", route=lambda z, top: route(z, top) / route(z, top).sum(-1, keepdims=True))
    assert all(v > 0.01 for v in moves.values()), moves
    # a state by hand: one head, two tokens
    y, S = P.state_space(np.array([[[2.0]], [[3.0]]]), np.array([[[1.0, 2.0]], [[0.5, 1.0]]]),
                         np.array([[[1.0, 1.0]], [[2.0, 0.0]]]), np.array([[0.5], [0.25]]), np.array([np.log(2.0)]), np.array([10.0]))
    s1 = 0.5 * 2.0 * np.array([1.0, 2.0])
    s2 = np.exp(-0.5) * s1 + 0.25 * 3.0 * np.array([0.5, 1.0])
    assert np.allclose(S[0, :, 0], s2) and np.allclose(y[:, 0, 0], [s1.sum() + 20.0, 2.0 * s2[0] + 30.0])
    # the constant counts as a key of score zero without a value
    q, k, v = (rng.standard_normal((5, 1, 4)) for _ in range(3))
    e = np.exp(0.5 * (q[4, 0] @ k[:, 0].T))
    assert np.allclose(P.softmax_attention(q, k, v, 0.5)[4, 0], (e[:, None] * v[:, 0]).sum(0) / (1 + e.sum()))
    # streams from the old ones: what stream 0 became does not enter stream 1
    X = rng.standard_normal((2, 1, 3))
    got = P.streams_write(X, np.ones((1, 3)), np.array([0.5, -1.0]), np.array([[0.1, 0.2], [0.3, 0.4]]))
    assert np.allclose(got[1], 0.2 * X[0] + 0.4 * X[1] - 1.0) and np.allclose(got[0], 0.1 * X[0] + 0.3 * X[1] + 0.5)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_test_models_are_decided_by_more_than_rounding(tmp_path, name):
    """The whole-model tests compare logits: their models' choices must not all be close calls, and some gates
    must reach their bounds."""
    cfg, w = P.read_model_dir(make_dir(tmp_path, name))
    margins, bounded = [], []
    route, gate = P.route, P.clamped_gate

    def watch(z, top):
        s = np.exp(z - z.max(-1, keepdims=True))
        s = np.sort(s / s.sum(-1, keepdims=True), -1)
        if top < z.shape[1]:
            margins.extend(s[:, -top] - s[:, -top - 1])
        return route(z, top)

    def watch_gate(g, u, limit):
        bounded.append([(g > limit).mean(), (g < -limit).mean(), (u > limit).mean(), (u < -limit).mean()])
        return gate(g, u, limit)
    try:
        P.route, P.clamped_gate = watch, watch_gate
        P.forward(cfg, w, np.random.default_rng(5).integers(0, cfg["vocab"], 120))
    finally:
        P.route, P.clamped_gate = route, gate
    assert np.median(margins) > 0.03
    assert (np.array(bounded).max(0) > 0.01).all(), bounded
