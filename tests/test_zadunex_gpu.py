"""Zadunex on the device: every mechanism's kernel alone against the plain implementation's function,
then whole models through the engine's step function in every cut (whole prompts, last tokens one by
one, portions down to two tokens, mixed batches with pages and state slots used again, long decoding),
models whose constants make a lost key or a lost state show, and greedy generation through the scheduler
and the command line."""
import math

import numpy as np
import pytest
import torch

import plain_zadunex as P
import traces
from zadunex_models import PAGE, ZAD, make_dir, make_sharp_dir

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
# Errors are a position's largest difference against the size of the logits (their standard deviation
# over the whole run).  The 32-bit bound is the sharp one: 98 in 100 positions lie within it, and none is
# twenty times beyond (a position whose gated row happens to be small is normed up with its rounding; a
# lost key or state moves the logits by forty times the bound and more).  In bfloat16 these narrow random models are
# noisy: the bound there is on the median, on 98 in 100 and on the worst, and only says that nothing is
# lost (single positions whose routing is a close call choose another expert); edges and states are
# pinned by the 32-bit runs of the same code.
TOL = {"float32": 5e-5}
WORST = 20
BF16_MEDIAN, BF16_MOST, BF16_WORST = 0.06, 0.3, 2.0
LENGTHS = {"A": [1, 2, 3, 17, 49, 130, 211], "B": [5, 129, 321, 16], "C": [1, 9, 40, 63, 150], "D": [1, 65, 200]}


def dev(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device=DEV)


def i32(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def f64(t):
    return t.float().cpu().numpy().astype(np.float64)


def cuts(lens, sizes):
    """Steps of portions of several requests side by side: [[(request, from, to)]]."""
    done, k, out = [0] * len(lens), 0, []
    while any(d < n for d, n in zip(done, lens)):
        step = []
        for r, n in enumerate(lens):
            take = min(sizes[(k + r) % len(sizes)], n - done[r])
            if take > 0:
                step.append((r, done[r], done[r] + take))
                done[r] += take
        k += 1
        out.append(step)
    return out


def step_arrays(step, slots):
    n = [hi - lo for _, lo, hi in step]
    return i32(np.repeat(np.arange(len(step)), n)), i32(np.concatenate([[0], np.cumsum(n)])), i32([slots[r] for r, _, _ in step])


def rows_of(step, data):
    return dev(np.concatenate([data[r][lo:hi] for r, lo, hi in step]))


# ---------------------------------------------------------------------------- residual streams
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("S,E", [(1, 64), (2, 50), (3, 128), (4, 772), (5, 36), (7, 7), (11, 260), (4, 2080)])
def test_streams_are_read_written_and_summed(S, E, dtype):
    """The first read of copies, writes with the next read behind them in place, and the last write with
    the sum for some rows only."""
    from sglang_c_b200.csrc import ops
    rng = np.random.default_rng(S * 100 + E)
    T, eps = 9, 1e-5
    x0 = rng.standard_normal((T, E)) * 3
    X = np.stack([x0] * S)
    src = dev(x0).unsqueeze(1).expand(T, S, E)
    buf, h = torch.zeros((T, S, E), device=DEV), torch.zeros((T, E), dtype=dtype, device=DEV)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    gain = 1.0 + 0.3 * rng.standard_normal(E)
    weights = lambda: (rng.standard_normal(S), rng.standard_normal(S), rng.standard_normal((S, S)))
    w_in, w_out, w_mix = weights()
    ops.stream_step(src, h, dev(w_in), dev(gain), eps)
    want = P.rms_norm(P.streams_read(X, w_in), gain, eps)
    assert np.abs(f64(h) - want).max() < tol * np.abs(want).max()
    for _ in range(3):
        y = rng.standard_normal((T, E))
        n_in, n_out, n_mix = weights()
        X = P.streams_write(X, y, w_out, w_mix)
        ops.stream_step(src, h, dev(n_in), dev(gain), eps, write=(dev(y), dev(w_out), dev(w_mix), buf))
        src, w_out, w_mix = buf, n_out, n_mix
        want = P.rms_norm(P.streams_read(X, n_in), gain, eps)
        assert np.abs(f64(buf).transpose(1, 0, 2) - X).max() < 4e-6 * np.abs(X).max()
        assert np.abs(f64(h) - want).max() < 2 * tol * np.abs(want).max()
    y = rng.standard_normal((T, E))
    before, out = buf.clone(), torch.full((T, E), 5.0, device=DEV)
    ops.stream_step(src, out, torch.ones(S, device=DEV), write=(dev(y), dev(w_out), dev(w_mix), None), rows=i32([7, 2]))
    want = P.streams_write(X, y, w_out, w_mix).sum(0)
    assert np.abs(f64(out)[[7, 2]] - want[[7, 2]]).max() < 8e-6 * np.abs(want).max()
    assert float((out[[0, 1, 3, 4, 5, 6, 8]] - 5.0).abs().max()) == 0.0 and torch.equal(before, buf)


# ---------------------------------------------------------------------------- state space
@pytest.mark.parametrize("K", [1, 2, 3, 4, 6, 9])
@pytest.mark.parametrize("C,heads", [(132, 5), (57, 3), (1028, 40)])
def test_convolution_with_bias_and_step_sizes_in_portions(K, C, heads):
    """Requests side by side in shuffled slots, whole and in portions down to one token (portions shorter than
    the taps reach into what earlier ones left); the gates from the columns behind the channels."""
    from sglang_c_b200.csrc import ops
    rng = np.random.default_rng(C + K)
    lens, slots = [45, 1, 70, 12], [4, 0, 5, 2]
    A_log, dt_bias = rng.standard_normal(heads) * 0.5, rng.standard_normal(heads)
    taps, bias = rng.standard_normal((C, K)) * 0.5, rng.standard_normal(C)
    front = 4                                                # columns ahead of the channels (a gate's)
    data = [rng.standard_normal((n, front + C + heads + 3)) for n in lens]
    chan = [d[:, front:front + C] for d in data]
    want = [P.silu(P.short_convolution(u, taps, bias)) for u in chan]
    dts = [P.softplus(d[:, front + C:front + C + heads] + dt_bias) for d in data]
    for sizes in ((100,), (7, 2, 1, 3), (1,), (2, 40, 5)):
        tail = torch.zeros((7, K - 1, C), device=DEV)
        tail[[1, 3, 6]] = 9.0
        for step in cuts(lens, sizes):
            tr, qs, sl = step_arrays(step, slots)
            x = rows_of(step, data)
            T = x.shape[0]
            y, gates = torch.zeros((T, C), device=DEV), torch.zeros((T, 2 * heads), device=DEV)
            ops.conv_silu(x[:, front:front + C + heads], dev(taps.T.copy()), dev(bias), tail, y, tr, qs, sl, len(step),
                          gates=(heads, C, dev(A_log), dev(dt_bias), gates))
            w = np.concatenate([want[r][lo:hi] for r, lo, hi in step])
            dt = np.concatenate([dts[r][lo:hi] for r, lo, hi in step])
            assert np.abs(f64(y) - w).max() < 1e-5, (sizes, step)
            assert np.abs(f64(gates)[:, :heads] - dt).max() < 1e-5
            assert np.abs(f64(gates)[:, heads:] - np.exp(-np.exp(A_log) * dt)).max() < 1e-5
        for r, n in enumerate(lens):                          # the last K-1 inputs, zeros ahead of the first
            left = np.concatenate([np.zeros((K - 1, C)), chan[r]], 0)[n:]
            assert K == 1 or np.abs(f64(tail[slots[r]]) - left).max() < 1e-6
        assert K == 1 or float((tail[[1, 3, 6]] - 9.0).abs().max()) == 0.0


def _space_case(rng, n, H, G, N, V):
    """Steps small enough that the first tokens still count at the end, but for one large one now and then."""
    x, B, C = rng.standard_normal((n, H, V)), rng.standard_normal((n, G, N)), rng.standard_normal((n, G, N))
    dt = np.exp(rng.standard_normal((n, H)) * 0.7 - 5.0)
    x[0] *= 30.0
    return x, B, C, dt


@pytest.mark.parametrize("form", ["tokens", "chunks", "single"])
@pytest.mark.parametrize("H,G,N,V", [(4, 2, 24, 20), (3, 1, 7, 5), (2, 2, 128, 64), (2, 1, 160, 72), (6, 3, 64, 64), (1, 1, 256, 130),
                                     (8, 1, 16, 128)])
def test_state_space_in_portions_by_tokens_and_by_chunks(form, H, G, N, V):
    """The forms of the recurrence (and the one for single tokens behind the others): three requests of unequal lengths in shuffled slots, whole and in portions
    (down to one token, across chunks' borders), states carried through their slots; the first token,
    which is large, still shows at the end."""
    from sglang_c_b200.csrc import ops
    rng = np.random.default_rng(H * 1000 + N)
    lens, slots = [301, 1, 130], [4, 2, 5]
    A_log, D = rng.standard_normal(H) * 0.3, rng.standard_normal(H)
    cases = [_space_case(rng, n, H, G, N, V) for n in lens]
    want = [P.state_space(*c, A_log, D) for c in cases]
    x, B, C, dt = cases[0]
    lost = P.state_space(x[1:], B[1:], C[1:], dt[1:], A_log, D)[0]
    assert np.abs(lost[-1] - want[0][0][-1]).max() > 1e-2 * np.abs(want[0][0]).std()
    flat = [[c[0].reshape(n, -1) for c, n in zip(cases, lens)], [c[1].reshape(n, -1) for c, n in zip(cases, lens)],
            [c[2].reshape(n, -1) for c, n in zip(cases, lens)], [c[3] for c in cases]]
    for sizes in ((400,), (64, 128, 65), (63, 2, 1, 129)) if form != "single" else ((298, 1, 1, 1, 64, 1),):
        state = torch.zeros((6, H, N, V), device=DEV)
        state[[0, 1, 3]] = 7.0
        for step in cuts(lens, sizes):
            _, qs, sl = step_arrays(step, slots)
            xs, Bs, Cs, dts = (rows_of(step, f) for f in flat)
            T, R = xs.shape[0], len(step)
            gates = torch.cat([dts, torch.exp(-torch.exp(dev(A_log)) * dts)], 1).contiguous()
            out = torch.zeros((T, H * V), device=DEV)
            if T == R and form == "single":
                ops.state_step(Cs, Bs, xs, gates, out, state, sl, H, G, N, V, skip=dev(D))
            elif form != "chunks":
                ops.matrix_state("gated", Cs, Bs, xs, out, state, qs, sl, R, H, G, N, V, gates=gates, skip=dev(D))
            else:
                ws = torch.full((ops.state_chunks_workspace(T, R, H, G, N, V),), float("nan"), device=DEV)
                ops.state_chunks(Cs, Bs, xs, gates, dev(A_log), out, state, qs, sl, R, H, G, N, V, ws, skip=dev(D))
            w = np.concatenate([want[r][0][lo:hi].reshape(hi - lo, -1) for r, lo, hi in step])
            assert np.abs(f64(out) - w).max() < 2e-5 * np.abs(w).max() * math.sqrt(N), (sizes, step)
        for r in range(3):
            assert np.abs(f64(state[slots[r]]) - want[r][1]).max() < 1e-4 * np.abs(want[r][1]).max()
        assert float((state[[0, 1, 3]] - 7.0).abs().max()) == 0.0


def test_chunks_with_large_and_small_steps():
    """Sums of logarithms that run far down within a chunk: what follows them is as exact as without them."""
    from sglang_c_b200.csrc import ops
    rng = np.random.default_rng(9)
    n, H, N, V = 128, 2, 16, 16
    x, B, C = rng.standard_normal((n, H, V)), rng.standard_normal((n, 1, N)), rng.standard_normal((n, 1, N))
    dt = np.full((n, H), 1e-3)
    dt[10:40] = 60.0                                # thirty tokens that forget everything
    A_log = np.log(np.array([16.0, 3.0]))
    dt = dt.astype(np.float32).astype(np.float64)
    want = P.state_space(x, B, C, dt, A_log, np.zeros(H))[0]
    gates = torch.cat([dev(dt), torch.exp(-torch.exp(dev(A_log)) * dev(dt))], 1).contiguous()
    out, state = torch.zeros((n, H * V), device=DEV), torch.zeros((1, H, N, V), device=DEV)
    ws = torch.empty(ops.state_chunks_workspace(n, 1, H, 1, N, V), device=DEV)
    ops.state_chunks(dev(C.reshape(n, -1)), dev(B.reshape(n, -1)), dev(x.reshape(n, -1)), gates, dev(A_log), out, state,
                     i32([0, n]), i32([0]), 1, H, 1, N, V, ws)
    err = np.abs(f64(out).reshape(n, H, V) - want)
    assert np.isfinite(err).all()
    for lo, hi in ((0, 10), (10, 40), (45, 64), (64, 128)):
        assert err[lo:hi].max() < 2e-5 * np.abs(want[lo:hi]).max(), (lo, hi)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups,width", [(1, 64), (5, 24), (3, 5), (2, 1536), (6, 6)])
@pytest.mark.parametrize("act", ["silu", "sigmoid"])
def test_gate_ahead_of_a_norm_in_groups(groups, width, dtype, act):
    from sglang_c_b200.csrc import ops
    rng = np.random.default_rng(groups * width)
    W = groups * width
    o, z = rng.standard_normal((7, W)) * np.linspace(0.01, 20.0, W), rng.standard_normal((7, W + 3)) * 2
    gain = 1.0 + 0.3 * rng.standard_normal(W)
    fn = P.silu if act == "silu" else P.sigmoid
    want = P.group_rms_norm(o * fn(z[:, :W]), gain, 1e-5, groups)
    y = torch.zeros((7, W), dtype=dtype, device=DEV)
    ops.gate_then_norm(dev(o), dev(z)[:, :W], dev(gain), y, groups, width, 1e-5, act)
    assert np.abs(f64(y) - want).max() < (1e-5 if dtype == torch.float32 else 1e-2) * np.abs(want).max()
    assert np.abs(P.group_rms_norm(o, gain, 1e-5, groups) * fn(z[:, :W]) - want).max() > 0.1      # not the other order


# ---------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("F,dtype", [(33, torch.float32), (64, torch.bfloat16), (40, torch.float32)])
@pytest.mark.parametrize("limit,slope,mult", [(0.7, 1.702, 1.0), (3.0, 0.9, 0.5)])
def test_bounded_gate(F, dtype, limit, slope, mult):
    from sglang_c_b200.csrc import ops
    rng = np.random.default_rng(F)
    gu = torch.tensor(rng.standard_normal((9, 2 * F)) * 2.5, dtype=dtype, device=DEV)
    gu[0, :4] = torch.tensor([-200.0, 200.0, limit, -limit])
    z = torch.zeros((9, F), dtype=dtype, device=DEV)
    ops.gated_act(gu, z, act="clamped", slope=slope, limit=limit, mult=mult)
    g, u = f64(gu)[:, :F], f64(gu)[:, F:]
    gb, ub = np.minimum(g, limit), np.clip(u, -limit, limit)
    want = gb / (1.0 + np.exp(np.minimum(-slope * gb, 600.0))) * (ub + 1.0) * mult
    if slope == 1.702 and mult == 1.0:
        assert np.abs(want - P.clamped_gate(g, u, limit)).max() < 1e-12
    assert np.abs(f64(z) - want).max() < (2e-6 if dtype == torch.float32 else 1e-2) * np.abs(want).max()


# ---------------------------------------------------------------------------- attention
def _standing_out(rng, n, H, G, D, V, key_at, strength=3.5):
    """Small queries and keys but for the last query and the key at `key_at`, whose score is strength^2."""
    q, k, v = rng.standard_normal((n, H, D)) * 0.1, rng.standard_normal((n, G, D)) * 0.1, rng.standard_normal((n, G, V))
    d = rng.standard_normal(D)
    d /= np.linalg.norm(d)
    q[-1], k[key_at] = strength * d, strength * d
    return q, k, v


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,V,page", [(6, 2, 32, 20, 16), (2, 1, 64, 64, 16), (3, 1, 10, 6, 8), (16, 1, 64, 64, 16)])
def test_a_constant_in_the_softmax_and_keys_far_back(dtype, H, G, D, V, page):
    """One key carries nearly all the weight of the last query: the first of all, at a page's border on either
    side, in the last portion.  The prompt whole, as a last portion, and the last token alone."""
    from sglang_c_b200.csrc import ops
    rng = np.random.default_rng(D + H)
    n = 391
    for at in (0, n // 2 // page * page, n // 2 // page * page - 1, n - 3):
        q, k, v = _standing_out(rng, n, H, G, D, V, at)
        if dtype == torch.bfloat16:
            q, k, v = (f64(dev(a, dtype)) for a in (q, k, v))
        want = P.softmax_attention(q, k, v, 1.0)
        assert np.abs(want[-1, 0] - v[at, 0]).max() < 0.5           # the key carries the query
        s0 = np.exp((q[0] * k[0].repeat(H // G, 0)).sum(-1, keepdims=True))
        assert np.abs(want[0] - v[0].repeat(H // G, 0) * s0 / (1.0 + s0)).max() < 1e-12     # one key beside the constant
        n_pages = (n + page - 1) // page + 3
        table = rng.permutation(n_pages)[:(n + page - 1) // page]
        pages = np.zeros((n_pages, G * page * (D + V)))
        for t in range(n):
            pg, off = table[t // page], t % page
            pages[pg, :G * page * D].reshape(G, page, D)[:, off] = k[t]
            pages[pg, G * page * D:].reshape(G, page, V)[:, off] = v[t]
        cache, qd, one = dev(pages, dtype), dev(q.reshape(n, -1), dtype), torch.zeros(H, device=DEV)
        tol = 1e-4 if dtype == torch.float32 else 2e-2
        for lo, hi in ((0, n), (n - 70, n), (n - 2, n), (n - 1, n)):
            T = hi - lo
            splits = ops.attention_ext_splits(hi, None, None, G) if T == 1 else 1
            ws = torch.empty(T * H * splits * (V + 2), device=DEV) if splits > 1 else None
            out = torch.zeros((T, H * V), dtype=dtype, device=DEV)
            ops.attention_ext(qd[lo:hi], cache, i32(table[None, :]), i32([0] * T), i32(np.arange(lo, hi)), out, H, G, D, V, page,
                              1.0, None, None, one, hi, max_q_len=T, splits=splits, workspace=ws)
            assert np.abs(f64(out).reshape(T, H, V) - want[lo:hi]).max() < tol, (at, lo)
            if dtype == torch.bfloat16 and D == V == 64 and T > 1:
                o = torch.zeros((T, H * V), dtype=dtype, device=DEV)
                ops.attention_prefill_tc(qd[lo:hi], cache.view(n_pages, 2, G, page, D), i32(table[None, :]), i32([0, T]), i32([n]),
                                         o, H, 1.0, None, 1, T, sinks=one)
                assert np.abs(f64(o).reshape(T, H, V) - want[lo:hi]).max() < tol, (at, lo)


# ---------------------------------------------------------------------------- whole models
def requests_for(name):
    V = ZAD[name]["vocab"]
    return {f"r{i}": traces.random_tokens(7 * i + ord(name), n, V) for i, n in enumerate(LENGTHS[name])}


_ref = {}


def forward_dir(model_dir, toks):
    key = (model_dir, tuple(toks))
    if key not in _ref:
        cfg, w = P.read_model_dir(model_dir)
        _ref[key] = P.forward(cfg, w, toks)
    return _ref[key]


def reference(model_dir, requests):
    return {rid: forward_dir(model_dir, toks) for rid, toks in requests.items()}


def check_errors(got, ref, dtype, what, factor=1.0):
    """Every produced position's largest difference over the vocabulary, against the logits' size."""
    traces.max_error(got, ref)                     # (checks that every position was produced)
    size = float(np.concatenate([r.ravel() for r in ref.values()]).std())
    e = np.array([np.abs(got[rid][p].astype(np.float64) - ref[rid][p]).max() / size for rid in ref for p in sorted(got[rid])])
    assert np.isfinite(e).all(), what
    if dtype == "float32":
        tol = factor * TOL[dtype]
        assert np.quantile(e, 0.98) < tol and e.max() < WORST * TOL[dtype], \
            f"{what}: 98 in 100 under {np.quantile(e, 0.98)} of the logits' size, worst {e.max()} at position {e.argmax()}"
    else:
        assert np.median(e) < BF16_MEDIAN and np.quantile(e, 0.98) < BF16_MOST and e.max() < BF16_WORST, \
            f"{what}: errors of the logits' size: median {np.median(e)}, 98 in 100 under {np.quantile(e, 0.98)}, worst {e.max()}"


def run_trace(model_dir, dtype, name, steps, tmp_path, max_tokens=None, max_step_tokens=1024, max_requests=4):
    from sglang_c_b200.engine import Engine
    from sglang_c_b200.engine.replay import replay
    ps = PAGE[name]
    n_pages = (max_tokens or traces.peak_tokens(steps)) // ps
    eng = Engine.from_dir(model_dir, dtype=dtype, page_size=ps, n_pages=n_pages, max_requests=max_requests,
                          max_step_tokens=max_step_tokens)
    out = str(tmp_path / "out")
    done = []
    replay(eng, traces.to_lines(steps), out, emit=done.append)
    assert done == [f"done {st['step']}" for st in steps]
    eng.cache.check()
    assert eng.cache.n_free_pages() == n_pages and eng.cache.n_free_slots() == max_requests
    return traces.collect(steps, out, ZAD[name]["vocab"]), eng


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    base = tmp_path_factory.mktemp("zadunex")
    return lambda name, store="float32", sharp=False: (make_sharp_dir if sharp else make_dir)(base, name, store)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
@pytest.mark.parametrize("mode", ["whole", "tail", "portions"])
def test_each_request_alone(dirs, tmp_path, name, dtype, mode):
    d = dirs(name, dtype)
    reqs = requests_for(name)
    steps = {"whole": traces.whole, "tail": traces.tail_decoded, "portions": traces.portions}[mode](reqs)
    got, _ = run_trace(d, dtype, name, steps, tmp_path)
    check_errors(got, reference(d, reqs), dtype, mode)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_mixed_batches_with_pages_and_slots_used_again(dirs, tmp_path, name, dtype):
    d = dirs(name, dtype)
    V = ZAD[name]["vocab"]
    lens = [37, 64, 150, 21, 128, 55, 33, 131, 48]
    reqs = {f"m{i}": traces.random_tokens(2000 + i, n, V) for i, n in enumerate(lens)}
    prompt_len = {rid: max(1, len(t) - 20 - 3 * i) for i, (rid, t) in enumerate(reqs.items())}
    steps = traces.mixed(reqs, prompt_len, seed=5, max_live=3, sizes=(5, 2, 11, 3, 140, 2, 8))
    peak = traces.peak_tokens(steps)
    assert peak < sum((n + 63) // 64 * 64 for n in lens)
    got, eng = run_trace(d, dtype, name, steps, tmp_path, max_tokens=peak, max_requests=3)
    check_errors(got, reference(d, reqs), dtype, "mixed")


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_sharp_model_in_every_cut(dirs, tmp_path, name, dtype="float32"):
    """Keys that carry weight and states that remember: first what the change does to the plain logits (tokens
    changed far back must move the last logits), then every cut.  (32-bit only: with scores this large the
    rounding of bfloat16 queries and keys moves the logits as much as a lost key.)"""
    d = dirs(name, sharp=True)
    V = ZAD[name]["vocab"]
    reqs = {f"s{i}": traces.random_tokens(900 + i, n, V) for i, n in enumerate([200, 45, 131])}
    ref = reference(d, reqs)
    toks = list(reqs["s0"])
    toks[3:30] = [(t + 1) % V for t in toks[3:30]]
    moved = np.abs(forward_dir(d, toks)[-50:] - ref["s0"][-50:]).max()
    size = float(ref["s0"].std())
    assert moved > 40 * TOL["float32"] * size, moved / size
    prompt_len = {"s0": 150, "s1": 20, "s2": 129}
    for steps in (traces.whole(reqs), traces.tail_decoded(reqs, 40), traces.portions(reqs, sizes=(2, 127, 3, 2, 64, 23)),
                  traces.mixed(reqs, prompt_len, seed=2, sizes=(130, 2, 16, 3))):
        got, _ = run_trace(d, dtype, name, steps, tmp_path)
        check_errors(got, ref, dtype, "sharp", factor=4.0)


def test_mixed_results_do_not_depend_on_the_batch_in_32_bit(dirs, tmp_path):
    d = dirs("A")
    V = ZAD["A"]["vocab"]
    reqs = {f"q{i}": traces.random_tokens(500 + i, n, V) for i, n in enumerate([90, 33, 140, 7])}
    prompt_len = {rid: len(t) - 5 for rid, t in reqs.items()}
    mixed, _ = run_trace(d, "float32", "A", traces.mixed(reqs, prompt_len, seed=9), tmp_path)
    alone, _ = run_trace(d, "float32", "A", traces.whole(reqs), tmp_path)
    size = float(reference(d, reqs)["q2"].std())
    for rid in reqs:
        for p in alone[rid]:
            assert np.abs(mixed[rid][p] - alone[rid][p]).max() < 3e-5 * size


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_long_decoding_replays_graphs(dirs, tmp_path, name, dtype):
    """240 tokens one by one for two requests."""
    d = dirs(name, dtype)
    V = ZAD[name]["vocab"]
    reqs = {"long": traces.random_tokens(31, 300, V), "other": traces.random_tokens(32, 240, V)}
    steps = []
    for s in range(240):
        entries = []
        for rid, first in (("long", 60), ("other", 1)):
            if s == 0:
                entries.append({"id": rid, "tokens": reqs[rid][:first], "want": list(range(first))})
            elif first + s <= len(reqs[rid]):
                entries.append({"id": rid, "tokens": [reqs[rid][first + s - 1]], "want": [0]})
        steps.append({"step": s, "entries": entries, "end": []})
    steps[-1]["end"] = ["long", "other"]
    got, eng = run_trace(d, dtype, name, steps, tmp_path, max_tokens=640)
    ref = {"long": forward_dir(d, reqs["long"][:299]), "other": forward_dir(d, reqs["other"])}
    check_errors(got, ref, dtype, "long decoding")
    assert eng.graph_replays > 150, "steady decoding did not replay captured graphs"


def test_steps_whose_logits_nobody_wants(dirs, tmp_path):
    """Portions without a wanted place still move caches and states."""
    d = dirs("A")
    toks = traces.random_tokens(77, 100, ZAD["A"]["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:70], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[70:99], "want": [3]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[99:], "want": [0]}], "end": ["a"]}]
    got, _ = run_trace(d, "float32", "A", steps, tmp_path)
    ref = forward_dir(d, toks)
    assert sorted(got["a"]) == [73, 99]
    for p in (73, 99):
        assert np.abs(got["a"][p] - ref[p]).max() < TOL["float32"] * ref.std()


def check_greedy(model_dir, prompt, got, tie):
    cfg, w = P.read_model_dir(model_dir)
    seq = list(prompt)
    for t in got:
        lg = P.forward(cfg, w, seq)[-1]
        best = int(np.argmax(lg))
        assert t == best or lg[best] - lg[t] < tie * lg.std(), (t, best, float(lg[best] - lg[t]))
        seq.append(t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_scheduler(dirs, name, dtype):
    """The entry point a user calls: prompts of unequal lengths in one batch, prompt portions of 24
    tokens, few pages (so requests wait for pages and slots that others give back)."""
    from sglang_c_b200.engine import generate, sched_new
    from sglang_c_b200.sampling import SamplingParams
    d = dirs(name, dtype)
    V = ZAD[name]["vocab"]
    prompts = [traces.random_tokens(70 + i, n, V) for i, n in enumerate([5, 40, 1, 63, 100, 17])]
    s = sched_new(d, dtype=dtype, page_size=PAGE[name], max_tokens=384, max_requests=3, max_step_tokens=64,
                  prefill_chunk=24)
    got = generate(s, prompts, SamplingParams(temperature=0.0), max_new=10)
    for p, g in zip(prompts, got):
        assert len(g) == 10
        check_greedy(d, p, g, 2e-4 if dtype == "float32" else 0.5)
    st = s.get_stats()
    assert st.n_finished == len(prompts) and st.pool_free == st.pool_pages


def test_command_line_generates_from_a_random_folder(tmp_path):
    """bin/sglc: a random folder written from a config.json, then greedy generation from it."""
    import json
    import os
    import subprocess
    import sys
    from conftest import ROOT
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(ZAD["C"]))
    d = str(tmp_path / "model")
    prompt = [5, 17, 3, 99, 42]
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "sglc"), "--random-weights", "11", "--config", str(cfg),
                           "--init", "varied", "--save-model", d, "--dtype", "float32", "--prompt",
                           " ".join(map(str, prompt)), "--max-new", "8", "--temperature", "0", "--page-size", "8"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    ids = [int(t) for t in proc.stdout.strip().splitlines()[-1].split()]
    assert ids[:len(prompt)] == prompt and len(ids) == len(prompt) + 8
    check_greedy(d, prompt, ids[len(prompt):], 1e-4)
