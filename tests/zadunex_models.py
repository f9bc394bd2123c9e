"""Small Zadunex configurations for the tests, random model folders for them, and "sharp" variants whose
constants and weights are changed so that a lost key, a lost state, a dropped constant of the softmax or a
stream that is read or written in the wrong order shows in the logits."""
import copy
import json
import os

import numpy as np
import torch


def _ssm(mlp, heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                                    "conv": conv, "norm_groups": norm_groups}}


def _attn(mlp, heads, kv_heads, dim, vdim, scale, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


# A: every kind of layer; three streams; a loop in the middle that holds both mixers; value sizes that
# differ from the key sizes; partial rotation; a layer of each mixer without a feed-forward
ZAD_A = {"architecture": "Zadunex", "vocab": 300, "width": 64, "streams": 3, "norm": {"eps": 1e-5}, "logit_scale": 1.75,
         "loop": {"start": 1, "stop": 3, "times": 2},
         "layers": [_ssm(_moe(6, 3, 40), 6, 20, 24, 3, 4, 5), _attn(_dense(72, 0.8), 6, 2, 32, 20, 0.3, (5000.0, 12)),
                    _ssm(None, 4, 16, 40, 1, 2, 1), _attn(None, 4, 4, 16, 24, 0.2, (100.0, 16)),
                    _ssm(_dense(48, 0.5), 2, 36, 16, 2, 3, 4)]}
# B: sizes the tensor-core kernels take (heads of 64 on both sides); two streams; the last layer repeats; a
# state of 128 rows and one of 160 (two row tiles); value rows of two column tiles
ZAD_B = {"architecture": "Zadunex", "vocab": 257, "width": 96, "streams": 2, "norm": {"eps": 1e-6}, "logit_scale": 0.6,
         "loop": {"start": 3, "stop": 4, "times": 3},
         "layers": [_attn(_moe(4, 1, 32), 6, 3, 64, 64, 0.125, (10000.0, 64)), _ssm(_dense(64, 1.2), 2, 72, 128, 2, 4, 2),
                    _attn(_dense(40, 2.5), 5, 1, 64, 64, 0.1, (300.0, 24)), _ssm(_moe(3, 2, 24), 4, 64, 160, 1, 3, 4)]}
# C: sizes that no vector load and no tensor-core tile fits; five streams; one tap and six; one head a
# group and one group for all; all experts chosen; no rotation; no loop
ZAD_C = {"architecture": "Zadunex", "vocab": 101, "width": 50, "streams": 5, "norm": {"eps": 1e-5}, "logit_scale": 1.0,
         "layers": [_ssm(_moe(3, 3, 11), 3, 5, 7, 3, 6, 3), _attn(_moe(5, 2, 9), 3, 1, 10, 6, 0.5),
                    _ssm(_dense(13, 0.3), 4, 9, 10, 1, 1, 6), _attn(_dense(21, 1.0), 6, 3, 6, 10, 0.6, (50.0, 2))]}
# D: one stream (the combinations are numbers), one layer run twice
ZAD_D = {"architecture": "Zadunex", "vocab": 61, "width": 32, "streams": 1, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
         "loop": {"start": 0, "stop": 1, "times": 2}, "layers": [_ssm(_dense(40, 1.0), 2, 16, 8, 1, 4, 1)]}
ZAD = {"A": ZAD_A, "B": ZAD_B, "C": ZAD_C, "D": ZAD_D}
SEED = {"A": 710, "B": 707, "C": 701, "D": 768}
PAGE = {"A": 16, "B": 16, "C": 8, "D": 4}


def _rewrite(src, out, store_dtype, change, cfg_change=None):
    """The folder `src` (32-bit) written again as `out` with change(name, array) applied to every tensor."""
    import plain_zadunex
    from sglang_c_b200.weights.safetensors_io import write_safetensors
    cfg, w = plain_zadunex.read_model_dir(src)
    cfg = copy.deepcopy(cfg)
    if cfg_change is not None:
        cfg_change(cfg)
    tensors = {}
    for k, v in w.items():
        t = torch.from_numpy(np.ascontiguousarray(change(k, np.array(v, dtype=np.float32)), dtype=np.float32))
        tensors[k] = t.to(torch.bfloat16) if (store_dtype == "bfloat16" and t.dim() >= 2) else t
    os.makedirs(out, exist_ok=True)
    with open(os.path.join(out, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(out, "model.safetensors"), tensors, metadata={"format": "pt"})
    return out


def _lively(k, a):
    """Random weights of the usual small size leave much of this design without effect: sublayers that hardly
    move the streams, streams that stay copies of one another, bounds that nothing reaches, decays all alike,
    routers whose choices are all close calls.  So what decides how much a mechanism shows is spread out."""
    if k == "embed":
        return a * 50.0
    if k.endswith((".hc1.in", ".hc2.in", ".hc1.out", ".hc2.out")):
        return 0.7 + (a - 1.0) * 3.5
    if k.endswith((".hc1.mix", ".hc2.mix")):
        return a * 0.8
    if k.endswith(".mlp.router"):
        return a * 8.0
    if k.endswith(".mix.A_log"):
        return a * 40.0
    if k.endswith(".mix.dt_bias"):
        return a * 40.0 - 2.5
    if k.endswith(".mix.D"):
        return (a - 1.0) * 4.0
    if k.endswith((".q.b", ".k.b", ".v.b", ".conv.b")):
        return a * 20.0
    if k.endswith((".mlp.gate", ".mlp.up")):
        return a * 10.0
    if k.endswith((".mix.in", ".mix.o", ".down", ".up", ".gate", ".mix.v")):
        return a * 6.0
    return a


def make_dir(tmp, name, store_dtype="float32"):
    from sglang_c_b200.config import resolve_architecture
    from sglang_c_b200.weights import write_random_model
    d = ZAD[name]
    arch = resolve_architecture(d)
    out = os.path.join(str(tmp), f"zad_{name}_{store_dtype}")
    if not os.path.exists(os.path.join(out, "model.safetensors")):
        raw = write_random_model(out + "_raw", arch, arch.config_class.from_dict(d), SEED[name], scheme="varied",
                                 store_dtype="float32")
        _rewrite(raw, out, store_dtype, _lively)
    return out


def make_sharp_dir(tmp, name, store_dtype="float32"):
    """The model `name` with attention scores several times as large (queries and keys are normed, so the
    config's multiplier is what sharpens the softmax) and states that remember: small steps, so that the
    decays are close to one, and no share of the token's own value to drown what they recall."""
    base = make_dir(tmp, name, "float32")
    out = os.path.join(str(tmp), f"zad_sharp_{name}_{store_dtype}")
    if os.path.exists(os.path.join(out, "model.safetensors")):
        return out

    def sharper(cfg):
        for entry in cfg["layers"]:
            if entry["type"] == "attention":
                entry["mixer"]["scale"] *= 5.0

    def change(k, a):
        if k.endswith(".mix.dt_bias"):
            return a - 3.5
        if k.endswith(".mix.D"):
            return a * 0.05
        return a
    return _rewrite(base, out, store_dtype, change, sharper)
