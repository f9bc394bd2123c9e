"""Small Fupapel configurations for the tests, random model folders for them, and "sharp" variants
whose constants and weights are changed so that a lost key, a chunk edge that is one token off, a
dropped sink or a lost state shows in the logits."""
import copy
import json
import os

import numpy as np
import torch


def _rot(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def _mixer(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None, **more):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = rot
    m.update(more)
    return m


def _gated(mlp, *a, **k):
    return {"type": "attention", "mixer": _mixer(*a, **k), "mlp": mlp}


def _conv(mlp, *a, **k):
    return {"type": "attention_2", "mixer": _mixer(*a, **k), "mlp": mlp}


def _latent(mlp, heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": scale, "rot": _rot(base, rot_dim)}}


def _moe(experts, top, ff, identity=0, groups=None):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


# A: every kind of layer; a chunk that is no multiple of a page; keys and values read from an earlier
# layer by one with a wider chunk, with other layers in between; partial rotations; value sizes that
# differ from the key sizes; identity experts in the last group only; a layer without feed-forward
FUP_A = {"architecture": "Fupapel", "vocab": 300, "width": 64, "norm": {"eps": 1e-6}, "residual_mult": 0.45,
         "layers": [
             _conv(_moe(6, 3, 40, 3, (3, 2)), 4, 2, 32, 16, 0.2, 24, _rot(10000.0, 16, (6.0, 1.0, 5.0, 128)), conv=3),
             _latent(_moe(5, 2, 24, 1, (2, 1)), 4, 24, 16, 20, 40, 24, 0.17, 3000.0),
             _gated(None, 4, 2, 24, 16, 0.25, 20, _rot(500.0, 12)),
             _conv(_moe(8, 1, 16, 4, (4, 1)), 4, 2, 32, 16, 0.3, 36, _rot(10000.0, 16, (6.0, 1.0, 5.0, 128)), conv=3,
                   kv_from=0),
             _latent(None, 2, 40, 8, 12, 24, 56, 0.2, 100.0)]}
# B: sizes the tensor-core kernels take (heads of 64 on both sides, a cached latent row of 128 and one of
# 64), a chunk of several pages, no chunk, full rotations with and without scaling, a reader with a chunk
# of a layer without one; a residual multiplier of one; no groups
FUP_B = {"architecture": "Fupapel", "vocab": 257, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 1.0,
         "layers": [
             _gated(_moe(4, 2, 32, 2), 2, 1, 64, 64, 0.125, 128, _rot(500000.0, 64)),
             _latent(_moe(6, 1, 64), 3, 64, 32, 64, 96, 40, 0.1, 10000.0),
             _conv(_moe(4, 4, 24, 0, (2, 2)), 2, 2, 64, 64, 0.125, None, _rot(20.0, 64), conv=4),
             _latent(_moe(2, 1, 48, 4, (3, 1)), 2, 32, 16, 48, 48, 24, 0.14, 77.0),
             _conv(_moe(3, 2, 32, 1), 2, 2, 64, 64, 0.15, 160, _rot(20.0, 64), conv=4, kv_from=2)]}
# C: sizes that no vector load and no tensor-core tile fits; a chunk shorter than a page; one head over a
# tiny latent; one tap, and readers with other numbers of taps than their source; all experts chosen; no
# rotation; a multiplier above one
FUP_C = {"architecture": "Fupapel", "vocab": 101, "width": 50, "norm": {"eps": 1e-5}, "residual_mult": 2.5,
         "layers": [
             _conv(_moe(3, 5, 11, 2), 3, 1, 10, 6, 0.4, 5, _rot(100.0, 6, (3.0, 0.5, 0.5, 10)), conv=2),
             _latent(_moe(2, 1, 7, 1), 1, 7, 2, 5, 9, 4, 0.5, 100.0),
             _gated(_moe(5, 2, 9, 0, (5, 3)), 6, 3, 10, 6, 0.4, 7),
             _conv(None, 3, 1, 10, 6, 0.3, 15, _rot(100.0, 6, (3.0, 0.5, 0.5, 10)), conv=5, kv_from=0),
             _conv(_moe(1, 1, 13, 1, (2, 1)), 3, 1, 10, 6, 0.3, 3, _rot(100.0, 6, (3.0, 0.5, 0.5, 10)), conv=1, kv_from=0)]}
FUP = {"A": FUP_A, "B": FUP_B, "C": FUP_C}
PAGE = {"A": 16, "B": 16, "C": 8}


def _rewrite(src, out, store_dtype, change, cfg_change=None):
    """The folder `src` (32-bit) written again as `out` with change(name, array) applied to every tensor."""
    import plain_fupapel
    from sglang_c_b200.weights.safetensors_io import write_safetensors
    cfg, w = plain_fupapel.read_model_dir(src)
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
    """Random weights of the usual small size leave much of this design without effect: sublayers that
    hardly move the stream, gates at one half, sinks at zero, factors at one, routers whose choices are
    all close calls.  So the tables and matrices that decide how much a mechanism shows are spread out."""
    if k == "embed":
        return a * 50.0
    if k.endswith(".mlp.router"):
        return a * 15.0
    if k.endswith(".correction"):
        return a * 8.0
    if k.endswith((".norm1", ".norm2")) or k == "final.norm":
        return (a - 1.0) * 2.0                       # stored around zero
    if k.endswith(".mix.temp"):
        return 1.0 + (a - 1.0) * 5.0
    if k.endswith(".mix.sink"):
        return a * 50.0
    if k.endswith((".mix.g", ".mix.uq", ".mix.uk")):
        return a * 8.0
    if k.endswith((".mix.o", ".down", ".up", ".gate", ".mix.v", ".mix.uv")):
        return a * 6.0
    return a


def make_dir(tmp, name, store_dtype="float32", seed=None):
    from sglang_c_b200.config import resolve_architecture
    from sglang_c_b200.weights import write_random_model
    d = FUP[name]
    arch = resolve_architecture(d)
    out = os.path.join(str(tmp), f"fup_{name}_{store_dtype}")
    if not os.path.exists(os.path.join(out, "model.safetensors")):
        raw = write_random_model(out + "_raw", arch, arch.config_class.from_dict(d),
                                 seed if seed is not None else 900 + ord(name), scheme="varied", store_dtype="float32")
        _rewrite(raw, out, store_dtype, _lively)
    return out


LATENT_SHARP = {"A": 6.0, "B": 6.0, "C": 25.0}


def make_sharp_dir(tmp, name, store_dtype="float32"):
    """The model `name` with attention scores several times as large (queries and keys are normed, so
    the config's multiplier is what sharpens the softmax: a key lost, misplaced, read from a stale page
    or let in across a chunk's edge then moves the logits by far more than rounding) and sinks raised so
    that they carry weight against such scores."""
    base = make_dir(tmp, name, "float32")
    out = os.path.join(str(tmp), f"fup_sharp_{name}_{store_dtype}")
    if os.path.exists(os.path.join(out, "model.safetensors")):
        return out

    def sharper(cfg):
        for entry in cfg["layers"]:
            entry["mixer"]["scale"] *= LATENT_SHARP[name] if entry["type"] == "latent_attention" else 5.0

    return _rewrite(base, out, store_dtype, lambda k, a: a + 1.5 if k.endswith(".mix.sink") else a, sharper)
