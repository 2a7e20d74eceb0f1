"""Model folders (config.json + model.safetensors): a writer, and seeded random models of the designs the library reads.

The reader is C++ (``csrc/safetensors.hpp``, ``csrc/layered_spec.hpp``); this module only makes folders, for tests and measurements.
"""
from __future__ import annotations

import json
import os
import struct

import numpy as np

ROW_LIMIT = 1 << 20  # values drawn per tensor; larger tensors repeat them from shifting offsets (measurements only)


def bf16_bits(a) -> np.ndarray:
    """float32 -> bfloat16 bit patterns, round to nearest even."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).reshape(np.shape(a))
    return np.asarray((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_floats(bits: np.ndarray) -> np.ndarray:
    return np.asarray(bits.astype(np.uint32) << 16).view(np.float32)


def write_safetensors(path: str, tensors: dict) -> None:
    """``tensors``: name -> float32 array (stored as F32) or uint16 array (bfloat16 bit patterns, stored as BF16)."""
    header, at = {}, 0
    for name, a in tensors.items():
        n = a.size * a.itemsize
        header[name] = {"dtype": {"float32": "F32", "uint16": "BF16"}[a.dtype.name], "shape": list(a.shape), "data_offsets": [at, at + n]}
        at += n
    raw = json.dumps(header).encode()
    raw += b" " * (-len(raw) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(raw)))
        f.write(raw)
        for a in tensors.values():
            np.ascontiguousarray(a).tofile(f)


def write_folder(path: str, config: dict, tensors: dict) -> str:
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(config, f)
    write_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return path


# ---- Lasosun -----------------------------------------------------------------------------------------------------------------------------
def mamba2(heads, vdim, state, groups=1, conv=4, norm_groups=1, ff=0) -> dict:
    return _layer("mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}, ff)


def hgrn2(heads, dim, vdim, ff=0) -> dict:
    return _layer("hgrn2", {"heads": heads, "dim": dim, "vdim": vdim}, ff)


def attention(heads, kv_heads, dim, vdim, window, pool, scale=None, ff=0) -> dict:
    return _layer("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                                "mask": {"size": window, "pool": pool}}, ff)


def _layer(kind: str, mixer: dict, ff: int) -> dict:
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def lasosun_config(layers, width, vocab, max_positions, eps=1e-6, embed_scale=1.0) -> dict:
    return {"architecture": "Lasosun", "width": width, "vocab": vocab, "max_positions": max_positions, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}


def lasosun_shapes(config: dict) -> dict:
    """Tensor name -> shape, in file order."""
    W = config["width"]
    out = {"embed": (config["vocab"], W), "pos": (config["max_positions"], W)}
    for i, l in enumerate(config["layers"]):
        p, m = f"l{i}.", l["mixer"]
        h, v = m["heads"], m["vdim"]
        out[p + "norm1"] = (W,)
        if l["mlp"]:
            out[p + "norm2"] = (W,)
        if l["type"] == "mamba2":
            inner, bc = h * v, 2 * m["groups"] * m["state"]
            out |= {p + "mix.in": (2 * inner + bc + h, W), p + "mix.conv": (inner + bc, m["conv"]), p + "mix.conv.b": (inner + bc,), p + "mix.dt_bias": (h,),
                    p + "mix.A_log": (h,), p + "mix.D": (h,), p + "mix.norm": (inner,)}
        elif l["type"] == "hgrn2":
            hd = h * m["dim"]
            out |= {p + "mix.q": (hd, W), p + "mix.f": (hd, W), p + "mix.f.b": (hd,), p + "mix.lower": (hd,), p + "mix.v": (h * v, W), p + "mix.norm": (v,)}
        else:
            g = m["kv_heads"]
            out |= {p + "mix.q": (h * m["dim"], W), p + "mix.k": (g * m["dim"], W), p + "mix.v": (g * v, W), p + "mix.g": (h, W)}
        out[p + "mix.o"] = (W, h * v)
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            out |= {p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)}
        for k in "12" if l["mlp"] else "1":
            out |= {p + f"rg{k}": (W, W), p + f"rg{k}.b": (W,)}
    out["final.norm"] = (W,)
    return out


def random_lasosun(config: dict, seed: int) -> dict:
    """Seeded bfloat16 weights (bit patterns): matrices with unit output variance for unit inputs, gates and decays spread over their range."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in lasosun_shapes(config).items():
        leaf = name.split(".", 1)[1] if name[0] == "l" and "." in name else name
        n = int(np.prod(shape))
        if leaf in ("norm1", "norm2", "mix.norm", "norm", "final.norm"):
            a = rng.uniform(0.7, 1.3, n)
        elif leaf == "mix.A_log":
            a = rng.uniform(-4.0, 1.0, n)
        elif leaf == "mix.dt_bias":
            a = rng.uniform(-3.0, 0.5, n)
        elif leaf == "mix.lower":
            a = rng.uniform(0.0, 0.95, n)
        elif leaf == "mix.f.b":
            a = rng.uniform(-1.0, 4.0, n)
        elif leaf in ("mix.D", "mix.conv.b", "rg1.b", "rg2.b"):
            a = rng.normal(0, 0.5, n)
        elif leaf == "mix.conv":
            a = rng.normal(0, shape[1] ** -0.5, n)
        elif leaf in ("embed", "pos"):
            a = rng.normal(0, 1.0 if leaf == "embed" else 0.3, min(n, ROW_LIMIT))
        else:
            a = rng.normal(0, shape[1] ** -0.5, min(n, ROW_LIMIT))
        bits = bf16_bits(a)
        if bits.size < n:
            bits = np.resize(bits, n)
        out[name] = bits.reshape(shape)
    return out


# ---- Tosevik -----------------------------------------------------------------------------------------------------------------------------
def retention(heads, dim, vdim, decay=None, rot=None, base=10000.0) -> dict:
    """decay: one number per head (default: memories of 32 tokens and up); rot: rotated dimensions (default: all)."""
    decay = [1.0 - 2.0 ** -(5 + 5 * h / max(heads - 1, 1)) for h in range(heads)] if decay is None else list(decay)
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"dims": dim if rot is None else rot, "base": base}}


def logistic(heads, kv_heads, dim, vdim, coef=0.3, every=64, scale=None) -> dict:
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "q_temp": {"coef": coef, "every": every}}


def experts(count, top, ff, shared_ff, groups=1, keep=1, scale=1.0) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared_ff}, "router": {"experts": count, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}


def retention_layer(mixer: dict, mlp: dict | None = None) -> dict:
    return {"type": "retention", "mixer": mixer, "mlp": mlp}


def parallel_layer(left: dict, right: dict, mlp: dict | None = None) -> dict:
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def tosevik_config(layers, width, vocab, eps=1e-6) -> dict:
    return {"architecture": "Tosevik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def tosevik_shapes(config: dict) -> dict:
    """Tensor name -> shape, in file order."""
    W = config["width"]
    norm = lambda name: {name: (W,), name + ".b": (W,), name + ".alpha": ()}

    def ret(m, p):
        qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        return {p + "q": (qk, W), p + "k": (qk, W), p + "v": (v, W), p + "g": (v, W), p + "o": (W, v)}

    def swiglu(p, ff):
        return {p + "gate": (ff, W), p + "up": (ff, W), p + "down": (W, ff)}

    out = {"embed": (config["vocab"], W)} | norm("embed.norm")
    for i, l in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", l["mixer"], l["mlp"]
        out |= norm(p + "norm1") | (norm(p + "norm2") if mlp else {})
        if l["type"] == "retention":
            out |= ret(m, p + "mix.")
        else:
            a = m["left"]
            q, k, v = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
            x = p + "mix.left."
            out |= {x + "q": (q, W), x + "k": (k, W), x + "v": (v, W), x + "q.norm": (q,), x + "k.norm": (k,), x + "pb": (a["heads"],), x + "o": (W, a["heads"] * a["vdim"])}
            out |= ret(m["right"], p + "mix.right.") | {x + "out": (W,), p + "mix.right.out": (W,)}
        if mlp:
            for e in range(mlp["router"]["experts"]):
                out |= swiglu(p + f"mlp.e{e}.", mlp["expert"]["ff"])
            out |= {p + "mlp.router": (mlp["router"]["experts"], W)} | swiglu(p + "mlp.shared.", mlp["shared"]["ff"]) | {p + "mlp.shared.sg": (1, W)}
        out[p + "dwa"] = (i + 2,)
    return out | norm("final.norm") | {"head": (config["vocab"], W)}


def random_tosevik(config: dict, seed: int) -> dict:
    """Seeded bfloat16 weights (bit patterns): matrices with unit output variance for unit inputs; averages over depth that add up to one."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tosevik_shapes(config).items():
        leaf, n = name.rsplit(".", 1)[-1], int(np.prod(shape))
        if leaf == "alpha":
            a = rng.uniform(0.4, 0.9, n)
        elif leaf == "b":
            a = rng.normal(0, 0.1, n)
        elif leaf in ("norm", "norm1", "norm2", "out"):
            a = rng.uniform(0.7, 1.3, n)
        elif leaf == "pb":
            a = rng.normal(-3.0, 0.5, n)
        elif leaf == "dwa":
            a = rng.normal(0, 0.3, n)
            a[-1] = 1.0 - a[:-1].sum()
        elif leaf == "embed":
            a = rng.normal(0, 1.0, min(n, ROW_LIMIT))
        elif leaf == "router":
            a = rng.normal(0, 2.0 * shape[1] ** -0.5, min(n, ROW_LIMIT))
        else:
            a = rng.normal(0, shape[1] ** -0.5, min(n, ROW_LIMIT))
        bits = bf16_bits(a)
        out[name] = (np.resize(bits, n) if bits.size < n else bits).reshape(shape)
    return out
