"""Configuration and seeded synthetic weights of the Zozonex design.

A decoder whose config.json lists its layers one by one: gated delta-rule mixers and sliding-window attention with a softmax
sink (some layers reading the keys and values of an earlier one), a norm on every sublayer's output, squared-ReLU
feed-forwards, scaled embeddings with sinusoidal positions and a tied head.
"""
from __future__ import annotations

import json
import zlib
from typing import Iterator, List, Tuple

import numpy as np

ARCHITECTURE = "Zozonex"


class ZozonexConfig:
    """The parsed config.json with the attribute names the session code asks every config for."""

    def __init__(self, raw: dict, max_seq_len: int = 2048):
        self.raw = raw
        self.vocab_size = int(raw["vocab"])
        self.d_model = int(raw["width"])
        self.n_layers = len(raw["layers"])
        self.max_seq_len = max_seq_len
        self.byte_level = False

    def to_json(self) -> str:
        return json.dumps(self.raw)

    @staticmethod
    def from_json(text: str) -> "ZozonexConfig":
        return ZozonexConfig(json.loads(text))


def delta(heads: int, dim: int, vdim: int, kv_heads: int = 0, conv: int = 4, ff: int = 0) -> dict:
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads or heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention(heads: int, dim: int, window: int, vdim: int = 0, kv_heads: int = 0, ff: int = 0, kv_from=None, scale=None) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads or heads, "dim": dim, "vdim": vdim or dim, "mask": {"size": window},
         "scale": float(scale if scale is not None else dim ** -0.5)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width: int, vocab: int, layers: List[dict], eps: float = 1e-5, embed_scale: float = 1.0, max_seq_len: int = 2048) -> ZozonexConfig:
    return ZozonexConfig({"architecture": ARCHITECTURE, "width": width, "vocab": vocab, "norm": {"eps": eps},
                          "embedding": {"scale": embed_scale}, "layers": layers}, max_seq_len)


def tensor_specs(cfg: ZozonexConfig) -> List[Tuple[str, Tuple[int, ...], str]]:
    """(name, shape, kind) of every tensor."""
    D = cfg.d_model
    out: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (cfg.vocab_size, D), "embed")]
    for i, L in enumerate(cfg.raw["layers"]):
        p, m = "l%d." % i, L["mixer"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.append((p + "norm1", (D,), "norm"))
        if L.get("mlp"):
            out += [(p + "norm2", (D,), "norm"), (p + "mlp.up", (L["mlp"]["ff"], D), "matrix"), (p + "mlp.down", (D, L["mlp"]["ff"]), "matrix")]
        if L["type"] == "delta":
            for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                out += [(p + "mix." + n, (rows, D), "matrix"), (p + "mix." + n + ".conv", (rows, m["conv"]), "conv")]
            out += [(p + "mix.b", (H, D), "matrix"), (p + "mix.a", (H, D), "matrix"), (p + "mix.A_log", (H,), "a_log"),
                    (p + "mix.dt_bias", (H,), "dt_bias"), (p + "mix.norm", (dv,), "weight"), (p + "mix.g", (H * dv, D), "matrix")]
        else:
            out.append((p + "mix.q", (H * dk, D), "matrix"))
            if m.get("kv_from") is None:
                out += [(p + "mix.k", (G * dk, D), "matrix"), (p + "mix.v", (G * dv, D), "matrix")]
        out.append((p + "mix.o", (D, H * dv), "matrix"))
    out.append(("final.norm", (D,), "norm"))
    return out


def iter_tensors(cfg: ZozonexConfig, seed: int = 0, weights_dtype: str = "bf16") -> Iterator[Tuple[str, int, np.ndarray]]:
    """(name, dtype code, array) with seeded random values of a sensible size; bf16 tensors as uint16 bit patterns.  Values are
    rounded to bf16 in either case, so that an fp32 model holds the same numbers."""
    from . import synth
    for name, shape, kind in tensor_specs(cfg):
        g = np.random.Generator(np.random.Philox(key=[seed, zlib.crc32(name.encode())]))
        if kind == "a_log":
            a = g.uniform(-3.0, 2.0, shape)
        elif kind == "dt_bias":
            a = g.uniform(-4.0, 1.0, shape)
        else:
            a = g.standard_normal(shape, dtype=np.float32)
            if kind == "matrix":
                a *= shape[1] ** -0.5
            elif kind == "embed":
                a *= 0.3
            elif kind == "conv":
                a *= 0.6
            elif kind == "norm":
                a *= 0.2
            elif kind == "weight":
                a = 1.0 + 0.2 * a
        bits = synth.f32_to_bf16_bits(np.asarray(a, dtype=np.float32))
        if weights_dtype == "bf16":
            yield name, synth.BF16, bits
        else:
            yield name, synth.F32, synth.bf16_bits_to_f32(bits)


def write_model_dir(dirpath: str, cfg: ZozonexConfig, seed: int = 0, weights_dtype: str = "bf16") -> Tuple[str, str]:
    """Write `config.json` and `model.safetensors`; returns their paths."""
    import os
    from . import synth
    os.makedirs(dirpath, exist_ok=True)
    cpath, mpath = os.path.join(dirpath, "config.json"), os.path.join(dirpath, "model.safetensors")
    with open(cpath, "w") as f:
        f.write(cfg.to_json())
    synth.write_safetensors(mpath, {n: (dt, a) for n, dt, a in iter_tensors(cfg, seed, weights_dtype)})
    return cpath, mpath
