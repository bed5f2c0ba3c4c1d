"""Configuration and seeded synthetic weights of the Zutazen design.

A decoder whose config.json lists its layers one by one: retention (linear attention with fixed decays), gated linear
recurrences over channels, and sliding-window attention over a cached latent, behind norms of the residual stream; gated
feed-forwards, dense with biases or a mixture of experts whose weight multiplies the expert's input; a head of its own.  A
layer may use the weights of an earlier one.
"""
from __future__ import annotations

import json
import zlib
from typing import Iterator, List, Optional, Tuple

import numpy as np

ARCHITECTURE = "Zutazen"


class ZutazenConfig:
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
    def from_json(text: str) -> "ZutazenConfig":
        return ZutazenConfig(json.loads(text))


def dense(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(experts: int, top: int, ff: int) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def retention(heads: int, dim: int, vdim: int, decay: Optional[List[float]] = None, rot_dims: Optional[int] = None, base: float = 10000.0,
              mlp: Optional[dict] = None) -> dict:
    if decay is None:
        decay = [1.0 - 2.0 ** -(5 + 5.0 * h / max(1, heads - 1)) for h in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay),
                                           "rot": {"dims": dim if rot_dims is None else rot_dims, "base": base}}, "mlp": mlp}


def rglru(width: int, blocks: int, conv: int = 4, mlp: Optional[dict] = None) -> dict:
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def latent_attention(heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, window: int, base: float = 10000.0, scale: Optional[float] = None,
                     mlp: Optional[dict] = None) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"dims": rot_dim, "base": base},
         "scale": float(scale if scale is not None else (dim + rot_dim) ** -0.5)}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def again(layers: List[dict], of: int) -> dict:
    """A further layer with the weights of layer `of`."""
    src = of
    while "weights_of" in layers[src]:
        src = layers[src]["weights_of"]
    return dict(layers[src], weights_of=of)


def config(width: int, vocab: int, layers: List[dict], eps: float = 1e-6, embed_scale: float = 1.0, max_seq_len: int = 2048) -> ZutazenConfig:
    return ZutazenConfig({"architecture": ARCHITECTURE, "width": width, "vocab": vocab, "norm": {"eps": eps},
                          "embedding": {"scale": embed_scale}, "layers": layers}, max_seq_len)


def tensor_specs(cfg: ZutazenConfig) -> List[Tuple[str, Tuple[int, ...], str]]:
    """(name, shape, kind) of every tensor."""
    D = cfg.d_model
    out: List[Tuple[str, Tuple[int, ...], str]] = [("embed", (cfg.vocab_size, D), "embed")]
    for i, L in enumerate(cfg.raw["layers"]):
        if "weights_of" in L:
            continue
        p, m, f = "l%d." % i, L["mixer"], L.get("mlp")
        out.append((p + "norm1", (D,), "norm"))
        if L["type"] == "retention":
            k, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out += [(p + "mix." + n, (r, D), "matrix") for n, r in (("q", k), ("k", k), ("v", v), ("g", v))] + [(p + "mix.o", (D, v), "matrix")]
        elif L["type"] == "rglru":
            C, s = m["width"], m["width"] // m["blocks"]
            for n in ("y", "x"):
                out += [(p + "mix." + n, (C, D), "matrix"), (p + "mix." + n + ".b", (C,), "bias")]
            out += [(p + "mix.conv", (C, m["conv"]), "conv"), (p + "mix.conv.b", (C,), "bias")]
            for n in ("ra", "ri"):
                out += [(p + "mix." + n, (m["blocks"], s, s), "matrix"), (p + "mix." + n + ".b", (m["blocks"], s), "bias")]
            out += [(p + "mix.lam", (C,), "lam"), (p + "mix.o", (D, C), "matrix")]
        else:
            H, r = m["heads"], m["kv_rank"]
            out += [(p + "mix.q", (H * (m["dim"] + m["rot_dim"]), D), "matrix"), (p + "mix.dkv", (r + m["rot_dim"], D), "matrix"),
                    (p + "mix.dkv.norm", (r,), "norm"), (p + "mix.uk", (H * m["dim"], r), "matrix"), (p + "mix.uv", (H * m["vdim"], r), "matrix"),
                    (p + "mix.g", (H * m["vdim"], D), "matrix"), (p + "mix.o", (D, H * m["vdim"]), "matrix")]
        if f is None:
            continue
        out.append((p + "norm2", (D,), "norm"))
        if f["kind"] == "dense":
            for n in ("gate", "up"):
                out += [(p + "mlp." + n, (f["ff"], D), "matrix"), (p + "mlp." + n + ".b", (f["ff"],), "bias")]
            out += [(p + "mlp.down", (D, f["ff"]), "matrix"), (p + "mlp.down.b", (D,), "bias")]
        else:
            for e in range(f["router"]["experts"]):
                q, w = p + "mlp.e%d." % e, f["expert"]["ff"]
                out += [(q + "gate", (w, D), "matrix"), (q + "up", (w, D), "matrix"), (q + "down", (D, w), "matrix")]
            out.append((p + "mlp.router", (f["router"]["experts"], D), "matrix"))
    return out + [("final.norm", (D,), "norm"), ("head", (cfg.vocab_size, D), "matrix")]


def iter_tensors(cfg: ZutazenConfig, seed: int = 0, weights_dtype: str = "bf16") -> Iterator[Tuple[str, int, np.ndarray]]:
    """(name, dtype code, array) with seeded random values of a sensible size; bf16 tensors as uint16 bit patterns.  Values are
    rounded to bf16 in either case, so that an fp32 model holds the same numbers."""
    from . import synth
    for name, shape, kind in tensor_specs(cfg):
        g = np.random.Generator(np.random.Philox(key=[seed, zlib.crc32(name.encode())]))
        if kind == "lam":
            a = g.uniform(-6.0, 0.0, shape)
        else:
            a = g.standard_normal(shape, dtype=np.float32)
            if kind == "matrix":
                a *= shape[-1] ** -0.5
            elif kind == "embed":
                a *= 0.3
            elif kind == "conv":
                a *= 0.6
            elif kind == "bias":
                a *= 0.3
            else:
                a = 1.0 + 0.2 * a
        bits = synth.f32_to_bf16_bits(np.asarray(a, dtype=np.float32))
        if weights_dtype == "bf16":
            yield name, synth.BF16, bits
        else:
            yield name, synth.F32, synth.bf16_bits_to_f32(bits)


def write_model_dir(dirpath: str, cfg: ZutazenConfig, seed: int = 0, weights_dtype: str = "bf16") -> Tuple[str, str]:
    """Write `config.json` and `model.safetensors`; returns their paths."""
    import os
    from . import synth
    os.makedirs(dirpath, exist_ok=True)
    cpath, mpath = os.path.join(dirpath, "config.json"), os.path.join(dirpath, "model.safetensors")
    with open(cpath, "w") as f:
        f.write(cfg.to_json())
    synth.write_safetensors(mpath, {n: (dt, a) for n, dt, a in iter_tensors(cfg, seed, weights_dtype)})
    return cpath, mpath
