"""Bisuzen: a decoder whose config.json lists its layers one by one.  Every norm is elementwise, dyt(x) = tanh(alpha x) w + b with
one number alpha; a layer is pre-normed and its sublayers follow each other:
    x <- x + mixer(dyt1(x));   x <- x + ff(dyt2(x)).
A span of layers ("loop") may run several passes in a row on the same weights, every pass with keys / values / state of its own.

  "parallel"    two mixers on the same input, each output normed over the width, averaged: grouped-query attention (biased
                projections, interleaved rotary pairs, a sliding window plus the first tokens of the sequence, a learned sink
                per head) beside lightning attention (an outer-product memory with one fixed decay per head)
  "attention"   grouped-query attention without rotation inside chunks of the sequence, queries and keys of unit root mean square

The feed-forward is dense (gelu-gated) or a mixture of experts: softmax scores over experts and identity experts, a choice by
score + correction limited to the best groups, exact-gelu experts.

This module only reads the configuration: sizes and constants go to the native engine as `tgis_model_spec` /
`tgis_layer_spec` (include/tgis_engine.h), the arithmetic is csrc/engine.cu `dyt_layer`, keys and values live in the engine's
paged cache (one set per layer RUN), recurrent state in its sequence slots.
"""
from __future__ import annotations

import ctypes as C
import dataclasses
import math

from . import _lib
from .core import ModelConfig
from .sikazen import layer_runs


@dataclasses.dataclass
class LayerSpec:
    kind: str                 # "parallel" | "attention"
    heads: int = 0            # attention (of "parallel": its left side)
    kv_heads: int = 0
    dim: int = 0
    vdim: int = 0
    scale: float = 1.0
    window: int = 0           # "parallel": the last `window` positions ...
    keep_first: int = 0       # ... and the first `keep_first` of the sequence
    chunk: int = 0            # "attention": positions of the query's own chunk
    rot_dims: int = 0
    rot_base: float = 10000.0
    # "parallel", right side: lightning attention
    lin_heads: int = 0
    lin_dim: int = 0
    lin_vdim: int = 0
    decay: tuple = ()
    # feed-forward: dense (ff > 0), mixture of experts (experts + identity > 0), or none
    ff: int = 0
    experts: int = 0
    identity: int = 0
    top: int = 0
    expert_ff: int = 0
    groups: int = 1
    groups_keep: int = 1

    @property
    def moe(self) -> bool:
        return self.experts + self.identity > 0


def layer_from_json(i: int, entry: dict) -> LayerSpec:
    kind, m = entry.get("type"), entry["mixer"]
    if kind == "parallel":
        a, r = m["left"], m["right"]
        mask, rot = a.get("mask") or {}, a.get("rot") or {}
        spec = LayerSpec(kind, window=int(mask.get("size", 0)), keep_first=int(mask.get("keep_first", 0)), rot_dims=int(rot.get("dims", 0)),
                         rot_base=float(rot.get("base", 10000.0)), lin_heads=int(r["heads"]), lin_dim=int(r["dim"]),
                         lin_vdim=int(r["vdim"]), decay=tuple(float(x) for x in r["decay"]))
        if len(spec.decay) != spec.lin_heads:
            raise ValueError(f"layer {i}: one decay per head expected, got {len(spec.decay)} for {spec.lin_heads} heads")
    elif kind == "attention":
        a = m
        spec = LayerSpec(kind, chunk=int((m.get("mask") or {}).get("size", 0)))
    else:
        raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
    spec.heads, spec.kv_heads = int(a["heads"]), int(a.get("kv_heads", a["heads"]))
    spec.dim, spec.vdim, spec.scale = int(a["dim"]), int(a["vdim"]), float(a["scale"])
    mlp = entry.get("mlp")
    if mlp is None:
        return spec
    if mlp.get("kind") == "dense":
        spec.ff = int(mlp["ff"])
    elif mlp.get("kind") == "moe":
        r = mlp["router"]
        groups = r.get("groups") or {}
        spec.experts, spec.identity, spec.top = int(r["experts"]), int(r.get("identity", 0)), int(r["top"])
        spec.groups, spec.groups_keep = int(groups.get("count", 1)), int(groups.get("keep", 1))
        spec.expert_ff = int(mlp["expert"]["ff"])
    else:
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    return spec


def model_config_from_json(cfg: dict, max_model_len: int | None, dtype: str = "bfloat16") -> ModelConfig:
    layers = [layer_from_json(i, e) for i, e in enumerate(cfg["layers"])]
    if not layers:
        raise ValueError("config.json lists no layers")
    loop = cfg.get("loop") or {}
    return ModelConfig(n_layers=len(layers), hidden=int(cfg["width"]), n_q_heads=1, n_kv_heads=1, ffn=64, vocab=int(cfg["vocab"]),
                       rms_eps=float(cfg["norm"]["eps"]), max_model_len=max_model_len or 4096, arch="bisuzen", layers=layers,
                       dtype=dtype, logit_scale=float(cfg.get("logit_scale", 1.0)),
                       loop=(int(loop.get("start", 0)), int(loop.get("stop", 0)), int(loop.get("times", 1))))


def config_json(mc: ModelConfig) -> dict:
    """The config.json of `mc` (what model_config_from_json reads back)."""
    out = []
    for l in mc.layers:
        a = {"heads": l.heads, "kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale}
        if l.kind == "parallel":
            a["mask"] = {"size": l.window, "keep_first": l.keep_first}
            a["rot"] = {"base": l.rot_base, "dims": l.rot_dims}
            m = {"left": a, "right": {"heads": l.lin_heads, "dim": l.lin_dim, "vdim": l.lin_vdim, "decay": list(l.decay)}}
        else:
            a["mask"] = {"size": l.chunk}
            m = a
        mlp = None
        if l.moe:
            mlp = {"kind": "moe", "expert": {"ff": l.expert_ff},
                   "router": {"experts": l.experts, "identity": l.identity, "top": l.top,
                              "groups": {"count": l.groups, "keep": l.groups_keep}}}
        elif l.ff > 0:
            mlp = {"kind": "dense", "ff": l.ff}
        out.append({"type": l.kind, "mixer": m, "mlp": mlp})
    cfg = {"architecture": "Bisuzen", "width": mc.hidden, "vocab": mc.vocab, "norm": {"eps": mc.rms_eps},
           "logit_scale": mc.logit_scale, "layers": out}
    if mc.loop[2] > 1:
        cfg["loop"] = dict(zip(("start", "stop", "times"), mc.loop))
    return cfg


def model_spec(mc: ModelConfig):
    """(TgisModelSpec, the ctypes arrays it points into)."""
    if mc.dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {mc.dtype!r}: bfloat16 or float32")
    arr = (_lib.TgisLayerSpec * len(mc.layers))()
    keep = [arr]
    for a, l in zip(arr, mc.layers):
        a.heads, a.kv_heads, a.dim, a.vdim, a.scale = l.heads, l.kv_heads, l.dim, l.vdim, l.scale
        if l.kind == "parallel":
            a.mixer = _lib.MIXER_WINDOW_LIGHTNING
            a.flags = _lib.LAYER_QKV_BIAS | _lib.LAYER_OUT_BIAS | _lib.LAYER_ROT_INTERLEAVED | _lib.LAYER_SINK
            a.window, a.keep_first, a.rot_dims, a.rot_base = l.window, l.keep_first, l.rot_dims, l.rot_base
            a.mm_heads, a.mm_dim, a.mm_vdim = l.lin_heads, l.lin_dim, l.lin_vdim
            decay = (C.c_float * max(l.lin_heads, 1))(*l.decay)
            a.decay = C.cast(decay, C.POINTER(C.c_float))
            keep.append(decay)
        else:
            a.mixer = _lib.MIXER_POOLED_ATTENTION
            a.flags, a.chunk = _lib.LAYER_UNIT_QK, l.chunk
        if l.moe:
            a.mlp = _lib.MLP_MOE_GROUPED
            a.experts, a.identity, a.top, a.expert_ff = l.experts, l.identity, l.top, l.expert_ff
            a.expert_groups, a.expert_groups_keep = l.groups, l.groups_keep
        else:
            a.mlp, a.ff = (_lib.MLP_DENSE_GELU, l.ff) if l.ff > 0 else (_lib.MLP_NONE, 0)
    spec = _lib.TgisModelSpec()
    spec.n_layers = len(mc.layers)
    spec.dtype = _lib.DTYPE_F32 if mc.dtype == "float32" else _lib.DTYPE_BF16
    spec.embed_scale, spec.residual_mult, spec.norm_eps = 1.0, 1.0, mc.rms_eps
    spec.logit_scale = mc.logit_scale
    spec.style = _lib.STYLE_PRE_DYT
    spec.loop_start, spec.loop_stop, spec.loop_times = mc.loop if mc.loop[1] > mc.loop[0] else (0, 0, 1)   # (an empty span: no loop)
    spec.layers = C.cast(arr, C.POINTER(_lib.TgisLayerSpec))
    return spec, keep


def cache_row_elems(mc: ModelConfig) -> int:
    """Cache elements of one token over all layer RUNS: keys and values of every run's attention."""
    return sum(mc.layers[i].kv_heads * (mc.layers[i].dim + mc.layers[i].vdim) for i in layer_runs(mc))


def tensor_shapes(mc: ModelConfig) -> dict[str, tuple[int, ...]]:
    """Every parameter of the checkpoint with its shape ([out, in] for matrices; () for a single number)."""
    w, out = mc.hidden, {}

    def norm(name):
        out[name], out[name + ".b"], out[name + ".alpha"] = (w,), (w,), ()

    out["embed"] = (mc.vocab, w)
    for i, l in enumerate(mc.layers):
        p, m = f"l{i}.", f"l{i}.mix."
        norm(p + "norm1")
        left = m + "left." if l.kind == "parallel" else m
        for s, n in (("q", l.heads * l.dim), ("k", l.kv_heads * l.dim), ("v", l.kv_heads * l.vdim)):
            out[left + s] = (n, w)
            if l.kind == "parallel":
                out[left + s + ".b"] = (n,)
        out[left + "o"] = (w, l.heads * l.vdim)
        if l.kind == "parallel":
            r, hd, hv = m + "right.", l.lin_heads * l.lin_dim, l.lin_heads * l.lin_vdim
            out[left + "o.b"] = (w,)
            out[left + "sink"] = (l.heads,)
            out[r + "q"] = out[r + "k"] = (hd, w)
            out[r + "v"] = out[r + "g"] = (hv, w)
            out[r + "norm"] = (hv,)
            out[r + "o"] = (w, hv)
            out[left + "out"] = out[r + "out"] = (w,)
        if l.moe or l.ff > 0:
            norm(p + "norm2")
        if l.moe:
            out[p + "mlp.router"] = (l.experts + l.identity, w)
            out[p + "mlp.correction"] = (l.experts + l.identity,)
            for e in range(l.experts):
                out[p + f"mlp.e{e}.up"] = (l.expert_ff, w)
                out[p + f"mlp.e{e}.down"] = (w, l.expert_ff)
        elif l.ff > 0:
            out[p + "mlp.gate"] = out[p + "mlp.up"] = (l.ff, w)
            out[p + "mlp.down"] = (w, l.ff)
    norm("final.norm")
    out["head"] = (mc.vocab, w)
    return out


def iter_synthetic_weights(mc: ModelConfig, seed: int, device: str = "cpu"):
    """Seeded random bf16 weights of the architecture, one (name, tensor) at a time, drawn on `device`: matrices
    ~ N(0, 1 / fan_in), norm weights around one, alphas around 1/2, biases and router corrections small, sinks around zero."""
    import torch

    gen = torch.Generator(device=device).manual_seed(seed)

    def randn(shape):
        return torch.randn(shape, generator=gen, device=device)

    for name, shape in tensor_shapes(mc).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "alpha":
            t = 0.5 + 0.2 * torch.rand(shape, generator=gen, device=device)
        elif leaf == "sink":
            t = randn(shape)
        elif leaf == "b":
            t = randn(shape) * 0.1
        elif leaf == "correction":
            t = randn(shape) * 0.05
        elif len(shape) <= 1:
            t = 1.0 + randn(shape) * 0.1
        elif name == "embed":
            t = randn(shape)
        else:
            t = randn(shape) * shape[1] ** -0.5
        yield name, t.to(torch.bfloat16)


def synthetic_weights(mc: ModelConfig, seed: int, device: str = "cpu") -> dict:
    return dict(iter_synthetic_weights(mc, seed, device))


def _stack(hidden: int, vocab: int, layers: list[LayerSpec], loop: tuple[int, int, int], logit_scale: float = 1.0) -> ModelConfig:
    return ModelConfig(n_layers=len(layers), hidden=hidden, n_q_heads=1, n_kv_heads=1, ffn=64, vocab=vocab, rms_eps=1e-5,
                       max_model_len=4096, arch="bisuzen", layers=layers, logit_scale=logit_scale, loop=loop)


def _decays(heads: int) -> tuple:
    return tuple(math.exp(-(2.0 ** (-1.0 - 7.0 * h / max(heads - 1, 1)))) for h in range(heads))


def _par(heads: int, kv_heads: int, dim: int, window: int, keep: int, lin_heads: int, lin_dim: int, **ff) -> LayerSpec:
    return LayerSpec("parallel", heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, window=window, keep_first=keep,
                     rot_dims=dim, rot_base=10000.0, lin_heads=lin_heads, lin_dim=lin_dim, lin_vdim=lin_dim, decay=_decays(lin_heads), **ff)


def _att(heads: int, kv_heads: int, dim: int, chunk: int, **ff) -> LayerSpec:
    return LayerSpec("attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, chunk=chunk, **ff)


def _moe(experts: int, identity: int, top: int, ff: int, groups: int, keep: int) -> dict:
    return dict(experts=experts, identity=identity, top=top, expert_ff=ff, groups=groups, groups_keep=keep)


# Sizes that resemble the layers of real hybrid models (random weights; `--model <name> --synthetic-weights`,
# bench.py --arch-compare): four layers of which the first two run two passes -- six layer runs -- at the hidden size,
# vocabulary and active feed-forward width of the Llama twin
PRESETS: dict[str, ModelConfig] = {
    "bisuzen-tiny": _stack(128, 512, [
        LayerSpec("parallel", heads=4, kv_heads=2, dim=32, vdim=24, scale=0.3, window=20, keep_first=3, rot_dims=16, rot_base=1000.0,
                  lin_heads=2, lin_dim=24, lin_vdim=40, decay=(0.7, 0.97), **_moe(5, 1, 2, 48, 2, 1)),
        LayerSpec("attention", heads=4, kv_heads=4, dim=16, vdim=32, scale=0.9, chunk=24, ff=160),
        LayerSpec("attention", heads=6, kv_heads=2, dim=24, vdim=24, scale=1.1, chunk=40)], loop=(1, 3, 2), logit_scale=0.5),
    "bisuzen-1k": _stack(1024, 32768, [
        _par(8, 2, 128, 256, 4, 8, 128, ff=3072),
        _att(8, 2, 128, 2048, **_moe(15, 1, 2, 1536, 2, 1)),
        _par(8, 2, 128, 256, 4, 8, 128, **_moe(15, 1, 2, 1536, 2, 1)),
        _att(8, 2, 128, 2048, ff=3072)], loop=(0, 2, 2)),
    "bisuzen-2k": _stack(2048, 32768, [
        _par(16, 4, 128, 256, 4, 16, 128, ff=11264),
        _att(16, 4, 128, 2048, **_moe(60, 4, 6, 1408, 8, 4)),
        _par(16, 4, 128, 256, 4, 16, 128, **_moe(60, 4, 6, 1408, 8, 4)),
        _att(16, 4, 128, 2048, ff=11264)], loop=(0, 2, 2)),
}
