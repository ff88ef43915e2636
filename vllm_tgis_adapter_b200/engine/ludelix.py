"""Ludelix: a decoder whose config.json lists its layers one by one.  Layers are pre-normed with plain RMS weights and their
sublayers follow each other:
    x <- x + mixer(rms(x) norm1);   x <- x + ff(rms(x) norm2)
and the logits read the embedding table.

  "parallel"    two mixers on the same input, weighed by two constants: grouped-query attention inside chunks of the sequence
                (YaRN-scaled rotary positions, a sigmoid gate per head) beside retention (an outer-product memory with one fixed
                decay per head on rotated queries and keys)
  "attention"   sliding-window attention with a sink whose values are the keys as projected; queries and keys are normed over
                all heads at once and turned as interleaved pairs (frequencies scaled by wavelength)
  "gla"         gated linear attention: an outer-product memory whose key channels decay one by one

The feed-forward is dense (squared relu) or a mixture of experts that a table chooses by the token id, plus a gated shared expert.

This module only reads the configuration: sizes and constants go to the native engine as `tgis_model_spec` /
`tgis_layer_spec` (include/tgis_engine.h), the arithmetic is csrc/engine.cu `rms_layer`, keys and values live in the engine's
paged cache, recurrent state in its sequence slots.
"""
from __future__ import annotations

import ctypes as C
import dataclasses

from . import _lib
from .core import ModelConfig
from .falerax import checkpoint_shapes  # noqa: F401  (the loader asks the family's module for it)


@dataclasses.dataclass
class LayerSpec:
    kind: str                 # "parallel" | "attention" | "gla"
    heads: int = 0            # attention (of "parallel": its left side), gla
    kv_heads: int = 0
    dim: int = 0
    vdim: int = 0
    scale: float = 1.0
    window: int = 0           # "attention": the last `window` positions
    chunk: int = 0            # "parallel": positions of the query's own chunk
    rot_dims: int = 0
    rot_base: float = 10000.0
    # "parallel": YaRN (yarn_factor 0: plain); "attention": scaling by wavelength (band_factor 0: plain)
    yarn_factor: float = 0.0
    yarn_original: float = 0.0
    yarn_fast: float = 0.0
    yarn_slow: float = 0.0
    band_factor: float = 0.0
    band_original: float = 0.0
    band_low: float = 0.0
    band_high: float = 0.0
    # "parallel", right side: retention
    ret_heads: int = 0
    ret_dim: int = 0
    ret_vdim: int = 0
    ret_rot_dims: int = 0
    ret_rot_base: float = 10000.0
    decay: tuple = ()
    left_scale: float = 1.0
    right_scale: float = 1.0
    # "gla"
    tau: float = 1.0
    rank: int = 0             # inner size of the decay's low-rank map (from the checkpoint)
    # feed-forward: dense (ff > 0), mixture of experts (experts > 0), or none
    ff: int = 0
    experts: int = 0
    top: int = 0
    expert_ff: int = 0
    shared_ff: int = 0

    @property
    def moe(self) -> bool:
        return self.experts > 0


def _attention(spec: LayerSpec, m: dict) -> LayerSpec:
    spec.heads, spec.kv_heads = int(m["heads"]), int(m.get("kv_heads", m["heads"]))
    spec.dim, spec.vdim, spec.scale = int(m["dim"]), int(m["vdim"]), float(m["scale"])
    rot = m.get("rot") or {}
    spec.rot_dims, spec.rot_base = int(rot.get("dims", 0)), float(rot.get("base", 10000.0))
    return spec


def layer_from_json(i: int, entry: dict) -> LayerSpec:
    kind, m = entry.get("type"), entry["mixer"]
    if kind == "parallel":
        left, r = m["left"], m["right"]
        spec = _attention(LayerSpec(kind, chunk=int((left.get("mask") or {}).get("size", 0)), left_scale=float(m["left_scale"]),
                                    right_scale=float(m["right_scale"]), ret_heads=int(r["heads"]), ret_dim=int(r["dim"]),
                                    ret_vdim=int(r["vdim"]), decay=tuple(float(x) for x in r["decay"])), left)
        if len(spec.decay) != spec.ret_heads:
            raise ValueError(f"layer {i}: one decay per head expected, got {len(spec.decay)} for {spec.ret_heads} heads")
        rot = r.get("rot") or {}
        spec.ret_rot_dims, spec.ret_rot_base = int(rot.get("dims", 0)), float(rot.get("base", 10000.0))
        sc = (left.get("rot") or {}).get("scaling")
        if sc:
            spec.yarn_factor, spec.yarn_original = float(sc["factor"]), float(sc["original"])
            spec.yarn_fast, spec.yarn_slow = float(sc["fast"]), float(sc["slow"])
    elif kind == "attention":
        spec = _attention(LayerSpec(kind, window=int((m.get("mask") or {}).get("size", 0))), m)
        if spec.vdim != spec.dim:
            raise ValueError(f"layer {i}: values are the keys, but vdim {spec.vdim} is not dim {spec.dim}")
        sc = (m.get("rot") or {}).get("scaling")
        if sc:
            spec.band_factor, spec.band_original = float(sc["factor"]), float(sc["original"])
            spec.band_low, spec.band_high = float(sc["low"]), float(sc["high"])
    elif kind == "gla":
        spec = LayerSpec(kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]))
    else:
        raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
    mlp = entry.get("mlp")
    if mlp is None:
        return spec
    if mlp.get("kind") == "dense":
        spec.ff = int(mlp["ff"])
    elif mlp.get("kind") == "moe":
        spec.experts, spec.top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
        spec.expert_ff = int(mlp["expert"]["ff"])
        spec.shared_ff = int((mlp.get("shared") or {}).get("ff", 0))
    else:
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
    return spec


def model_config_from_json(cfg: dict, max_model_len: int | None, dtype: str = "bfloat16",
                           shapes: dict[str, tuple[int, ...]] | None = None) -> ModelConfig:
    layers = [layer_from_json(i, e) for i, e in enumerate(cfg["layers"])]
    if not layers:
        raise ValueError("config.json lists no layers")
    for i, l in enumerate(layers):
        if l.kind == "gla":   # the low-rank map's inner size is known from its first matrix alone
            name = f"l{i}.mix.a1"
            if not shapes or name not in shapes:
                raise ValueError(f"the checkpoint holds no {name}: the decay's low-rank map has no size without it")
            l.rank = int(shapes[name][0])
    return ModelConfig(n_layers=len(layers), hidden=int(cfg["width"]), n_q_heads=1, n_kv_heads=1, ffn=64, vocab=int(cfg["vocab"]),
                       rms_eps=float(cfg["norm"]["eps"]), max_model_len=max_model_len or 4096, arch="ludelix", layers=layers, dtype=dtype)


def config_json(mc: ModelConfig) -> dict:
    """The config.json of `mc` (what model_config_from_json reads back)."""
    out = []
    for l in mc.layers:
        if l.kind == "gla":
            m = {"heads": l.heads, "dim": l.dim, "vdim": l.vdim, "tau": l.tau}
        else:
            rot: dict = {"base": l.rot_base, "dims": l.rot_dims}
            if l.yarn_factor > 0:
                rot["scaling"] = {"factor": l.yarn_factor, "original": l.yarn_original, "fast": l.yarn_fast, "slow": l.yarn_slow}
            if l.band_factor > 0:
                rot["scaling"] = {"factor": l.band_factor, "original": l.band_original, "low": l.band_low, "high": l.band_high}
            m = {"heads": l.heads, "kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale, "rot": rot,
                 "mask": {"size": l.chunk if l.kind == "parallel" else l.window}}
        if l.kind == "parallel":
            m = {"left": m, "left_scale": l.left_scale, "right_scale": l.right_scale,
                 "right": {"heads": l.ret_heads, "dim": l.ret_dim, "vdim": l.ret_vdim, "decay": list(l.decay),
                           "rot": {"base": l.ret_rot_base, "dims": l.ret_rot_dims}}}
        mlp = None
        if l.moe:
            mlp = {"kind": "moe", "expert": {"ff": l.expert_ff}, "router": {"experts": l.experts, "top": l.top}}
            if l.shared_ff > 0:
                mlp["shared"] = {"ff": l.shared_ff}
        elif l.ff > 0:
            mlp = {"kind": "dense", "ff": l.ff}
        out.append({"type": l.kind, "mixer": m, "mlp": mlp})
    return {"architecture": "Ludelix", "width": mc.hidden, "vocab": mc.vocab, "norm": {"eps": mc.rms_eps}, "layers": out}


def model_spec(mc: ModelConfig):
    """(TgisModelSpec, the ctypes arrays it points into)."""
    if mc.dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {mc.dtype!r}: bfloat16 or float32")
    arr = (_lib.TgisLayerSpec * len(mc.layers))()
    keep = [arr]
    for a, l in zip(arr, mc.layers):
        a.heads, a.dim, a.vdim = l.heads, l.dim, l.vdim
        if l.kind == "gla":
            a.mixer, a.tau, a.decay_rank = _lib.MIXER_GLA, l.tau, l.rank
        else:
            a.kv_heads, a.scale, a.rot_dims, a.rot_base, a.window, a.chunk = l.kv_heads, l.scale, l.rot_dims, l.rot_base, l.window, l.chunk
            a.yarn_factor, a.yarn_original, a.yarn_fast, a.yarn_slow = l.yarn_factor, l.yarn_original, l.yarn_fast, l.yarn_slow
            a.band_factor, a.band_original, a.band_low, a.band_high = l.band_factor, l.band_original, l.band_low, l.band_high
        if l.kind == "attention":
            a.mixer = _lib.MIXER_POOLED_ATTENTION
            a.flags = (_lib.LAYER_QKV_BIAS | _lib.LAYER_ROT_INTERLEAVED | _lib.LAYER_SINK | _lib.LAYER_SHARED_KV
                       | _lib.LAYER_FULL_QK_NORM)
        elif l.kind == "parallel":
            a.mixer, a.flags = _lib.MIXER_CHUNK_RETENTION, _lib.LAYER_HEAD_GATE
            a.mm_heads, a.mm_dim, a.mm_vdim = l.ret_heads, l.ret_dim, l.ret_vdim
            a.mm_rot_dims, a.mm_rot_base = l.ret_rot_dims, l.ret_rot_base
            a.left_scale, a.right_scale = l.left_scale, l.right_scale
            decay = (C.c_float * max(l.ret_heads, 1))(*l.decay)
            a.decay = C.cast(decay, C.POINTER(C.c_float))
            keep.append(decay)
        if l.moe:
            a.mlp = _lib.MLP_MOE_TABLE
            a.experts, a.top, a.expert_ff, a.shared_ff = l.experts, l.top, l.expert_ff, l.shared_ff
        else:
            a.mlp, a.ff = (_lib.MLP_DENSE_RELU2, l.ff) if l.ff > 0 else (_lib.MLP_NONE, 0)
    spec = _lib.TgisModelSpec()
    spec.n_layers = len(mc.layers)
    spec.dtype = _lib.DTYPE_F32 if mc.dtype == "float32" else _lib.DTYPE_BF16
    spec.embed_scale, spec.residual_mult, spec.norm_eps, spec.logit_scale = 1.0, 1.0, mc.rms_eps, 1.0
    spec.style = _lib.STYLE_PRE_RMS | _lib.STYLE_TIED_HEAD
    spec.layers = C.cast(arr, C.POINTER(_lib.TgisLayerSpec))
    return spec, keep


def cache_row_elems(mc: ModelConfig) -> int:
    """Cache elements of one token over all layers: keys and values of every attention."""
    return sum(l.kv_heads * (l.dim + l.vdim) for l in mc.layers if l.kind != "gla")


def tensor_shapes(mc: ModelConfig) -> dict[str, tuple[int, ...]]:
    """Every parameter of the checkpoint with its shape ([out, in] for matrices)."""
    w, out = mc.hidden, {"embed": (mc.vocab, mc.hidden)}
    for i, l in enumerate(mc.layers):
        p, m = f"l{i}.", f"l{i}.mix."
        out[p + "norm1"] = (w,)
        hd, hv, gd = l.heads * l.dim, l.heads * l.vdim, l.kv_heads * l.dim
        if l.kind == "gla":
            out[m + "q"] = out[m + "k"] = (hd, w)
            out[m + "v"] = out[m + "g"] = (hv, w)
            out[m + "o"] = (w, hv)
            out[m + "norm"] = (l.vdim,)
            out[m + "a1"], out[m + "a2"], out[m + "a2.b"] = (l.rank, w), (hd, l.rank), (hd,)
        elif l.kind == "attention":
            for s, n in (("q", hd), ("k", gd)):
                out[m + s], out[m + s + ".b"], out[m + s + ".norm"] = (n, w), (n,), (n,)
            out[m + "sink"], out[m + "o"] = (l.heads,), (w, hv)
        else:
            left, right, rd, rv = m + "left.", m + "right.", l.ret_heads * l.ret_dim, l.ret_heads * l.ret_vdim
            out[left + "q"], out[left + "k"], out[left + "v"] = (hd, w), (gd, w), (l.kv_heads * l.vdim, w)
            out[left + "g"], out[left + "o"] = (l.heads, w), (w, hv)
            out[right + "q"] = out[right + "k"] = (rd, w)
            out[right + "v"] = out[right + "g"] = (rv, w)
            out[right + "o"] = (w, rv)
        if l.moe or l.ff > 0:
            out[p + "norm2"] = (w,)
        if l.moe:
            for e in [f"e{j}" for j in range(l.experts)] + (["shared"] if l.shared_ff > 0 else []):
                ff = l.shared_ff if e == "shared" else l.expert_ff
                out[p + f"mlp.{e}.gate"] = out[p + f"mlp.{e}.up"] = (ff, w)
                out[p + f"mlp.{e}.down"] = (w, ff)
            out[p + "mlp.table"] = (mc.vocab, l.top)
            if l.shared_ff > 0:
                out[p + "mlp.shared.sg"] = (1, w)
        elif l.ff > 0:
            out[p + "mlp.up"], out[p + "mlp.down"] = (l.ff, w), (w, l.ff)
    out["final.norm"] = (w,)
    return out


def iter_synthetic_weights(mc: ModelConfig, seed: int, device: str = "cpu"):
    """Seeded random weights of the architecture, one (name, tensor) at a time, drawn on `device`: bf16 matrices
    ~ N(0, 1 / fan_in), norm weights around one, biases small, sinks around zero, decay biases around two; int32 expert tables
    whose rows hold `top` different experts."""
    import torch

    gen = torch.Generator(device=device).manual_seed(seed)

    def randn(shape):
        return torch.randn(shape, generator=gen, device=device)

    for name, shape in tensor_shapes(mc).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "table":
            l = mc.layers[int(name[1:].split(".", 1)[0])]
            first = torch.randint(l.experts, (shape[0], 1), generator=gen, device=device)
            yield name, ((first + torch.arange(l.top, device=device)) % l.experts).to(torch.int32)
            continue
        if leaf == "sink":
            t = randn(shape)
        elif name.endswith("a2.b"):
            t = 2.0 + randn(shape)
        elif leaf == "b":
            t = randn(shape) * 0.1
        elif len(shape) == 1:
            t = 1.0 + randn(shape) * 0.1
        elif name == "embed":
            t = randn(shape)
        else:
            t = randn(shape) * shape[1] ** -0.5
        yield name, t.to(torch.bfloat16)


def synthetic_weights(mc: ModelConfig, seed: int, device: str = "cpu") -> dict:
    return dict(iter_synthetic_weights(mc, seed, device))


def _stack(hidden: int, vocab: int, layers: list[LayerSpec]) -> ModelConfig:
    return ModelConfig(n_layers=len(layers), hidden=hidden, n_q_heads=1, n_kv_heads=1, ffn=64, vocab=vocab, rms_eps=1e-5,
                       max_model_len=4096, arch="ludelix", layers=layers)


def _par(heads: int, kv_heads: int, dim: int, chunk: int, ret_heads: int, ret_dim: int, **ff) -> LayerSpec:
    return LayerSpec("parallel", heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, chunk=chunk, rot_dims=dim,
                     rot_base=10000.0, yarn_factor=4.0, yarn_original=4096.0, yarn_fast=32.0, yarn_slow=1.0, ret_heads=ret_heads,
                     ret_dim=ret_dim, ret_vdim=ret_dim, ret_rot_dims=ret_dim, ret_rot_base=10000.0,
                     decay=tuple(1.0 - 2.0 ** (-5.0 - 4.0 * h / ret_heads) for h in range(ret_heads)), left_scale=0.8, right_scale=0.7, **ff)


def _att(heads: int, kv_heads: int, dim: int, window: int, **ff) -> LayerSpec:
    return LayerSpec("attention", heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=dim ** -0.5, window=window, rot_dims=dim,
                     rot_base=500000.0, band_factor=8.0, band_original=8192.0, band_low=1.0, band_high=4.0, **ff)


def _gla(heads: int, dim: int, vdim: int, rank: int = 16, tau: float = 16.0, **ff) -> LayerSpec:
    return LayerSpec("gla", heads=heads, dim=dim, vdim=vdim, rank=rank, tau=tau, **ff)


def _moe(experts: int, top: int, ff: int, shared: int) -> dict:
    return dict(experts=experts, top=top, expert_ff=ff, shared_ff=shared)


# Sizes that resemble the layers of real hybrid models (random weights; `--model <name> --synthetic-weights`,
# bench.py --arch-compare): four layers at the hidden size, vocabulary and active feed-forward width of the Llama twin
PRESETS: dict[str, ModelConfig] = {
    "ludelix-tiny": _stack(128, 500, [
        LayerSpec("parallel", heads=4, kv_heads=2, dim=32, vdim=24, scale=0.3, chunk=40, rot_dims=16, rot_base=1000.0, yarn_factor=3.0,
                  yarn_original=64.0, yarn_fast=8.0, yarn_slow=1.0, ret_heads=2, ret_dim=24, ret_vdim=40, ret_rot_dims=12,
                  ret_rot_base=500.0, decay=(0.8, 0.97), left_scale=0.7, right_scale=1.3, **_moe(5, 2, 48, 72)),
        LayerSpec("gla", heads=3, dim=32, vdim=24, tau=4.0, rank=5, ff=160),
        LayerSpec("attention", heads=6, kv_heads=3, dim=32, vdim=32, scale=0.4, window=24, rot_dims=24, rot_base=2000.0, band_factor=2.0,
                  band_original=96.0, band_low=1.0, band_high=3.0, **_moe(4, 1, 40, 0)),
        LayerSpec("gla", heads=2, dim=16, vdim=32, tau=16.0, rank=8)]),
    "ludelix-1k": _stack(1024, 32768, [
        _par(8, 2, 128, 2048, 8, 128, ff=3072),
        _gla(4, 128, 256, **_moe(16, 2, 1024, 1024)),
        _att(8, 2, 128, 256, **_moe(16, 2, 1024, 1024)),
        _par(8, 2, 128, 2048, 8, 128, **_moe(16, 2, 1024, 1024))]),
    "ludelix-2k": _stack(2048, 32768, [
        _par(16, 4, 128, 2048, 16, 128, ff=11264),
        _gla(16, 128, 128, **_moe(64, 6, 1408, 2816)),
        _att(16, 4, 128, 256, **_moe(64, 6, 1408, 2816)),
        _par(16, 4, 128, 2048, 16, 128, **_moe(64, 6, 1408, 2816))]),
}
