"""CPU-side checks of the Ludelix family: config.json -> engine specs, the parameter list, cache accounting, presets, and properties
of the plain oracle that the GPU tests lean on (edges of windows and chunks, the sink, both rotary layouts and frequency scalings,
values that are the keys as projected, decays, the expert table, state carried token by token)."""
import copy
import math

import pytest
import torch

from oracle import ludelix_oracle as O
from vllm_tgis_adapter_b200.engine import _lib
from vllm_tgis_adapter_b200.engine.core import cache_block_bytes
from vllm_tgis_adapter_b200.engine.ludelix import (PRESETS, cache_row_elems, config_json, model_config_from_json, model_spec,
                                                   synthetic_weights, tensor_shapes)

F64 = torch.float64
LEFT = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "scale": 0.9, "mask": {"size": 7},
        "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.5, "original": 30, "fast": 3.0, "slow": 0.5}}}
RIGHT = {"heads": 3, "dim": 5, "vdim": 4, "decay": [0.5, 0.9, 0.95], "rot": {"base": 40.0, "dims": 2}}
ATT = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 6, "scale": 0.7, "mask": {"size": 5},
       "rot": {"base": 60.0, "dims": 6, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40}}}
GLA = {"heads": 2, "dim": 5, "vdim": 7, "tau": 3.0}
MOE = {"kind": "moe", "expert": {"ff": 9}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 11}}
CFG = {
    "architecture": "Ludelix", "width": 24, "vocab": 50, "norm": {"eps": 1e-3},
    "layers": [
        {"type": "gla", "mixer": GLA, "mlp": None},
        {"type": "parallel", "mixer": {"left": LEFT, "right": RIGHT, "left_scale": 0.8, "right_scale": 1.4}, "mlp": MOE},
        {"type": "attention", "mixer": ATT, "mlp": {"kind": "dense", "ff": 13}},
        {"type": "gla", "mixer": {**GLA, "heads": 1}, "mlp": {k: v for k, v in MOE.items() if k != "shared"}},
    ],
}
SHAPES = {"l0.mix.a1": (4, 24), "l3.mix.a1": (1, 24)}


def _mc(dtype="float32"):
    return model_config_from_json(CFG, 256, dtype, SHAPES)


def test_config_json_to_specs():
    mc = _mc()
    assert (mc.arch, mc.hidden, mc.vocab, mc.n_layers, mc.max_model_len, mc.rms_eps, mc.dtype) == ("ludelix", 24, 50, 4, 256, 1e-3, "float32")
    a, b, c, d = mc.layers
    assert (a.kind, a.heads, a.dim, a.vdim, a.tau, a.rank, a.ff, a.moe) == ("gla", 2, 5, 7, 3.0, 4, 0, False) and d.rank == 1
    assert (b.kind, b.heads, b.kv_heads, b.dim, b.vdim, b.chunk, b.window, b.rot_dims, b.rot_base) == ("parallel", 4, 2, 6, 3, 7, 0, 4, 100.0)
    assert (b.yarn_factor, b.yarn_original, b.yarn_fast, b.yarn_slow, b.band_factor) == (2.5, 30.0, 3.0, 0.5, 0.0)
    assert (b.ret_heads, b.ret_dim, b.ret_vdim, b.ret_rot_dims, b.ret_rot_base, b.decay) == (3, 5, 4, 2, 40.0, (0.5, 0.9, 0.95))
    assert (b.left_scale, b.right_scale, b.experts, b.top, b.expert_ff, b.shared_ff) == (0.8, 1.4, 5, 2, 9, 11)
    assert (c.window, c.chunk, c.band_factor, c.band_low, c.band_high, c.band_original, c.ff) == (5, 0, 4.0, 1.0, 3.0, 40.0, 13)
    assert (d.shared_ff, d.experts) == (0, 5)
    spec, keep = model_spec(mc)
    specs = keep[0]
    assert (spec.n_layers, spec.dtype, spec.style) == (4, _lib.DTYPE_F32, _lib.STYLE_PRE_RMS | _lib.STYLE_TIED_HEAD)
    assert [s.mixer for s in specs] == [_lib.MIXER_GLA, _lib.MIXER_CHUNK_RETENTION, _lib.MIXER_POOLED_ATTENTION, _lib.MIXER_GLA]
    assert [s.mlp for s in specs] == [_lib.MLP_NONE, _lib.MLP_MOE_TABLE, _lib.MLP_DENSE_RELU2, _lib.MLP_MOE_TABLE]
    assert (specs[0].tau, specs[0].decay_rank) == (3.0, 4)
    assert specs[1].flags == _lib.LAYER_HEAD_GATE and (specs[1].chunk, specs[1].window) == (7, 0) and abs(specs[1].right_scale - 1.4) < 1e-6
    assert [round(specs[1].decay[i], 6) for i in range(3)] == [0.5, 0.9, 0.95] and specs[1].mm_rot_dims == 2
    assert specs[2].flags == (_lib.LAYER_QKV_BIAS | _lib.LAYER_ROT_INTERLEAVED | _lib.LAYER_SINK | _lib.LAYER_SHARED_KV | _lib.LAYER_FULL_QK_NORM)
    assert (specs[2].window, specs[2].chunk, specs[2].band_factor, specs[2].yarn_factor) == (5, 0, 4.0, 0.0)
    back = model_config_from_json(config_json(mc), 256, "float32", SHAPES)
    assert back.layers == mc.layers                              # round trip
    for bad in ({"type": "something_else"}, {"mlp": {"kind": "other"}}):
        with pytest.raises(ValueError):
            model_config_from_json({**CFG, "layers": [{**CFG["layers"][0], **bad}]}, None, "float32", SHAPES)
    for mixer in ({"left": LEFT, "right": {**RIGHT, "heads": 2}, "left_scale": 1, "right_scale": 1},):   # one decay per head
        with pytest.raises(ValueError):
            model_config_from_json({**CFG, "layers": [{**CFG["layers"][1], "mixer": mixer}]}, None)
    with pytest.raises(ValueError):                              # values are the keys
        model_config_from_json({**CFG, "layers": [{**CFG["layers"][2], "mixer": {**ATT, "vdim": 4}}]}, None)
    with pytest.raises(ValueError):                              # the low-rank map's size comes from the checkpoint
        model_config_from_json(CFG, None)


def test_parameter_list_cache_accounting_and_presets():
    mc = _mc("bfloat16")
    shapes = tensor_shapes(mc)
    assert shapes["embed"] == (50, 24) and "head" not in shapes and shapes["final.norm"] == (24,) and "l0.norm2" not in shapes
    assert shapes["l0.mix.a1"] == (4, 24) and shapes["l0.mix.a2"] == (10, 4) and shapes["l0.mix.a2.b"] == (10,) and shapes["l0.mix.norm"] == (7,)
    assert shapes["l1.mix.left.g"] == (4, 24) and shapes["l1.mix.left.v"] == (6, 24) and shapes["l1.mix.right.o"] == (24, 12)
    assert shapes["l1.mlp.table"] == (50, 2) and shapes["l1.mlp.shared.sg"] == (1, 24) and shapes["l1.mlp.shared.down"] == (24, 11)
    assert shapes["l2.mix.q.norm"] == (24,) and shapes["l2.mix.k.norm"] == shapes["l2.mix.k.b"] == (12,) and "l2.mix.v" not in shapes
    assert shapes["l2.mlp.up"] == (13, 24) and "l2.mlp.gate" not in shapes and "l3.mlp.shared.sg" not in shapes
    w = synthetic_weights(mc, 3)
    assert set(w) == set(shapes) and all(tuple(w[k].shape) == shapes[k] for k in shapes)
    t = w["l1.mlp.table"]
    assert t.dtype == torch.int32 and int(t.min()) >= 0 and int(t.max()) == 4 and bool((t[:, 0] != t[:, 1]).all())
    assert all(v.dtype == torch.bfloat16 for k, v in w.items() if not k.endswith("table"))
    assert cache_row_elems(mc) == 2 * (6 + 3) + 2 * (6 + 6)      # keys and values of the two attentions
    assert cache_block_bytes(mc) == 32 * 2 * cache_row_elems(mc) and cache_block_bytes(_mc()) == 32 * 4 * cache_row_elems(mc)
    for name, p in PRESETS.items():
        ranks = {f"l{i}.mix.a1": (l.rank, p.hidden) for i, l in enumerate(p.layers) if l.kind == "gla"}
        assert p.arch == "ludelix" and model_config_from_json(config_json(p), None, "bfloat16", ranks).layers == p.layers, name


def test_oracle_masks_and_sink():
    T = 40
    win, chunk = O.window_mask(T, 5), O.chunk_mask(T, 7)
    for i in range(T):
        assert win[i].nonzero().flatten().tolist() == list(range(max(0, i - 4), i + 1))
        assert chunk[i].nonzero().flatten().tolist() == list(range(i // 7 * 7, i + 1))
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(6, 2, 4, generator=g, dtype=F64) for _ in range(3))
    mask = O.window_mask(6, 6)
    none = O.attend(q, k, v, mask, 0.5)
    assert torch.allclose(O.attend(q, k, v, mask, 0.5, torch.full((2,), -1e9, dtype=F64)), none, atol=1e-12)
    s0 = float(q[0, 1] @ k[0, 1] * 0.5)                       # the first token: itself and the sink, which the scale does not touch
    one = O.attend(q, k, v, mask, 0.5, torch.tensor([0.0, 1.25], dtype=F64))
    assert torch.allclose(one[0, 1], v[0, 1] * math.exp(s0) / (math.exp(s0) + math.exp(1.25)), atol=1e-12)


def test_oracle_rotary_layouts_and_scalings():
    x = torch.randn(5, 1, 6, dtype=F64, generator=torch.Generator().manual_seed(2))
    f = O.plain_freqs({"base": 9.0, "dims": 4})
    assert f[0] == 1.0 and abs(f[1] - 1.0 / 3.0) < 1e-15
    c, s = math.cos(3 / 3.0), math.sin(3 / 3.0)
    r = O.rotate(x, f, True)                                  # pair 1 = entries 2 and 3
    assert abs(float(r[3, 0, 2] - (x[3, 0, 2] * c - x[3, 0, 3] * s))) < 1e-12 and abs(float(r[3, 0, 3] - (x[3, 0, 3] * c + x[3, 0, 2] * s))) < 1e-12
    r = O.rotate(x, f, False, 2.0)                            # pair 1 = entries 1 and 3, doubled
    assert abs(float(r[3, 0, 1] - 2 * (x[3, 0, 1] * c - x[3, 0, 3] * s))) < 1e-12 and torch.equal(r[..., 4:], x[..., 4:])
    rot = {"base": 10000.0, "dims": 16, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 100}}
    plain, band = O.plain_freqs(rot), O.banded_freqs(rot)
    kinds = set()
    for p, b in zip(plain, band):
        wave = 2 * math.pi / p
        kinds.add("keep" if wave < 25 else "div" if wave > 100 else "mix")
        if wave < 25:
            assert b == p
        elif wave > 100:
            assert b == p / 8
        else:
            assert p / 8 < b < p
    assert kinds == {"keep", "div", "mix"}
    yf, mag = O.yarn_freqs({"base": 10000.0, "dims": 16, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}})
    assert abs(mag - (0.1 * math.log(8.0) + 1)) < 1e-15 and yf[0] == plain[0] and abs(yf[-1] - plain[-1] / 8) < 1e-12
    assert any(p / 8 * 1.001 < y < p * 0.999 for p, y in zip(plain, yf))


def test_oracle_values_are_projected_keys_and_table_experts():
    g = torch.Generator().manual_seed(3)
    h = torch.randn(1, 8, generator=g, dtype=F64)
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0, "mask": {"size": 3}, "rot": {**ATT["rot"], "dims": 4}}
    w = {n: torch.randn(*s, generator=g, dtype=F64) for n, s in
         {"q": (8, 8), "k": (4, 8), "q.b": (8,), "k.b": (4,), "q.norm": (8,), "k.norm": (4,)}.items()}
    w.update(sink=torch.full((2,), -1e9, dtype=F64), o=torch.eye(8, dtype=F64))
    got = O.shared_attention(h, w, m, 1e-5)[0]                # one token, no sink: the value itself, once per head
    assert torch.allclose(got, (h[0] @ w["k"].T + w["k.b"]).repeat(2), atol=1e-9)
    names = {f"e{e}.{p}": torch.randn(*s, generator=g, dtype=F64) for e in range(3) for p, s in {"gate": (5, 8), "up": (5, 8), "down": (8, 5)}.items()}
    names["table"] = torch.tensor([[0, 2], [1, 0], [2, 1]], dtype=torch.int32)
    y = O.table_ff(h.repeat(2, 1), names, {}, [1, 2])
    assert torch.allclose(y[0], (O.expert(h, names, "e1") + O.expert(h, names, "e0"))[0] / 2, atol=1e-12)
    assert torch.allclose(y[1], (O.expert(h, names, "e2") + O.expert(h, names, "e1"))[0] / 2, atol=1e-12)


def test_oracle_decays_state_and_every_constant_matters():
    q = torch.ones(3, 1, 2, dtype=F64)
    o = O.outer_memory(q, q, torch.ones(3, 1, 1, dtype=F64), torch.tensor([[[0.5, 0.1]]] * 3, dtype=F64))
    assert torch.allclose(o.flatten(), torch.tensor([2.0, 2.6, 1 + 0.5 * 1.5 + 1 + 0.1 * 1.1], dtype=F64))   # rows decay one by one
    mc = _mc()
    weights = synthetic_weights(mc, 5)
    for k in weights:    # sharp attention: single keys decide
        if k.endswith(("left.q", "left.k", "l2.mix.q.norm", "l2.mix.k.norm")):
            weights[k] = weights[k] * 2
    toks = [3, 9, 1, 40, 22, 7, 7, 30, 2, 11, 5, 48, 19, 33, 0, 8, 27, 14, 6, 41]
    runs = []
    logits = O.forward(CFG, weights, toks, runs)
    assert logits.shape == (20, 50) and len(runs) == 4
    assert torch.allclose(O.forward(CFG, weights, toks[:5]), logits[:5], atol=1e-9)         # causal through every mechanism
    assert O.greedy(CFG, weights, toks[:4], 3) == O.greedy(CFG, weights, toks[:4], 5)[:3]

    def changed(edit):
        cfg = copy.deepcopy(CFG)
        edit(cfg)
        return float((O.forward(cfg, weights, toks) - logits).abs().max())

    par, att = (lambda c: c["layers"][1]["mixer"]), (lambda c: c["layers"][2]["mixer"])
    edits = {
        "window + 1": lambda c: att(c)["mask"].update(size=6), "window - 1": lambda c: att(c)["mask"].update(size=4),
        "chunk + 1": lambda c: par(c)["left"]["mask"].update(size=8), "chunk - 1": lambda c: par(c)["left"]["mask"].update(size=6),
        "left base": lambda c: par(c)["left"]["rot"].update(base=150.0), "left dims": lambda c: par(c)["left"]["rot"].update(dims=2),
        "right base": lambda c: par(c)["right"]["rot"].update(dims=4), "band base": lambda c: att(c)["rot"].update(base=90.0),
        "band factor": lambda c: att(c)["rot"]["scaling"].update(factor=2.0), "band low": lambda c: att(c)["rot"]["scaling"].update(low=2.0),
        "band high": lambda c: att(c)["rot"]["scaling"].update(high=6.0), "band original": lambda c: att(c)["rot"]["scaling"].update(original=20),
        "yarn factor": lambda c: par(c)["left"]["rot"]["scaling"].update(factor=4.0), "yarn slow": lambda c: par(c)["left"]["rot"]["scaling"].update(slow=0.05),
        "yarn original": lambda c: par(c)["left"]["rot"]["scaling"].update(original=300),
        "left scale": lambda c: par(c).update(left_scale=0.9), "right scale": lambda c: par(c).update(right_scale=1.5),
        "scale": lambda c: att(c).update(scale=0.8), "decay": lambda c: par(c)["right"].update(decay=[0.5, 0.9, 0.96]),
        "tau": lambda c: c["layers"][0]["mixer"].update(tau=4.0), "eps": lambda c: c["norm"].update(eps=1e-2),
    }
    for name, edit in edits.items():
        assert changed(edit) > 1e-4, name
    for leaf in ("l2.mix.sink", "l2.mix.k.b", "l2.mix.q.b", "l2.mix.q.norm", "l0.mix.norm", "l0.mix.a2.b", "l1.mix.left.g", "l1.mlp.shared.sg", "final.norm"):
        w2 = {**weights, leaf: weights[leaf] + 0.5}
        assert float((O.forward(CFG, w2, toks) - logits).abs().max()) > 1e-3, leaf
    w2 = {**weights, "l1.mlp.table": (weights["l1.mlp.table"] + 1) % 5}
    assert float((O.forward(CFG, w2, toks) - logits).abs().max()) > 1e-3
