"""CPU-side checks of the Bisuzen family: config.json -> engine specs, the parameter list, layer runs of a loop, cache accounting,
presets, and properties of the plain oracle that the GPU tests lean on (edges of windows, kept first tokens and chunks, the sink, the
rotary layout, the router's groups and identity experts, state carried token by token)."""
import copy
import math

import pytest
import torch

from oracle import bisuzen_oracle as O
from vllm_tgis_adapter_b200.engine import _lib
from vllm_tgis_adapter_b200.engine.bisuzen import (PRESETS, cache_row_elems, config_json, layer_runs, model_config_from_json, model_spec,
                                                   synthetic_weights, tensor_shapes)
from vllm_tgis_adapter_b200.engine.core import cache_block_bytes

F64 = torch.float64
LEFT = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "scale": 0.9, "mask": {"size": 7, "keep_first": 2}, "rot": {"base": 100.0, "dims": 4}}
RIGHT = {"heads": 2, "dim": 5, "vdim": 4, "decay": [0.5, 0.95]}
MOE = {"kind": "moe", "expert": {"ff": 9},
       "router": {"experts": 5, "identity": 1, "top": 2, "groups": {"count": 3, "keep": 2}}}
CFG = {
    "architecture": "Bisuzen", "width": 24, "vocab": 50, "norm": {"eps": 1e-3}, "logit_scale": 0.4,
    "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [
        {"type": "attention", "mixer": {"heads": 3, "kv_heads": 1, "dim": 4, "vdim": 5, "scale": 0.7, "mask": {"size": 6}}, "mlp": None},
        {"type": "parallel", "mixer": {"left": LEFT, "right": RIGHT}, "mlp": {"kind": "dense", "ff": 11}},
        {"type": "attention", "mixer": {"heads": 2, "kv_heads": 2, "dim": 4, "vdim": 4, "scale": 1.5, "mask": {"size": 9}}, "mlp": MOE},
        {"type": "parallel", "mixer": {"left": {**LEFT, "heads": 2}, "right": {**RIGHT, "heads": 1, "decay": [0.9]}}, "mlp": MOE},
    ],
}


def test_config_json_to_specs():
    mc = model_config_from_json(CFG, 256, "float32")
    assert (mc.arch, mc.hidden, mc.vocab, mc.n_layers, mc.max_model_len, mc.rms_eps, mc.dtype) == ("bisuzen", 24, 50, 4, 256, 1e-3, "float32")
    assert (mc.logit_scale, mc.loop) == (0.4, (1, 3, 3))
    a, b, c, d = mc.layers
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.window, a.ff, a.moe) == ("attention", 3, 1, 4, 5, 0.7, 6, 0, 0, False)
    assert (b.kind, b.heads, b.kv_heads, b.dim, b.vdim, b.window, b.keep_first, b.rot_dims, b.rot_base, b.ff) == \
        ("parallel", 4, 2, 6, 3, 7, 2, 4, 100.0, 11)
    assert (b.lin_heads, b.lin_dim, b.lin_vdim, b.decay) == (2, 5, 4, (0.5, 0.95))
    assert (c.experts, c.identity, c.top, c.expert_ff, c.groups, c.groups_keep, c.ff) == (5, 1, 2, 9, 3, 2, 0)
    spec, keep = model_spec(mc)
    specs = keep[0]
    assert (spec.n_layers, spec.dtype, spec.style, spec.loop_add_embed) == (4, _lib.DTYPE_F32, _lib.STYLE_PRE_DYT, 0)
    assert (spec.loop_start, spec.loop_stop, spec.loop_times) == (1, 3, 3) and abs(spec.logit_scale - 0.4) < 1e-7
    assert [s.mixer for s in specs] == [_lib.MIXER_POOLED_ATTENTION, _lib.MIXER_WINDOW_LIGHTNING, _lib.MIXER_POOLED_ATTENTION,
                                        _lib.MIXER_WINDOW_LIGHTNING]
    assert [s.mlp for s in specs] == [_lib.MLP_NONE, _lib.MLP_DENSE_GELU, _lib.MLP_MOE_GROUPED, _lib.MLP_MOE_GROUPED]
    assert specs[0].flags == _lib.LAYER_UNIT_QK and (specs[0].chunk, specs[0].window) == (6, 0)
    assert specs[1].flags == _lib.LAYER_QKV_BIAS | _lib.LAYER_OUT_BIAS | _lib.LAYER_ROT_INTERLEAVED | _lib.LAYER_SINK
    assert (specs[1].window, specs[1].keep_first, specs[1].chunk, specs[1].pool) == (7, 2, 0, 0)
    assert [round(specs[1].decay[i], 6) for i in range(2)] == [0.5, 0.95]
    assert (specs[2].experts, specs[2].identity, specs[2].expert_groups, specs[2].expert_groups_keep) == (5, 1, 3, 2)
    back = model_config_from_json(config_json(mc), 256, "float32")
    assert back.layers == mc.layers and back.loop == mc.loop and back.logit_scale == mc.logit_scale      # round trip
    for bad in ({"type": "something_else"}, {"mlp": {"kind": "other"}}):
        with pytest.raises(ValueError):
            model_config_from_json({**CFG, "layers": [{**CFG["layers"][0], **bad}]}, None)
    with pytest.raises(ValueError):   # one decay per head
        model_config_from_json({**CFG, "layers": [{**CFG["layers"][1], "mixer": {"left": LEFT, "right": {**RIGHT, "heads": 3}}}]}, None)
    empty, _ = model_spec(model_config_from_json({**CFG, "loop": {"start": 2, "stop": 2, "times": 4}}, None))
    assert (empty.loop_start, empty.loop_stop, empty.loop_times) == (0, 0, 1)
    plain = model_config_from_json({k: v for k, v in CFG.items() if k not in ("loop", "logit_scale")}, None)
    assert (plain.loop[2], plain.logit_scale) == (1, 1.0)


def test_layer_runs_and_cache_accounting():
    mc = model_config_from_json(CFG, 256)
    assert layer_runs(mc) == [0, 1, 2, 1, 2, 1, 2, 3] == O.layer_runs(CFG)
    # rows per token: one run of layer 0 (1 kv head x (4 + 5)), three of layer 1 (2 x (6 + 3)) and 2 (2 x (4 + 4)), one of layer 3
    assert cache_row_elems(mc) == 9 + 3 * 18 + 3 * 16 + 18
    assert cache_block_bytes(mc) == 32 * 2 * cache_row_elems(mc)
    assert layer_runs(model_config_from_json({**CFG, "loop": {"start": 0, "stop": 4, "times": 1}}, 256)) == [0, 1, 2, 3]
    assert layer_runs(model_config_from_json({**CFG, "loop": {"start": 0, "stop": 4, "times": 2}}, 256)) == [0, 1, 2, 3, 0, 1, 2, 3]


def test_parameter_list_and_presets():
    mc = model_config_from_json(CFG, 256)
    shapes = tensor_shapes(mc)
    assert shapes["embed"] == shapes["head"] == (50, 24) and shapes["final.norm"] == shapes["final.norm.b"] == (24,) and shapes["final.norm.alpha"] == ()
    assert "l0.norm2" not in shapes and "l0.mix.q.b" not in shapes and shapes["l1.norm2.alpha"] == ()
    assert shapes["l1.mix.left.k.b"] == (12,) and shapes["l1.mix.left.o.b"] == (24,) and shapes["l1.mix.left.sink"] == (4,)
    assert shapes["l1.mix.right.q"] == (10, 24) and shapes["l1.mix.right.g"] == (8, 24) and shapes["l1.mix.right.norm"] == (8,)
    assert shapes["l2.mlp.router"] == (6, 24) and shapes["l2.mlp.correction"] == (6,) and "l2.mlp.e4.up" in shapes and "l2.mlp.e5.up" not in shapes
    w = synthetic_weights(mc, 3)
    assert set(w) == set(shapes) and all(tuple(w[k].shape) == shapes[k] and w[k].dtype == torch.bfloat16 for k in shapes)
    for name, p in PRESETS.items():
        assert p.arch == "bisuzen" and model_config_from_json(config_json(p), None).layers == p.layers, name
        for l in p.layers:
            assert l.rot_dims % 2 == 0 and l.heads % l.kv_heads == 0 and (l.experts + l.identity) % l.groups == 0
            assert not l.moe or l.top <= (l.experts + l.identity) // l.groups * l.groups_keep


def test_oracle_masks():
    T = 40
    win, chunk = O.window_mask(T, 5, 3), O.chunk_mask(T, 7)
    for i in range(T):
        assert win[i].nonzero().flatten().tolist() == sorted({j for j in range(i + 1) if i - j < 5} | {j for j in range(3) if j <= i})
        assert chunk[i].nonzero().flatten().tolist() == list(range(i // 7 * 7, i + 1))
    assert O.window_mask(T, 5, 0).sum() == O.window_mask(T, 5, 1).sum() - (T - 5)


def test_oracle_sink_and_rotary_layout():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(6, 2, 4, generator=g, dtype=F64) for _ in range(3))
    mask = O.chunk_mask(6, 6)
    none = O.attend(q, k, v, mask, 0.5)
    assert torch.allclose(O.attend(q, k, v, mask, 0.5, torch.full((2,), -1e9, dtype=F64)), none, atol=1e-12)
    assert float(O.attend(q, k, v, mask, 0.5, torch.full((2,), 60.0, dtype=F64)).abs().max()) < 1e-20
    s0 = float(q[0, 1] @ k[0, 1] * 0.5)                       # the first token: itself and the sink, which the scale does not touch
    one = O.attend(q, k, v, mask, 0.5, torch.tensor([0.0, 1.25], dtype=F64))
    assert torch.allclose(one[0, 1], v[0, 1] * math.exp(s0) / (math.exp(s0) + math.exp(1.25)), atol=1e-12)
    x = torch.randn(5, 1, 6, generator=g, dtype=F64)
    r = O.rotate_pairs(x, {"base": 9.0, "dims": 4})
    c, s = math.cos(3 / 3.0), math.sin(3 / 3.0)               # pair 1 (entries 2 and 3) turns by t / 3
    assert abs(float(r[3, 0, 2] - (x[3, 0, 2] * c - x[3, 0, 3] * s))) < 1e-12 and abs(float(r[3, 0, 3] - (x[3, 0, 3] * c + x[3, 0, 2] * s))) < 1e-12
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.equal(r[0], x[0])


def test_oracle_router_groups_and_identity():
    r = dict(experts=4, identity=2, top=2, groups=dict(count=3, keep=1))
    z = torch.log(torch.tensor([[0.05, 0.30, 0.25, 0.24, 0.10, 0.06]], dtype=F64))
    zero = torch.zeros(6, dtype=F64)
    (pairs,) = O.route(z, zero, r)
    assert [e for e, _ in pairs] == [1, 0] and abs(pairs[0][1] - 0.30 / 0.35) < 1e-12      # the best group holds 0.30; its weak member follows
    (pairs,) = O.route(z, torch.tensor([0, 0, 0, 0, 0.0, 0.5], dtype=F64), r)
    assert [e for e, _ in pairs] == [5, 4] and abs(pairs[0][1] - 0.06 / 0.16) < 1e-12      # the correction chooses, it does not weigh
    (pairs,) = O.route(z, torch.full((6,), -2.0, dtype=F64), r)                            # negative choice scores: the others are out, not zero
    assert [e for e, _ in pairs] == [1, 0]
    h = torch.randn(1, 3, dtype=F64)
    w = {"router": torch.zeros(2, 3, dtype=F64), "correction": torch.tensor([0.0, 1.0], dtype=F64)}
    assert torch.allclose(O.moe_ff(h, w, dict(experts=0, identity=2, top=1)), h)           # an identity expert hands its input on


def test_oracle_state_loop_and_every_constant_matters():
    mc = model_config_from_json(CFG, 64)
    weights = synthetic_weights(mc, 5)
    for k in weights:    # sharp attention: single keys decide
        if k.endswith((".mix.q", ".mix.k", "left.q", "left.k")):
            weights[k] = weights[k] * 3
    toks = [3, 9, 1, 40, 22, 7, 7, 30, 2, 11, 5, 48, 19, 33, 0, 8, 27, 14, 6, 41]
    runs = []
    logits = O.forward(CFG, weights, toks, runs)
    assert logits.shape == (20, 50) and len(runs) == 8
    assert torch.allclose(O.forward(CFG, weights, toks[:5]), logits[:5], atol=1e-9)         # causal through every mechanism
    assert O.greedy(CFG, weights, toks[:4], 3) == O.greedy(CFG, weights, toks[:4], 5)[:3]

    def changed(edit):
        cfg = copy.deepcopy(CFG)
        edit(cfg)
        return float((O.forward(cfg, weights, toks) - logits).abs().max())

    left, right = (lambda c: c["layers"][1]["mixer"]["left"]), (lambda c: c["layers"][1]["mixer"]["right"])
    edits = {
        "window + 1": lambda c: left(c)["mask"].update(size=8), "window - 1": lambda c: left(c)["mask"].update(size=6),
        "kept + 1": lambda c: left(c)["mask"].update(keep_first=3), "kept - 1": lambda c: left(c)["mask"].update(keep_first=1),
        "chunk + 1": lambda c: c["layers"][0]["mixer"]["mask"].update(size=7), "chunk - 1": lambda c: c["layers"][2]["mixer"]["mask"].update(size=8),
        "rotary base": lambda c: left(c)["rot"].update(base=101.0), "rotary dims": lambda c: left(c)["rot"].update(dims=2),
        "scale": lambda c: left(c).update(scale=0.91), "decay": lambda c: right(c).update(decay=[0.5, 0.96]),
        "passes": lambda c: c["loop"].update(times=2), "span": lambda c: c["loop"].update(stop=2), "logit scale": lambda c: c.update(logit_scale=0.41),
        "groups kept": lambda c: c["layers"][2]["mlp"]["router"]["groups"].update(keep=1), "eps": lambda c: c["norm"].update(eps=1e-2),
    }
    for name, edit in edits.items():
        assert changed(edit) > 1e-3, name
    for leaf in ("l1.mix.left.sink", "l1.mix.left.o.b", "l1.mix.left.v.b", "l1.mix.right.norm", "l2.mlp.correction", "l3.norm2.b", "final.norm.alpha"):
        w2 = {**weights, leaf: weights[leaf] + 0.5}
        assert float((O.forward(CFG, w2, toks) - logits).abs().max()) > 1e-3, leaf
