"""-m gpu parity of the Bisuzen architecture against oracle/bisuzen_oracle.py.

Kernel level (include/tgis_kernels.h hooks): windowed attention with kept first tokens and a sink, and chunked attention, over a paged
cache in portions, on random inputs and on inputs built so that ONE key decides a query's output -- just inside and just outside a
window or a chunk, among the kept first tokens, on both sides of a cache page's border, far away --, in fp32 and in bf16; the
lightning scan in portions through two state slots; the group-limited router; the sublayer tails.
Engine level (trace replay = the engine's own step function, sequence slots and block manager): every mechanism alone, whole prompts
in fp32 and bf16, portions down to two tokens, token-by-token decoding, mixed batches against each alone with pages and state slots
that are used again, long decoding across window, chunk and page borders, a far kept token that decides, other sizes, loops and
layer orders (values equal to 1, parts absent), and greedy generation through add_request + the step loop with and without
CUDA-graph replay, over gRPC, and through the trace runner's command line."""
import ctypes as C
import json

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

F32, BF16 = 0, 1
KV_BLOCK = 32
F64 = torch.float64
EPS = 1e-5


def _lib():
    from vllm_tgis_adapter_b200.engine import _lib as L

    return L.load_library()


def _p(t):
    return C.c_void_p(t.data_ptr()) if t is not None else None


def _ok(rc):
    assert rc == 0, (_lib().tgis_k_last_error() or b"").decode()


_KEEP = []   # device tensors whose pointers went into a C call stay alive until the test ends


@pytest.fixture(autouse=True)
def _release_device_tensors():
    yield
    _KEEP.clear()


def _dev(t, dt=torch.float32):
    d = t.to(dt).cuda().contiguous()
    _KEEP.append(d)
    return d


def _ints(v):
    return (C.c_int32 * len(v))(*v)


def _i32(v):
    d = torch.tensor(v, dtype=torch.int32).cuda()
    _KEEP.append(d)
    return d


def _portions(total, sizes):
    out, at, i = [], 0, 0
    while at < total:
        n = min(sizes[i % len(sizes)], total - at)
        out.append((at, n))
        at += n
        i += 1
    return out


# ====================================================================================================== attention kernels
def _win(heads, kv_heads, dim, vdim, size, keep, rot_dims, base=300.0, scale=0.3):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size, keep_first=keep),
                rot=dict(base=base, dims=rot_dims))


def _chk(heads, kv_heads, dim, vdim, size, scale=0.6):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size))


def _reference(h, bias, m, sink):
    """The heads' outputs [T, heads * vdim] of columns [q | k | v] through the oracle's functions."""
    from oracle import bisuzen_oracle as O

    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = h.double() + (bias.double() if bias is not None else 0.0)
    q, k, v = h[:, :H * d].view(T, H, d), h[:, H * d:H * d + G * d].view(T, G, d), h[:, H * d + G * d:].view(T, G, dv)
    if "rot" in m:
        q, k = O.rotate_pairs(q, m["rot"]), O.rotate_pairs(k, m["rot"])
        mask = O.window_mask(T, m["mask"]["size"], m["mask"]["keep_first"])
    else:
        q, k = O.rms(q, EPS), O.rms(k, EPS)
        mask = O.chunk_mask(T, m["mask"]["size"])
    return O.attend(q, k, v, mask, m["scale"], sink.double() if sink is not None else None).reshape(T, H * dv)


def _run(h, bias, m, sink, dt, sizes, pool_pages=40, seed=0):
    """h [T, width] = [q | k | v] goes through the kernels in portions over a paged cache whose pages are scattered through the pool."""
    from vllm_tgis_adapter_b200.engine._lib import TgisKPoolAttnGeom

    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    win = "rot" in m
    rd = m["rot"]["dims"] if win else 0
    tdt = torch.bfloat16 if dt == BF16 else torch.float32
    s = _dev(sink) if sink is not None else None
    geom = TgisKPoolAttnGeom(H, G, d, dv, m["mask"]["size"] if win else 0, 0, rd, float(m["scale"]), 0 if win else 1,
                             m["mask"]["keep_first"] if win else 0, 0 if win else m["mask"]["size"], 1, s.data_ptr() if s is not None else None)
    table = None
    if rd > 0:
        f = torch.tensor([m["rot"]["base"] ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=F64)
        ang = torch.arange(T, dtype=F64)[:, None] * f[None, :]
        table = _dev(torch.cat([torch.cos(ang), torch.sin(ang)], -1))
    n_pages = (T + KV_BLOCK - 1) // KV_BLOCK
    pages = torch.randperm(pool_pages, generator=torch.Generator().manual_seed(seed))[:n_pages].tolist()
    kc = torch.randn(pool_pages * KV_BLOCK, G * d, device="cuda").to(tdt)     # stale rows of earlier owners: finite, never visible
    vc = torch.randn(pool_pages * KV_BLOCK, G * dv, device="cuda").to(tdt)
    y = _dev(h)
    b = _dev(bias) if bias is not None else None
    out = torch.full((T, H * dv), float("nan"), dtype=tdt, device="cuda")
    for at, n in _portions(T, sizes):
        pos = list(range(at, at + n))
        slots = [pages[p // KV_BLOCK] * KV_BLOCK + p % KV_BLOCK for p in pos]
        q = torch.zeros(n, H * d, dtype=tdt, device="cuda")
        yp = y[at:at + n].contiguous()
        _ok(_lib().tgis_k_poolattn_prep(_p(yp), y.shape[1], 0, H * d, H * d + G * d, _p(b), C.byref(geom), _p(table), EPS,
                                        _p(_i32(pos)), _p(_i32(slots)), _p(q), _p(kc), _p(vc), dt, n))
        o = torch.full((n, H * dv), float("nan"), dtype=tdt, device="cuda")
        _ok(_lib().tgis_k_poolattn(_p(q), _p(kc), _p(vc), None, None, dt, _ints([0, n, at + n, 0]), 1, _ints(pages), 1, len(pages),
                                   _p(o), C.byref(geom)))
        out[at:at + n] = o
    return out


def _width(m):
    return m["heads"] * m["dim"] + m["kv_heads"] * (m["dim"] + m["vdim"])


_ATTN = [
    _win(4, 2, 6, 10, 9, 3, 4, base=50.0),
    _win(3, 1, 40, 33, 70, 40, 40, base=1000.0, scale=0.2),       # kept tokens on two cache pages
    _win(2, 2, 5, 140, 1, 1, 0),                                  # a window of one token, one kept token, nothing rotates
    _win(2, 1, 8, 8, 33, 0, 8),                                   # no kept tokens
    _chk(3, 1, 7, 9, 10),
    _chk(2, 2, 20, 6, 1),                                         # chunks of one token
    _chk(4, 4, 12, 40, 45, scale=2.0),
    # sizes the tensor-core kernel takes in bf16: several query heads per key/value head in one tile, or one
    _win(6, 2, 96, 200, 100, 5, 96, base=500.0, scale=0.1),
    _win(4, 2, 32, 48, 24, 70, 16, base=20000.0, scale=0.2),
    _win(8, 1, 16, 24, 32, 32, 8),
    _chk(4, 2, 64, 64, 64, scale=0.3),
    _chk(3, 3, 48, 72, 100, scale=0.4),
]


@pytest.mark.parametrize("m", _ATTN)
def test_window_and_chunk_attention_in_portions_matches_oracle(m):
    g = torch.Generator().manual_seed(5)
    T = 300
    h = torch.randn(T, _width(m), generator=g)
    win = "rot" in m
    bias = torch.randn(_width(m), generator=g) * 0.3 if win else None
    sink = torch.randn(m["heads"], generator=g) * 2 + 1 if win else None
    ref = _reference(h, bias, m, sink)
    for sizes in ([T], [3, 1, 40, 2, 64, 1, 1, 17], [1]):
        got = _run(h, bias, m, sink, F32, sizes).double().cpu()
        assert float((got - ref).abs().max()) < 2e-5 * max(1.0, float(ref.abs().max())), sizes
    if m["dim"] % 16 == 0:
        for sizes in ([T], [3, 1, 40, 2, 64, 1, 1, 17], [1]):
            got = _run(h, bias, m, sink, BF16, sizes).double().cpu()
            assert float((got - ref).abs().max()) < 0.06 * max(1.0, float(ref.abs().max())), sizes


@pytest.mark.parametrize("dt,m", [(F32, _ATTN[0]), (F32, _ATTN[1]), (F32, _ATTN[4]), (F32, _ATTN[6]), (BF16, _ATTN[8]), (BF16, _ATTN[9]),
                                  (BF16, _ATTN[10]), (BF16, _ATTN[11])])
def test_one_key_decides_at_window_first_token_chunk_and_page_edges(dt, m):
    """Every key but one points along one axis, the marked key along another, and so does the query under test (nothing rotates
    here); the marked value stands out.  The query either sees the marked key or not at all: a window, a chunk, a kept token or
    a page that is one off changes the output by the marked value's size."""
    m = dict(m, scale=60.0 / m["dim"])
    win = "rot" in m
    if win:
        m["rot"] = dict(m["rot"], dims=0)
    H, G, d, dv, W = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"]
    K = m["mask"].get("keep_first", 0)
    T = 3 * KV_BLOCK + 2 * W + K + 5
    cases = set()
    for j in {0, 1, KV_BLOCK - 1, KV_BLOCK, K - 1, K, K + 1, W - 1, W, 2 * W - 1, 2 * W, 2 * KV_BLOCK + 1}:
        for i in (j, j + 1, j + W - 1, j + W, j + W + 1, W - 1, W, 2 * W - 1, 2 * W, j + 3 * KV_BLOCK, T - 1):
            if 0 <= j <= i < T:
                cases.add((j, i))
    unit = d ** 0.5 if win else 1.0     # (chunked attention norms its queries and keys itself)
    seen = 0
    for j, i in sorted(cases):
        h = torch.zeros(T, _width(m), dtype=F64)
        h[:, 1:H * d:d] = unit                      # every query along axis 1 ...
        h[:, H * d + 1:H * d + G * d:d] = unit      # ... and every key
        h[:, H * d + G * d:] = torch.linspace(-0.1, 0.1, G * dv, dtype=F64)
        h[j, H * d:H * d + G * d] = 0.0
        h[j, H * d:H * d + G * d:d] = unit          # the marked key along axis 0
        h[j, H * d + G * d:] = 7.0                  # its value
        h[i, :H * d] = 0.0
        h[i, 0:H * d:d] = unit                      # the query under test along axis 0
        sink = torch.full((H,), 3.0) if win else None
        ref = _reference(h, None, m, sink)[i]
        seen += int(float(ref[0]) > 5.0)
        got = _run(h.float(), None, m, sink, dt, [j + 1, 2, 33, 1], seed=j)[i].double().cpu()
        assert float((got - ref).abs().max()) < (3e-4 if dt == F32 else 0.08), (j, i, float(ref[0]), float(got[0]))
    assert 0 < seen < len(cases)     # both outcomes occur


def test_sink_of_each_head_takes_its_weight():
    """Sinks that hold from none to all of the softmax's weight, another one per head, among one and among hundreds of keys."""
    for m, dt, tol in ((_win(4, 2, 32, 48, 200, 4, 16), F32, 2e-5), (_win(4, 2, 32, 48, 200, 4, 16), BF16, 0.03), (_win(3, 3, 7, 9, 200, 2, 2), F32, 2e-5)):
        g = torch.Generator().manual_seed(2)
        h = torch.randn(260, _width(m), generator=g)
        sink = torch.tensor([-30.0, 2.0, 5.0, 40.0])[:m["heads"]]
        ref = _reference(h, None, m, sink)
        without = _reference(h, None, m, None)
        per_head = (ref - without).view(260, m["heads"], -1).abs().amax((0, 2))
        assert float(per_head[0]) < 1e-9 and all(float(x) > 0.5 for x in per_head[1:])
        for sizes in ([260], [1]):
            got = _run(h, None, m, sink, dt, sizes).double().cpu()
            assert float((got - ref).abs().max()) < tol * max(1.0, float(ref.abs().max())), (m, dt, sizes)


# ====================================================================================================== lightning attention
@pytest.mark.parametrize("chunked,H,d,dv", [(1, 2, 16, 8), (1, 3, 48, 72), (1, 2, 128, 128), (1, 4, 64, 64), (1, 1, 80, 136), (1, 1, 32, 200)] + [
    (0, *s) for s in [(3, 6, 5), (2, 70, 40), (1, 1, 1), (2, 130, 33), (4, 48, 64), (2, 128, 128), (1, 64, 200)]])
def test_lightning_scan_in_portions_and_two_slots_matches_oracle(chunked, H, d, dv):
    """chunked: the tensor-core form rounds q, k and v to bf16 after silu, and so does the reference here; everything the recurrence
    adds stays fp32-like, so the bound is far below bf16's."""
    from oracle import bisuzen_oracle as O

    g = torch.Generator().manual_seed(3)
    width = 2 * H * d + H * dv
    decay = torch.tensor([0.6, 0.99, 0.999, 0.02][:H]) if H > 1 else torch.tensor([0.97])
    seqs = [torch.randn(330, width, generator=g) * 2.0, torch.randn(150, width, generator=g) * 2.0]
    refs = []
    for h in seqs:
        h = h.double()
        q, k, v = O.silu(h[:, :H * d]).view(-1, H, d), O.silu(h[:, H * d:2 * H * d]).view(-1, H, d), O.silu(h[:, 2 * H * d:]).view(-1, H, dv)
        if chunked:
            q, k, v = (x.float().to(torch.bfloat16).double() for x in (q, k, v))
        S = torch.zeros(H, d, dv, dtype=F64)
        o = []
        for t in range(h.shape[0]):
            S = decay.double()[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            o.append(torch.einsum("hdv,hd->hv", S, q[t]).reshape(-1))
        refs.append(torch.stack(o))
    ys, dec = [_dev(s) for s in seqs], _dev(decay)
    for sizes in ([[5, 1, 40, 2, 17], [33, 1, 1, 64]], [[330], [150]], [[1], [150]], [[16, 100, 15, 65], [2, 3]]):
        S_dev = torch.randn(4, H, d, dv, device="cuda")       # slots 1 and 3 are used; what an earlier owner left is never read
        outs = [torch.zeros(s.shape[0], H * dv, device="cuda") for s in seqs]
        at, step = [0, 0], 0
        while at[0] < seqs[0].shape[0] or at[1] < seqs[1].shape[0]:
            rows, meta, tok_slot, dst = [], [], [], []
            for s in (0, 1):
                n = min(sizes[s][step % len(sizes[s])], seqs[s].shape[0] - at[s])
                if n <= 0:
                    continue
                meta += [sum(r.shape[0] for r in rows), n, at[s] + n, 0]
                rows.append(ys[s][at[s]:at[s] + n])
                tok_slot += [1 + 2 * s] * n
                dst.append((s, at[s], n))
                at[s] += n
            y = torch.cat(rows).contiguous()
            _KEEP.append(y)
            out = torch.zeros(y.shape[0], H * dv, device="cuda")
            _ok(_lib().tgis_k_lightning_scan(_p(y), _p(y[:, H * d:]), _p(y[:, 2 * H * d:]), width, width, width, _p(dec), _p(S_dev), _p(out),
                                             H * dv, H, d, dv, _ints(meta), len(meta) // 4, _p(_i32(tok_slot)), chunked))
            o = 0
            for s, a, n in dst:
                outs[s][a:a + n] = out[o:o + n]
                o += n
            step += 1
        for s in (0, 1):
            err = (outs[s].double().cpu() - refs[s]).abs().max()
            # (a value that sits on a bf16 rounding boundary may round the other way than the reference's)
            assert float(err) < (2e-4 if chunked else 2e-5) * max(1.0, float(refs[s].abs().max())), (sizes, s)


# ====================================================================================================== router and tails
@pytest.mark.parametrize("E,top,count,keep", [(6, 2, 3, 2), (15, 3, 3, 1), (1, 1, 1, 1), (64, 6, 8, 4), (40, 32, 1, 1), (130, 5, 65, 3), (12, 3, 4, 1)])
def test_grouped_router_matches_oracle(E, top, count, keep):
    from oracle import bisuzen_oracle as O

    g = torch.Generator().manual_seed(E)
    T = 37
    for shift in (0.0, -1.5):      # corrections that make every choice score negative
        z = torch.randn(T, E, generator=g) * 2
        corr = torch.randn(E, generator=g) * 0.3 + shift
        ids = torch.full((T, top), -1, dtype=torch.int32, device="cuda")
        w = torch.zeros(T, top, device="cuda")
        _ok(_lib().tgis_k_moe_route_grouped(_p(_dev(z)), E, _p(_dev(corr)), E, top, count, keep, _p(ids), _p(w), T))
        ref = O.route(z.double(), corr.double(), dict(top=top, groups=dict(count=count, keep=keep)))
        for t in range(T):
            got = dict(zip(ids[t].tolist(), w[t].tolist()))
            assert set(got) == {e for e, _ in ref[t]} and len(got) == top, t
            assert all(abs(got[e] - p) < 2e-6 for e, p in ref[t]), t


@pytest.mark.parametrize("hidden", [40, 37, 2048])
def test_sublayer_tails_match_oracle(hidden):
    from oracle import bisuzen_oracle as O

    g = torch.Generator().manual_seed(7)
    T, top, E = 9, 3, 4
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    w = {"n": 1 + rnd(hidden) * 0.1, "n.b": rnd(hidden) * 0.2, "n.alpha": torch.tensor(0.7),
         "i": 1 + rnd(hidden) * 0.1, "i.b": rnd(hidden) * 0.2, "i.alpha": torch.tensor(1.3)}
    d = {k: _dev(v.reshape(-1)) for k, v in w.items()}
    x, ya, yb, ba, wa, wb = rnd(T, hidden) * 2, rnd(T, hidden) * 3, rnd(T, hidden), rnd(hidden), 1 + rnd(hidden) * 0.2, 1 + rnd(hidden) * 0.2
    rows = rnd(T * top, hidden)
    ids = torch.randint(0, E + 2, (T, top), generator=g)        # outputs E and E + 1 are identity experts
    inv = torch.randperm(T * top, generator=g).view(T, top)
    mix = torch.rand(T, top, generator=g)
    X = x.double()
    h = O.dyt(X, w, "i")
    moe = torch.stack([sum(mix[t, k].double() * (rows[inv[t, k]].double() if ids[t, k] < E else h[t]) for k in range(top)) for t in range(T)])
    pair = 0.5 * (O.rms(ya.double() + ba.double(), EPS) * wa.double() + O.rms(yb.double(), EPS) * wb.double())
    cases = {"none": (0.0, [None] * 5, [None] * 4), "plain": (ya.double(), [ya, None, None, None, None], [None] * 4),
             "bias": (ya.double() + ba.double(), [ya, ba, None, None, None], [None] * 4),
             "pair": (pair, [ya, ba, yb, wa, wb], [None] * 4), "moe": (moe, [None] * 5, [rows, inv, ids, mix])}
    for name, (y, mains, mixes) in cases.items():
        for dt, tol in ((F32, 1e-5), (BF16, 1e-2)):
            r = _dev(x)
            out = torch.zeros(T, hidden, dtype=torch.bfloat16 if dt == BF16 else torch.float32, device="cuda")
            m = [_dev(t) if t is not None else None for t in mains]
            q = [_dev(t, torch.int32 if i in (1, 2) else torch.float32) if t is not None else None for i, t in enumerate(mixes)]
            _ok(_lib().tgis_k_dyt_tail(*[_p(t) for t in m], EPS, *[_p(t) for t in q], top, E, _p(d["i"]), _p(d["i.b"]), _p(d["i.alpha"]), _p(r),
                                       _p(d["n"]), _p(d["n.b"]), _p(d["n.alpha"]), 0.5, _p(out), dt, T, hidden))
            new = X + y
            assert float((r.double().cpu() - new).abs().max()) < 1e-5, name
            assert float((out.double().cpu() - 0.5 * O.dyt(new, w, "n")).abs().max()) < tol, name


# ====================================================================================================== engine level
def _par(left, heads=2, dim=5, vdim=4, decay=(0.5, 0.97)):
    return {"left": left, "right": dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay))}


def _moe(experts, identity, top, ff, count=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top,
                                                            "groups": {"count": count, "keep": keep}}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _lay(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _cfg(layers=None, width=40, vocab=97, logit_scale=0.3, loop=(1, 3, 2)):
    if layers is None:
        layers = [_lay("attention", _chk(4, 2, 6, 5, 21), _moe(4, 2, 2, 18, 3, 2)),
                  _lay("parallel", _par(_win(4, 2, 6, 10, 9, 3, 4, base=50.0)), _dense(24)),
                  _lay("attention", _chk(3, 3, 8, 7, 40, scale=1.1), _moe(7, 1, 3, 10)),
                  _lay("parallel", _par(_win(3, 1, 8, 5, 33, 2, 8), heads=1, dim=12, vdim=9, decay=(0.9,)))]
    cfg = {"architecture": "Bisuzen", "width": width, "vocab": vocab, "norm": {"eps": EPS}, "logit_scale": logit_scale, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def _model(cfg, dtype="float32", max_model_len=512):
    from vllm_tgis_adapter_b200.engine.bisuzen import model_config_from_json

    return model_config_from_json(cfg, max_model_len, dtype)


def _weights(mc, seed):
    """Seeded weights whose attention is sharp enough that single keys decide."""
    from vllm_tgis_adapter_b200.engine.bisuzen import synthetic_weights

    w = synthetic_weights(mc, seed)
    for k in w:
        if k.endswith(("left.q", "left.k")):
            w[k] = w[k] * 2
    return w


def _engine(mc, weights, *, blocks=16, seqs=4, graphs=False, tokens=512):
    from vllm_tgis_adapter_b200.engine.core import NativeEngine, cache_block_bytes

    eng = NativeEngine(mc, max_num_seqs=seqs, max_batched_tokens=tokens, kv_cache_bytes=cache_block_bytes(mc) * blocks,
                       use_cuda_graphs=graphs)
    eng.load_weights(weights)
    return eng


def _tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _rel(got, ref):
    """Error of logit rows the way a user sees it: mean removed, root mean square, relative to the rows' own spread."""
    d = torch.as_tensor(got).double() - ref
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / ref.std(-1)).max())


def _bf16_close(got, ref):
    """bf16 operands on widths this small: rounding alone moves single rows by several percent of their spread, and a row whose
    choice of experts is close may take another expert; so the bound is on the typical row and on the bulk (the sharp comparison
    is the float32 one)."""
    rows = sorted(_rel(got[t:t + 1], ref[t:t + 1]) for t in range(len(ref)))
    return rows[len(rows) // 2] < 4e-2 and rows[int(0.9 * len(rows))] < 0.2


def _whole(eng, toks, rid="w"):
    return eng.trace_step([(rid, toks, list(range(len(toks))))], [rid])


def _in_parts(eng, toks, sizes, rid="p"):
    return np.concatenate([eng.trace_step([(rid, toks[a:a + n], list(range(n)))], [rid] if a + n == len(toks) else [])
                           for a, n in _portions(len(toks), sizes)])


TOL = 3e-5


def test_whole_prompt_matches_oracle_fp32_and_bf16():
    from oracle import bisuzen_oracle as O

    cfg = _cfg()
    toks = _tokens(150, 97, 1)
    for dtype in ("float32", "bfloat16"):
        mc = _model(cfg, dtype)
        weights = _weights(mc, 11)
        ref = O.forward(cfg, weights, toks)
        eng = _engine(mc, weights)
        got = _whole(eng, toks)
        if dtype == "float32":
            for n in (1, 2, 3, 4, 5):    # the first tokens of a sequence on their own
                assert _rel(_whole(eng, toks[:n]), O.forward(cfg, weights, toks[:n])) < TOL
        eng.close()
        assert _rel(got, ref) < TOL if dtype == "float32" else _bf16_close(got, ref), dtype


def _alone():
    one = _chk(1, 1, 1, 1, 1)
    return {
        "parallel": dict(layers=[_lay("parallel", _par(_win(4, 2, 6, 10, 9, 3, 4, base=50.0)))]),
        "parallel_whole_head_rotates": dict(layers=[_lay("parallel", _par(_win(3, 3, 8, 5, 40, 1, 8), heads=4, dim=3, vdim=11, decay=(0.1, 0.5, 0.9, 1.0)))]),
        "parallel_nothing_kept": dict(layers=[_lay("parallel", _par(_win(2, 1, 8, 8, 11, 0, 2)))]),
        "parallel_keys_of_70": dict(layers=[_lay("parallel", _par(_win(2, 2, 4, 4, 20, 5, 4), heads=2, dim=70, vdim=35))]),
        "attention": dict(layers=[_lay("attention", _chk(4, 2, 6, 10, 19))]),
        "attention_one_chunk": dict(layers=[_lay("attention", _chk(4, 1, 6, 10, 1000))]),
        "dense": dict(layers=[_lay("attention", one, _dense(50))]),
        "experts": dict(layers=[_lay("attention", one, _moe(6, 0, 2, 30))]),
        "experts_groups_identity": dict(layers=[_lay("attention", one, _moe(9, 3, 3, 16, 4, 2))]),
        "identity_experts_only": dict(layers=[_lay("attention", one, _moe(0, 4, 2, 8, 2, 1))]),
        "loop_of_one_layer_three_passes": dict(layers=[_lay("parallel", _par(_win(2, 1, 8, 8, 11, 3, 4)), _moe(3, 1, 2, 16, 2, 1))], loop=(0, 1, 3)),
    }


@pytest.mark.parametrize("name", list(_alone()))
def test_each_mechanism_alone_whole_and_in_portions(name):
    from oracle import bisuzen_oracle as O

    cfg = _cfg(width=24, vocab=61, **{"loop": None, **_alone()[name]})
    toks = _tokens(90, 61, 4)
    mc = _model(cfg)
    weights = _weights(mc, 17)
    ref = O.forward(cfg, weights, toks)
    eng = _engine(mc, weights)
    whole = _whole(eng, toks)
    parts = _in_parts(eng, toks, [3, 1, 40, 2])
    single = _in_parts(eng, toks[:45], [1])
    eng.close()
    assert _rel(whole, ref) < TOL and _rel(parts, ref) < TOL and _rel(single, ref[:45]) < TOL, name


def _variants():
    return {
        "ones": _cfg([_lay("parallel", _par(_win(1, 1, 2, 1, 1, 1, 2), heads=1, dim=1, vdim=1, decay=(0.5,)), _dense(1)),
                      _lay("attention", _chk(1, 1, 1, 1, 1), _moe(1, 1, 1, 1, 2, 1))], width=6, vocab=11, logit_scale=1.0, loop=(0, 2, 1)),
        "no_loop_no_feed_forward": _cfg([_lay("attention", _chk(2, 2, 10, 6, 16)), _lay("parallel", _par(_win(4, 4, 10, 6, 16, 16, 6), heads=5, dim=9, vdim=10,
                                                                                                    decay=(0.3, 0.5, 0.7, 0.9, 0.99)))], width=30, loop=None),
        "whole_stack_loops_four_times": _cfg([_lay("parallel", _par(_win(2, 1, 12, 12, 50, 4, 6)), _moe(3, 1, 2, 40)),
                                              _lay("attention", _chk(4, 4, 8, 8, 24), _dense(40))], width=32, loop=(0, 2, 4)),
        "loop_in_the_middle_window_longer_than_the_prompt": _cfg(
            [_lay("attention", _chk(2, 2, 32, 32, 70), _dense(64)), _lay("parallel", _par(_win(4, 1, 16, 24, 1000, 8, 16, base=20000.0)), _moe(8, 2, 4, 48, 5, 3)),
             _lay("attention", _chk(4, 1, 16, 24, 33)), _lay("parallel", _par(_win(4, 2, 16, 24, 50, 50, 8), heads=1, dim=64, vdim=64, decay=(0.999,)), _dense(32))],
            width=64, vocab=130, loop=(1, 4, 2)),
        "tensor_core_sizes": _cfg([_lay("parallel", _par(_win(4, 2, 64, 64, 64, 4, 64, scale=0.125), heads=4, dim=64, vdim=64, decay=(0.6, 0.9, 0.97, 0.999)), _dense(512)),
                                   _lay("attention", _chk(4, 4, 32, 96, 100, scale=0.2), _moe(14, 2, 4, 256, 4, 2)),
                                   _lay("parallel", _par(_win(6, 2, 48, 80, 30, 40, 32, scale=0.15), heads=2, dim=128, vdim=128, decay=(0.8, 0.99)), _moe(5, 1, 2, 128, 2, 1)),
                                   _lay("attention", _chk(8, 2, 64, 64, 37, scale=0.2), _dense(256))],
                                  width=256, vocab=300, loop=(0, 2, 2)),
    }


@pytest.mark.parametrize("name", list(_variants()))
def test_other_sizes_orders_loops_and_absent_parts(name):
    from oracle import bisuzen_oracle as O

    cfg = _variants()[name]
    V = cfg["vocab"]
    toks = _tokens(140, V, 6)
    for dtype in ("float32", "bfloat16") if name == "tensor_core_sizes" else ("float32",):
        mc = _model(cfg, dtype)
        weights = _weights(mc, 23)
        ref = O.forward(cfg, weights, toks)
        eng = _engine(mc, weights)
        whole = _whole(eng, toks)
        parts = _in_parts(eng, toks, [2, 45, 1, 1, 33])
        eng.close()
        if dtype == "float32":
            assert _rel(whole, ref) < TOL and _rel(parts, ref) < TOL, name
        else:
            assert _bf16_close(whole, ref) and _bf16_close(parts, ref), name


def test_prefill_portions_and_token_by_token_agree_with_whole_prompt():
    from oracle import bisuzen_oracle as O

    cfg = _cfg()
    mc = _model(cfg)
    weights = _weights(mc, 31)
    toks = _tokens(131, 97, 3)
    ref = O.forward(cfg, weights, toks)
    eng = _engine(mc, weights)
    for sizes in ([2], [1], [31, 33, 2, 64, 1], [64, 1, 1, 1, 1, 1, 1], [9, 37, 8], [20, 2, 19, 2]):
        assert _rel(_in_parts(eng, toks, sizes, "s"), ref) < TOL, sizes
    eng.close()


def test_long_decoding_crosses_window_chunk_and_page_borders_bf16_stays_close():
    from oracle import bisuzen_oracle as O

    cfg = _cfg()
    toks = _tokens(300, 97, 9)
    for dtype in ("float32", "bfloat16"):
        mc = _model(cfg, dtype)
        weights = _weights(mc, 37)
        ref = O.forward(cfg, weights, toks)
        eng = _engine(mc, weights)
        got = [eng.trace_step([("d", toks[:30], list(range(30)))], [])]
        for t in range(30, 300):
            got.append(eng.trace_step([("d", [toks[t]], [0])], ["d"] if t == 299 else []))
        eng.close()
        got = np.concatenate(got)
        assert _rel(got, ref) < TOL if dtype == "float32" else _bf16_close(got, ref), dtype


def test_far_kept_token_decides_hundreds_of_tokens_later():
    """The embedding of one token turns its key towards every query: as one of the kept first tokens it decides the output at any
    distance, in a prompt and decoded; one place further it is gone with the window."""
    from oracle import bisuzen_oracle as O

    cfg = _cfg([_lay("parallel", _par(_win(2, 1, 16, 16, 24, 3, 2, base=1e6, scale=0.5)))], width=64, vocab=61, loop=None)
    for dtype in ("float32", "bfloat16"):
        mc = _model(cfg, dtype)
        weights = _weights(mc, 19)
        weights["l0.mix.left.q.b"] = torch.full((32,), 1.5).to(torch.bfloat16)         # a direction all queries share ...
        weights["l0.mix.left.k"] = weights["l0.mix.left.k"] * 0.2
        v = weights["l0.mix.left.k"].float()
        # ... and a token whose key lies along it: solve for a normed input that maps to it, stretched so that tanh keeps its signs
        x = torch.linalg.lstsq(v, torch.full((16, 1), 2.0)).solution[:, 0]
        weights["embed"][60] = (x * 20).to(torch.bfloat16)
        base = _tokens(390, 60, 8)
        for place in (2, 3):       # the last kept token, and the first one that is not
            toks = list(base)
            toks[place] = 60
            ref, plain = O.forward(cfg, weights, toks), O.forward(cfg, weights, base)
            far = _rel(plain[340:].numpy(), ref[340:])     # what the marked token changes behind the window
            assert far > 0.05 if place == 2 else far < 0.01
            eng = _engine(mc, weights)
            got = [eng.trace_step([("d", toks[:350], list(range(350)))], [])]
            for t in range(350, 390):
                got.append(eng.trace_step([("d", [toks[t]], [0])], ["d"] if t == 389 else []))
            eng.close()
            got = np.concatenate(got)
            assert _rel(got, ref) < TOL if dtype == "float32" else _bf16_close(got, ref), (dtype, place)


def test_mixed_batches_of_unequal_requests_match_each_alone_and_reuse_pages_and_slots():
    from oracle import bisuzen_oracle as O

    cfg = _cfg()
    mc = _model(cfg)
    weights = _weights(mc, 41)
    reqs = {f"q{i}": _tokens(n, 97, 50 + i) for i, n in enumerate([97, 40, 3, 130, 64, 33, 71, 1, 90])}
    ref = {k: O.forward(cfg, weights, v) for k, v in reqs.items()}
    # 3 slots and a pool of 10 pages: the requests only fit because finished ones give their state slot and pages back
    eng = _engine(mc, weights, blocks=10, seqs=3)
    at = {k: 0 for k in reqs}
    got = {k: [] for k in reqs}
    nb = lambda k: (len(reqs[k]) + KV_BLOCK - 1) // KV_BLOCK  # noqa: E731
    waiting, live, step = list(reqs), [], 0
    while waiting or live:
        while waiting and len(live) < 3 and sum(nb(k) for k in live) + nb(waiting[0]) <= 10:
            live.append(waiting.pop(0))
        entries, ends = [], []
        for j, k in enumerate(live):
            if (step + j) % 5 == 4:
                continue                                        # a request may sit a step out
            n = min(len(reqs[k]) - at[k], [1, 7, 2, 29, 1, 33][(step + 2 * j) % 6])   # single tokens beside portions
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(reqs[k]):
                ends.append(k)
        if entries:
            out = eng.trace_step(entries, ends)
            o = 0
            for k, t, _ in entries:
                got[k].append(out[o:o + len(t)])
                o += len(t)
        live = [k for k in live if k not in ends]
        step += 1
    st = eng.status()
    eng.close()
    assert st.free_blocks == st.total_blocks == 10
    for k in reqs:
        assert _rel(np.concatenate(got[k]), ref[k]) < TOL, k


def test_greedy_generation_through_the_scheduler_matches_oracle():
    from oracle import bisuzen_oracle as O
    from vllm_tgis_adapter_b200.engine.core import make_sampling_params

    cfg = _cfg(logit_scale=1.5)
    mc = _model(cfg)
    weights = _weights(mc, 61)
    prompts = [_tokens(45, 97, 70), _tokens(3, 97, 71), _tokens(80, 97, 72)]
    n_new = 40
    want = [O.greedy(cfg, weights, p, n_new) for p in prompts]
    for graphs in (False, True):
        eng = _engine(mc, weights, graphs=graphs, tokens=64)     # 64-token steps: the prompts are prefilled in portions
        sp = make_sampling_params(greedy=True, max_tokens=n_new, min_tokens=n_new, eos_token_id=-1, num_logprobs=1)
        outs = eng.generate_sync(prompts, sp)
        st = eng.status()
        eng.close()
        assert st.errored == 0 and (st.graph_launches > 0) == graphs
        for p, w, recs in zip(prompts, want, outs):
            toks = [r.new_token for r in recs if r.new_token is not None]
            assert toks == w, graphs
            lp = torch.log_softmax(O.forward(cfg, weights, p + toks[:-1])[len(p) - 1:], -1)
            for i, r in enumerate([r for r in recs if r.new_token is not None]):
                assert abs(r.logprob - float(lp[i, r.new_token])) < 1e-3


def test_generate_over_grpc_matches_oracle():
    """grpc client -> TextGenerationService -> AsyncTGISEngine -> the engine's step loop on a Bisuzen preset (float32): greedy
    tokens and their logprobs of a batched Generate call against the oracle."""
    from test_server_gpu import LiveServer

    from oracle import bisuzen_oracle as O
    from vllm_tgis_adapter_b200.engine.bisuzen import config_json
    from vllm_tgis_adapter_b200.engine.tokenizer import synthetic_prompt
    from vllm_tgis_adapter_b200.grpc.pb import generation_pb2 as pb

    srv = LiveServer("bisuzen-tiny", seed=29)
    try:
        cfg = config_json(srv.cfg.model_config)
        rs = np.random.RandomState(5)
        prompts = [rs.randint(3, srv.cfg.vocab, size=n).tolist() for n in (12, 70, 7)]     # 70: prefilled in two portions
        params = pb.Parameters()
        params.stopping.max_new_tokens = 10
        params.stopping.min_new_tokens = 10
        params.response.generated_tokens = True
        params.response.token_logprobs = True
        call = srv.channel.unary_unary("/fmaas.GenerationService/Generate",
                                       request_serializer=pb.BatchedGenerationRequest.SerializeToString,
                                       response_deserializer=pb.BatchedGenerationResponse.FromString)
        resp = call(pb.BatchedGenerationRequest(model_id="m", requests=[pb.GenerationRequest(text=synthetic_prompt(p)) for p in prompts],
                                                params=params), timeout=120)
    finally:
        srv.close()
    assert len(resp.responses) == 3
    for p, r in zip(prompts, resp.responses):
        assert r.input_token_count == len(p) and r.generated_token_count == 10
        got = [int(t.text[1:]) for t in r.tokens]
        assert got == O.greedy(cfg, srv.weights, p, 10)
        lp = torch.log_softmax(O.forward(cfg, srv.weights, p + got[:-1])[len(p) - 1:], -1)
        for i, t in enumerate(r.tokens):
            assert abs(t.logprob - float(lp[i, got[i]])) < 1e-3


def test_trace_runner_command_line_on_a_model_directory(tmp_path):
    """bin/trace_run on a directory with config.json + model.safetensors: the family, the loop and every size come from the
    files, a mixed schedule with a reused slot goes through standard input, the logits land in the output folder."""
    import subprocess
    import sys
    from pathlib import Path

    from safetensors.torch import save_file

    from oracle import bisuzen_oracle as O

    cfg = _cfg()
    weights = _weights(_model(cfg), 71)
    model = tmp_path / "model"
    model.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(model / "model.safetensors"))
    a, b, c = _tokens(70, 97, 1), _tokens(9, 97, 2), _tokens(40, 97, 3)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}, {"id": "b", "tokens": b[:2], "want": [1]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [6]}, {"id": "a", "tokens": a[33:69], "want": []}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[69:], "want": [0]}, {"id": "c", "tokens": c, "want": [39]}], "end": ["a", "c"]},
    ]
    want = {0: [("a", 0), ("a", 32), ("b", 1)], 1: [("b", 8)], 2: [("a", 69), ("c", 39)]}
    ref = {"a": O.forward(cfg, weights, a), "b": O.forward(cfg, weights, b), "c": O.forward(cfg, weights, c)}
    root = Path(__file__).resolve().parent.parent
    for dtype, tol in (("float32", TOL), ("bfloat16", 0.3)):
        out = tmp_path / f"out_{dtype}"
        p = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        for n, rows in want.items():
            got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(rows), -1)
            for g, (rid, pos) in zip(got, rows):
                assert _rel(g[None], ref[rid][pos:pos + 1]) < tol, (dtype, n, rid, pos)
