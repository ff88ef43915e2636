"""-m gpu parity of the Ludelix architecture against oracle/ludelix_oracle.py.

Kernel level (include/tgis_kernels.h hooks): windowed attention with a sink whose values are the projected keys (queries and keys
normed over all heads, frequencies scaled by wavelength) and chunked attention with a gate per head, over a paged cache in portions,
on random inputs and on inputs built so that ONE key decides a query's output -- just inside and just outside a window or a chunk, on
both sides of a cache page's border --, in fp32 and in bf16; retention and gated linear attention in portions through two state
slots, chunk by chunk and token by token, strong decays among them; the row lists of table-routed experts; the sublayer tail.
Engine level (trace replay = the engine's own step function, sequence slots and block manager): every mechanism alone, whole prompts
in fp32 and bf16, portions down to two tokens, token-by-token decoding, mixed batches against each alone with pages and state slots
that are used again, long decoding across window, chunk and page borders, a far token that decides through each memory, other sizes
and layer orders (values equal to 1, parts absent), and greedy generation through add_request + the step loop with and without
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
def _win(heads, kv_heads, dim, size, rot_dims, base=300.0, scale=0.3, factor=4.0, low=1.0, high=3.0, original=80):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, mask=dict(size=size), rot=dict(base=base, dims=rot_dims))
    m["rot"]["scaling"] = dict(factor=factor, low=low, high=high, original=original)
    return m


def _chk(heads, kv_heads, dim, vdim, size, rot_dims, base=200.0, scale=0.4, factor=2.5, original=90, fast=6.0, slow=1.0):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=size), rot=dict(base=base, dims=rot_dims))
    m["rot"]["scaling"] = dict(factor=factor, original=original, fast=fast, slow=slow)
    return m


def _is_win(m):
    return "low" in m["rot"]["scaling"]


def _width(m):   # windowed: [q | k]; chunked: [q | k | v | gate logits]
    w = (m["heads"] + m["kv_heads"]) * m["dim"]
    return w if _is_win(m) else w + m["kv_heads"] * m["vdim"] + m["heads"]


def _freqs(m):
    from oracle import ludelix_oracle as O

    if m["rot"]["dims"] == 0:
        return [], 1.0
    return (O.banded_freqs(m["rot"]), 1.0) if _is_win(m) else O.yarn_freqs(m["rot"])


def _reference(h, bias, m, sink, norms, mul):
    """The heads' outputs [T, heads * vdim] of the projected columns through the oracle's functions."""
    from oracle import ludelix_oracle as O

    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = h.double()
    nq, nk = H * d, G * d
    if bias is not None:
        h = torch.cat([h[:, :nq + nk] + bias.double(), h[:, nq + nk:]], 1)
    q, k = h[:, :nq], h[:, nq:nq + nk]
    f, mag = _freqs(m)
    if _is_win(m):
        v = k.view(T, G, d)
        if norms is not None:
            q, k = O.rms(q, EPS) * norms[0].double(), O.rms(k, EPS) * norms[1].double()
        q, k = O.rotate(q.reshape(T, H, d), f, True), O.rotate(k.reshape(T, G, d), f, True)
        return O.attend(q, k, v, O.window_mask(T, m["mask"]["size"]), m["scale"], sink.double()).reshape(T, H * d) * mul
    q, k = O.rotate(q.reshape(T, H, d), f, False, mag), O.rotate(k.reshape(T, G, d), f, False, mag)
    v, gate = h[:, nq + nk:nq + nk + G * dv].reshape(T, G, dv), torch.sigmoid(h[:, nq + nk + G * dv:])
    o = O.attend(q, k, v, O.chunk_mask(T, m["mask"]["size"]), m["scale"])
    return (o * gate[:, :, None] * mul).reshape(T, H * dv)


def _run(h, bias, m, sink, norms, mul, dt, sizes, pool_pages=40, seed=0, pad=6):
    """h [T, width] goes through the kernels in portions over a paged cache whose pages are scattered through the pool; output rows
    are `pad` elements further apart than they are long."""
    from vllm_tgis_adapter_b200.engine._lib import TgisKPoolAttnGeom

    T = h.shape[0]
    H, G, d, dv, win = m["heads"], m["kv_heads"], m["dim"], m["vdim"], _is_win(m)
    nq, nk, rd = H * d, G * d, m["rot"]["dims"]
    tdt = torch.bfloat16 if dt == BF16 else torch.float32
    y, ld = _dev(h), H * dv + pad
    s = _dev(sink) if win else None
    nrm = [_dev(n) for n in norms] if norms is not None else [None, None]
    geom = TgisKPoolAttnGeom(H, G, d, dv, m["mask"]["size"] if win else 0, 0, rd, float(m["scale"]), 0, 0, 0 if win else m["mask"]["size"],
                             1 if win else 0, s.data_ptr() if win else None, None, y.shape[1], ld, float(mul), 0,
                             *[n.data_ptr() if n is not None else None for n in nrm])
    table = None
    if rd > 0:
        f, mag = _freqs(m)
        ang = torch.arange(T, dtype=F64)[:, None] * torch.tensor(f, dtype=F64)[None, :]
        table = _dev(torch.cat([mag * torch.cos(ang), mag * torch.sin(ang)], -1))
    n_pages = (T + KV_BLOCK - 1) // KV_BLOCK
    pages = torch.randperm(pool_pages, generator=torch.Generator().manual_seed(seed))[:n_pages].tolist()
    kc = torch.randn(pool_pages * KV_BLOCK, nk, device="cuda").to(tdt)         # stale rows of earlier owners: finite, never visible
    vc = torch.randn(pool_pages * KV_BLOCK, G * dv, device="cuda").to(tdt)
    b = _dev(bias) if bias is not None else None
    out = torch.full((T, H * dv), float("nan"), dtype=tdt, device="cuda")
    for at, n in _portions(T, sizes):
        pos = list(range(at, at + n))
        slots = [pages[p // KV_BLOCK] * KV_BLOCK + p % KV_BLOCK for p in pos]
        q = torch.zeros(n, nq, dtype=tdt, device="cuda")
        yp = y[at:at + n].contiguous()
        if not win:
            geom.head_gate = yp.data_ptr() + 4 * (nq + nk + G * dv)
        _ok(_lib().tgis_k_poolattn_prep(_p(yp), y.shape[1], 0, nq, nq if win else nq + nk, _p(b), C.byref(geom), _p(table), EPS,
                                        _p(_i32(pos)), _p(_i32(slots)), _p(q), _p(kc), _p(vc), dt, n))
        o = torch.full((n, ld), float("nan"), dtype=tdt, device="cuda")
        _ok(_lib().tgis_k_poolattn(_p(q), _p(kc), _p(vc), None, None, dt, _ints([0, n, at + n, 0]), 1, _ints(pages), 1, len(pages),
                                   _p(o), C.byref(geom)))
        assert bool(o[:, H * dv:].isnan().all())       # nothing beside the row is touched
        out[at:at + n] = o[:, :H * dv]
    return out


_ATTN = [
    _win(4, 2, 6, 9, 4, base=50.0),
    _win(3, 1, 40, 70, 40, base=1000.0, scale=0.2),
    _win(2, 2, 5, 1, 0),                                          # a window of one token, nothing rotates
    _win(2, 1, 8, 33, 8, factor=1.0),
    _chk(3, 1, 7, 9, 10, 4),
    _chk(2, 2, 20, 6, 1, 20),                                     # chunks of one token
    _chk(4, 4, 12, 40, 45, 6, scale=1.0),
    # sizes the tensor-core kernel takes in bf16: several query heads per key/value head in one tile, or one
    _win(6, 2, 80, 100, 64, base=500.0, scale=0.1),
    _win(4, 2, 32, 24, 16, base=20000.0, scale=0.2),
    _win(8, 1, 16, 32, 8),
    _chk(4, 2, 64, 64, 64, 64, scale=0.2),
    _chk(3, 3, 48, 72, 100, 24, scale=0.2),
    _chk(10, 2, 128, 128, 130, 128, scale=0.1),
]


@pytest.mark.parametrize("m", _ATTN)
def test_window_and_chunk_attention_in_portions_matches_oracle(m):
    g = torch.Generator().manual_seed(5)
    T = 300
    h = torch.randn(T, _width(m), generator=g)
    nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
    win = _is_win(m)
    bias = torch.randn(nq + nk, generator=g) * 0.3 if win else None
    sink = torch.randn(m["heads"], generator=g) * 2 + 1 if win else None
    norms = (1.5 + torch.randn(nq, generator=g) * 0.3, 1.5 + torch.randn(nk, generator=g) * 0.3) if win else None
    mul = 1.0 if win else 0.6
    ref = _reference(h, bias, m, sink, norms, mul)
    for dt in (F32, BF16) if m["dim"] % 16 == 0 else (F32,):
        for sizes in ([T], [3, 1, 40, 2, 64, 1, 1, 17], [1]):
            got = _run(h, bias, m, sink, norms, mul, dt, sizes).double().cpu()
            tol = 2e-5 if dt == F32 else 0.06
            assert float((got - ref).abs().max()) < tol * max(1.0, float(ref.abs().max())), (dt, sizes)


@pytest.mark.parametrize("dt,m", [(F32, _ATTN[0]), (F32, _ATTN[1]), (F32, _ATTN[4]), (F32, _ATTN[6]), (BF16, _ATTN[8]), (BF16, _ATTN[9]),
                                  (BF16, _ATTN[10]), (BF16, _ATTN[11])])
def test_one_key_decides_at_window_chunk_and_page_edges(dt, m):
    """Every key but one points along one axis, the marked key along another, and so does the query under test (nothing rotates and
    nothing is normed here); the marked value stands out.  The query either sees the marked key or not at all: a window, a chunk or
    a page that is one off changes the output by the marked value's size."""
    win = _is_win(m)
    m = dict(m, scale=60.0, rot=dict(m["rot"], dims=0))
    H, G, d, dv, W = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"]
    nq, nk = H * d, G * d
    T = 3 * KV_BLOCK + 2 * W + 5
    cases = set()
    for j in {0, 1, KV_BLOCK - 1, KV_BLOCK, W - 1, W, 2 * W - 1, 2 * W, 2 * KV_BLOCK + 1}:
        for i in (j, j + 1, j + W - 1, j + W, j + W + 1, W - 1, W, 2 * W - 1, 2 * W, j + 3 * KV_BLOCK, T - 1):
            if 0 <= j <= i < T:
                cases.add((j, i))
    seen = 0
    for j, i in sorted(cases):
        h = torch.zeros(T, _width(m), dtype=F64)
        h[:, 1:nq:d] = 1.0                      # every query along axis 1 ...
        h[:, nq + 1:nq + nk:d] = 1.0            # ... and every key
        h[j, nq:nq + nk] = 0.0
        h[j, nq:nq + nk:d] = 1.0                # the marked key along axis 0
        h[i, :nq] = 0.0
        h[i, 0:nq:d] = 1.0                      # the query under test along axis 0
        if win:                                 # values are the keys: theirs stands out by the third axis, which no query asks for
            h[j, nq + 2:nq + nk:d] = 7.0
        else:
            h[:, nq + nk:nq + nk + G * dv] = torch.linspace(-0.1, 0.1, G * dv, dtype=F64)
            h[j, nq + nk:nq + nk + G * dv] = 7.0
            h[:, nq + nk + G * dv:] = 2.0
        sink = torch.full((H,), 3.0) if win else None
        ref = _reference(h, None, m, sink, None, 1.0)[i]
        seen += int(float(ref.max()) > 5.0)
        got = _run(h.float(), None, m, sink, None, 1.0, dt, [j + 1, 2, 33, 1], seed=j)[i].double().cpu()
        assert float((got - ref).abs().max()) < (3e-4 if dt == F32 else 0.08), (j, i, float(ref.max()), float(got.max()))
    assert 0 < seen < len(cases)     # both outcomes occur


def test_sink_of_each_head_takes_its_weight_and_each_gate_its_head():
    g = torch.Generator().manual_seed(2)
    for m, dt, tol in ((_win(4, 2, 32, 200, 16), F32, 2e-5), (_win(4, 2, 32, 200, 16), BF16, 0.03), (_win(3, 3, 7, 200, 2), F32, 2e-5)):
        h = torch.randn(260, _width(m), generator=g)
        sink = torch.tensor([-30.0, 2.0, 5.0, 40.0])[:m["heads"]]
        ref, without = _reference(h, None, m, sink, None, 1.0), _reference(h, None, m, torch.full((m["heads"],), -1e9), None, 1.0)
        per_head = (ref - without).view(260, m["heads"], -1).abs().amax((0, 2))
        assert float(per_head[0]) < 1e-9 and all(float(x) > 0.5 for x in per_head[1:])
        for sizes in ([260], [1]):
            got = _run(h, None, m, sink, None, 1.0, dt, sizes).double().cpu()
            assert float((got - ref).abs().max()) < tol * max(1.0, float(ref.abs().max())), (m, dt, sizes)
    m = _chk(4, 2, 32, 48, 50, 16)
    h = torch.randn(120, _width(m), generator=g)
    h[:, -4:] = torch.tensor([-30.0, 0.0, 3.0, 30.0])       # closed, half, almost and wholly open
    ref = _reference(h, None, m, None, None, 1.0)
    assert float(ref.view(120, 4, -1)[:, 0].abs().max()) < 1e-9
    for dt, tol in ((F32, 2e-5), (BF16, 0.03)):
        for sizes in ([120], [1]):
            assert float((_run(h, None, m, None, None, 1.0, dt, sizes).double().cpu() - ref).abs().max()) < tol * float(ref.abs().max())


# ====================================================================================================== recurrent mixers
def _walk(seqs, sizes, run):
    """Both sequences through state slots 1 and 3 in portions, two at a time: run(rows, meta, slots, positions) -> outputs."""
    outs = [[] for _ in seqs]
    at, step = [0] * len(seqs), 0
    while any(a < s.shape[0] for a, s in zip(at, seqs)):
        rows, meta, slots, pos, dst = [], [], [], [], []
        for s in range(len(seqs)):
            n = min(sizes[s][step % len(sizes[s])], seqs[s].shape[0] - at[s])
            if n <= 0:
                continue
            meta += [sum(r.shape[0] for r in rows), n, at[s] + n, 0]
            rows.append(seqs[s][at[s]:at[s] + n])
            slots += [1 + 2 * s] * n
            pos += list(range(at[s], at[s] + n))
            dst.append((s, n))
            at[s] += n
        out, o = run(torch.cat(rows).contiguous(), meta, slots, pos), 0
        for s, n in dst:
            outs[s].append(out[o:o + n])
            o += n
        step += 1
    return [torch.cat(o).double().cpu() for o in outs]


_CUTS = ([[5, 1, 40, 2, 17], [33, 1, 1, 64]], [[330], [150]], [[1], [150]], [[16, 100, 15, 65], [2, 3]], [[32], [31, 33]])


@pytest.mark.parametrize("chunked,H,d,dv,rd", [(1, 2, 16, 8, 16), (1, 3, 48, 72, 20), (1, 2, 128, 128, 128), (1, 1, 80, 136, 0)] + [
    (0, *s) for s in [(3, 6, 5, 4), (2, 70, 40, 70), (1, 1, 1, 0), (2, 130, 33, 64), (2, 128, 128, 128)]])
def test_retention_in_portions_and_two_slots_matches_oracle(chunked, H, d, dv, rd):
    """chunked: the tensor-core form rounds q, k (after the turn) and v to bf16, and so does the reference here; everything the
    recurrence adds stays fp32-like, so the bound is far below bf16's."""
    from oracle import ludelix_oracle as O

    g = torch.Generator().manual_seed(3)
    width, kmul = 2 * H * d + H * dv, d ** -0.5
    decay = torch.tensor([0.6, 0.99, 0.999][:H]) if H > 1 else torch.tensor([0.97])
    rot = {"base": 70.0, "dims": max(rd, 1)}
    f = O.plain_freqs(rot) if rd else []
    seqs = [torch.randn(330, width, generator=g), torch.randn(150, width, generator=g)]
    refs = []
    for h in seqs:
        h = h.double()
        q, k = O.rotate(h[:, :H * d].reshape(-1, H, d), f, False), O.rotate(h[:, H * d:2 * H * d].reshape(-1, H, d), f, False) * kmul
        v = h[:, 2 * H * d:].reshape(-1, H, dv)
        if chunked:
            q, k, v = (x.float().to(torch.bfloat16).double() for x in (q, k, v))
        refs.append(O.outer_memory(q, k, v, decay.double()[None, :, None].expand(h.shape[0], H, d)).reshape(-1, H * dv))
    ang = torch.arange(330, dtype=F64)[:, None] * torch.tensor(f, dtype=F64)[None, :]
    table, dec = _dev(torch.cat([torch.cos(ang), torch.sin(ang)], -1)) if rd else None, _dev(decay)
    for sizes in _CUTS:
        S = torch.randn(4, H, d, dv, device="cuda")       # slots 1 and 3 are used; what an earlier owner left is never read

        def run(rows, meta, slots, pos):
            x, out = _dev(rows), torch.zeros(rows.shape[0], H * dv, device="cuda")
            _ok(_lib().tgis_k_retention_scan(_p(x), width, 0, H * d, 2 * H * d, _p(table), _p(_i32(pos)), rd, kmul, _p(dec), _p(S), _p(out),
                                             H * dv, H, d, dv, _ints(meta), len(meta) // 4, _p(_i32(slots)), rows.shape[0], chunked))
            return out

        for got, ref in zip(_walk(seqs, sizes, run), refs):
            # (a value that sits on a bf16 rounding boundary may round the other way than the reference's)
            assert float((got - ref).abs().max()) < (2e-3 if chunked else 2e-5) * max(1.0, float(ref.abs().max())), sizes


@pytest.mark.parametrize("bias", [3.0, -4.0, -30.0])
@pytest.mark.parametrize("chunked,H,d,dv,rank", [(1, 2, 16, 8, 1), (1, 3, 48, 72, 16), (1, 2, 128, 128, 16), (1, 1, 80, 136, 64), (1, 4, 64, 64, 7)] + [
    (0, *s) for s in [(3, 6, 5, 2), (2, 70, 40, 16), (1, 1, 1, 1), (2, 130, 33, 8), (2, 128, 128, 16)]])
def test_gated_linear_attention_in_portions_and_two_slots_matches_oracle(chunked, H, d, dv, rank, bias):
    """Decays from almost one to almost nothing (bias -30: a token's decay is e^-20, sixteen of them leave the range of fp32), channel by
    channel; chunked: v is rounded to bf16 and so is the reference's."""
    from oracle import ludelix_oracle as O

    g = torch.Generator().manual_seed(3)
    hd, hv, tau = H * d, H * dv, 1.5
    width = 2 * hd + hv + rank + 3
    width += width % 2
    a2 = (torch.randn(hd, rank, generator=g) * rank ** -0.5).to(torch.bfloat16)
    b = bias + torch.randn(hd, generator=g) * 2
    seqs = [torch.randn(330, width, generator=g), torch.randn(150, width, generator=g)]
    refs = []
    for h in seqs:
        h = h.double()
        z = h[:, 2 * hd + hv:2 * hd + hv + rank] @ a2.double().T + b.double()
        decay = (torch.sigmoid(z) ** (1.0 / tau)).reshape(-1, H, d)
        v = h[:, 2 * hd:2 * hd + hv].reshape(-1, H, dv)
        if chunked:
            v = v.float().to(torch.bfloat16).double()
        refs.append(O.outer_memory(h[:, :hd].reshape(-1, H, d) * d ** -0.5, h[:, hd:2 * hd].reshape(-1, H, d), v, decay).reshape(-1, hv))
    w2, bd = _dev(a2, torch.bfloat16), _dev(b)
    for sizes in _CUTS:
        S = torch.randn(4, H, d, dv, device="cuda")

        def run(rows, meta, slots, pos):
            x, out = _dev(rows), torch.full((rows.shape[0], hv), float("nan"), device="cuda")
            _ok(_lib().tgis_k_gla_scan(_p(x), width, 0, hd, 2 * hd, 2 * hd + hv, d ** -0.5, _p(w2), rank, _p(bd), 1.0 / tau, _p(S), _p(out), hv,
                                       H, d, dv, _ints(meta), len(meta) // 4, _p(_i32(slots)), rows.shape[0], chunked))
            return out

        for got, ref in zip(_walk(seqs, sizes, run), refs):
            assert float((got - ref).abs().max()) < (2e-4 if chunked else 3e-5) * max(1.0, float(ref.abs().max())), sizes


# ====================================================================================================== experts and tails
@pytest.mark.parametrize("E,top,T,vocab", [(5, 2, 37, 50), (1, 1, 9, 3), (64, 6, 700, 1000), (1500, 3, 300, 40), (4, 4, 1, 7)])
def test_table_chosen_experts_fill_their_row_segments(E, top, T, vocab):
    g = torch.Generator().manual_seed(E)
    table = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(vocab)]).to(torch.int32)
    tok = torch.randint(0, vocab, (T,), generator=g)
    seg, order, inv = (torch.full((n,), -1, dtype=torch.int32, device="cuda") for n in (E + 1, T * top, T * top))
    _ok(_lib().tgis_k_moe_table_align(_p(_dev(table, torch.int32)), vocab, _p(_dev(tok, torch.int32)), T, top, E, _p(seg), _p(order), _p(inv)))
    want = table[tok].reshape(-1).long()
    assert seg.tolist() == [0] + torch.bincount(want, minlength=E).cumsum(0).tolist()
    order, inv, seg = order.cpu().long(), inv.cpu().long(), seg.cpu().long()
    assert sorted(order.tolist()) == list(range(T * top)) and torch.equal(order[inv], torch.arange(T * top))
    for p in range(T * top):
        e = int(want[order[p]])
        assert seg[e] <= p < seg[e + 1]


@pytest.mark.parametrize("hidden", [40, 37, 2048])
def test_plain_sublayer_tail_matches_oracle(hidden):
    from oracle import ludelix_oracle as O

    g = torch.Generator().manual_seed(7)
    T, top = 9, 3
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    x, y, rows, side, gate = rnd(T, hidden) * 2, rnd(T, hidden) * 3, rnd(T * top, hidden), rnd(T, hidden), torch.rand(T, generator=g)
    w, dot = 1 + rnd(hidden) * 0.1, rnd(hidden) * hidden ** -0.5
    inv = torch.randperm(T * top, generator=g).view(T, top)
    X, moe = x.double(), rows.double()[inv].sum(1) / top
    cases = {"plain": (y.double(), y, None, None, None), "experts": (moe, None, rows, None, None),
             "experts and shared": (moe + gate.double()[:, None] * side.double(), None, rows, side, gate)}
    for name, (add, main, er, sd, sg) in cases.items():
        for dt, tol in ((F32, 1e-5), (BF16, 3e-2)):
            r = _dev(x)
            out = torch.zeros(T, hidden, dtype=torch.bfloat16 if dt == BF16 else torch.float32, device="cuda")
            dots = torch.zeros(T, device="cuda")
            d = [_dev(t) if t is not None else None for t in (main, er)]
            _ok(_lib().tgis_k_resid_tail_plain(_p(d[0]), _p(d[1]), _p(_dev(inv, torch.int32)), 1.0 / top, top, _p(_dev(sd)) if sd is not None else None,
                                               _p(_dev(sg)) if sg is not None else None, _p(_dev(w)), _p(r), _p(out), dt, _p(_dev(dot)), _p(dots),
                                               EPS, T, hidden))
            new = X + add
            n = O.rms(new, EPS) * w.double()
            assert float((r.double().cpu() - new).abs().max()) < 1e-5, name
            assert float((out.double().cpu() - n).abs().max()) < tol, name
            assert float((dots.double().cpu() - torch.sigmoid(n @ dot.double())).abs().max()) < 1e-5, name    # from the fp32 row in both types


# ====================================================================================================== engine level
def _par(left, heads=2, dim=6, vdim=4, rd=4, decay=(0.5, 0.97), base=90.0, scales=(0.8, 1.3)):
    return {"left": left, "right": dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay), rot=dict(base=base, dims=rd)),
            "left_scale": scales[0], "right_scale": scales[1]}


def _gla(heads=2, dim=6, vdim=5, tau=4.0):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def _moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _lay(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _cfg(layers=None, width=40, vocab=97):
    if layers is None:
        layers = [_lay("attention", _win(4, 2, 6, 13, 4, base=50.0), _moe(4, 2, 18, 14)),
                  _lay("parallel", _par(_chk(4, 2, 6, 10, 21, 4, base=50.0)), _dense(24)),
                  _lay("gla", _gla(3, 7, 6), _moe(7, 3, 10)),
                  _lay("parallel", _par(_chk(3, 1, 8, 5, 40, 8), heads=1, dim=12, vdim=9, rd=12, decay=(0.9,)), _moe(3, 1, 12, 8)),
                  _lay("gla", _gla(1, 12, 20, 16.0))]
    return {"architecture": "Ludelix", "width": width, "vocab": vocab, "norm": {"eps": EPS}, "layers": layers}


def _model(cfg, dtype="float32", max_model_len=512, ranks=(5, 3, 8)):
    from vllm_tgis_adapter_b200.engine.ludelix import model_config_from_json

    shapes = {f"l{i}.mix.a1": (ranks[i % len(ranks)], cfg["width"]) for i in range(len(cfg["layers"]))}
    return model_config_from_json(cfg, max_model_len, dtype, shapes)


def _weights(mc, seed):
    """Seeded weights whose attention is sharp enough that single keys decide."""
    from vllm_tgis_adapter_b200.engine.ludelix import synthetic_weights

    w = synthetic_weights(mc, seed)
    for k in w:
        if k.endswith(("left.q", "left.k", "mix.q.norm", "mix.k.norm")):
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
    """bf16 operands on widths this small: rounding alone moves single rows by several percent of their spread; so the bound is on
    the typical row and on the bulk (the sharp comparison is the float32 one)."""
    rows = sorted(_rel(got[t:t + 1], ref[t:t + 1]) for t in range(len(ref)))
    return rows[len(rows) // 2] < 4e-2 and rows[int(0.9 * len(rows))] < 0.2


def _whole(eng, toks, rid="w"):
    return eng.trace_step([(rid, toks, list(range(len(toks))))], [rid])


def _in_parts(eng, toks, sizes, rid="p"):
    return np.concatenate([eng.trace_step([(rid, toks[a:a + n], list(range(n)))], [rid] if a + n == len(toks) else [])
                           for a, n in _portions(len(toks), sizes)])


TOL = 3e-5


def test_whole_prompt_matches_oracle_fp32_and_bf16():
    from oracle import ludelix_oracle as O

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
    one = _gla(1, 1, 1, 1.0)
    return {
        "parallel": [_lay("parallel", _par(_chk(4, 2, 6, 10, 19, 4, base=50.0)))],
        "parallel_whole_heads_rotate": [_lay("parallel", _par(_chk(3, 3, 8, 5, 40, 8), heads=4, dim=4, vdim=11, rd=4, decay=(0.1, 0.5, 0.9, 1.0)))],
        "parallel_nothing_rotates_one_chunk": [_lay("parallel", _par(_chk(2, 1, 8, 8, 1000, 0), rd=0, scales=(1.0, 1.0)))],
        "parallel_keys_of_70": [_lay("parallel", _par(_chk(2, 2, 4, 4, 20, 4), heads=2, dim=70, vdim=35, rd=30))],
        "parallel_left_only_right_only": [_lay("parallel", _par(_chk(2, 2, 4, 4, 20, 4), scales=(1.5, 0.0))),
                                          _lay("parallel", _par(_chk(2, 2, 4, 4, 20, 4), scales=(0.0, 1.5)))],
        "attention": [_lay("attention", _win(4, 2, 6, 19, 4))],
        "attention_every_head_its_own": [_lay("attention", _win(5, 5, 10, 1000, 10, factor=8.0, low=2.0, high=5.0, original=200))],
        "attention_window_of_one": [_lay("attention", _win(2, 1, 4, 1, 2))],
        "gla": [_lay("gla", _gla(3, 8, 10))],
        "gla_keys_of_70": [_lay("gla", _gla(2, 70, 9, 1.0))],
        "dense": [_lay("gla", one, _dense(50))],
        "experts": [_lay("gla", one, _moe(6, 2, 30))],
        "experts_and_shared": [_lay("gla", one, _moe(5, 1, 16, 22))],
        "one_expert": [_lay("gla", one, _moe(1, 1, 8))],
    }


@pytest.mark.parametrize("name", list(_alone()))
def test_each_mechanism_alone_whole_and_in_portions(name):
    from oracle import ludelix_oracle as O

    cfg = _cfg(_alone()[name], width=24, vocab=61)
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
        "ones": _cfg([_lay("parallel", _par(_chk(1, 1, 2, 1, 1, 2), heads=1, dim=1, vdim=1, rd=0, decay=(0.5,)), _dense(1)),
                      _lay("gla", _gla(1, 1, 1, 1.0), _moe(1, 1, 1, 1)), _lay("attention", _win(1, 1, 2, 1, 2), _moe(2, 1, 1))], width=6, vocab=11),
        "no_feed_forward": _cfg([_lay("attention", _win(2, 2, 10, 16, 6)), _lay("gla", _gla(4, 5, 3, 2.0)),
                                 _lay("parallel", _par(_chk(4, 4, 10, 6, 16, 6), heads=5, dim=9, vdim=10, rd=8, decay=(0.3, 0.5, 0.7, 0.9, 0.99)))], width=30),
        "all_experts_chosen_chunk_longer_than_the_prompt": _cfg(
            [_lay("parallel", _par(_chk(4, 1, 16, 24, 1000, 16, base=20000.0)), _moe(4, 4, 48, 20)), _lay("attention", _win(6, 3, 16, 33, 8), _dense(64)),
             _lay("gla", _gla(4, 16, 24), _moe(9, 5, 16))], width=64, vocab=130),
        "tensor_core_sizes": _cfg([_lay("parallel", _par(_chk(4, 2, 64, 64, 70, 64, scale=0.125), heads=4, dim=64, vdim=64, rd=64, decay=(0.6, 0.9, 0.97, 0.999)),
                                        _dense(512)),
                                   _lay("gla", _gla(4, 64, 80, 16.0), _moe(14, 2, 256, 512)),
                                   _lay("attention", _win(8, 4, 32, 50, 16, scale=0.2), _moe(5, 1, 128, 256)),
                                   _lay("parallel", _par(_chk(6, 2, 48, 80, 37, 32, scale=0.15), heads=2, dim=128, vdim=128, rd=32, decay=(0.8, 0.99)), _moe(6, 3, 128)),
                                   _lay("gla", _gla(2, 128, 128, 8.0), _dense(256)), _lay("attention", _win(4, 1, 128, 100, 128, scale=0.1))],
                                  width=256, vocab=300),
    }


@pytest.mark.parametrize("name", list(_variants()))
def test_other_sizes_orders_and_absent_parts(name):
    from oracle import ludelix_oracle as O

    cfg = _variants()[name]
    toks = _tokens(140, cfg["vocab"], 6)
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
    from oracle import ludelix_oracle as O

    cfg = _cfg()
    mc = _model(cfg)
    weights = _weights(mc, 31)
    toks = _tokens(131, 97, 3)
    ref = O.forward(cfg, weights, toks)
    eng = _engine(mc, weights)
    for sizes in ([2], [1], [31, 33, 2, 64, 1], [64, 1, 1, 1, 1, 1, 1], [13, 37, 8], [20, 2, 19, 2]):
        assert _rel(_in_parts(eng, toks, sizes, "s"), ref) < TOL, sizes
    eng.close()


def test_long_decoding_crosses_window_chunk_and_page_borders_bf16_stays_close():
    from oracle import ludelix_oracle as O

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


@pytest.mark.parametrize("memory", ["chunk", "retention", "gla"])
def test_far_token_decides_hundreds_of_tokens_later(memory):
    """One large early token: through a long chunk, through a retention head that hardly decays or through key channels that hardly
    decay, it reaches outputs hundreds of tokens later, in a prompt, in portions and decoded."""
    from oracle import ludelix_oracle as O

    layers = {"chunk": [_lay("parallel", _par(_chk(2, 1, 16, 16, 1000, 4, base=1e6, scale=0.5), scales=(2.0, 0.0)))],
              "retention": [_lay("parallel", _par(_chk(2, 1, 16, 16, 8, 4), heads=2, dim=16, vdim=16, rd=4, base=1e6, decay=(0.9998, 1.0), scales=(0.0, 1.0)))],
              "gla": [_lay("gla", _gla(2, 16, 16, 16.0))]}[memory]
    cfg = _cfg(layers, width=64, vocab=61)
    for dtype in ("float32", "bfloat16"):
        mc = _model(cfg, dtype)
        weights = _weights(mc, 19)
        # every token shares a direction that queries read; the marked token alone has another one that keys and values read
        common, mark = torch.linalg.qr(torch.randn(64, 2, generator=torch.Generator().manual_seed(4)))[0].T
        emb = weights["embed"].float() + 3 * common
        emb[60] = 8 * mark + 3 * common
        weights["embed"] = emb.to(torch.bfloat16)
        side = {"chunk": "left.", "retention": "right.", "gla": ""}[memory]
        for part, row, d in (("q", 10, 1.5 * common), ("k", 10, 0.5 * mark), ("v", 3, mark)):
            w = weights[f"l0.mix.{side}{part}"].float()
            w[row::16] += d           # entry `row` of every head (past the entries that turn)
            weights[f"l0.mix.{side}{part}"] = w.to(torch.bfloat16)
        weights[f"l0.mix.{side}o"] = weights[f"l0.mix.{side}o"] * 4       # the mixer's output beside the token's own embedding
        if memory == "gla":
            weights["l0.mix.a2.b"] = torch.full((32,), 9.0).to(torch.bfloat16)           # decays of about e^(-1e-5)
            weights["l0.mix.a2"] = weights["l0.mix.a2"] * 0.1
        base = _tokens(390, 60, 8)
        toks = list(base)
        toks[7] = 60
        ref, plain = O.forward(cfg, weights, toks), O.forward(cfg, weights, base)
        assert _rel(plain[340:].numpy(), ref[340:]) > 0.05    # what the marked token changes far away
        eng = _engine(mc, weights)
        got = [eng.trace_step([("d", toks[:200], list(range(200)))], []), eng.trace_step([("d", toks[200:350], list(range(150)))], [])]
        for t in range(350, 390):
            got.append(eng.trace_step([("d", [toks[t]], [0])], ["d"] if t == 389 else []))
        eng.close()
        got = np.concatenate(got)
        assert _rel(got, ref) < TOL if dtype == "float32" else _bf16_close(got, ref), dtype


def test_mixed_batches_of_unequal_requests_match_each_alone_and_reuse_pages_and_slots():
    from oracle import ludelix_oracle as O

    for cfg, dtype in ((_cfg(), "float32"), (_variants()["tensor_core_sizes"], "bfloat16")):
        V = cfg["vocab"]
        mc = _model(cfg, dtype)
        weights = _weights(mc, 41)
        reqs = {f"q{i}": _tokens(n, V, 50 + i) for i, n in enumerate([97, 40, 3, 130, 64, 33, 71, 1, 90])}
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
            g = np.concatenate(got[k])
            assert _rel(g, ref[k]) < TOL if dtype == "float32" else _bf16_close(g, ref[k]), (dtype, k)


def test_bad_tables_are_refused():
    mc = _model(_cfg())
    weights = _weights(mc, 5)
    for bad in (4, -1):
        t = weights["l0.mlp.table"].clone()
        t[3, 1] = bad
        with pytest.raises(Exception, match="out of range"):
            _engine(mc, {**weights, "l0.mlp.table": t})
    with pytest.raises(Exception, match="shape mismatch"):
        _engine(mc, {**weights, "l0.mlp.table": weights["l0.mlp.table"][:, :1]})


def test_greedy_generation_through_the_scheduler_matches_oracle():
    from oracle import ludelix_oracle as O
    from vllm_tgis_adapter_b200.engine.core import make_sampling_params

    cfg = _cfg()
    mc = _model(cfg)
    weights = _weights(mc, 61)
    weights["embed"] = weights["embed"] * 0.5     # (logits read this table as well)
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
    """grpc client -> TextGenerationService -> AsyncTGISEngine -> the engine's step loop on a Ludelix preset (float32): greedy
    tokens and their logprobs of a batched Generate call against the oracle."""
    from test_server_gpu import LiveServer

    from oracle import ludelix_oracle as O
    from vllm_tgis_adapter_b200.engine.ludelix import config_json
    from vllm_tgis_adapter_b200.engine.tokenizer import synthetic_prompt
    from vllm_tgis_adapter_b200.grpc.pb import generation_pb2 as pb

    srv = LiveServer("ludelix-tiny", seed=29)
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
    """bin/trace_run on a directory with config.json + model.safetensors: the family, the low-rank maps' sizes and every other size come
    from the files, a mixed schedule with a reused slot goes through standard input, the logits land in the output folder."""
    import subprocess
    import sys
    from pathlib import Path

    from safetensors.torch import save_file

    from oracle import ludelix_oracle as O

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
