"""GPU: the Gebasun decoder's mechanisms one by one against the plain implementation (tests/plain_gebasun.py)."""

import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_gebasun as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F = torch.float64


def _rel(got, want):
    got = got.detach().cpu().numpy() if torch.is_tensor(got) else got
    want = np.asarray(want, dtype=np.float64)
    return float(np.abs(np.asarray(got, dtype=np.float64) - want).max() / max(np.abs(want).max(), 1e-30))


def _exact(t, dtype=torch.float32):
    """Numbers that the given dtype holds exactly, as float64."""
    return t.to(dtype).to(F)


def _f32(t):
    return t.float().to(DEV).contiguous()


def _i32(x):
    return torch.tensor(np.asarray(x), dtype=torch.int32, device=DEV)


def _ctx(past, counts, slots=None):
    """The step's index arrays for sequences that hold ``past`` positions and bring ``counts`` tokens."""
    token_seq = [b for b, n in enumerate(counts) for _ in range(n)]
    token_pos = [past[b] + k for b, n in enumerate(counts) for k in range(n)]
    starts = np.concatenate([[0], np.cumsum(counts)])
    return SimpleNamespace(token_seq=_i32(token_seq), token_pos=_i32(token_pos), seq_start=_i32(starts),
                           seq_past=_i32(past), seq_slot=_i32(slots if slots is not None else range(len(counts))),
                           n_seqs=len(counts), n_tokens=int(sum(counts)), max_new=max(counts),
                           is_decode=all(n == 1 for n in counts))


def _store(lens, G, *dims, dtype, seed=0):
    """Empty paged stores (one per entry of ``dims``) for sequences of those lengths, pages dealt out in any order."""
    g = torch.Generator().manual_seed(seed)
    per = [max(1, -(-n // 64)) for n in lens]
    order = torch.randperm(sum(per) + 2, generator=g).tolist()
    table = torch.full((len(per), max(per)), -1, dtype=torch.int32)
    at = 0
    for b, n in enumerate(per):
        table[b, :n] = torch.tensor(order[at : at + n], dtype=torch.int32)
        at += n
    # rows nobody has written hold NaN: whoever reads one shows it
    stores = [torch.full((sum(per) + 2, G, 64, d), float("nan"), dtype=dtype, device=DEV) for d in dims]
    return table.to(DEV), stores


def _rows(table, store, b, n):
    """[n, G, D]: positions 0 .. n-1 of sequence b."""
    pages = table[b].cpu().tolist()
    return torch.stack([store[pages[p // 64], :, p % 64] for p in range(n)]).cpu()


# ---------------------------------------------------------------------------------------------------------
# both norms of a block, and what two sublayers owe the stream
# ---------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("d, na, nb, bias", [(40, 1, 3, True), (101, 2, 2, True), (2048, 0, 9, False), (4096, 9, 3, True),
                                             (9000, 1, 2, False), (96, 0, 0, True), (7000, 4, 5, True)])
@pytest.mark.parametrize("act", [torch.float32, torch.bfloat16])
def test_two_results_join_the_stream_and_two_norms_read_it(d, na, nb, bias, act):
    from llmoxide_b200 import kernels

    g = torch.Generator().manual_seed(d)
    T, eps = 19, 1e-3
    h = _exact(torch.randn(T, d, generator=g) * 0.1)                       # small: eps shows
    a = _exact(torch.randn(na, T, d, generator=g) * 0.03, torch.bfloat16 if na == 1 else torch.float32)
    b = _exact(torch.randn(nb, T, d, generator=g) * 0.03)
    bv = _exact(torch.randn(d, generator=g) * 0.05)
    g0, g1 = _exact(torch.randn(d, generator=g)), _exact(torch.randn(d, generator=g))
    want = h + a.sum(0) + b.sum(0) + (bv if bias else 0.0)
    groups = ([a[0].to(torch.bfloat16).to(DEV).contiguous() if na == 1 else _f32(a)] if na else []) + ([_f32(b)] if nb else [])
    hd = _f32(h)
    out0, out1 = (torch.empty((T, d), dtype=act, device=DEV) for _ in range(2))
    kernels.dual_norm(hd, groups, _f32(bv) if bias else None, _f32(g0), eps, out0, _f32(g1), out1)
    tol = 2e-6 if act == torch.float32 else 6e-3
    assert _rel(hd, want) < 2e-6
    assert _rel(out0.float(), plain.rms_norm(want, g0, eps)) < tol and _rel(out1.float(), plain.rms_norm(want, g1, eps)) < tol
    # rows asked for, one norm, the stream left alone
    hd, rows = _f32(h), [7, 0, 18]
    kernels.dual_norm(hd, groups, _f32(bv) if bias else None, _f32(g0), eps, out0[:3], rows=_i32(rows), write_h=False)
    assert _rel(out0[:3].float(), plain.rms_norm(want, g0, eps)[rows]) < tol and torch.equal(hd, _f32(h))
    # only the sum
    kernels.dual_norm(hd, groups, _f32(bv) if bias else None, None, eps, None)
    assert _rel(hd, want) < 2e-6
    kernels.check_status()


# ---------------------------------------------------------------------------------------------------------
# keys that are values: bias, rotation, unit norm, cache write; the output's gate
# ---------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("H, G, D, rot, n_split, extra", [(4, 2, 24, 8, 1, 96), (3, 1, 18, 0, 3, 0), (6, 6, 14, 14, 2, 84),
                                                          (16, 4, 128, 64, 1, 2048), (8, 4, 64, 64, 9, 0), (2, 1, 200, 2, 1, 8),
                                                          (5, 5, 256, 128, 2, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("counts", [[9, 8, 1], [70, 3, 2]])
def test_unit_norm_rotation_and_keys_stored_twice(H, G, D, rot, n_split, extra, dtype, counts):
    from llmoxide_b200 import kernels

    g = torch.Generator().manual_seed(H * 100 + D)
    past, eps, base = [0, 60, 199], 1e-2, 700.0
    T, N = sum(counts), (H + G) * D + extra
    proj = _exact(torch.randn(n_split, T, N, generator=g) * 0.2, torch.float32 if n_split > 1 else dtype)
    bias = _exact(torch.randn((H + G) * D, generator=g) * 0.3)
    pos = torch.tensor([p + k for p, n in zip(past, counts) for k in range(n)])
    row = proj.sum(0)[:, : (H + G) * D] + bias
    x = row.reshape(T, H + G, D)
    turned = x
    if rot:
        # positions of different sequences may coincide: turn them one at a time
        turned = torch.stack([plain.rotate_halves(torch.cat([torch.zeros((int(p), H + G, D), dtype=F), x[i : i + 1]]), rot,
                                                  base)[-1] for i, p in enumerate(pos)])
    unit = plain.unit_rms(turned, eps)
    cos = sin = None
    if rot:
        ang = np.arange(300, dtype=np.float32)[:, None] * np.array([base ** (-2.0 * i / rot) for i in range(rot // 2)],
                                                                  dtype=np.float32)
        cos, sin = (_f32(torch.from_numpy(f(ang.astype(np.float64)))) for f in (np.cos, np.sin))
    table, (kc, vc) = _store([p + n for p, n in zip(past, counts)], G, D, D, dtype=dtype)
    pd = (proj[0] if n_split == 1 else proj).to(torch.float32 if n_split > 1 else dtype).to(DEV).contiguous()
    q = torch.empty((T, H * D), dtype=dtype, device=DEV)
    ctx = _ctx(past, counts)
    kernels.qk_unit_rope_cache(pd, _f32(bias), q, kc, vc, table, ctx, eps, cos, sin, rot, H, G, D)
    # (angles are float32 products of position and frequency: up to 200 radians here)
    tol = 2e-5 if dtype == torch.float32 else 6e-3
    assert _rel(q.float().reshape(T, H, D), unit[:, :H]) < tol
    at = 0
    for b, (p, n) in enumerate(zip(past, counts)):
        ks, vs = _rows(table, kc, b, p + n), _rows(table, vc, b, p + n)
        assert torch.isnan(ks[:p].float()).all() and torch.isnan(vs[:p].float()).all()      # earlier rows are not touched
        assert _rel(ks[p:].float(), unit[at : at + n, H:]) < tol
        assert _rel(vs[p:].float(), x[at : at + n, H:]) < tol                # the key as projected, bias included
        at += n
    written = sum(counts)
    assert int((~torch.isnan(kc.float())).sum()) == written * G * D
    if extra:
        out = _exact(torch.randn(T, extra, generator=g), dtype)
        od = out.to(dtype).to(DEV).contiguous()
        kernels.gate_rows(od, pd[..., (H + G) * D :])
        assert _rel(od.float(), out * torch.sigmoid(proj.sum(0)[:, (H + G) * D :])) < tol
    kernels.check_status()


def test_a_bad_page_is_reported_and_nothing_is_written():
    from llmoxide_b200 import kernels
    from llmoxide_b200.errors import KernelError

    table, (kc, vc) = _store([5], 1, 16, 16, dtype=torch.float32)
    q = torch.zeros((1, 16), device=DEV)
    pd = torch.ones((1, 32), device=DEV)
    table[0, 0] = 99
    kernels.qk_unit_rope_cache(pd, None, q, kc, vc, table, _ctx([4], [1]), 1e-5, None, None, 0, 1, 1, 16)
    torch.cuda.synchronize()
    assert torch.isnan(kc).all() and torch.isnan(vc).all()
    with pytest.raises(KernelError, match="qk_unit"):
        kernels.check_status()
    kernels.check_status()


# ---------------------------------------------------------------------------------------------------------
# attention with distance biases and learned sinks
# ---------------------------------------------------------------------------------------------------------

def _paged(lens, G, D, dtype, seed):
    table, (kc, vc) = _store(lens, G, D, D, dtype=dtype, seed=seed)
    g = torch.Generator().manual_seed(seed)
    ks, vs = [], []
    for b, n in enumerate(lens):
        k = plain.unit_rms(torch.randn(n, G, D, generator=g, dtype=F), 1e-6)
        v = torch.randn(n, G, D, generator=g, dtype=F)
        ks.append(_exact(k, dtype)), vs.append(_exact(v, dtype))
    return table, kc, vc, ks, vs


def _fill(table, store, b, rows):
    pages = table[b].cpu().tolist()
    for p in range(rows.shape[0]):
        store[pages[p // 64], :, p % 64] = rows[p].to(store.dtype).to(DEV)


def _want(q, k, v, G, scale, window, keep, sinks, lut, first):
    """Plain attention of the last rows of one sequence: q [n, H, D] at positions first .., k, v [T, G, D]."""
    T, H = k.shape[0], q.shape[1]
    seen = plain.window_mask(T, window, keep)[first:]
    i, j = torch.arange(first, T)[:, None], torch.arange(T)[None, :]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if lut is not None:
            s = s + lut[h][(i - j).clamp(0, lut.shape[1] - 1)]
        s = s.masked_fill(~seen, -math.inf)
        m = torch.maximum(s.max(1, keepdim=True).values, sinks[h])
        e = torch.exp(s - m)
        out.append((e @ v[:, g]) / (e.sum(1, keepdim=True) + torch.exp(sinks[h] - m)))
    return torch.stack(out, 1)


EDGES = [("window's last key", lambda p, w: p - w + 1), ("first key outside", lambda p, w: p - w), ("itself", lambda p, w: p),
         ("first", lambda p, w: 0), ("page border", lambda p, w: p // 64 * 64), ("before a page border", lambda p, w: p // 64 * 64 - 1)]


@pytest.mark.parametrize("H, G, D, window, keep, bias_len", [(4, 2, 20, 37, 0, 37), (3, 1, 18, None, 0, 91), (6, 3, 32, 50, 3, 34),
                                                             (8, 4, 64, 100, 0, 80), (4, 1, 128, 130, 66, 200)])
def test_general_attention_one_key_stands_out(H, G, D, window, keep, bias_len):
    """One key of the newest query's is scaled so that its score dominates, and the bias of its distance is lifted: the
    result moves to its value when it is seen, and not at all when it is just outside."""
    from llmoxide_b200 import kernels

    g = torch.Generator().manual_seed(D)
    lens = [300, 65, 64, 1, 131]
    table, kc, vc, ks, vs = _paged(lens, G, D, torch.float32, D)
    sinks = torch.randn(H, generator=g, dtype=F)
    lut = _exact(torch.randn(H, bias_len, generator=g, dtype=F))
    scale = 0.4
    for name, where in EDGES:
        for b, n in enumerate(lens):
            p = n - 1
            j = where(p, window or n)
            q = _exact(torch.randn(1, H, D, generator=g, dtype=F))
            k, lut_b = ks[b].clone(), lut.clone()
            if 0 <= j <= p:
                k[j] = k[j] + 6.0 * plain.unit_rms(q[0, :: H // G][:G], 1e-6)
                lut_b[:, min(p - j, bias_len - 1)] += 3.0
            k, lut_b = _exact(k), _exact(lut_b)
            _fill(table, kc, b, k), _fill(table, vc, b, vs[b])
            out = torch.empty((1, H * D), device=DEV)
            kernels.attention_paged(_f32(q.reshape(1, -1)), out, kc, vc, table[b : b + 1], _i32([0]), _i32([p]), H, G, D, window,
                                    scale, keep_first=keep, sinks=_f32(sinks), score_bias=_f32(lut_b))
            want = _want(q, k, vs[b], G, scale, window, keep, sinks, lut_b, p)
            assert _rel(out.reshape(1, H, D), want) < 5e-6, (name, b)
    kernels.check_status()


def _tiled_case(H, G, D, lens, counts, seed, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    table, kc, vc, ks, vs = _paged(lens, G, D, dtype, seed)
    for b in range(len(lens)):
        _fill(table, kc, b, ks[b]), _fill(table, vc, b, vs[b])
    past = [n - c for n, c in zip(lens, counts)]
    q = _exact(plain.unit_rms(torch.randn(sum(counts), H, D, generator=g, dtype=F), 1e-6), dtype)
    return table, kc, vc, ks, vs, past, q


def _check_tiled(kernel, H, G, D, window, keep, lens, counts, biased, seed, **kw):
    from llmoxide_b200 import kernels

    table, kc, vc, ks, vs, past, q = _tiled_case(H, G, D, lens, counts, seed)
    g = torch.Generator().manual_seed(seed + 1)
    reach = max(lens) + 1
    for name, bump in (("edge of the window", (window or reach) - 1), ("one beyond it", window or reach - 1), ("itself", 0),
                       ("a page back", 64), ("far", 199), ("none", None)):
        lut = None
        if biased:
            n = min(window, reach) if window and not keep else reach
            lut = torch.randn(H, n, generator=g, dtype=F) * 0.5
            if bump is not None and bump < n:
                lut[:, bump] += 6.0                     # one distance stands out
            lut = _exact(lut)
        sinks = _exact(torch.randn(H, generator=g, dtype=F) * 2)
        qd, out = q.reshape(q.shape[0], -1).to(torch.bfloat16).to(DEV), torch.empty((q.shape[0], H * D), dtype=torch.bfloat16, device=DEV)
        ctx = _ctx(past, counts)
        extra = dict(keep_first=keep, sinks=_f32(sinks), score_bias=_f32(lut) if biased else None, **kw)
        if kernel == "decode":
            kernels.attention_decode(qd, out, kc, vc, table, ctx.seq_past, H, G, D, window, 0.15, **extra)
        else:
            getattr(kernels, kernel)(qd, out, kc, vc, table, ctx.seq_start, ctx.seq_past, ctx.n_seqs, ctx.max_new, H, G, D, window,
                                     0.15, **extra)
        at = 0
        for b, (n, c) in enumerate(zip(lens, counts)):
            want = _want(q[at : at + c], ks[b], vs[b], G, 0.15, window, keep, sinks, lut, n - c)
            err = _rel(out[at : at + c].float().reshape(c, H, D), want)
            assert err < 1.2e-2, (kernel, name, b, err)
            at += c
    kernels.check_status()


@pytest.mark.parametrize("n_chunks", [0, 1, 3, 8, 11])
@pytest.mark.parametrize("H, G, D, window, keep, biased", [(4, 1, 128, 100, 0, True), (8, 4, 64, 129, 0, True), (18, 2, 32, 70, 0, True),
                                                           (6, 3, 48, None, 0, True), (8, 4, 64, 64, 3, False), (10, 5, 80, 90, 1, False),
                                                           (4, 2, 128, 150, 65, True), (3, 3, 112, 33, 0, True)])
def test_decode_attention_with_biases_and_sinks(H, G, D, window, keep, biased, n_chunks):
    lens = [300, 65, 64, 1, 33, 230]
    _check_tiled("decode", H, G, D, window, keep, lens, [1] * len(lens), biased, seed=D + H, n_chunks=n_chunks)


@pytest.mark.parametrize("window, keep, biased", [(100, 0, True), (64, 0, True), (129, 3, True), (None, 0, True), (150, 65, True), (33, 0, True),
                                                  (90, 4, False)])
@pytest.mark.parametrize("lens, counts", [([300, 65, 17], [300, 65, 17]), ([260, 131, 70, 5], [2, 129, 6, 5])])
def test_prompt_attention_with_biases_and_sinks(window, keep, biased, lens, counts):
    _check_tiled("attention_prefill", 8, 4, 64, window, keep, lens, counts, biased, seed=3)
    _check_tiled("attention_prefill", 4, 1, 128, window, keep, lens, counts, biased, seed=4)
    _check_tiled("attention_prefill_tc", 4, 1, 128, window, keep, lens, counts, biased, seed=4)
    _check_tiled("attention_prefill_tc", 6, 3, 128, window, keep, lens, counts, biased, seed=5)


def test_biases_are_refused_where_they_are_not_built():
    from llmoxide_b200 import kernels
    from llmoxide_b200.errors import Unsupported

    table, kc, vc, *_ = _paged([5], 1, 64, torch.bfloat16, 0)
    q = torch.zeros((1, 64), dtype=torch.bfloat16, device=DEV)
    lut = torch.zeros((1, 8), device=DEV)
    with pytest.raises(Unsupported):
        kernels.attention_decode(q, q.clone(), kc, vc, table, _i32([4]), 1, 1, 64, 4, 0.1, score_bias=lut, softcap=3.0)
    with pytest.raises(Unsupported):
        kernels.attention_paged(q, q.clone(), kc, vc, table, _i32([0]), _i32([4]), 1, 1, 64, 4, 0.1, score_bias=lut, softcap=3.0)


# ---------------------------------------------------------------------------------------------------------
# feed-forwards without a gate
# ---------------------------------------------------------------------------------------------------------

def _runtime(dtype):
    from llmoxide_b200.parts import Runtime

    return Runtime(dtype="float32" if dtype == torch.float32 else "bfloat16", device=torch.device(DEV), max_positions=256)


@pytest.mark.parametrize("activation, f", [("relu_squared", plain.relu_squared), ("silu", plain.silu),
                                           ("relu", lambda z: torch.clamp(z, min=0))])
@pytest.mark.parametrize("T", [1, 16, 50, 128, 300])
def test_activation_in_the_products_epilogue_and_behind_partials(activation, f, T):
    from llmoxide_b200 import kernels

    g = torch.Generator().manual_seed(T)
    for N, K in ((64, 136), (200, 320), (1000, 72)):
        x, w = (_exact(torch.randn(n, K, generator=g) * 0.3, torch.bfloat16) for n in (T, N))
        out = torch.empty((T, N), dtype=torch.bfloat16, device=DEV)
        xd, wd = x.to(torch.bfloat16).to(DEV), w.to(torch.bfloat16).to(DEV)
        kernels.gemm_tc(xd, wd, out, gated=3, pair=T > 128, activation=activation)
        want = f(x @ w.T)
        assert _rel(out.float(), want) < 6e-3
        parts = _f32(torch.stack([x @ w.T - 1.25, torch.full((T, N), 1.25, dtype=F)]))
        kernels.plain_act(parts, out, activation)
        assert _rel(out.float(), want) < 6e-3
        full = torch.empty((T, N), device=DEV)
        kernels.plain_act(parts, full, activation)
        assert _rel(full, want) < 4e-6
    kernels.check_status()


@pytest.mark.parametrize("T", [1, 5, 40, 129, 700])
@pytest.mark.parametrize("d, ff, E, top, shared", [(96, 40, 6, 2, 24), (100, 20, 7, 3, 28), (256, 64, 8, 8, 128), (64, 72, 3, 1, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_without_gates_and_a_shared_one(T, d, ff, E, top, shared, dtype):
    from llmoxide_b200 import kernels
    from llmoxide_b200.config.spec import PartSpec, TensorSpec
    from llmoxide_b200.parts.experts import RoutedExperts

    g = torch.Generator().manual_seed(T + d)
    x = _exact(torch.randn(T, d, generator=g), dtype)
    w = {"mlp.router": torch.randn(E, d, generator=g) * 0.5, "mlp.router.b": torch.randn(E, generator=g)}
    for e in list(range(E)) + (["shared"] if shared else []):
        n, f = (f"mlp.e{e}", ff) if e != "shared" else ("mlp.shared", shared)
        w[n + ".up"], w[n + ".down"] = torch.randn(f, d, generator=g) * 0.1, torch.randn(d, f, generator=g) * 0.2
    w = {k: _exact(v, dtype) for k, v in w.items()}
    tensors = {"router": TensorSpec("mlp.router", (E, d)), "router_bias": TensorSpec("mlp.router.b", (E,), "vector")}
    for e in range(E):
        tensors[f"up{e}"], tensors[f"down{e}"] = TensorSpec(f"mlp.e{e}.up", (ff, d)), TensorSpec(f"mlp.e{e}.down", (d, ff))
    if shared:
        tensors.update(shared_up=TensorSpec("mlp.shared.up", (shared, d)), shared_down=TensorSpec("mlp.shared.down", (d, shared)))
    part = RoutedExperts(PartSpec("routed_experts", dict(
        hidden_size=d, intermediate_size=ff, n_experts=E, top=top, score="softmax_top", gated=False, activation="relu_squared",
        shared_size=shared), tensors), {k: v.to(dtype).to(DEV).contiguous() for k, v in w.items()}, _runtime(dtype))
    want = plain.experts(w, "", dict(router=dict(experts=E, top=top), shared=dict(ff=shared) if shared else None), x)
    xd, ctx = x.to(dtype).to(DEV).contiguous(), SimpleNamespace(probe=None)
    y = part.forward(xd, ctx)
    assert y.shape[0] >= top and y.shape[1:] == (T, d)
    tol = 5e-6 if dtype == torch.float32 else 1.2e-2
    assert _rel(y.double().sum(0), want) < tol
    # with the stream at hand the shared expert may add to it; the sum is the same
    h = torch.randn(T, d, generator=g).to(DEV)
    h0 = h.clone()
    y = part.forward(xd, ctx, residual=h)
    assert _rel((h - h0).double() + y.double().sum(0), want) < tol
    assert part.adds_to_residual == bool(shared)
    kernels.check_status()


# ---------------------------------------------------------------------------------------------------------
# the state-space recurrence
# ---------------------------------------------------------------------------------------------------------

SHAPES = [  # H, G, N, P, taps, parts
    (4, 2, 12, 20, 3, 4), (5, 5, 7, 13, 1, 5), (2, 1, 30, 9, 2, 3), (8, 2, 64, 64, 4, 2), (2, 1, 128, 128, 4, 1),
    (12, 4, 96, 8, 4, 3), (6, 3, 68, 36, 3, 8), (1, 1, 1, 1, 5, 1), (3, 1, 200, 130, 6, 2), (16, 1, 128, 64, 4, 1)]


def _ssm_weights(H, G, N, P, taps, seed):
    g = torch.Generator().manual_seed(seed)
    C, inner = H * P + 2 * G * N, H * P
    r = lambda *s: torch.randn(*s, generator=g)
    w = {"mix.conv": r(C, taps) * 0.5, "mix.conv.b": r(C) * 0.2, "mix.dt_bias": r(H) * 0.5 - 1.5, "mix.A_log": r(H) * 0.7,
         "mix.D": r(H), "mix.norm": 1 + 0.2 * r(inner)}
    return {k: _exact(v) for k, v in w.items()}, g


def _plain_ssm(w, H, G, N, P, proj):
    """(gated outputs [T, inner] before the norm, S of every head) of one sequence from its projected rows."""
    T, inner = proj.shape[0], H * P
    z, xbc, dt = proj[:, :inner], proj[:, inner : 2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N :]
    xbc = plain.silu(plain.causal_conv(xbc, w["mix.conv"], w["mix.conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B, C = (xbc[:, inner + i * G * N : inner + (i + 1) * G * N].reshape(T, G, N) for i in (0, 1))
    dt = plain.softplus(dt + w["mix.dt_bias"])
    ys, S = [], []
    for h in range(H):
        y, s = plain.state_space(x[:, h], B[:, h // (H // G)], C[:, h // (H // G)], dt[:, h], w["mix.A_log"][h], w["mix.D"][h])
        ys.append(y), S.append(s)
    return torch.cat(ys, 1) * plain.silu(z), torch.stack(S)


class _Ssm:
    """The kernels on a state area of their own."""

    def __init__(self, w, H, G, N, P, taps, n_slots):
        self.dims, self.C = (H, G, N, P), H * P + 2 * G * N
        self.conv_w, self.taps = _f32(w["mix.conv"].t()), taps
        self.vec = [_f32(w[k]) for k in ("mix.conv.b", "mix.A_log", "mix.dt_bias", "mix.D")]
        self.ring_off = (H * N * P + 3) // 4 * 4
        self.state = torch.zeros((n_slots, (self.ring_off + taps * self.C + 3) // 4 * 4), device=DEV)

    def run(self, proj, past, counts, slots):
        from llmoxide_b200 import kernels

        ctx = _ctx(past, counts, slots)
        y = torch.full((sum(counts), self.dims[0] * self.dims[3]), float("nan"), device=DEV)
        f = kernels.ss_decode if ctx.is_decode else kernels.ss_prompt
        f(proj, self.conv_w, *self.vec, self.state, self.ring_off, y, ctx, *self.dims)
        return y

    def S(self, slot):
        H, G, N, P = self.dims
        return self.state[slot, : H * N * P].reshape(H, N, P)

    def ring(self, slot, pos):
        return self.state[slot, self.ring_off + (pos % self.taps) * self.C :][: self.C]


CUTS = {"whole": lambda n: [n], "one by one": lambda n: [1] * n, "twos": lambda n: [2] * (n // 2) + [1] * (n % 2),
        "chunks' edges": lambda n: [63, 1, 64, 1, n - 129] if n > 129 else [n],
        "uneven": lambda n: [5, 70, n - 75] if n > 75 else [n - 1, 1], "tail": lambda n: [n - 3, 1, 1, 1]}


@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("shape", SHAPES)
def test_state_space_under_every_cutting(shape, cut):
    """Two sequences of unequal lengths side by side, in slots that are neither first nor in order."""
    from llmoxide_b200 import kernels

    H, G, N, P, taps, parts = shape
    w, g = _ssm_weights(H, G, N, P, taps, seed=N + P)
    width = 2 * H * P + 2 * G * N + H
    lens = [150, 131] if cut != "one by one" else [70, 66]
    rows = [_exact(torch.randn(n, width, generator=g)) for n in lens]
    want = [_plain_ssm(w, H, G, N, P, r) for r in rows]
    k = _Ssm(w, H, G, N, P, taps, 4)
    k.state[0] += 7.0                                     # another owner's slot stays as it is
    before, slots = k.state[0].clone(), [3, 1]
    got, past = [[], []], [0, 0]
    steps = [CUTS[cut](n) for n in lens]
    for i in range(max(len(s) for s in steps)):
        live = [b for b in (0, 1) if i < len(steps[b]) and steps[b][i] > 0]
        counts = [steps[b][i] for b in live]
        proj = _f32(torch.cat([rows[b][past[b] : past[b] + c] for b, c in zip(live, counts)]))
        y = k.run(proj, [past[b] for b in live], counts, [slots[b] for b in live])
        at = 0
        for b, c in zip(live, counts):
            got[b].append(y[at : at + c])
            past[b] += c
            at += c
    for b in (0, 1):
        y, S = want[b]
        assert _rel(torch.cat(got[b]), y) < 2e-5, b
        assert _rel(k.S(slots[b]), S) < 1e-5, b
        for p in range(max(0, lens[b] - taps + 1), lens[b]):              # the rows a next token would read
            assert torch.equal(k.ring(slots[b], p), _f32(rows[b][p, H * P : H * P + k.C])), (b, p)
    assert torch.equal(k.state[0], before)
    y = torch.cat(got[0])
    for act in (torch.float32, torch.bfloat16):
        out = torch.empty(y.shape, dtype=act, device=DEV)
        kernels.ss_norm(y.contiguous(), _f32(w["mix.norm"]), 1e-3, parts, out)
        T, n = y.shape
        unit = plain.unit_rms(want[0][0].reshape(T, parts, n // parts), 1e-3).reshape(T, n) * w["mix.norm"]
        assert _rel(out.float(), unit) < (3e-5 if act == torch.float32 else 6e-3)
    kernels.check_status()


def test_state_space_takes_partials_and_rows_of_any_stride():
    H, G, N, P, taps = 4, 2, 16, 24, 4
    w, g = _ssm_weights(H, G, N, P, taps, 3)
    width = 2 * H * P + 2 * G * N + H
    row = _exact(torch.randn(90, width, generator=g))
    want, S = _plain_ssm(w, H, G, N, P, row)
    parts = _exact(torch.randn(5, 90, width, generator=g) * 0.3)
    parts[4] = _exact(row - parts[:4].sum(0))
    want, S = _plain_ssm(w, H, G, N, P, parts.sum(0))
    k = _Ssm(w, H, G, N, P, taps, 1)
    pd = _f32(parts)
    got = [k.run(pd[:, :80].contiguous(), [0], [80], [0])] + [k.run(pd[:, t : t + 1].contiguous(), [t], [1], [0]) for t in range(80, 90)]
    assert _rel(torch.cat(got), want) < 2e-5 and _rel(k.S(0), S) < 1e-5


def test_state_space_many_sequences_with_every_remainder_of_a_chunk():
    """Lengths that end before, at and behind a chunk's edge, packed behind one another, with pasts of their own."""
    H, G, N, P, taps = 2, 1, 20, 12, 3
    w, g = _ssm_weights(H, G, N, P, taps, 9)
    width = 2 * H * P + 2 * G * N + H
    lens = [1, 63, 64, 65, 2, 127, 128, 129, 16, 15, 17]
    past = [0, 5, 64, 0, 77, 1, 0, 3, 130, 0, 12]
    k = _Ssm(w, H, G, N, P, taps, len(lens))
    rows = [_exact(torch.randn(p + n, width, generator=g)) for p, n in zip(past, lens)]
    for b, p in enumerate(past):
        if p:
            k.run(_f32(rows[b][:p]), [0], [p], [b])
    y = k.run(_f32(torch.cat([r[p:] for r, p in zip(rows, past)])), past, lens, list(range(len(lens))))
    at = 0
    for b, n in enumerate(lens):
        want, S = _plain_ssm(w, H, G, N, P, rows[b])
        assert _rel(y[at : at + n], want[past[b] :]) < 2e-5, b
        assert _rel(k.S(b), S) < 1e-5, b
        at += n


@pytest.mark.parametrize("cut", ["whole", "one by one", "uneven"])
def test_state_space_decays_at_their_ends_and_a_far_write(cut):
    """One head forgets everything between tokens (a underflows), one nothing (a is one to the last bit) while almost
    nothing is written, except one token that writes strongly and is read hundreds of positions later."""
    H, G, N, P, taps = 3, 1, 8, 8, 2
    w, g = _ssm_weights(H, G, N, P, taps, 4)
    T = 400
    width = 2 * H * P + 2 * G * N + H
    w["mix.A_log"] = torch.tensor([6.0, -12.0, -3.0], dtype=F)
    w["mix.dt_bias"] = torch.tensor([3.0, -14.0, -6.0], dtype=F)
    row = _exact(torch.randn(T, width, generator=g))
    row[17, -1] = row[17, -2] = 22.0                       # heads 1 and 2 write at position 17
    row = _exact(row)
    want, S = _plain_ssm(w, H, G, N, P, row)
    k = _Ssm(w, H, G, N, P, taps, 1)
    got, past = [], 0
    for c in CUTS[cut](T):
        got.append(k.run(_f32(row[past : past + c]), [past], [c], [0]))
        past += c
    got = torch.cat(got)
    for h in range(H):
        cols = slice(h * P, (h + 1) * P)
        assert _rel(got[:, cols], want[:, cols]) < 2e-5, h
        assert _rel(k.S(0)[h], S[h]) < 2e-5, h
    # the far write is what head 1 still reads at the end
    without = row.clone()
    without[17, -2] = 0.0
    far, _ = _plain_ssm(w, H, G, N, P, without)
    assert (far[-1, P : 2 * P] - want[-1, P : 2 * P]).abs().max() > 0.1 * want[-1, P : 2 * P].abs().max()


def test_state_space_bad_slots_are_reported_and_touch_nothing():
    from llmoxide_b200 import kernels
    from llmoxide_b200.errors import KernelError

    H, G, N, P, taps = 2, 1, 8, 8, 2
    w, g = _ssm_weights(H, G, N, P, taps, 4)
    width = 2 * H * P + 2 * G * N + H
    k = _Ssm(w, H, G, N, P, taps, 2)
    for counts in ([3], [1]):
        k.run(_f32(torch.randn(counts[0], width, generator=g)), [0], counts, [5])
        torch.cuda.synchronize()
        assert not k.state.any()
        with pytest.raises(KernelError, match="state_space"):
            kernels.check_status()
    kernels.check_status()
