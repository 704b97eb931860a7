"""GPU: the Soputar decoder's mechanisms one by one against the plain implementation (tests/plain_soputar.py)."""

import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_soputar as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F = torch.float64


def _rel(got, want):
    want = np.asarray(want, dtype=np.float64)
    return float(np.abs(np.asarray(got, dtype=np.float64) - want).max() / max(np.abs(want).max(), 1e-30))


def _exact(t, dtype=torch.float32):
    """Numbers that the given dtype holds exactly, as float64."""
    return t.to(dtype).to(F)


def _i32(x):
    return torch.tensor(np.asarray(x), dtype=torch.int32, device=DEV)


def _ctx(past, counts, slots=None):
    """The step's index arrays for sequences that hold ``past`` positions and bring ``counts`` tokens."""
    token_seq = [b for b, n in enumerate(counts) for _ in range(n)]
    token_pos = [past[b] + k for b, n in enumerate(counts) for k in range(n)]
    starts = np.concatenate([[0], np.cumsum(counts)])
    pages = sum(-(-(p + n) // 64) for p, n in zip(past, counts))
    return SimpleNamespace(token_seq=_i32(token_seq), token_pos=_i32(token_pos), seq_start=_i32(starts),
                           seq_past=_i32(past), seq_slot=_i32(slots if slots is not None else range(len(counts))),
                           n_seqs=len(counts), n_tokens=int(sum(counts)), max_new=max(counts), ctx_pages=pages,
                           is_decode=all(n == 1 for n in counts))


def _store(lens, G, *dims, dtype, seed=0, width=None):
    """Empty paged stores (one per entry of ``dims``) for sequences of those lengths, pages dealt out in any order."""
    g = torch.Generator().manual_seed(seed)
    per = [max(1, -(-n // 64)) for n in lens]
    order = torch.randperm(sum(per) + 2, generator=g).tolist()
    table = torch.full((len(per), width or max(per)), -1, dtype=torch.int32)
    at = 0
    for b, n in enumerate(per):
        table[b, :n] = torch.tensor(order[at : at + n], dtype=torch.int32)
        at += n
    # rows nobody has written hold NaN: whoever reads one shows it
    stores = [torch.full((sum(per) + 2, G, 64, d), float("nan"), dtype=dtype, device=DEV) for d in dims]
    return table.to(DEV), stores


def _fill(table, store, b, rows, first=0):
    """rows [n, G, D] of sequence b from position ``first``."""
    for j in range(rows.shape[0]):
        p = first + j
        store[int(table[b, p // 64]), :, p % 64] = rows[j].to(store.dtype).to(DEV)


# ---------------------------------------------------------------------------------------------------------
# the norm behind a sublayer whose reader takes the stream itself
# ---------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("d, n_split", [(40, 1), (96, 3), (101, 2), (1000, 5), (4100, 1), (9000, 2)])
@pytest.mark.parametrize("act", [torch.float32, torch.bfloat16])
def test_result_normed_and_added_stream_handed_on_as_it_is(d, n_split, act):
    from llmoxide_b200 import kernels
    from llmoxide_b200.parts.norm import PostNormed, stream_rows

    g = torch.Generator().manual_seed(d)
    T, eps = 23, 1e-3
    h = _exact(torch.randn(T, d, generator=g) * 3)
    y = _exact(torch.randn(n_split, T, d, generator=g) * 0.05)          # small: eps and the norm show
    w = _exact(torch.randn(d, generator=g) * 0.3)
    want = h + plain.rms_norm_zero_centred(y.sum(0), w, eps)
    hd = h.float().to(DEV).contiguous()
    owed = PostNormed([(y.float().to(DEV).contiguous(), 1.0)], None, (1.0 + w).float().to(DEV), False, eps)
    out = stream_rows(hd, owed, act)
    assert _rel(hd.cpu().numpy(), want.numpy()) < 2e-6
    assert torch.equal(out.cpu(), hd.cpu().to(act)) and (out is hd) == (act == torch.float32)
    before = hd.clone()
    out = stream_rows(hd, None, act)                                      # nothing owed: the rows alone
    assert torch.equal(out.cpu(), before.cpu().to(act)) and torch.equal(hd, before)
    kernels.check_status()


# ---------------------------------------------------------------------------------------------------------
# whole-row norm of q and k, query temperature, cache write
# ---------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("H, G, D, Dv, temp, n_split", [(4, 2, 32, 16, (0.4, 3), 1), (3, 3, 20, 40, (0.9, 1), 3),
                                                        (5, 1, 18, 7, None, 1), (16, 4, 128, 128, (0.2, 100), 2),
                                                        (1, 1, 64, 64, (-0.3, 70), 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_row_norm_with_temperature_and_cache_write(H, G, D, Dv, temp, n_split, dtype):
    from llmoxide_b200 import kernels

    g = torch.Generator().manual_seed(H * 100 + D)
    past, counts, eps = [0, 60, 199], [9, 8, 1], 1e-4
    T, N = sum(counts), (H + G) * D + G * Dv
    proj = _exact(torch.randn(n_split, T, N, generator=g) * 0.1, torch.float32 if n_split > 1 else dtype)
    # one head much larger than the others: a norm per head would show
    proj[:, :, :D] *= 8
    qg, kg = _exact(torch.randn(H * D, generator=g)), _exact(torch.randn(G * D, generator=g))
    pos = [p + k for p, n in zip(past, counts) for k in range(n)]
    row = proj.sum(0)
    q = plain.unit_rms(row[:, : H * D], eps) * qg
    if temp:
        q = q * torch.tensor([plain.query_temperature(p, *temp) for p in pos], dtype=F)[:, None]
    k = (plain.unit_rms(row[:, H * D : (H + G) * D], eps) * kg).reshape(T, G, D)
    v = row[:, (H + G) * D :].reshape(T, G, Dv)
    table, (kc, vc) = _store([p + n for p, n in zip(past, counts)], G, D, Dv, dtype=dtype)
    pd = (proj[0] if n_split == 1 else proj).to(torch.float32 if n_split > 1 else dtype).to(DEV).contiguous()
    ctx = _ctx(past, counts)
    out = torch.empty((T, H * D), dtype=dtype, device=DEV)
    kernels.qk_row_norm(pd, out, kc, vc, table, ctx, qg.float().to(DEV), kg.float().to(DEV), eps, temp, H, G, D, Dv, True)
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    assert _rel(out.float().cpu().numpy(), q.numpy()) < tol
    written = torch.zeros(kc.shape[0], 64, dtype=torch.bool)
    for t in range(T):
        b, p = int(ctx.token_seq[t]), pos[t]
        page = int(table[b, p // 64])
        written[page, p % 64] = True
        assert _rel(kc[page, :, p % 64].float().cpu().numpy(), k[t].numpy()) < tol * 4
        assert _rel(vc[page, :, p % 64].float().cpu().numpy(), v[t].numpy()) < tol * 4
    assert bool(torch.isnan(kc[:, 0, :, 0].cpu()[~written]).all())        # and nothing else was
    # a borrower's row is the query alone
    alone = pd[..., : H * D].contiguous()
    out2 = torch.empty_like(out)
    kernels.qk_row_norm(alone, out2, kc, vc, table, ctx, qg.float().to(DEV), None, eps, temp, H, G, D, Dv, False)
    assert _rel(out2.float().cpu().numpy(), q.numpy()) < tol
    kernels.check_status()


# ---------------------------------------------------------------------------------------------------------
# capped scores and learned sinks, every attention kernel
# ---------------------------------------------------------------------------------------------------------

def _attention_case(lens, H, G, D, Dv, dtype, seed):
    """Keys and values of sequences of those lengths; per sequence one key made to stand out for the last query."""
    g = torch.Generator().manual_seed(seed)
    ks = [_exact(torch.randn(n, G, D, generator=g), dtype) for n in lens]
    vs = [_exact(torch.randn(n, G, Dv, generator=g), dtype) for n in lens]
    qs = [_exact(torch.randn(n, H, D, generator=g), dtype) for n in lens]
    return qs, ks, vs


def _plain_heads(q, k, v, scale, softcap, sinks):
    H, G = q.shape[1], k.shape[1]
    return torch.stack([plain.attend_causal(q[:, h], k[:, h // (H // G)], v[:, h // (H // G)], scale, softcap=softcap,
                                            sink=None if sinks is None else sinks[h]) for h in range(H)], dim=1)


CAPS = [(4.0, False), (None, True), (2.0, True)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("softcap, with_sinks", CAPS)
@pytest.mark.parametrize("H, G, D, Dv", [(4, 2, 32, 16), (3, 3, 20, 41), (8, 1, 64, 64)])
def test_general_attention_with_capped_scores_and_sinks(H, G, D, Dv, softcap, with_sinks, dtype):
    """One key at a time stands out (the first, both sides of a page border, the query's own, the one after it), large
    enough that the cap decides the result."""
    from llmoxide_b200 import kernels

    lens = [130, 64, 1, 65]
    qs, ks, vs = _attention_case(lens, H, G, D, Dv, dtype, 5)
    for b, j in ((0, 0), (0, 63), (0, 64), (0, 129), (1, 63), (3, 64)):
        ks[b][j] = _exact(ks[b][j] * 2 + qs[b][-1][:: H // G], dtype)
    sinks = _exact(torch.linspace(-2, 6, H)) if with_sinks else None
    table, (kc, vc) = _store(lens, G, D, Dv, dtype=dtype)
    for b in range(len(lens)):
        _fill(table, kc, b, ks[b]), _fill(table, vc, b, vs[b])
    q = torch.cat(qs).reshape(-1, H * D).to(dtype).to(DEV).contiguous()
    out = torch.empty((q.shape[0], H * Dv), dtype=dtype, device=DEV)
    ctx = _ctx([0] * len(lens), lens)
    kernels.attention_paged(q, out, kc, vc, table, ctx.token_seq, ctx.token_pos, H, G, D, None, 0.3, v_head_dim=Dv,
                            softcap=softcap or 0.0, sinks=None if sinks is None else sinks.float().to(DEV))
    want = torch.cat([_plain_heads(q_, k_, v_, 0.3, softcap, sinks) for q_, k_, v_ in zip(qs, ks, vs)]).reshape(-1, H * Dv)
    assert _rel(out.float().cpu().numpy(), want.numpy()) < (3e-6 if dtype == torch.float32 else 6e-3)
    kernels.check_status()


@pytest.mark.parametrize("softcap, with_sinks", CAPS)
@pytest.mark.parametrize("D, H, G", [(64, 8, 1), (128, 4, 4), (48, 6, 2), (16, 20, 2), (256, 2, 1)])
def test_decode_attention_with_capped_scores_and_sinks(D, H, G, softcap, with_sinks):
    """Lengths on both sides of a tile's and a page's border, every way of sharing the keys out."""
    from llmoxide_b200 import kernels

    lens = [1, 32, 33, 64, 65, 200, 641]
    qs, ks, vs = _attention_case(lens, H, G, D, D, torch.bfloat16, 6)
    scale = 1.5 / math.sqrt(D)
    for b, n in enumerate(lens):
        for j in (0, n // 2, n - 1):
            ks[b][j] = _exact(ks[b][j] + qs[b][-1][:: H // G], torch.bfloat16)
    sinks = _exact(torch.linspace(-3, 5, H)) if with_sinks else None
    table, (kc, vc) = _store(lens, G, D, D, dtype=torch.bfloat16, width=12)
    for b in range(len(lens)):
        _fill(table, kc, b, ks[b]), _fill(table, vc, b, vs[b])
    q = torch.stack([x[-1] for x in qs]).reshape(-1, H * D).to(torch.bfloat16).to(DEV).contiguous()
    want = torch.stack([_plain_heads(q_, k_, v_, scale, softcap, sinks)[-1] for q_, k_, v_ in zip(qs, ks, vs)])
    for n_chunks in (0, 1, 2, 3, 5, 8, 11, 32):
        out = torch.empty_like(q)
        kernels.attention_decode(q, out, kc, vc, table, _i32([n - 1 for n in lens]), H, G, D, None, scale, n_chunks=n_chunks,
                                 softcap=softcap or 0.0, sinks=None if sinks is None else sinks.float().to(DEV))
        assert _rel(out.float().cpu().numpy(), want.reshape(-1, H * D).numpy()) < 8e-3, n_chunks
    kernels.check_status()


@pytest.mark.parametrize("softcap, with_sinks", CAPS)
@pytest.mark.parametrize("kernel, D, H, G", [("mma", 64, 8, 1), ("mma", 128, 4, 2), ("tc", 128, 4, 4), ("tc", 128, 6, 2)])
def test_prompt_attention_with_capped_scores_and_sinks(kernel, D, H, G, softcap, with_sinks):
    """Whole prompts and later portions of prompts, lengths around a tile's and a page's border."""
    from llmoxide_b200 import kernels

    past, counts = [0, 0, 100, 63, 0, 5], [130, 1, 65, 2, 64, 200]
    lens = [p + n for p, n in zip(past, counts)]
    qs, ks, vs = _attention_case(lens, H, G, D, D, torch.bfloat16, 7)
    scale = 1.5 / math.sqrt(D)
    for b, n in enumerate(lens):
        for j in (0, n // 2, n - 1):
            ks[b][j] = _exact(ks[b][j] + qs[b][-1][:: H // G], torch.bfloat16)
    sinks = _exact(torch.linspace(-3, 5, H)) if with_sinks else None
    table, (kc, vc) = _store(lens, G, D, D, dtype=torch.bfloat16)
    for b in range(len(lens)):
        _fill(table, kc, b, ks[b]), _fill(table, vc, b, vs[b])
    q = torch.cat([x[p:] for x, p in zip(qs, past)]).reshape(-1, H * D).to(torch.bfloat16).to(DEV).contiguous()
    want = torch.cat([_plain_heads(q_, k_, v_, scale, softcap, sinks)[p:] for q_, k_, v_, p in zip(qs, ks, vs, past)])
    ctx = _ctx(past, counts)
    out = torch.empty_like(q)
    f = kernels.attention_prefill_tc if kernel == "tc" else kernels.attention_prefill
    f(q, out, kc, vc, table, ctx.seq_start, ctx.seq_past, ctx.n_seqs, ctx.max_new, H, G, D, None, scale,
      softcap=softcap or 0.0, sinks=None if sinks is None else sinks.float().to(DEV))
    assert _rel(out.float().cpu().numpy(), want.reshape(-1, H * D).numpy()) < 8e-3
    kernels.check_status()


def test_a_cap_far_beyond_the_scores_changes_nothing_and_saturated_scores_stay_finite():
    from llmoxide_b200 import kernels

    H, G, D, n = 4, 2, 64, 150
    qs, ks, vs = _attention_case([n], H, G, D, D, torch.bfloat16, 8)
    table, (kc, vc) = _store([n], G, D, D, dtype=torch.bfloat16)
    _fill(table, kc, 0, ks[0]), _fill(table, vc, 0, vs[0])
    q = qs[0].reshape(n, H * D).to(torch.bfloat16).to(DEV).contiguous()
    ctx = _ctx([0], [n])
    outs = []
    for cap in (0.0, 1e4):
        out = torch.empty_like(q)
        kernels.attention_prefill(q, out, kc, vc, table, ctx.seq_start, ctx.seq_past, 1, n, H, G, D, None, 0.1, softcap=cap)
        outs.append(out.float().cpu().numpy())
    assert _rel(outs[1], outs[0]) < 6e-3
    big = (q * 500).contiguous()                  # every score is at +-cap
    out = torch.empty_like(q)
    kernels.attention_prefill(big, out, kc, vc, table, ctx.seq_start, ctx.seq_past, 1, n, H, G, D, None, 1.0, softcap=5.0)
    want = _plain_heads(_exact(big.cpu()).reshape(n, H, D), ks[0], vs[0], 1.0, 5.0, None).reshape(n, H * D)
    assert _rel(out.float().cpu().numpy(), want.numpy()) < 8e-3
    kernels.check_status()


# ---------------------------------------------------------------------------------------------------------
# the gated delta rule
# ---------------------------------------------------------------------------------------------------------

class _Delta:
    """A delta layer's tensors, its sequences' projected rows, and the plain outputs before and behind norm and gate."""

    def __init__(self, H, G, D, Dv, taps, lens, seed, decay=(-2.0, 1.0), beta_shift=0.0):
        g = torch.Generator().manual_seed(seed)
        self.H, self.G, self.D, self.Dv, self.taps, self.lens = H, G, D, Dv, taps, lens
        C = self.C = 2 * G * D + H * Dv
        N = C + H * Dv + 2 * H
        self.offsets = (0, G * D, 2 * G * D, C + H * Dv, C + H * Dv + H, C)          # q, k, v, b, a, gate
        self.rows = [_exact(torch.randn(n, N, generator=g)) for n in lens]
        for x in self.rows:
            x[:, C + H * Dv : C + H * Dv + H] += beta_shift
        self.conv = _exact(torch.randn(C, taps, generator=g) * 0.7)
        self.a_log = _exact(torch.randn(H, generator=g) * 0.5)
        self.dt = _exact(torch.randn(H, generator=g) * decay[1] + decay[0])
        self.gain = _exact(torch.randn(Dv, generator=g))
        self.eps, self.unit_eps = 1e-5, 1e-6
        self.ring_off = (H * D * Dv + 3) // 4 * 4
        self.floats = (self.ring_off + taps * C + 3) // 4 * 4

    def want(self, b):
        H, G, D, Dv, C = self.H, self.G, self.D, self.Dv, self.C
        x = self.rows[b]
        u = plain.silu(plain.causal_conv(x[:, :C], self.conv))
        q = plain.unit_vectors(u[:, : G * D].reshape(-1, G, D)) * D ** -0.5
        k = plain.unit_vectors(u[:, G * D : 2 * G * D].reshape(-1, G, D))
        v = u[:, 2 * G * D :].reshape(-1, H, Dv)
        beta = torch.sigmoid(x[:, self.offsets[3] : self.offsets[3] + H])
        g = torch.exp(-torch.exp(self.a_log) * plain.softplus(x[:, self.offsets[4] : self.offsets[4] + H] + self.dt))
        o, S = zip(*(plain.delta_rule(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], beta[:, h], g[:, h]) for h in range(H)))
        o = torch.stack(o, dim=1)
        y = plain.unit_rms(o, self.eps) * self.gain * plain.silu(x[:, self.offsets[5] :][:, : H * Dv]).reshape(-1, H, Dv)
        return o.reshape(-1, H * Dv), y.reshape(-1, H * Dv), torch.stack(S)

    def run(self, cuts, dtype=torch.float32, split=1):
        """``cuts[b]``: how many tokens sequence b brings in each step (0: it sits the step out).  Steps of single tokens
        go through the single-token kernel.  Returns y per sequence and the state area (slot 2 b is sequence b's)."""
        from llmoxide_b200 import kernels

        H, G, D, Dv = self.H, self.G, self.D, self.Dv
        dev = lambda t: t.float().to(DEV).contiguous()
        state = torch.zeros((2 * len(self.lens), self.floats), device=DEV)
        state[1::2] = 7.0
        args = (dev(self.conv.t()), self.taps, dev(self.a_log), dev(self.dt), D ** -0.5, self.unit_eps)
        fed, outs = [0] * len(self.lens), [[] for _ in self.lens]
        for j in range(max(len(c) for c in cuts)):
            live = [b for b, c in enumerate(cuts) if j < len(c) and c[j] > 0]
            counts = [cuts[b][j] for b in live]
            ctx = _ctx([fed[b] for b in live], counts, slots=[2 * b for b in live])
            proj = torch.cat([self.rows[b][fed[b] : fed[b] + cuts[b][j]] for b in live])
            if split > 1:        # float32 partials that add up to the rows
                parts = [proj * (0.25 * (s + 1)) for s in range(split - 1)]
                proj = torch.stack(parts + [proj - sum(parts)])
            proj = proj.to(dtype if split == 1 else torch.float32).to(DEV).contiguous()
            y = torch.empty((sum(counts), H * Dv), device=DEV)
            if ctx.is_decode:
                kernels.delta_decode(proj, self.offsets, *args, state, self.ring_off, dev(self.gain), self.eps, y, ctx, H, G, D, Dv)
            else:
                o = torch.empty_like(y)
                kernels.delta_prompt(proj, self.offsets, *args, state, self.ring_off, o, ctx, H, G, D, Dv)
                kernels.gated_norm(o, proj, self.offsets[5], dev(self.gain).repeat(H), self.eps, "silu", True, y, H, Dv)
            at = 0
            for b, n in zip(live, counts):
                outs[b].append(y[at : at + n].cpu())
                at += n
                fed[b] += n
        torch.cuda.synchronize()
        kernels.check_status()
        assert float(state[1::2].min()) == float(state[1::2].max()) == 7.0        # nobody's slots stay as they were
        return [torch.cat(o) for o in outs], state


CUTTINGS = {"whole": lambda n: [n], "one by one": lambda n: [1] * n, "twos": lambda n: [2] * (n // 2) + [1] * (n % 2),
            "sevens": lambda n: [7] * (n // 7) + ([n % 7] if n % 7 else []),
            "all but the last five, then one by one": lambda n: ([n - 5] if n > 5 else []) + [1] * min(5, n),
            "one, then eight, then the rest": lambda n: [1, 8, n - 9] if n > 9 else [n]}


@pytest.mark.parametrize("H, G, D, Dv, taps", [(4, 2, 24, 16, 3), (1, 1, 30, 41, 1), (2, 2, 128, 128, 4), (6, 1, 64, 64, 2),
                                               (3, 3, 140, 20, 5), (2, 1, 256, 136, 4), (5, 5, 3, 5, 16), (8, 4, 32, 6, 4)])
def test_delta_rule_under_every_cutting(H, G, D, Dv, taps):
    """Two sequences of unequal lengths side by side; prompts (chunks of eight tokens from a step's start) and single
    tokens; the state left behind is the plain one."""
    case = _Delta(H, G, D, Dv, taps, [37, 18], seed=D)
    want = [case.want(b) for b in range(2)]
    for what, cut in CUTTINGS.items():
        got, state = case.run([cut(37), cut(18)])
        for b in range(2):
            # relative to each position's own size: a position whose read-out is small counts as well
            assert _rel(got[b].numpy(), want[b][1].numpy()) < 3e-5, (what, b)
            S = state[2 * b][: H * D * Dv].reshape(H, D, Dv).cpu()
            assert _rel(S.numpy(), want[b][2].numpy()) < 3e-6, (what, b)
            ring = state[2 * b][case.ring_off : case.ring_off + taps * case.C].reshape(taps, case.C).cpu()
            for p in range(max(0, case.lens[b] - (taps - 1)), case.lens[b]):
                assert torch.equal(ring[p % taps], case.rows[b][p, : case.C].float()), (what, b, p)


@pytest.mark.parametrize("decay, beta_shift, what", [((4.0, 2.0), 0.0, "decays near zero"), ((-12.0, 0.5), 3.0, "decays near one"),
                                                     ((60.0, 1.0), 0.0, "decays that underflow"), ((-1.0, 0.5), -40.0, "no writes")])
def test_delta_rule_at_extreme_gates(decay, beta_shift, what):
    """Decays enter as products: none of these may give anything but the plain recurrence's numbers."""
    case = _Delta(4, 2, 32, 24, 4, [70], seed=3, decay=decay, beta_shift=beta_shift)
    want = case.want(0)
    for cut in ("whole", "sevens", "one by one"):
        got, state = case.run([CUTTINGS[cut](70)])
        assert bool(torch.isfinite(got[0]).all()) and bool(torch.isfinite(state[0]).all())
        S = state[0][: 4 * 32 * 24].reshape(4, 32, 24).cpu()
        assert np.abs(S.numpy() - want[2].numpy()).max() < 1e-5 * max(1.0, float(want[2].abs().max())), (what, cut)
        if what != "no writes":
            assert _rel(got[0].numpy(), want[1].numpy()) < 3e-5, (what, cut)


def test_delta_rule_out_of_partials_and_bfloat16_rows():
    case = _Delta(4, 2, 24, 16, 3, [21, 9], seed=11)
    want = [case.want(b)[1] for b in range(2)]
    for split in (2, 3, 9):
        for cut in ("whole", "one by one"):
            got, _ = case.run([CUTTINGS[cut](21), CUTTINGS[cut](9)], split=split)
            assert all(_rel(got[b].numpy(), want[b].numpy()) < 3e-5 for b in range(2)), (split, cut)
    case.rows = [_exact(x, torch.bfloat16) for x in case.rows]
    want = [case.want(b)[1] for b in range(2)]
    got, _ = case.run([[21], [9]], dtype=torch.bfloat16)
    assert all(_rel(got[b].numpy(), want[b].numpy()) < 3e-5 for b in range(2))


def test_delta_rule_many_unequal_sequences_against_each_alone():
    """A batch of eleven: chunk slots of neighbouring sequences must not meet, whatever their lengths' remainders."""
    lens = [1, 8, 9, 7, 16, 15, 17, 2, 31, 3, 24]
    case = _Delta(4, 4, 16, 12, 4, lens, seed=12)
    together, _ = case.run([[n] for n in lens])
    mixed, _ = case.run([[n - 1, 1] if n > 1 else [1] for n in lens])
    for b, n in enumerate(lens):
        want = case.want(b)[1].numpy()
        assert _rel(together[b].numpy(), want) < 3e-5 and _rel(mixed[b].numpy(), want) < 3e-5, (b, n)


def test_a_key_written_long_ago_is_read_and_can_be_replaced():
    """One direction is written at the first token with a large value, hundreds of other tokens follow, and the last
    token asks for it; then it is written anew."""
    case = _Delta(2, 1, 64, 32, 1, [400], seed=13, decay=(-30.0, 0.1))
    x, C, D = case.rows[0], case.C, case.D
    case.conv[:] = 1.0
    mark = torch.zeros(D, dtype=F)
    mark[5] = 40.0                                    # after silu and the unit norm: the unit vector of dim 5
    x[:, : 2 * D] = -x[:, : 2 * D].abs()              # other queries and keys: small negative, never near the mark
    x[:, 5], x[:, D + 5] = -20.0, -20.0
    for t in (0, 399):
        x[t, : 2 * D] = torch.cat([mark - 30.0 * (mark == 0), mark - 30.0 * (mark == 0)])
    x[0, 2 * D : C] = 9.0
    x[399, D : 2 * D] = -x[0, D : 2 * D].abs()        # the last token asks but writes elsewhere
    case.rows[0] = _exact(x)
    want = case.want(0)
    assert float(want[0][399].abs().min()) > 0.3      # the first value is still there to be read
    for cut in ("whole", "all but the last five, then one by one"):
        got, _ = case.run([CUTTINGS[cut](400)])
        assert _rel(got[0][399].numpy(), want[1][399].numpy()) < 1e-4, cut


# ---------------------------------------------------------------------------------------------------------
# attention over a cache of latents
# ---------------------------------------------------------------------------------------------------------

def _latent_rows(lens, rank, R, dtype, seed):
    g = torch.Generator().manual_seed(seed)
    return [_exact(torch.randn(n, rank + R, generator=g), dtype) for n in lens]


def _plain_latents(q, rows, rank, scale, sinks):
    """q [H, rank + R] of the last position, rows [n, rank + R] -> [H, rank]."""
    s = (q @ rows.T) * scale
    top = s.max(1, keepdim=True).values if sinks is None else torch.maximum(s.max(1, keepdim=True).values, sinks[:, None])
    e = torch.exp(s - top)
    den = e.sum(1, keepdim=True) + (0 if sinks is None else torch.exp(sinks[:, None] - top))
    return (e / den) @ rows[:, :rank]


@pytest.mark.parametrize("H, rank, R", [(3, 40, 8), (8, 96, 16), (16, 512, 64), (20, 304, 16), (5, 17, 6), (33, 128, 32),
                                        (2, 16, 16), (1, 600, 10)])
@pytest.mark.parametrize("with_sinks", [False, True])
def test_absorbed_attention_over_cached_latents(H, rank, R, with_sinks):
    """Lengths on both sides of a tile's and a page's border; a row far back, one at a page border and the newest stand
    out in turn; rows past the newest hold NaN.  The float32 kernel at every size, the tensor-core kernel at every way
    of sharing the rows out."""
    from llmoxide_b200 import kernels

    lens = [1, 31, 32, 33, 64, 65, 129, 700]
    scale = 1.0 / math.sqrt(rank + R)
    sinks = _exact(torch.linspace(-2, 4, H)) if with_sinks else None
    for dtype in (torch.float32, torch.bfloat16):
        rows = _latent_rows(lens, rank, R, dtype, rank)
        g = torch.Generator().manual_seed(9)
        q = _exact(torch.randn(len(lens), H, rank + R, generator=g), dtype)
        for b, n in enumerate(lens):
            for x, j in enumerate((n - 1, 0, n // 2, min(63, n - 1), min(64, n - 1))):
                rows[b][j] = _exact(rows[b][j] * 0.3 + q[b, x % H] * 1.2, dtype)
        table, (cache,) = _store(lens, 1, rank + R, dtype=dtype, width=12)
        for b in range(len(lens)):
            _fill(table, cache, b, rows[b][:, None, :])
        ctx = _ctx([n - 1 for n in lens], [1] * len(lens))
        want = torch.stack([_plain_latents(q[b], rows[b], rank, scale, sinks) for b in range(len(lens))])
        sd = None if sinks is None else sinks.float().to(DEV)
        lat = torch.empty((len(lens), H, rank), device=DEV)
        kernels.latent_paged(q.float().to(DEV).contiguous(), lat, cache, table, ctx, sd, scale, rank)
        assert _rel(lat.cpu().numpy(), want.numpy()) < 3e-6
        if dtype == torch.float32 or not kernels.latent_decode_supports(rank, R):
            continue
        for n_chunks in (0, 1, 2, 3, 7, 12, 40, 128):
            lat = torch.empty((len(lens), H, rank), dtype=torch.bfloat16, device=DEV)
            kernels.latent_decode(q.to(torch.bfloat16).to(DEV).contiguous(), lat, cache, table, ctx, sd, scale, rank,
                                  n_chunks=n_chunks)
            assert _rel(lat.float().cpu().numpy(), want.numpy()) < 8e-3, n_chunks
    kernels.check_status()


def test_absorbed_attention_of_several_new_tokens_of_a_sequence():
    """A portion of a prompt: every token sees the rows up to its own and none behind it, although those are written."""
    from llmoxide_b200 import kernels

    H, rank, R, past, counts = 6, 64, 16, [0, 61, 200], [9, 6, 3]
    lens = [p + n for p, n in zip(past, counts)]
    rows = _latent_rows(lens, rank, R, torch.bfloat16, 4)
    g = torch.Generator().manual_seed(5)
    q = _exact(torch.randn(sum(counts), H, rank + R, generator=g), torch.bfloat16)
    table, (cache,) = _store(lens, 1, rank + R, dtype=torch.bfloat16)
    for b in range(3):
        _fill(table, cache, b, rows[b][:, None, :])
    ctx = _ctx(past, counts)
    want = torch.stack([_plain_latents(q[t], rows[int(b)][: int(p) + 1], rank, 0.2, None)
                        for t, (b, p) in enumerate(zip(ctx.token_seq.tolist(), ctx.token_pos.tolist()))])
    lat = torch.empty((sum(counts), H, rank), device=DEV)
    kernels.latent_paged(q.float().to(DEV).contiguous(), lat, cache, table, ctx, None, 0.2, rank)
    assert _rel(lat.cpu().numpy(), want.numpy()) < 3e-6
    for n_chunks in (1, 3):
        lb = torch.empty((sum(counts), H, rank), dtype=torch.bfloat16, device=DEV)
        kernels.latent_decode(q.to(torch.bfloat16).to(DEV).contiguous(), lb, cache, table, ctx, None, 0.2, rank, n_chunks=n_chunks)
        assert _rel(lb.float().cpu().numpy(), want.numpy()) < 8e-3
    kernels.check_status()


@pytest.mark.parametrize("T, H, N, K", [(1, 3, 40, 16), (5, 16, 512, 96), (17, 4, 24, 40), (64, 2, 130, 128), (9, 7, 33, 17), (100, 3, 64, 8)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_product_per_head(T, H, N, K, dtype):
    """y[t, h] = W_h x[t, h] into the first N of wider rows; what lies behind them stays."""
    from llmoxide_b200 import kernels

    g = torch.Generator().manual_seed(T)
    x, w = _exact(torch.randn(T, H, K, generator=g), dtype), _exact(torch.randn(H, N, K, generator=g), dtype)
    y = torch.full((T, H, N + 5), 3.0, dtype=dtype, device=DEV)
    kernels.head_product(x.to(dtype).to(DEV).contiguous(), w.to(dtype).to(DEV).contiguous(), y[:, :, :N])
    want = torch.einsum("thk,hnk->thn", x, w)
    assert _rel(y[:, :, :N].float().cpu().numpy(), want.numpy()) < (2e-6 if dtype == torch.float32 else 6e-3)
    assert float(y[:, :, N:].min()) == float(y[:, :, N:].max()) == 3.0


@pytest.mark.parametrize("n_split", [1, 3])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_rows_are_normed_rotated_and_cached(n_split, dtype):
    from llmoxide_b200 import kernels

    H, D, R, rank, eps, base = 5, 12, 6, 28, 1e-3, 50.0
    past, counts = [0, 62], [4, 5]
    T = sum(counts)
    g = torch.Generator().manual_seed(2)
    row = _exact(torch.randn(n_split, T, rank + R + H * (R + D), generator=g) * 0.3)
    gain = _exact(torch.randn(rank, generator=g))
    whole = row.sum(0)
    pos = torch.tensor([p + k for p, n in zip(past, counts) for k in range(n)])

    def turn(x):          # the pairs (i, i + R/2), as rows reordered at load are paired
        f = torch.tensor([base ** (-2.0 * i / R) for i in range(R // 2)], dtype=F)
        a = (pos[:, None] * f).reshape(T, *([1] * (x.dim() - 2)), R // 2)
        lo, hi = x[..., : R // 2], x[..., R // 2 :]
        return torch.cat([lo * torch.cos(a) - hi * torch.sin(a), hi * torch.cos(a) + lo * torch.sin(a)], dim=-1)

    q = whole[:, rank + R :].reshape(T, H, R + D)
    want_cache = torch.cat([plain.unit_rms(whole[:, :rank], eps) * gain, turn(whole[:, rank : rank + R])], dim=1)
    f = torch.tensor([base ** (-2.0 * i / R) for i in range(R // 2)], dtype=F)
    angles = torch.arange(80, dtype=F)[:, None] * f
    table, (cache,) = _store([p + n for p, n in zip(past, counts)], 1, rank + R, dtype=dtype)
    ctx = _ctx(past, counts)
    rd = (row[0] if n_split == 1 else row).float().to(DEV).contiguous()
    rot_out = torch.full((T, H, rank + R), 9.0, dtype=dtype, device=DEV)
    plain_out = torch.empty((T, H, D), dtype=dtype, device=DEV)
    kernels.latent_prep(rd, rd[..., rank + R :], gain.float().to(DEV), eps, cache, rot_out[:, :, rank:], plain_out, table, ctx,
                        torch.cos(angles).float().to(DEV), torch.sin(angles).float().to(DEV), H, D, R, rank)
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    assert _rel(rot_out[:, :, rank:].float().cpu().numpy(), turn(q[..., :R]).numpy()) < tol
    assert _rel(plain_out.float().cpu().numpy(), q[..., R:].numpy()) < tol
    assert float(rot_out[:, :, :rank].min()) == float(rot_out[:, :, :rank].max()) == 9.0
    for t in range(T):
        b, p = int(ctx.token_seq[t]), int(pos[t])
        assert _rel(cache[int(table[b, p // 64]), 0, p % 64].float().cpu().numpy(), want_cache[t].numpy()) < 2 * tol
    assert bool(torch.isnan(cache[int(table[1, 0]), 0, 61, 0]))               # not a row more
    kernels.check_status()


@pytest.mark.parametrize("H, D, R, Dv, rank", [(3, 48, 16, 64, 40), (2, 96, 32, 128, 144), (2, 13, 7, 5, 9)])
def test_gathered_latents_and_assembled_pages(H, D, R, Dv, rank):
    """Sequences of unequal lengths into scratch pages: latents in order, zeros past each end, and every head's keys and
    values where the scratch block table says."""
    from llmoxide_b200 import kernels

    past, counts = [0, 70, 128], [65, 3, 1]
    lens = [p + n for p, n in zip(past, counts)]
    rows = _latent_rows(lens, rank, R, torch.bfloat16, 3)
    table, (cache,) = _store(lens, 1, rank + R, dtype=torch.bfloat16, width=4)
    for b in range(3):
        _fill(table, cache, b, rows[b][:, None, :])
    ctx = _ctx(past, counts)
    n = ctx.ctx_pages
    assert n == 2 + 2 + 3
    scratch = torch.full_like(table, -5)
    c = torch.empty((64 * n, rank), dtype=torch.bfloat16, device=DEV)
    kernels.latent_gather(cache, table, ctx, scratch, c, rank)
    first = [0, 2, 4]
    for b, L in enumerate(lens):
        assert scratch[b, : -(-L // 64)].tolist() == list(range(first[b], first[b] + -(-L // 64)))
        got = c[64 * first[b] : 64 * (first[b] + -(-L // 64))].double().cpu()
        assert torch.equal(got[:L], rows[b][:, :rank]) and float(got[L:].abs().max() if got[L:].numel() else 0.0) == 0.0
    g = torch.Generator().manual_seed(8)
    kv = torch.randn(64 * n, H * (D + Dv), generator=g).to(torch.bfloat16)
    keys = torch.empty((n, H, 64, R + D), dtype=torch.bfloat16, device=DEV)
    vals = torch.empty((n, H, 64, Dv), dtype=torch.bfloat16, device=DEV)
    kernels.latent_assemble(kv.to(DEV), cache, table, ctx, keys, vals, H, D, R, Dv, rank)
    keys, vals = keys.cpu(), vals.cpu()
    for b, L in enumerate(lens):
        for p in (0, L // 2, L - 1):
            at, r = first[b] + p // 64, p % 64
            src = kv[64 * at + r]
            for h in range(H):
                assert torch.equal(keys[at, h, r, :R].double(), rows[b][p, rank:])
                assert torch.equal(keys[at, h, r, R:], src[h * D : (h + 1) * D])
                assert torch.equal(vals[at, h, r], src[H * D + h * Dv : H * D + (h + 1) * Dv])
        if L % 64:
            assert float(vals[first[b] + L // 64, :, L % 64 :].float().abs().max()) == 0.0
    kernels.check_status()


# ---------------------------------------------------------------------------------------------------------
# waits that run out are reported, and the libraries go on
# ---------------------------------------------------------------------------------------------------------

def test_a_wait_that_runs_out_is_reported_and_the_library_goes_on():
    """One CTA of each kernel leaves out its first copy; its bounded wait runs out (a short limit), the kernel winds down
    and reports, and the next launch is right again."""
    from llmoxide_b200 import kernels
    from llmoxide_b200.errors import KernelError

    case = _Delta(2, 1, 32, 16, 2, [20], seed=21)
    want = case.want(0)[1].numpy()
    assert _rel(case.run([[20]])[0][0].numpy(), want) < 3e-5
    H, rank, R, n = 4, 64, 16, 150
    rows = _latent_rows([n], rank, R, torch.bfloat16, 1)
    q = _exact(torch.randn(1, H, rank + R, generator=torch.Generator().manual_seed(1)), torch.bfloat16)
    table, (cache,) = _store([n], 1, rank + R, dtype=torch.bfloat16)
    _fill(table, cache, 0, rows[0][:, None, :])
    ctx = _ctx([n - 1], [1])
    expect = _plain_latents(q[0], rows[0], rank, 0.1, None).numpy()

    def attend():
        lat = torch.empty((1, H, rank), dtype=torch.bfloat16, device=DEV)
        kernels.latent_decode(q.to(torch.bfloat16).to(DEV).contiguous(), lat, cache, table, ctx, None, 0.1, rank, n_chunks=2)
        torch.cuda.synchronize()
        return lat[0].float().cpu().numpy()

    assert _rel(attend(), expect) < 8e-3
    for lib, launch in (("delta_rule", lambda: case.run([[20]])), ("latent_cache", attend)):
        try:
            kernels.test_waits(lib, 1_000_000, True)
            with pytest.raises(KernelError, match=lib):
                launch()
                kernels.check_status()
        finally:
            kernels.test_waits(lib, 0, False)
        kernels.check_status()                      # the report was cleared
    assert _rel(case.run([[20]])[0][0].numpy(), want) < 3e-5 and _rel(attend(), expect) < 8e-3
    kernels.check_status()
