"""GPU: whole Gebasun models under every way of cutting the same requests into steps, against the plain implementation
(tests/plain_gebasun.py), and greedy generation through the package's own entry point."""

import copy

import numpy as np
import pytest
import torch

import plain_gebasun as plain
import replay_util as ru
from gebasun_configs import ALL, make_folder
from tiny_configs import prompts

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 2e-5, 3e-2
LENGTHS = {"A": [150, 1, 37, 64, 9, 201, 2], "B": [140, 70, 3, 65, 129], "C": [300, 40, 131, 17, 64], "D": [330, 12, 101, 55]}


def _rel(got, want):
    want = np.asarray(want, dtype=np.float64)
    return float(np.abs(np.asarray(got, dtype=np.float64) - want).max() / max(np.abs(want).max(), 1e-30))


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("gebasun")
    return {(n, d): make_folder(base, n, d) for n in ALL for d in ("float32", "bfloat16")}


_plain_cache: dict = {}


def _expected(folder, reqs):
    """The plain logits of every request (each computed once per folder)."""
    cfg, w = plain.read_model(folder)
    out = {}
    for rid, toks in reqs.items():
        key = (str(folder), tuple(toks))
        if key not in _plain_cache:
            _plain_cache[key] = plain.forward(cfg, w, toks).numpy()
        out[rid] = _plain_cache[key]
    return out


def _engine(folder, dtype, max_tokens=4096, **kw):
    from llmoxide_b200.engine.engine import Engine, LoadOptions

    return Engine.load(folder, LoadOptions(dtype=dtype, max_tokens=max_tokens, max_batch=8, **kw))


def _requests(name):
    return {f"r{i}": t for i, t in enumerate(prompts(ALL[name]["vocab"], LENGTHS[name], seed=21))}


def _rms_err(got, want):
    d = got - want
    w = want - want.mean(axis=1, keepdims=True)
    return (d - d.mean(axis=1, keepdims=True)).std(axis=1) / np.sqrt((w * w).mean())


def _compare(got, want, dtype, what):
    """float32: every logit of every position within rounding.  bfloat16: a position's error is the root mean square over
    the vocabulary of the difference (its mean taken off) against that of the logits.  A token whose router logits nearly
    tie at the last chosen place may choose another expert than the float64 implementation does (and later positions read
    what it left), so up to a tenth of the positions may lie beyond the tolerance; the median lies well within it."""
    errs = []
    for rid in want:
        assert got[rid].shape == want[rid].shape, (what, rid)
        errs.append(np.abs(got[rid] - want[rid]).max(axis=1) / np.abs(want[rid]).max() if dtype == "float32"
                    else _rms_err(got[rid], want[rid]))
    e = np.concatenate(errs)
    tol = F32_TOL if dtype == "float32" else BF16_TOL
    over, worst, med = int((e > tol).sum()), float(e.max()), float(np.median(e))
    print(f"{what}: worst {worst:.2e}, median {med:.2e}, {over} of {len(e)} beyond {tol}")
    if dtype == "float32":
        assert over == 0, f"{what}: {over} of {len(e)} positions differ from the plain implementation, worst {worst:.3e}"
    else:
        assert over <= max(2, 0.1 * len(e)) and worst < 0.3 and med < 1.5e-2, \
            f"{what}: {over} of {len(e)} positions beyond {tol}, worst {worst:.3e}, median {med:.3e}"


def test_layer_by_layer_against_the_plain_stream(folders):
    """The residual stream after every layer, as the step's named intermediates report it."""
    for name in ALL:
        folder = folders[(name, "float32")]
        cfg, w = plain.read_model(folder)
        toks = prompts(ALL[name]["vocab"], [75], seed=4)[0]
        layers = []
        plain.forward(cfg, w, toks, streams=layers)
        eng = _engine(folder, "float32", max_tokens=512)
        got = {}
        eng.step([(eng.acquire(), toks)], [[0]], probe=lambda n, t: got.__setitem__(n, t.detach().float().cpu().numpy()))
        for i, want in enumerate(layers):
            assert _rel(got[f"l_out-{i}"], want.numpy()) < 1e-5, (name, i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALL))
def test_every_cutting_matches_the_plain_implementation(folders, tmp_path, name, dtype):
    folder = folders[(name, dtype)]
    reqs = _requests(name)
    want = _expected(folder, reqs)
    vocab = ALL[name]["vocab"]
    eng = _engine(folder, dtype)
    results = {}
    # the same engine runs every trace: slots, pages and state are freed and used again
    for what, steps in (("whole", ru.trace_whole(reqs)),
                        ("last 48 one by one", ru.trace_tail_decode(reqs, 48)),
                        ("all but the first token one by one", ru.trace_tail_decode(reqs, 10 ** 6)),
                        ("unequal batches", ru.trace_batches(reqs, 4)),
                        ("unequal batches of 3, short prompts", ru.trace_batches(reqs, 3, 0.2)),
                        ("portions of 2", ru.trace_chunks({k: v for k, v in reqs.items() if len(v) <= 70}, 2, 3, tail=3)),
                        ("portions of 5", ru.trace_chunks(reqs, 5, 6, tail=4)),
                        ("portions of 48", ru.trace_chunks(reqs, 48, 3)),
                        ("portions of 64", ru.trace_chunks(reqs, 64, 4)),
                        ("portions of 100 beside single tokens", ru.trace_chunks(reqs, 100, 6, tail=40, mixed=True))):
        out = tmp_path / what.replace(" ", "_").replace(",", "")
        ru.run_in_process(eng, steps, out)
        for g in range(eng.cache.n_groups()):
            assert eng.cache.alloc.pages_held(g) == 0
        got = ru.collect(steps, out, vocab)
        _compare(got, {rid: want[rid] for rid in got}, dtype, f"{name}/{dtype}/{what}")
        results[what] = got
    for what, got in results.items():
        if dtype == "float32":      # how a prompt is cut changes the order of sums, nothing else
            for rid in got:
                assert ru.rel_err(got[rid], results["whole"][rid]) < 1e-5, (what, rid)
        else:
            e = np.concatenate([_rms_err(got[rid], results["whole"][rid]) for rid in got])
            assert (e > BF16_TOL).sum() <= max(2, 0.1 * len(e)) and np.median(e) < 1.5e-2, \
                (what, int((e > BF16_TOL).sum()), float(np.median(e)), float(e.max()))
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_gives_what_each_request_gives_alone(folders, dtype):
    """Unequal requests together, then alone, prompt and decode steps: equal to rounding, whatever else is in the step."""
    folder = folders[("C", dtype)]
    eng = _engine(folder, dtype)
    reqs = prompts(ALL["C"]["vocab"], [200, 33, 129, 3], seed=8)
    cut = [max(1, len(t) - 20) for t in reqs]
    slots = [eng.acquire() for _ in reqs]
    rows = [[r] for r in torch.split(eng.step([(s, t[:c]) for s, t, c in zip(slots, reqs, cut)],
                                              [list(range(c)) for c in cut]).cpu(), cut)]
    for i in range(20):
        live = [j for j, (t, c) in enumerate(zip(reqs, cut)) if c + i < len(t)]
        out = eng.step([(slots[j], [reqs[j][cut[j] + i]]) for j in live], [[0]] * len(live)).cpu()
        for j, r in zip(live, out):
            rows[j].append(r[None])
    for s in slots:
        eng.release(s)
    for j, t in enumerate(reqs):
        s = eng.acquire()
        alone = [eng.step([(s, t[: cut[j]])], [list(range(cut[j]))]).cpu()]
        alone += [eng.step([(s, [tok])], [[0]]).cpu() for tok in t[cut[j] :]]
        eng.release(s)
        a, b = torch.cat(rows[j]).numpy(), torch.cat(alone).numpy()
        if dtype == "float32":
            assert ru.rel_err(a, b) < 5e-6, j
        else:
            e = _rms_err(a, b)
            assert (e > BF16_TOL).sum() <= max(1, 0.05 * len(e)) and np.median(e) < 1e-2, (j, float(e.max()))
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_as_a_user_runs_it(folders, tmp_path, dtype):
    """``bin/trace_run`` as a subprocess on a Gebasun folder: unequal batches whose requests end at different steps, with
    ``--max-tokens`` the bare sum of the live requests' tokens."""
    folder = folders[("A", dtype)]
    reqs = _requests("A")
    steps = ru.trace_batches(reqs, 3, 0.6)
    ru.run_trace_run(folder, dtype, steps, tmp_path / "out", max_tokens=sum(len(t) for t in reqs.values()))
    got = ru.collect(steps, tmp_path / "out", ALL["A"]["vocab"])
    _compare(got, _expected(folder, reqs), dtype, f"trace_run/{dtype}")


def test_a_slot_used_again_starts_from_an_empty_state(folders):
    """One slot: a long request, then a short one in the same slot, then a part of the first; the later ones must see
    neither the earlier keys nor the recurrence's state nor the convolution's earlier rows."""
    for name in ("A", "D"):
        folder = folders[(name, "float32")]
        eng = _engine(folder, "float32", max_tokens=512)
        cfg, w = plain.read_model(folder)
        long_req, short_req = prompts(ALL[name]["vocab"], [200, 30], seed=5)
        for toks in (long_req, short_req, long_req[:90], short_req[:1]):
            slot = eng.acquire()
            assert slot == 0
            cut = max(1, len(toks) - 2)
            got = [eng.step([(slot, toks[:cut])], [list(range(cut))]).cpu().numpy()]
            got += [eng.step([(slot, [t])], [[0]]).cpu().numpy() for t in toks[cut:]]
            eng.release(slot)
            assert ru.rel_err(np.concatenate(got), plain.forward(cfg, w, toks).numpy()) < F32_TOL
        eng.cache.alloc.check_consistent()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_long_decoding(folders, name, dtype):
    """A short prompt and 330 single-token steps past every window; decode steps replay a CUDA graph, and pages that have
    left the windows are given back on the way."""
    folder = folders[(name, dtype)]
    eng = _engine(folder, dtype, max_tokens=1024)
    toks = prompts(ALL[name]["vocab"], [340], seed=9)[0]
    want = _expected(folder, {"r": toks})["r"]
    slot = eng.acquire()
    rows = [eng.step([(slot, toks[:10])], [list(range(10))]).cpu().numpy()]
    rows += [eng.step([(slot, [t])], [[0]]).cpu().numpy() for t in toks[10:]]
    eng.release(slot)
    _compare({"r": np.concatenate(rows)}, {"r": want}, dtype, f"long decoding/{name}/{dtype}")
    eng.check_status()


def test_prompt_steps_replayed_as_graphs(folders):
    """A prompt step's shape that comes back is captured: the same shapes behind different pasts and slots."""
    folder = folders[("C", "bfloat16")]
    eng = _engine(folder, "bfloat16", max_tokens=2048)
    toks = prompts(ALL["C"]["vocab"], [400], seed=15)[0]
    want = _expected(folder, {"r": toks})["r"]
    for cut in ([100, 100, 100, 100], [100, 100, 100, 100], [100, 300], [200, 100, 100], [100, 100, 200], [200, 200]):
        slot, rows, at = eng.acquire(), [], 0
        for n in cut:
            rows.append(eng.step([(slot, toks[at : at + n])], [list(range(n))]).cpu().numpy())
            at += n
        eng.release(slot)
        _compare({"r": np.concatenate(rows)}, {"r": want}, "bfloat16", f"portions {cut}")
    eng.check_status()


def test_a_changed_token_moves_nothing_before_it(folders):
    folder = folders[("A", "float32")]
    cfg, w = plain.read_model(folder)
    eng = _engine(folder, "float32", max_tokens=1024)
    toks = prompts(ALL["A"]["vocab"], [260], seed=12)[0]
    other = list(toks)
    other[100] = (toks[100] + 1) % ALL["A"]["vocab"]
    outs = []
    for seq in (toks, other):
        slot = eng.acquire()
        a = eng.step([(slot, seq[:150])], [list(range(150))]).cpu().numpy()
        b = [eng.step([(slot, [t])], [[0]]).cpu().numpy() for t in seq[150:]]
        eng.release(slot)
        outs.append(np.concatenate([a] + b))
        assert ru.rel_err(outs[-1], plain.forward(cfg, w, seq).numpy()) < F32_TOL
    moved = np.abs(outs[0] - outs[1]).max(axis=1) > 0
    assert not moved[:100].any() and moved[100]


def _one_attention_layer(tmp_path, kind, window, keep):
    """A folder with one attention layer and no feed-forward in which token 63's key stands out for every query: its
    embedding points along one direction, W_k carries that to a fixed key, and the query bias asks for that key."""
    from llmoxide_b200.config import read_config
    from llmoxide_b200.weights import write_model_folder
    from llmoxide_b200.weights.safetensors_io import SafetensorsWriter

    m = dict(heads=2, kv_heads=1, dim=32, vdim=32, scale=3.0)
    m["mask"] = dict(size=window, keep_first=keep) if keep else dict(size=window)
    if kind == "attention":
        m.update(bias_max=3 * window, bias_rows=12)
    else:
        m["rot"] = dict(dims=2, base=1e6)
    raw = dict(architecture="Gebasun", vocab=64, width=64, norm=dict(eps=1e-6), torch_dtype="float32",
               layers=[dict(type=kind, mixer=m, mlp=None)])
    folder = write_model_folder(tmp_path, read_config(raw), 5, "float32")
    _, w = plain.read_model(folder)
    g = torch.Generator().manual_seed(window)
    w = {n: t.float() for n, t in w.items()}
    w["embed"], w["head"], w["l0.mix.o"] = (torch.randn(w[n].shape, generator=g) for n in ("embed", "head", "l0.mix.o"))
    w["embed"][:, 0], w["embed"][63] = 0.0, 0.0
    w["embed"][63, 0] = 8.0
    key = torch.randn(32, generator=g)
    w["l0.mix.k"] = torch.randn(w["l0.mix.k"].shape, generator=g) * 0.1
    w["l0.mix.k"][:, 0] = key
    w["l0.mix.q.b"] = torch.cat([key, key])
    with SafetensorsWriter(folder / "model.safetensors", [(n, torch.float32, tuple(t.shape)) for n, t in w.items()], {}) as out:
        for n, t in w.items():
            out.write(n, t.contiguous())
    return folder


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind, window, keep", [("attention", 40, 0), ("attention", 64, 0), ("attention_2", 40, 3),
                                                ("attention_2", 65, 66)])
def test_one_token_seen_to_the_edge_of_the_window_and_not_beyond(tmp_path, kind, window, keep, dtype):
    """A token that occurs once is followed through prompt and decoding: the logits where it has just left the window equal
    those of a sequence without it to rounding, those where it is just inside do not; a kept token is seen for good."""
    folder = _one_attention_layer(tmp_path / f"{kind}{window}{dtype}", kind, window, keep)
    cfg, w = plain.read_model(folder)
    rng = np.random.default_rng(window)
    base = rng.integers(0, 60, 260).tolist()
    for mark in (100, 127, 128, 1):
        toks = list(base)
        toks[mark] = 63
        eng = _engine(folder, dtype, max_tokens=512)
        outs = []
        for seq in (toks, base):
            slot = eng.acquire()
            a = eng.step([(slot, seq[:150])], [list(range(150))]).cpu().numpy()
            b = [eng.step([(slot, [t])], [[0]]).cpu().numpy() for t in seq[150:]]
            eng.release(slot)
            outs.append(np.concatenate([a] + b))
        want = plain.forward(cfg, w, toks).numpy()
        assert ru.rel_err(outs[0], want) < (F32_TOL if dtype == "float32" else 8e-2), mark
        diff = np.abs(outs[0] - outs[1]).max(axis=1) / np.abs(want).max()
        seen = np.zeros(len(toks), bool)
        seen[mark : mark + window] = True
        if mark < keep:
            seen[mark:] = True
        assert (diff[~seen] == 0).all(), (mark, np.nonzero(diff * ~seen)[0][:5])
        assert diff[seen].min() > 1e-2, (mark, float(diff[seen].min()))
        eng.check_status()


@pytest.mark.parametrize("name, dtype", [("A", "float32"), ("C", "float32"), ("C", "bfloat16")])
def test_greedy_generation_through_the_session(folders, name, dtype):
    from llmoxide_b200 import LoadOptions, Request, Sampling, Session

    folder = folders[(name, dtype)]
    cfg, w = plain.read_model(folder)
    session = Session.load(folder, LoadOptions(dtype=dtype, max_tokens=2048, max_batch=4))
    reqs = prompts(ALL[name]["vocab"], [9, 1, 140, 40], seed=3)
    outs = session.generate([Request(p, 20, Sampling.greedy(), stop_ids=()) for p in reqs])
    for p, o in zip(reqs, outs):
        assert len(o.tokens) == 20
        ids = list(p) + list(o.tokens)
        logits = plain.forward(cfg, w, ids[:-1]).numpy()[len(p) - 1 :]
        for row, tok in zip(logits, o.tokens):
            slack = 1e-5 if dtype == "float32" else 0.1       # bfloat16 may differ where the plain logits nearly tie
            assert row.max() - row[tok] <= slack * np.abs(row).max(), (name, p[:4], o.tokens)
    info = session.info()
    assert info["architecture"] == "Gebasun" and info["n_layers"] == len(ALL[name]["layers"])


def test_random_weights_on_the_device_equal_the_folder(folders):
    from llmoxide_b200 import Engine, LoadOptions, read_config

    folder = folders[("A", "float32")]
    toks = prompts(ALL["A"]["vocab"], [50], seed=1)[0]
    opts = dict(dtype="float32", max_tokens=256, max_batch=2)
    a = Engine.load(folder, LoadOptions(**opts))
    b = Engine.random(read_config(dict(copy.deepcopy(ALL["A"]), torch_dtype="float32")), 4321, LoadOptions(**opts))
    la = a.step([(a.acquire(), toks)], [[49]])
    lb = b.step([(b.acquire(), toks)], [[49]])
    assert torch.equal(la, lb)


def _drawn_config(rng):
    """A configuration whose every size is drawn: odd and even head sizes, widths that are no multiple of eight, one to six
    taps, layers in any order, some without a feed-forward or without a shared expert, with and without masks."""
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    width, vocab = int(pick(40, 48, 72, 100, 136, 176, 200)), int(rng.integers(50, 400))
    layers = []
    for _ in range(int(rng.integers(3, 7))):
        E = int(rng.integers(1, 12))
        mlp = None if rng.random() < 0.2 else dict(kind="moe", expert=dict(ff=int(pick(8, 12, 20, 24, 40, 96))),
                                                   router=dict(experts=E, top=int(rng.integers(1, E + 1))))
        if mlp and rng.random() < 0.8:
            mlp["shared"] = dict(ff=int(pick(8, 20, 36, 64)))
        kind = rng.random()
        if kind < 0.6:
            G = int(pick(1, 2, 3))
            D = int(pick(16, 64, 128)) if rng.random() < 0.5 else 2 * int(rng.integers(2, 50))
            m = dict(heads=G * int(pick(1, 2, 3, 9)), kv_heads=G, dim=D, vdim=D, scale=float(rng.uniform(0.05, 0.5)))
            if rng.random() < 0.85:
                m["mask"] = dict(size=int(pick(1, 2, 17, 63, 64, 65, 100, 500)))
            if kind < 0.3:
                rows = int(rng.integers(2, 40))
                m.update(bias_rows=rows, bias_max=rows // 2 + int(rng.integers(1, 300)))
                layers.append(dict(type="attention", mixer=m, mlp=mlp))
            else:
                if "mask" in m:
                    m["mask"]["keep_first"] = int(pick(0, 1, 4, 64, 90))
                m["rot"] = dict(dims=2 * int(rng.integers(1, D // 2 + 1)), base=float(pick(30.0, 10000.0, 500000.0)))
                layers.append(dict(type="attention_2", mixer=m, mlp=mlp))
        else:
            G = int(pick(1, 2, 3))
            H, P = G * int(pick(1, 2, 4)), int(rng.integers(1, 90))
            parts = [n for n in range(1, H + 1) if (H * P) % n == 0]
            layers.append(dict(type="mamba2", mlp=mlp, mixer=dict(
                heads=H, vdim=P, state=int(rng.integers(1, 150)), groups=G, conv=int(rng.integers(1, 7)),
                norm_groups=int(pick(*parts)))))
    return dict(architecture="Gebasun", vocab=vocab, width=width, norm=dict(eps=float(pick(1e-5, 1e-6, 1e-3))), layers=layers)


@pytest.mark.parametrize("seed", range(16))
def test_drawn_configurations(tmp_path, seed):
    """Sixteen drawn configurations, each in both dtypes: whole prompts, the last 30 tokens one by one, an unequal batch
    and portions, against the plain implementation."""
    from llmoxide_b200.config import read_config
    from llmoxide_b200.weights import write_model_folder

    rng = np.random.default_rng(7000 + seed)
    raw = _drawn_config(rng)
    reqs = {f"r{i}": t for i, t in enumerate(prompts(raw["vocab"], [150, 37, 5, 70], seed=seed))}
    for dtype in ("float32", "bfloat16"):
        folder = write_model_folder(tmp_path / dtype, read_config(dict(raw, torch_dtype=dtype)), 99 + seed, dtype)
        want = _expected(folder, reqs)
        eng = _engine(folder, dtype, max_tokens=1024)
        for what, steps in (("whole", ru.trace_whole(reqs)), ("last 30 one by one", ru.trace_tail_decode(reqs, 30)),
                            ("an unequal batch", ru.trace_batches(reqs, 4, 0.4)), ("portions", ru.trace_chunks(reqs, 67, 3))):
            out = tmp_path / f"{dtype}_{what.replace(' ', '_')}"
            ru.run_in_process(eng, steps, out)
            got = ru.collect(steps, out, raw["vocab"])
            _compare(got, {rid: want[rid] for rid in got}, dtype, f"drawn {seed}/{dtype}/{what}: {raw}")
        eng.check_status()
