"""GPU: whole Soputar models under every way of cutting the same requests into steps, against the plain implementation
(tests/plain_soputar.py), and greedy generation through the package's own entry point."""

import copy

import numpy as np
import pytest
import torch

import plain_soputar as plain
import replay_util as ru
from soputar_configs import ALL, make_folder
from tiny_configs import prompts

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 3e-5, 4e-2
LENGTHS = {"A": [150, 1, 37, 64, 9, 201, 2], "B": [140, 70, 3, 65, 129], "C": [300, 40, 131, 17, 64], "D": [330, 12, 101, 55]}


def _rel(got, want):
    want = np.asarray(want, dtype=np.float64)
    return float(np.abs(np.asarray(got, dtype=np.float64) - want).max() / max(np.abs(want).max(), 1e-30))


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("soputar")
    return {(n, d): make_folder(base, n, d) for n in ALL for d in ("float32", "bfloat16")}


def _engine(folder, dtype, max_tokens=4096, **kw):
    from llmoxide_b200.engine.engine import Engine, LoadOptions

    return Engine.load(folder, LoadOptions(dtype=dtype, max_tokens=max_tokens, max_batch=8, **kw))


def _requests(name):
    return {f"r{i}": t for i, t in enumerate(prompts(ALL[name]["vocab"], LENGTHS[name], seed=21))}


def _expected(folder, reqs):
    cfg, w = plain.read_model(folder)
    return {rid: plain.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}


def _rms_err(got, want):
    d = got - want
    w = want - want.mean(axis=1, keepdims=True)
    return (d - d.mean(axis=1, keepdims=True)).std(axis=1) / np.sqrt((w * w).mean())


def _compare(got, want, dtype, what):
    """float32: every logit of every position within rounding.  bfloat16: a position's error is the root mean square over
    the vocabulary of the difference (its mean taken off) against that of the logits; nothing in the design can tip (no
    router), so at most a fiftieth of the positions lies beyond the tolerance, none beyond twice, the median within a
    third.  (A delta layer's read-out can be small against the norm behind it, which magnifies rounding at single
    positions: with one key head, rounding the sublayers' inputs alone moves a position's logits by a tenth in the plain
    implementation, so whole models here have several.)"""
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
        assert over <= 0.02 * len(e) and worst < 2 * tol and med < tol / 3, \
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
            assert _rel(got[f"l_out-{i}"], want.numpy()) < 2e-5, (name, i)


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
                assert ru.rel_err(got[rid], results["whole"][rid]) < 2e-5, (what, rid)
        else:
            e = np.concatenate([_rms_err(got[rid], results["whole"][rid]) for rid in got])
            assert (e > BF16_TOL).sum() <= 0.02 * len(e) and np.median(e) < BF16_TOL / 3, \
                (what, int((e > BF16_TOL).sum()), float(np.median(e)), float(e.max()))
    eng.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_as_a_user_runs_it(folders, tmp_path, dtype):
    """``bin/trace_run`` as a subprocess on a Soputar folder: unequal batches whose requests end at different steps, with
    ``--max-tokens`` the bare sum of the live requests' tokens."""
    folder = folders[("A", dtype)]
    reqs = _requests("A")
    steps = ru.trace_batches(reqs, 3, 0.6)
    ru.run_trace_run(folder, dtype, steps, tmp_path / "out", max_tokens=sum(len(t) for t in reqs.values()))
    got = ru.collect(steps, tmp_path / "out", ALL["A"]["vocab"])
    _compare(got, _expected(folder, reqs), dtype, f"trace_run/{dtype}")


def test_a_slot_used_again_starts_from_an_empty_state(folders):
    """One slot: a long request, then a short one in the same slot, then a part of the first; the later ones must see
    neither the earlier keys and latents nor the recurrence's state nor the convolution's earlier rows."""
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
    """A short prompt and 330 single-token steps, over page borders and the temperature's steps; decode steps replay a
    CUDA graph."""
    folder = folders[(name, dtype)]
    eng = _engine(folder, dtype, max_tokens=1024)
    cfg, w = plain.read_model(folder)
    toks = prompts(ALL[name]["vocab"], [340], seed=9)[0]
    want = plain.forward(cfg, w, toks).numpy()
    slot = eng.acquire()
    rows = [eng.step([(slot, toks[:10])], [list(range(10))]).cpu().numpy()]
    rows += [eng.step([(slot, [t])], [[0]]).cpu().numpy() for t in toks[10:]]
    eng.release(slot)
    _compare({"r": np.concatenate(rows)}, {"r": want}, dtype, f"long decoding/{name}/{dtype}")
    eng.check_status()


def test_prompt_steps_replayed_as_graphs(folders):
    """A prompt step's shape that comes back is captured; scratch pages are sized by the step's pages, which belong to
    the shape: the same tokens behind different pasts must not share a graph."""
    folder = folders[("C", "bfloat16")]
    eng = _engine(folder, "bfloat16", max_tokens=2048)
    cfg, w = plain.read_model(folder)
    toks = prompts(ALL["C"]["vocab"], [400], seed=15)[0]
    want = plain.forward(cfg, w, toks).numpy()
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
    assert not moved[:100].any() and moved[100] and moved[259]


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
    assert info["architecture"] == "Soputar" and info["n_layers"] == len(ALL[name]["layers"])


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
    """A configuration whose every size is drawn: odd and even head sizes, ranks and widths that are no multiple of
    eight, one to six taps, layers in any order, some without a feed-forward, with and without cap and temperature,
    borrowers of any earlier owner."""
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    width, vocab = int(pick(40, 48, 72, 100, 136, 176, 200)), int(rng.integers(50, 400))
    layers, owners = [], []
    for i in range(int(rng.integers(3, 7))):
        mlp = None if rng.random() < 0.2 else dict(kind="dense", ff=int(pick(8, 12, 20, 24, 40, 50, 96)),
                                                   limit=float(pick(0.5, 2.0, 7.0)))
        kind = rng.random()
        if kind < 0.4:
            temp = None if rng.random() < 0.3 else dict(coef=float(rng.uniform(-0.2, 0.8)), every=int(pick(1, 2, 7, 30, 64)))
            m = dict(scale=float(rng.uniform(0.05, 0.4)), q_temp=temp)
            if rng.random() < 0.7:
                m["softcap"] = float(pick(0.7, 2.0, 10.0, 50.0))
            if owners and rng.random() < 0.5:
                j = int(pick(*owners))
                o = layers[j]["mixer"]
                m.update(kv_from=j, heads=o["kv_heads"] * int(pick(1, 2, 4)), **{k: o[k] for k in ("kv_heads", "dim", "vdim")})
            else:
                G, same = int(pick(1, 2, 3)), rng.random() < 0.4
                D = int(pick(16, 64, 128)) if same else int(rng.integers(3, 80))
                m.update(heads=G * int(pick(1, 2, 3)), kv_heads=G, dim=D, vdim=D if same else int(rng.integers(3, 70)))
                owners.append(i)
            layers.append(dict(type="attention", mixer=m, mlp=mlp))
        elif kind < 0.7:
            E = int(pick(0, 0, 64, 128))                # 0: any sizes; else sizes the tiled prompt kernels take
            R = int(pick(8, 16, 32)) if E else 2 * int(rng.integers(1, 20))
            m = dict(heads=int(pick(1, 2, 5, 17)), rot_dim=R, dim=E - R if E else int(rng.integers(1, 60)),
                     vdim=E or int(rng.integers(3, 70)), kv_rank=int(pick(16, 48, 80, 200)) if E else int(rng.integers(5, 90)),
                     scale=float(rng.uniform(0.05, 0.4)), rot=dict(base=float(pick(30.0, 10000.0, 500000.0)), dims=R))
            layers.append(dict(type="latent_attention", mixer=m, mlp=mlp))
        else:
            G = int(pick(1, 2, 3))
            layers.append(dict(type="delta", mlp=mlp, mixer=dict(heads=G * int(pick(1, 2, 3)), kv_heads=G,
                                                                 dim=int(rng.integers(2, 150)), vdim=int(rng.integers(2, 150)),
                                                                 conv=int(rng.integers(1, 7)))))
    return dict(architecture="Soputar", vocab=vocab, width=width, norm=dict(eps=float(pick(1e-5, 1e-6, 1e-3))),
                embedding=dict(scale=float(rng.uniform(0.5, 14.0))), layers=layers)


@pytest.mark.parametrize("seed", range(16))
def test_drawn_configurations(tmp_path, seed):
    """Sixteen drawn configurations, each in both dtypes: whole prompts, the last 30 tokens one by one, an unequal batch
    and portions, against the plain implementation."""
    from llmoxide_b200.config import read_config
    from llmoxide_b200.weights import write_model_folder

    rng = np.random.default_rng(5000 + seed)
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
