"""CPU: the Gebasun configuration and its description as parts, the cache it asks for, distance buckets, and the plain
implementation's own mechanisms against closed forms."""

import copy
import math

import pytest
import torch

import plain_gebasun as plain
from gebasun_configs import ALL, GB_A, GB_B, GB_C, make_folder

from llmoxide_b200.config import GebasunConfig, read_config
from llmoxide_b200.errors import ConfigError

F = torch.float64


# ---------------------------------------------------------------------------------------------------------
# configuration and description
# ---------------------------------------------------------------------------------------------------------

def test_config_is_chosen_by_name_and_round_trips():
    for raw in ALL.values():
        cfg = read_config(copy.deepcopy(raw))
        assert isinstance(cfg, GebasunConfig)
        again = read_config(cfg.to_dict())
        assert again.to_dict() == cfg.to_dict()
        assert "gebasun" in cfg.summary()


def test_description_names_every_tensor_once_with_the_shapes_of_the_configuration():
    spec = read_config(copy.deepcopy(GB_A)).to_spec()
    names = [t.name for t in spec.tensors()]
    assert len(names) == len(set(names))
    shapes = {t.name: tuple(t.shape) for t in spec.tensors()}
    assert shapes["embed"] == (211, 96) and shapes["head"] == (211, 96) and shapes["final.norm"] == (96,)
    # rotated attention: no values, a gate, a sink, no output bias
    assert shapes["l0.mix.q"] == (96, 96) and shapes["l0.mix.k"] == (48, 96) and shapes["l0.mix.k.b"] == (48,)
    assert shapes["l0.mix.g"] == (96, 96) and shapes["l0.mix.sink"] == (4,) and shapes["l0.mix.o"] == (96, 96)
    assert not any(n in shapes for n in ("l0.mix.v", "l0.mix.o.b", "l0.mix.rel", "l0.mix.g.b"))
    # state space: z and x of 80 columns, B and C of 24 each, four step sizes
    assert shapes["l1.mix.in"] == (80 + 80 + 48 + 4, 96) and shapes["l1.mix.conv"] == (128, 3) and shapes["l1.mix.conv.b"] == (128,)
    assert shapes["l1.mix.A_log"] == shapes["l1.mix.D"] == shapes["l1.mix.dt_bias"] == (4,) and shapes["l1.mix.norm"] == (80,)
    # biased attention
    assert shapes["l2.mix.rel"] == (10, 6) and shapes["l2.mix.o.b"] == (96,) and "l2.mix.g" not in shapes
    assert shapes["l2.mlp.e3.up"] == (32, 96) and shapes["l2.mlp.e3.down"] == (96, 32) and shapes["l2.mlp.router.b"] == (4,)
    assert shapes["l2.mlp.shared.up"] == (16, 96) and not any(".gate" in n for n in shapes)
    # a layer without a feed-forward has one norm, and a file may carry the other
    assert "l3.norm1" in shapes and "l3.norm2" not in shapes and spec.is_ignored("l3.norm2") and not spec.is_ignored("l2.norm2")
    b0, b1, b2, b3 = spec.blocks
    assert all(b.arrangement == "parallel" for b in spec.blocks) and b3.feed_forward.kind == "none"
    assert set(b0.norms) == {"mixer", "feed_forward"} and set(b3.norms) == {"mixer"}
    assert b0.mixer.kind == b2.mixer.kind == "gqa_attention" and b1.mixer.kind == "state_space"
    assert (b0.mixer["window"], b0.mixer["keep_first"], b0.mixer["values"], b0.mixer["qk_norm"]) == (37, 70, "keys", "unit")
    assert b0.position["n_rot"] == 8 and b0.position["base"] == 1000.0 and b2.position is None and b2.mixer["bias_max"] == 33
    assert b0.feed_forward["gated"] is False and b0.feed_forward["activation"] == "relu_squared"
    none = read_config(copy.deepcopy(GB_B)).to_spec().blocks[0].feed_forward
    assert none["shared_size"] == 0 and "shared_up" not in none.tensors


def test_a_distance_table_of_any_length_is_what_the_file_has():
    raw = copy.deepcopy(GB_A)
    del raw["layers"][2]["mixer"]["bias_rows"]
    spec = read_config(raw).to_spec()
    assert next(t.shape for t in spec.tensors() if t.name == "l2.mix.rel") == (-1, 6)


@pytest.mark.parametrize("path, value, text", [
    (("layers", 0, "type"), "mamba", "this design has"),
    (("layers", 0, "mixer", "kv_heads"), 3, "not a multiple"),
    (("layers", 0, "mixer", "vdim"), 20, "must equal dim"),
    (("layers", 0, "mixer", "scale"), None, "lacks 'scale'"),
    (("layers", 0, "mixer", "rot"), None, "lacks 'rot'"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "must be even"),
    (("layers", 0, "mixer", "rot", "dims"), 26, "at most dim"),
    (("layers", 0, "mixer", "rot", "base"), 0.0, "base must be positive"),
    (("layers", 0, "mixer", "mask", "keep_first"), -1, "non-negative"),
    (("layers", 0, "mixer", "mask", "size"), 0, "positive integer"),
    (("layers", 1, "mixer", "groups"), 3, "not a multiple"),
    (("layers", 1, "mixer", "conv"), 0, "positive integer"),
    (("layers", 1, "mixer", "norm_groups"), 3, "do not fall into"),
    (("layers", 1, "mixer", "state"), None, "lacks 'state'"),
    (("layers", 2, "mixer", "bias_max"), 0, "bias_max must be positive"),
    (("layers", 2, "mixer", "bias_max"), None, "lacks 'bias_max'"),
    (("layers", 2, "mlp", "router", "top"), 5, "exceeds"),
    (("layers", 2, "mlp", "kind"), "dense", "'moe'"),
    (("layers", 2, "mlp", "expert"), None, "lacks 'expert'"),
    (("layers", 2, "mlp", "shared", "ff"), 0, "positive integer"),
    (("norm", "eps"), 0.0, "positive"),
    (("vocab",), None, "lacks 'vocab'"),
])
def test_inconsistent_configurations_are_refused(path, value, text):
    raw = copy.deepcopy(GB_A)
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=text):
        read_config(raw)


def _built(raw, tmp_path, monkeypatch=None):
    from llmoxide_b200.parts import Runtime, build_block

    spec = read_config(copy.deepcopy(raw)).to_spec()
    rt = Runtime(dtype="float32", device=torch.device("cpu"), max_positions=256, tensor_cores=False, n_sm=148)
    weights = {t.name: torch.zeros(tuple(t.shape)) for t in spec.tensors()}
    return [build_block(b, weights, rt) for b in spec.blocks], weights


def test_parts_ask_for_the_cache_the_design_needs(tmp_path):
    from llmoxide_b200.cache import KVNeed

    blocks, _ = _built(GB_A, tmp_path)
    kv, state = blocks[0].cache_need()
    assert kv == KVNeed(2, 24, 37, keep_first=70) and state is None
    kv, state = blocks[1].cache_need()
    # four heads' 12 x 20 states, then a ring of three rows of 128 channels
    assert kv is None and state.shape == (4 * 12 * 20 + 3 * 128,) and state.dtype == torch.float32
    kv, state = blocks[2].cache_need()
    assert kv == KVNeed(3, 20, 50) and state is None
    assert blocks[2].mixer.defer_out_bias and blocks[0].mixer.out_bias is None


def test_parts_take_exactly_their_tensors_and_name_their_libraries(tmp_path):
    for raw in ALL.values():
        blocks, weights = _built(raw, tmp_path)
        left = {n for n in weights if not n.endswith(("norm1", "norm2"))}
        assert left == {"embed", "head", "final.norm"}, left
        for b in blocks:
            assert "dual_norm" in b.libraries()


def test_distance_table_is_as_long_as_the_mask_or_the_scale():
    from llmoxide_b200.parts.attention import GQAttention

    fake = lambda **kw: type("M", (), dict(dict(H=3, window=None, keep_first=0, chunk=0), **kw))()
    table = torch.arange(30, dtype=torch.float32).reshape(10, 3)
    for kw, far, n in ((dict(window=20), 50, 20), (dict(), 50, 51), (dict(window=20, keep_first=2), 50, 51),
                       (dict(window=500), 50, 51), (dict(), 50.5, 52)):
        lut = GQAttention._distance_table(fake(**kw), table, far)
        assert lut.shape == (3, n) and lut.is_contiguous()
        for h in range(3):
            want = [float(table[plain.distance_bucket(d, 10, far), h]) for d in range(n)]
            assert lut[h].tolist() == want
    for bad in (torch.zeros(1, 3), torch.zeros(10, 2)):
        with pytest.raises(ConfigError, match="distance table"):
            GQAttention._distance_table(fake(), bad, 50)
    with pytest.raises(ConfigError, match="bias_max beyond"):
        GQAttention._distance_table(fake(), table, 5)


def test_distance_buckets():
    from llmoxide_b200.parts.attention import distance_buckets

    # eight rows, the scale ends at 64: 0..3 have rows of their own, then a row per doubling
    assert distance_buckets(70, 8, 64) == [0, 1, 2, 3] + [4] * 4 + [5] * 8 + [6] * 16 + [7] * 38
    for rows, far in ((6, 20), (12, 333), (31, 77), (2, 9), (40, 1000)):
        got = distance_buckets(far + 20, rows, far)
        assert got == [plain.distance_bucket(n, rows, far) for n in range(far + 20)]
        assert got[0] == 0 and got[-1] == rows - 1 and got[far] == rows - 1
        assert all(0 <= b - a <= max(1, rows - 1) for a, b in zip(got, got[1:]))


# ---------------------------------------------------------------------------------------------------------
# the plain implementation against closed forms
# ---------------------------------------------------------------------------------------------------------

def test_state_space_against_its_closed_form():
    """S_t = sum_s (prod_(s<r<=t) a_r) dt_s B_s x_s^T, read by C_t, plus D x_t."""
    g = torch.Generator().manual_seed(1)
    T, P, N = 9, 3, 4
    x, B, C = (torch.randn(T, n, generator=g, dtype=F) for n in (P, N, N))
    dt, A, D = torch.rand(T, generator=g, dtype=F), torch.tensor(0.3, dtype=F), torch.tensor(-0.7, dtype=F)
    y, S = plain.state_space(x, B, C, dt, A, D)
    a = torch.exp(-math.exp(0.3) * dt)
    for t in range(T):
        want = D * x[t]
        for s in range(t + 1):
            want = want + a[s + 1 : t + 1].prod() * dt[s] * (B[s] @ C[t]) * x[s]
        assert torch.allclose(y[t], want, atol=1e-12)
    # the state after some tokens, handed on, goes on as if nothing had been cut
    _, S4 = plain.state_space(x[:4], B[:4], C[:4], dt[:4], A, D)
    y2, S2 = plain.state_space(x[4:], B[4:], C[4:], dt[4:], A, D, S4)
    assert torch.allclose(y2, y[4:], atol=1e-12) and torch.allclose(S2, S, atol=1e-12)


def test_convolution_meets_the_current_token_with_its_last_tap():
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=F)
    w = torch.tensor([[3.0, 5.0]], dtype=F)
    assert plain.causal_conv(u, w, torch.tensor([0.5], dtype=F))[:, 0].tolist() == [5.5, 53.5, 530.5]


def test_norm_in_parts_takes_the_gated_rows():
    y = torch.tensor([[3.0, 4.0, 1.0, 1.0]], dtype=F)
    z = torch.full((1, 4), 50.0, dtype=F)                 # silu(50) = 50
    got = plain.gate_then_norm(y, z, torch.tensor([1.0, 1.0, 2.0, 2.0], dtype=F), 2, 1e-12)
    r = math.sqrt(12.5)
    assert torch.allclose(got, torch.tensor([[3 / r, 4 / r, 2.0, 2.0]], dtype=F))


def test_window_kept_tokens_bias_and_sink():
    m = plain.window_mask(8, 3, 2)
    assert m[6].tolist() == [True, True, False, False, True, True, True, False]
    assert plain.window_mask(5, 2)[4].tolist() == [False, False, False, True, True]
    # equal keys: weights are 1 / (n + exp(sink)); a bias of ln 3 triples one of them
    q = k = torch.zeros(3, 2, dtype=F)
    v = torch.tensor([[1.0], [2.0], [6.0]], dtype=F)
    out = plain.attend(q, k, v, 1.0, plain.window_mask(3, None), torch.tensor(math.log(2.0), dtype=F))
    assert torch.allclose(out[:, 0], torch.tensor([1 / 3, 3 / 4, 9 / 5], dtype=F))
    bias = torch.zeros(3, 3, dtype=F)
    bias[2, 0] = math.log(3.0)
    out = plain.attend(q, k, v, 1.0, plain.window_mask(3, None), torch.tensor(0.0, dtype=F), bias)
    assert torch.allclose(out[2, 0], torch.tensor((3 * 1 + 2 + 6) / 6.0, dtype=F))


def test_routing_weights_are_the_softmax_over_the_chosen():
    ids, w = plain.route(torch.tensor([0.0, math.log(3.0), -5.0, math.log(5.0)], dtype=F), 2)
    assert ids == [3, 1] and torch.allclose(w, torch.tensor([5 / 8, 3 / 8], dtype=F))


def test_rotation_turns_the_pairs_of_the_two_halves_and_leaves_the_rest():
    x = torch.zeros(3, 1, 6, dtype=F)
    x[:, 0, 0], x[:, 0, 4] = 1.0, 7.0
    y = plain.rotate_halves(x, 4, 100.0)
    for p in range(3):
        assert torch.allclose(y[p, 0, [0, 2, 4]], torch.tensor([math.cos(p), math.sin(p), 7.0], dtype=F))


def test_a_model_folder_is_written_and_read_by_the_plain_implementation(tmp_path):
    folder = make_folder(tmp_path, "A", "float32")
    cfg, w = plain.read_model(folder)
    streams = []
    logits = plain.forward(cfg, w, [1, 5, 9, 200], streams)
    assert logits.shape == (4, 211) and len(streams) == 4 and torch.isfinite(logits).all()
    # a prefix gives the same rows
    assert torch.allclose(plain.forward(cfg, w, [1, 5]), logits[:2], atol=1e-10)


def test_random_state_space_layers_forget_and_remember(tmp_path):
    """The random weights are such that a wrong state shows: over sixty tokens some heads keep more than a tenth and some
    lose nearly everything."""
    folder = make_folder(tmp_path, "C", "float32")
    cfg, w = plain.read_model(folder)
    rate = torch.exp(w["l0.mix.A_log"]) * plain.softplus(w["l0.mix.dt_bias"])
    kept = torch.exp(-rate * 60)
    assert kept.max() > 1e-3 and kept.min() < 0.1
    assert cfg["layers"][0]["type"] == GB_C["layers"][0]["type"] == "mamba2"
