"""CPU: the Soputar configuration and its description as parts, the cache's entries of latents and of recurrent state,
and the plain implementation's own mechanisms against closed forms."""

import copy
import math

import pytest
import torch

import plain_soputar as plain
from soputar_configs import ALL, SP_A, SP_B, make_folder

from llmoxide_b200.config import SoputarConfig, read_config
from llmoxide_b200.errors import ConfigError

F = torch.float64


# ---------------------------------------------------------------------------------------------------------
# configuration and description
# ---------------------------------------------------------------------------------------------------------

def test_config_is_chosen_by_name_and_round_trips():
    for raw in ALL.values():
        cfg = read_config(copy.deepcopy(raw))
        assert isinstance(cfg, SoputarConfig)
        again = read_config(cfg.to_dict())
        assert again.to_dict() == cfg.to_dict()
        assert "soputar" in cfg.summary()


def test_description_names_every_tensor_once_with_the_shapes_of_the_configuration():
    spec = read_config(copy.deepcopy(SP_A)).to_spec()
    names = [t.name for t in spec.tensors()]
    assert len(names) == len(set(names))
    shapes = {t.name: tuple(t.shape) for t in spec.tensors()}
    assert shapes["embed"] == (211, 96) and shapes["head"] == (211, 96) and shapes["final.norm"] == (96,)
    # delta: four heads on two key heads, three taps
    assert shapes["l0.mix.q"] == shapes["l0.mix.k"] == (2 * 24, 96) and shapes["l0.mix.v"] == (4 * 16, 96)
    assert shapes["l0.mix.q.conv"] == (48, 3) and shapes["l0.mix.v.conv"] == (64, 3)
    assert shapes["l0.mix.b"] == shapes["l0.mix.a"] == (4, 96) and shapes["l0.mix.A_log"] == shapes["l0.mix.dt_bias"] == (4,)
    assert shapes["l0.mix.norm"] == (16,) and shapes["l0.mix.g"] == (64, 96) and shapes["l0.mix.o"] == (96, 64)
    # attention: gains over whole rows
    assert shapes["l1.mix.q.norm"] == (4 * 32,) and shapes["l1.mix.k.norm"] == (2 * 32,) and shapes["l1.mix.o"] == (96, 64)
    # latent attention: queries straight from the stream
    assert shapes["l2.mix.q"] == (3 * 24, 96) and shapes["l2.mix.dkv"] == (48, 96) and shapes["l2.mix.dkv.norm"] == (40,)
    assert shapes["l2.mix.uk"] == (48, 40) and shapes["l2.mix.uv"] == (72, 40) and shapes["l2.mix.sink"] == (3,)
    # a borrower has no key and value tensors, a layer without a feed-forward no second norm
    assert shapes["l3.mix.q"] == (6 * 32, 96) and shapes["l3.mix.q.norm"] == (192,) and "l3.norm1" in shapes
    assert not any(n in shapes for n in ("l3.mix.k", "l3.mix.v", "l3.mix.k.norm", "l3.norm2", "l3.mlp.gate"))
    assert [(c.layer, c.cache, c.writes_cache) for c in spec.schedule] == [(0, 0, True), (1, 1, True), (2, 2, True),
                                                                            (3, 1, False)]
    b0, b1, b2, b3 = spec.blocks
    assert all(b.arrangement == "post_norm" for b in spec.blocks) and spec.blocks[3].feed_forward.kind == "none"
    assert all(n.kind == "rms_norm" and n["gain_offset"] == 1.0 for b in spec.blocks for n in b.norms.values())
    assert b0.mixer.kind == "gated_delta" and (b0.mixer["conv_taps"], b0.mixer["unit_eps"]) == (3, 1e-6)
    assert b0.mixer["q_scale"] == pytest.approx(24 ** -0.5)
    m = b1.mixer
    assert m.kind == "gqa_attention" and m["qk_norm"] == "rows" and m["softcap"] == 2.5 and m["q_temp"] == (0.4, 3)
    assert b3.mixer["own_kv"] is False and (b3.mixer["softcap"], b3.mixer["q_temp"], b3.mixer["scale"]) == (6.0, (0.2, 20), 0.5)
    assert b2.mixer.kind == "latent_attention" and b2.mixer["cache"] == "latent" and b2.mixer["q_rank"] == 0
    assert b2.position["pairing"] == "neighbours" and b2.position["n_rot"] == 8 and b2.position["base"] == 1000.0
    assert b0.feed_forward["activation"] == ("clamped_swish", 1.702, 1.5, 1.0)
    assert spec.embedding["scale"] == 3.0
    other = read_config(copy.deepcopy(SP_B)).to_spec().blocks[1].mixer
    assert other["softcap"] is None and other["q_temp"] is None


@pytest.mark.parametrize("path, value, text", [
    (("layers", 0, "type"), "mamba", "this design has"),
    (("layers", 0, "mixer", "kv_heads"), 3, "not a multiple"),
    (("layers", 0, "mixer", "conv"), 0, "positive integer"),
    (("layers", 1, "mixer", "scale"), None, "lacks 'scale'"),
    (("layers", 1, "mixer", "softcap"), -1.0, "softcap must be positive"),
    (("layers", 1, "mixer", "q_temp", "every"), 0, "positive integer"),
    (("layers", 1, "mixer", "q_temp", "coef"), "x", "must be a number"),
    (("layers", 2, "mixer", "rot", "dims"), 6, "equal rot_dim"),
    (("layers", 2, "mixer", "kv_rank"), None, "lacks 'kv_rank'"),
    (("layers", 3, "mixer", "kv_from"), 3, "an earlier layer"),
    (("layers", 3, "mixer", "kv_from"), 0, "no keys and values of its own"),
    (("layers", 3, "mixer", "vdim"), 8, "differs from layer 1"),
    (("layers", 0, "mlp", "limit"), 0.0, "limit must be positive"),
    (("layers", 0, "mlp", "kind"), "moe", "'dense'"),
    (("embedding",), None, "lacks 'embedding'"),
    (("norm", "eps"), 0.0, "positive"),
])
def test_inconsistent_configurations_are_refused(path, value, text):
    raw = copy.deepcopy(SP_A)
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=text):
        read_config(raw)


def test_a_borrower_may_not_lend_on():
    raw = copy.deepcopy(SP_A)
    raw["layers"].append(copy.deepcopy(raw["layers"][3]))
    raw["layers"][4]["mixer"]["kv_from"] = 3
    with pytest.raises(ConfigError, match="no keys and values of its own"):
        read_config(raw)


def test_parts_ask_for_the_cache_the_design_needs(tmp_path):
    """An entry of latents keeps kv_rank + rot_dim numbers a position and no values; a delta layer keeps state only; two
    attention layers on one entry ask for the same."""
    from llmoxide_b200.cache import KVNeed
    from llmoxide_b200.cache.storage import Cache
    from llmoxide_b200.parts import Runtime, build_block
    from llmoxide_b200.weights import load_checkpoint

    folder = make_folder(tmp_path, "A", "float32")
    spec = read_config(folder).to_spec()
    weights = load_checkpoint(folder, spec, "float32", "cpu")
    rt = Runtime(dtype="float32", device=torch.device("cpu"), max_positions=128)
    needs = [build_block(b, weights, rt).cache_need() for b in spec.blocks]
    kv, state = needs[0]
    C = 2 * 2 * 24 + 4 * 16
    assert kv is None and state.shape[0] >= 4 * 24 * 16 + 3 * C
    assert needs[2] == (KVNeed(1, 40 + 8, None, v_head_dim=0), None)
    assert needs[1] == needs[3] == (KVNeed(2, 32, None, v_head_dim=16), None)
    cache = Cache(needs[:3], n_slots=2, max_tokens=256, dtype=torch.float32, device="cpu")
    view = cache.view(2)
    assert view.k.shape == (4, 1, 64, 48) and view.v.shape == (4, 1, 64, 0)
    per_position = cache.k_store[view.group].numel() // 256
    assert per_position == 48
    cache.wipe()


def test_norm_gain_is_one_plus_the_stored_weight(tmp_path):
    from llmoxide_b200.parts import Runtime
    from llmoxide_b200.parts.norm import RMSNorm
    from llmoxide_b200.config import PartSpec, TensorSpec

    rt = Runtime(dtype="float32", device=torch.device("cpu"), max_positions=64)
    w = torch.tensor([0.25, -1.0, 0.0, 3.0], dtype=torch.bfloat16)
    tensors = dict(gain=TensorSpec("g", (4,), "vector"))
    assert RMSNorm(PartSpec("rms_norm", dict(size=4, eps=1e-6, gain_offset=1.0), tensors), {"g": w}, rt).gain.tolist() == [1.25, 0, 1, 4]
    assert RMSNorm(PartSpec("rms_norm", dict(size=4, eps=1e-6), tensors), {"g": w}, rt).gain.tolist() == [0.25, -1, 0, 3]


# ---------------------------------------------------------------------------------------------------------
# the plain implementation against closed forms
# ---------------------------------------------------------------------------------------------------------

def test_plain_temperature_steps_where_the_next_position_is_a_multiple():
    assert plain.query_temperature(0, 0.5, 4) == 1.0 and plain.query_temperature(2, 0.5, 4) == 1.0
    assert plain.query_temperature(3, 0.5, 4) == pytest.approx(1 + 0.5 * math.log(2))
    assert plain.query_temperature(10, 0.5, 4) == pytest.approx(1 + 0.5 * math.log(3))
    assert plain.query_temperature(0, 0.9, 1) == pytest.approx(1 + 0.9 * math.log(2))


def test_plain_attention_caps_scores_and_counts_the_sink_once():
    q = torch.tensor([[2.0], [2.0]], dtype=F)
    k = torch.tensor([[5.0], [-1.0]], dtype=F)
    v = torch.tensor([[1.0], [0.0]], dtype=F)
    s = [3.0 * math.tanh(x * 2.0 * 0.5 / 3.0) for x in (5.0, -1.0)]           # capped, scale 0.5
    got = plain.attend_causal(q, k, v, 0.5, softcap=3.0)
    assert got[0, 0] == pytest.approx(1.0) and got[1, 0] == pytest.approx(math.exp(s[0]) / (math.exp(s[0]) + math.exp(s[1])))
    got = plain.attend_causal(q, k, v, 0.5, sink=torch.tensor(1.5))
    e = [math.exp(5.0), math.exp(-1.0), math.exp(1.5)]
    assert got[0, 0] == pytest.approx(e[0] / (e[0] + e[2])) and got[1, 0] == pytest.approx(e[0] / sum(e))


def test_plain_delta_rule_replaces_what_a_key_held():
    """With beta 1, no decay and unit keys, a second write under a key replaces the first; an orthogonal key's value
    stays; the read-out sees its own token's write."""
    k = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 0.0]], dtype=F)
    v = torch.tensor([[3.0], [5.0], [-2.0]], dtype=F)
    one = torch.ones(3, dtype=F)
    o, S = plain.delta_rule(k, k, v, one, one)
    assert o.flatten().tolist() == [3.0, 5.0, -2.0] and S.flatten().tolist() == [-2.0, 5.0]
    # a decay acts on the state before the correction
    o, S = plain.delta_rule(k[:2], k[:2], v[:2], one[:2], torch.tensor([1.0, 0.5], dtype=F))
    assert S.flatten().tolist() == [1.5, 5.0]
    # continued from a state
    o2, S2 = plain.delta_rule(k[2:], k[2:], v[2:], one[2:], one[2:], state=torch.tensor([[3.0], [5.0]], dtype=F))
    assert o2.flatten().tolist() == [-2.0] and S2.flatten().tolist() == [-2.0, 5.0]


def test_plain_convolution_unit_vectors_and_rotation():
    u = torch.tensor([[1.0], [10.0], [100.0]], dtype=F)
    w = torch.tensor([[0.5, 2.0]], dtype=F)
    assert plain.causal_conv(u, w).flatten().tolist() == [2.0, 20.5, 205.0]
    x = torch.tensor([[3.0, 4.0], [0.0, 0.0]], dtype=F)
    assert torch.allclose(plain.unit_vectors(x)[0], torch.tensor([0.6, 0.8], dtype=F), atol=1e-7)
    assert plain.unit_vectors(x)[1].tolist() == [0.0, 0.0]
    r = plain.rotate_neighbours(torch.ones(4, 1, 6, dtype=F), 4, 100.0)
    assert r[0].flatten().tolist() == [1.0] * 6 and r[3, 0, 4:].tolist() == [1.0, 1.0]
    a = 3 * 100.0 ** -0.5
    assert r[3, 0, 2] == pytest.approx(math.cos(a) - math.sin(a)) and r[3, 0, 3] == pytest.approx(math.cos(a) + math.sin(a))


def test_plain_feed_forward_clamps_and_shifts():
    w = {"l0.mlp.gate": torch.tensor([[1.0]], dtype=F), "l0.mlp.up": torch.tensor([[-1.0]], dtype=F),
         "l0.mlp.down": torch.tensor([[1.0]], dtype=F)}
    got = plain.clamped_mlp(torch.tensor([[5.0], [-4.0], [0.5]], dtype=F), w, "l0.", 2.0).flatten()
    f = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert got.tolist() == pytest.approx([f(2.0, -2.0), f(-4.0, 2.0), f(0.5, -0.5)])


def test_plain_absorbed_attention_is_the_same_sum(tmp_path):
    """(W_uk c) . q = c . (W_uk^T q) and sum w (W_uv c) = W_uv sum w c: what the cache of latents rests on."""
    cfg, w = plain.read_model(make_folder(tmp_path, "C", "float32"))
    m, p = cfg["layers"][1]["mixer"], "l1."
    T, H, D, R, Dv, rank = 9, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    h = torch.randn(T, cfg["width"], dtype=F, generator=torch.Generator().manual_seed(1))
    want = plain.latent_attention_mixer(h, w, p, m, 1e-6)
    down = h @ w[p + "mix.dkv"].T
    c = plain.unit_rms(down[:, :rank], 1e-6) * w[p + "mix.dkv.norm"]
    rows = torch.cat([c, plain.rotate_neighbours(down[:, rank:], R, m["rot"]["base"])], dim=1)
    q = (h @ w[p + "mix.q"].T).reshape(T, H, D + R)
    q_rot = plain.rotate_neighbours(q[..., D:], R, m["rot"]["base"])
    absorbed = torch.einsum("thd,hdr->thr", q[..., :D], w[p + "mix.uk"].reshape(H, D, rank))
    out = []
    for hq in range(H):
        lat = plain.attend_causal(torch.cat([absorbed[:, hq], q_rot[:, hq]], dim=1), rows, c, m["scale"], sink=w[p + "mix.sink"][hq])
        out.append(lat @ w[p + "mix.uv"].reshape(H, Dv, rank)[hq].T)
    assert torch.allclose(torch.cat(out, dim=1) @ w[p + "mix.o"].T, want, atol=1e-10)
