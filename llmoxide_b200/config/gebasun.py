"""Typed configuration of the Gebasun decoder and its description as a
``ModelSpec``.

config.json of this design is nested: ``vocab``, ``width``, ``norm.eps`` and a
list ``layers``; every layer names its mixer (``type``: ``attention``,
``attention_2`` or ``mamba2``) with the mixer's sizes and constants (``mixer``)
and its feed-forward (``mlp``: ``kind`` ``moe``, or null for none).  Tensors:
``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``final.norm``, ``head``.

A layer's two sublayers read the same stream, each through an RMS norm of its
own, and their results join it together: h += mixer(rms_1(h)) + experts(rms_2(h)).

Mixers.  Both attentions project queries and keys only, with biases; a key as
projected is also the value; q and k are divided by their root mean square per
head, without a weight; every head has a learned sink in the softmax's
denominator.  ``attention``: no rotation, a learned bias per distance bucket
and head on the scaled score (``rel`` [rows, heads]: one row per distance in
the first half, then a logarithmic scale up to ``bias_max``), a sliding window
(``mask.size``), a bias on the output projection.  ``attention_2``: rotation of
halves over ``rot.dims`` dimensions before the norm, a window that keeps the
first ``mask.keep_first`` tokens, and the concatenated heads times sigmoid(W_g
h) before the output projection.  ``mamba2``: one input projection [z | x | B |
C | dt], a short convolution with bias and SiLU on x, B and C, the state-space
recurrence with a decay and a step size per head and token, times silu(z), an
RMS norm in ``norm_groups`` equal parts with a weight.

Feed-forward ``moe``: ``router.top`` of ``router.experts`` experts (largest
logits, bias included; weights softmax over the chosen logits), an expert is
W_down relu(W_up h)^2, and a shared expert of the same form (``shared.ff``) is
added for every token.

The distance table's rows come from the tensor's shape; ``bias_rows`` (optional,
this package's own key) names them for random weights.
"""

from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field

from ..errors import ConfigError
from .fusasun import _number
from .spec import BlockSpec, LayerCall, ModelSpec, PartSpec, TensorSpec
from .tifapel import _need, _positive_int

_MIXERS = ("attention", "attention_2", "mamba2")
# random weights: biases and distance tables around zero, taps around zero, decays of a few per cent, a skip near one
BIAS_INIT = (0.0, 0.05)
REL_INIT = (0.0, 0.5)
SINK_INIT = (0.0, 1.0)
CONV_INIT = (0.0, 0.5)
A_LOG_INIT = (0.0, 0.5)
DT_BIAS_INIT = (-2.0, 0.5)
ROUTER_BIAS_INIT = (0.0, 0.1)


@dataclass
class GebasunConfig:
    vocab: int
    width: int
    eps: float
    layers: list                       # as in config.json: dicts with type / mixer / mlp
    max_positions: int = 1 << 20       # the design has no limit of its own; the cache's size is the limit
    torch_dtype: str = "bfloat16"
    extra: dict = field(default_factory=dict)
    generation: dict = field(default_factory=dict)

    # ---- reading -----------------------------------------------------------

    @classmethod
    def from_dict(cls, d: dict) -> "GebasunConfig":
        norm = _need(d, "norm", "the top level")
        known = {"architecture", "architectures", "vocab", "width", "norm", "layers", "max_positions", "torch_dtype"}
        cfg = cls(vocab=_need(d, "vocab", "the top level"), width=_need(d, "width", "the top level"),
                  eps=_number(_need(norm, "eps", "norm"), "norm.eps"),
                  layers=copy.deepcopy(_need(d, "layers", "the top level")),
                  max_positions=int(d.get("max_positions") or (1 << 20)),
                  torch_dtype=d.get("torch_dtype") or "bfloat16",
                  extra={k: v for k, v in d.items() if k not in known})
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        d = dict(self.extra)
        d.update(architecture="Gebasun", vocab=self.vocab, width=self.width, norm={"eps": self.eps},
                 layers=copy.deepcopy(self.layers), torch_dtype=self.torch_dtype)
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        return d

    # ---- checks ------------------------------------------------------------

    def validate(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.eps!r}")
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("'layers' must be a non-empty list")
        if self.torch_dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"torch_dtype {self.torch_dtype!r}: supported are bfloat16 and float32")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}.type {kind!r}: this design has {', '.join(_MIXERS)}")
            m = _need(layer, "mixer", where)
            if kind == "mamba2":
                self._check_mamba2(m, where + ".mixer")
            else:
                self._check_attention(m, where + ".mixer", kind)
            if layer.get("mlp") is not None:
                self._check_mlp(layer["mlp"], where + ".mlp")

    @staticmethod
    def _check_attention(m: dict, where: str, kind: str) -> None:
        for key in ("heads", "kv_heads", "dim"):
            _positive_int(_need(m, key, where), f"{where}.{key}")
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
        if _positive_int(m.get("vdim", m["dim"]), where + ".vdim") != m["dim"]:
            raise ConfigError(f"{where}.vdim {m['vdim']} must equal dim {m['dim']}: the keys are the values")
        _number(_need(m, "scale", where), where + ".scale")
        mask = m.get("mask")
        if mask is not None:
            _positive_int(_need(mask, "size", where + ".mask"), where + ".mask.size")
            keep = mask.get("keep_first", 0)
            if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
                raise ConfigError(f"{where}.mask.keep_first must be a non-negative integer")
        if kind == "attention":
            if not _number(_need(m, "bias_max", where), where + ".bias_max") > 0:
                raise ConfigError(f"{where}.bias_max must be positive")
            if m.get("bias_rows") is not None:
                _positive_int(m["bias_rows"], where + ".bias_rows")
            return
        rot = _need(m, "rot", where)
        dims = _positive_int(_need(rot, "dims", where + ".rot"), where + ".rot.dims")
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f"{where}.rot.dims {dims} must be even and at most dim {m['dim']}")
        if not _number(_need(rot, "base", where + ".rot"), where + ".rot.base") > 0:
            raise ConfigError(f"{where}.rot.base must be positive")

    @staticmethod
    def _check_mamba2(m: dict, where: str) -> None:
        for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
            _positive_int(_need(m, key, where), f"{where}.{key}")
        if m["heads"] % m["groups"]:
            raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['groups']} groups")
        if (m["heads"] * m["vdim"]) % m["norm_groups"]:
            raise ConfigError(f"{where}: {m['heads'] * m['vdim']} columns do not fall into {m['norm_groups']} norm_groups")

    @staticmethod
    def _check_mlp(mlp: dict, where: str) -> None:
        kind = _need(mlp, "kind", where)
        if kind != "moe":
            raise ConfigError(f"{where}.kind {kind!r}: 'moe' (or null for no feed-forward)")
        _positive_int(_need(_need(mlp, "expert", where), "ff", where + ".expert"), where + ".expert.ff")
        r = _need(mlp, "router", where)
        E = _positive_int(_need(r, "experts", where + ".router"), where + ".router.experts")
        top = _positive_int(_need(r, "top", where + ".router"), where + ".router.top")
        if top > E:
            raise ConfigError(f"{where}.router.top {top} exceeds the {E} experts")
        if mlp.get("shared") is not None:
            _positive_int(_need(mlp["shared"], "ff", where + ".shared"), where + ".shared.ff")

    # ---- derived ----------------------------------------------------------------

    def n_params(self) -> int:
        return sum(math.prod(t.shape) for t in self.to_spec().tensors() if -1 not in t.shape)   # (tables of unknown length are left out)

    def summary(self) -> str:
        kinds = "".join({"attention": "a", "attention_2": "r", "mamba2": "m"}[layer["type"]] for layer in self.layers)
        return (f"gebasun: {len(self.layers)} layers ({kinds}), width {self.width}, vocab {self.vocab}, "
                f"eps {self.eps:g}, {self.n_params() / 1e6:.1f} M params, {self.torch_dtype}")

    # ---- description as parts ------------------------------------------------

    def _mixer(self, p: str, kind: str, m: dict):
        """(mixer, position) of one layer whose tensors start with ``p``."""
        d, eps = self.width, self.eps
        matrix = lambda name, *shape: TensorSpec(p + "mix." + name, shape)
        vector = lambda name, n, init=None: TensorSpec(p + "mix." + name, (n,), "vector", init)
        if kind == "mamba2":
            H, P, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            inner, channels = H * P, H * P + 2 * G * N
            tensors = {"in": matrix("in", inner + channels + H, d),
                       "conv": TensorSpec(p + "mix.conv", (channels, taps), "vector", CONV_INIT),
                       "conv_bias": vector("conv.b", channels, BIAS_INIT), "dt_bias": vector("dt_bias", H, DT_BIAS_INIT),
                       "a_log": vector("A_log", H, A_LOG_INIT), "skip": vector("D", H), "norm": vector("norm", inner),
                       "o": matrix("o", d, inner)}
            return PartSpec("state_space", dict(
                hidden_size=d, n_heads=H, v_head_dim=P, state_size=N, n_groups=G, conv_taps=taps,
                norm_groups=m["norm_groups"], eps=eps), tensors), None
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        mask = m.get("mask") or {}
        tensors = dict(q=matrix("q", H * D, d), k=matrix("k", G * D, d), q_bias=vector("q.b", H * D, BIAS_INIT),
                       k_bias=vector("k.b", G * D, BIAS_INIT), sink=vector("sink", H, SINK_INIT),
                       o=matrix("o", d, H * D))
        params = dict(hidden_size=d, n_heads=H, n_kv_heads=G, head_dim=D, scale=float(m["scale"]),
                      window=mask.get("size"), keep_first=mask.get("keep_first", 0), qk_norm_eps=eps, qk_norm="unit",
                      values="keys")
        if kind == "attention":
            tensors.update(o_bias=vector("o.b", d, BIAS_INIT),
                           score_bias=TensorSpec(p + "mix.rel", (m.get("bias_rows") or -1, H), "vector", REL_INIT))
            params["bias_max"] = m["bias_max"]
            return PartSpec("gqa_attention", params, tensors), None
        tensors["gate"] = matrix("g", H * D, d)
        return PartSpec("gqa_attention", params, tensors), PartSpec("rope_neox", dict(
            n_rot=m["rot"]["dims"], base=float(m["rot"]["base"]), angles="float32"))

    def _feed_forward(self, p: str, mlp):
        if mlp is None:
            return PartSpec("none", {}, {})
        d, F, E = self.width, mlp["expert"]["ff"], mlp["router"]["experts"]
        tensors = {"router": TensorSpec(p + "mlp.router", (E, d)),
                   "router_bias": TensorSpec(p + "mlp.router.b", (E,), "vector", ROUTER_BIAS_INIT)}
        for e in range(E):
            tensors[f"up{e}"] = TensorSpec(f"{p}mlp.e{e}.up", (F, d))
            tensors[f"down{e}"] = TensorSpec(f"{p}mlp.e{e}.down", (d, F))
        shared = mlp.get("shared")
        if shared is not None:
            tensors.update(shared_up=TensorSpec(p + "mlp.shared.up", (shared["ff"], d)),
                           shared_down=TensorSpec(p + "mlp.shared.down", (d, shared["ff"])))
        return PartSpec("routed_experts", dict(
            hidden_size=d, intermediate_size=F, n_experts=E, top=mlp["router"]["top"], score="softmax_top", gated=False,
            activation="relu_squared", shared_size=shared["ff"] if shared is not None else 0), tensors)

    def to_spec(self) -> ModelSpec:
        d, eps = self.width, self.eps
        norm = lambda name: PartSpec("rms_norm", dict(size=d, eps=eps), dict(gain=TensorSpec(name, (d,), "vector")))
        blocks, schedule, ignored = [], [], []
        for i, layer in enumerate(self.layers):
            p, mlp = f"l{i}.", layer.get("mlp")
            mixer, position = self._mixer(p, layer["type"], layer["mixer"])
            norms = dict(mixer=norm(p + "norm1"))
            if mlp is not None:
                norms["feed_forward"] = norm(p + "norm2")
            else:
                ignored.append(p + "norm2")          # a layer without a feed-forward has no use for it
            blocks.append(BlockSpec("parallel", mixer, self._feed_forward(p, mlp), norms, position))
            schedule.append(LayerCall(layer=i, cache=i))
        return ModelSpec(
            architecture="Gebasun", hidden_size=d, vocab_size=self.vocab,
            embedding=PartSpec("gather", dict(scale=None), dict(table=TensorSpec("embed", (self.vocab, d)))),
            blocks=tuple(blocks), schedule=tuple(schedule), final_norm=norm("final.norm"),
            head=PartSpec("linear", dict(softcap=None), dict(weight=TensorSpec("head", (self.vocab, d)))),
            max_positions=self.max_positions, stop_ids=(), storage_dtype=self.torch_dtype, default_sampling={},
            ignored_tensors=tuple(ignored),
        )
