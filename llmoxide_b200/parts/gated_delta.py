"""The gated delta rule as a mixer: linear attention whose state first forgets,
then corrects what it holds for a key, in place of keys and values.

    q, k: [kv heads, D], v: [heads, Dv], gate: [heads * Dv], b, a: [heads]       one fused projection of the layer's input
    q, k, v <- silu(conv(q)), silu(conv(k)), silu(conv(v))     causal convolution over time per channel, ``conv_taps``
    q <- q / sqrt(sum q^2 + unit_eps) * q_scale,  k <- k / sqrt(sum k^2 + unit_eps)           per head
    beta = sigmoid(b),  g = exp(-exp(A_log) * softplus(a + dt_bias))                          per head
    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          S [D, Dv] per head, starts at zero
    y = W_o ( o / sqrt(mean(o^2) + eps) * gain * silu(gate) )             mean over a head's Dv, one gain [Dv] for all

Value head h uses key/query head h // (heads / kv heads).  Per sequence the
state is S of every head and the convolution's last projected rows, float32,
in the cache's state area.  The fused projection leaves float32 rows, and
everything from there to the gated norm is float32 whatever the compute dtype
(csrc/delta_rule.cu).
"""

from __future__ import annotations

import torch

from .. import kernels
from ..cache import StateNeed
from ..errors import Unsupported
from .linear import Linear
from .registry import register_mixer


@register_mixer("gated_delta")
class GatedDelta:
    def __init__(self, spec, position, weights: dict, rt):
        self.rt = rt
        self.H, self.G, self.D, self.Dv = spec["n_heads"], spec["n_kv_heads"], spec["head_dim"], spec["v_head_dim"]
        self.taps = int(spec["conv_taps"])
        if self.H % self.G:
            raise Unsupported(f"{self.H} heads are not a multiple of {self.G} kv heads")
        if self.D > 256:
            raise Unsupported(f"head_dim {self.D}: the recurrence kernels take sizes up to 256")
        if not 1 <= self.taps <= kernels.DELTA_MAX_TAPS:
            raise Unsupported(f"{self.taps} taps: the recurrence kernels take 1 to {kernels.DELTA_MAX_TAPS}")
        if position is not None and position.rotary_tables() is not None:
            raise Unsupported("a rotation inside the delta rule is not built")
        self.eps, self.unit_eps = float(spec["eps"]), float(spec.get("unit_eps", 1e-6))
        self.q_scale = float(spec.get("q_scale", self.D ** -0.5))
        t = spec.tensors
        ws = [weights.pop(t[r].name) for r in ("q", "k", "v", "g", "b", "a")]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.float() for w in ws]
        # one matrix product for q, k, v, the output gate, the step sizes and the decays: rows in that order
        self.proj = Linear(torch.cat(ws, dim=0), rt)
        del ws
        self.o = Linear(weights.pop(t["o"].name), rt)
        vec = lambda r: weights.pop(t[r].name).to(torch.float32).contiguous()
        # [channels of q | k | v, taps] -> tap-major [taps, channels]: neighbouring threads read neighbouring channels
        self.conv_w = torch.cat([vec(r) for r in ("q_conv", "k_conv", "v_conv")], dim=0).t().contiguous()
        self.a_log, self.dt_bias, self.gain = vec("a_log"), vec("dt_bias"), vec("norm")
        self.gain_rows = self.gain.repeat(self.H).contiguous()           # as the norm over whole rows takes it
        GD, HDv = self.G * self.D, self.H * self.Dv
        self.g_off = 2 * GD + HDv
        # columns of q, k, v, b, a and the gate, as the kernels take them
        self.offsets = (0, GD, 2 * GD, self.g_off + HDv, self.g_off + HDv + self.H, self.g_off)
        self.ring_off = (self.H * self.D * self.Dv + 3) // 4 * 4
        self.state_floats = (self.ring_off + self.taps * (2 * GD + HDv) + 3) // 4 * 4

    def cache_need(self):
        return None, StateNeed((self.state_floats,))

    def libraries(self) -> set:
        return {"delta_rule", "linear_attention"} | self.proj.libraries() | self.o.libraries()

    adds_to_residual = True      # forward() takes ``residual`` and may return None: "already added"

    def forward(self, x, ctx, view, writes_cache=True, residual=None):
        if not writes_cache:
            raise Unsupported("a recurrent state has one writer: the layer that owns it")
        T, H, G, D, Dv = x.shape[0], self.H, self.G, self.D, self.Dv
        proj = self.proj(x, out_dtype=torch.float32, splits_ok=True)
        y = torch.empty((T, H * Dv), dtype=self.rt.act_dtype, device=x.device)
        common = (proj, self.offsets, self.conv_w, self.taps, self.a_log, self.dt_bias, self.q_scale, self.unit_eps,
                  view.state, self.ring_off)
        if ctx.is_decode:
            kernels.delta_decode(*common, self.gain, self.eps, y, ctx, H, G, D, Dv)
        else:
            o = torch.empty((T, H * Dv), dtype=torch.float32, device=x.device)
            kernels.delta_prompt(*common, o, ctx, H, G, D, Dv)
            kernels.gated_norm(o, proj, self.g_off, self.gain_rows, self.eps, "silu", True, y, H, Dv)
        if residual is not None and self.o.add_into(y, residual):
            return None
        return self.o(y, splits_ok=True)
