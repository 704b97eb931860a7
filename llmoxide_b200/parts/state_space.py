"""The state-space recurrence of Mamba-2 as a mixer: a decay and a step size per
token and head, a state of fixed size per sequence in place of keys and values.

    [z: inner | x: inner | B: groups N | C: groups N | dt: heads]        one projection of the layer's input, inner = heads P
    x, B, C <- silu(conv(x, B, C) + conv_bias)         causal convolution over time per channel, ``conv_taps``
    dt <- softplus(dt + dt_bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x      S [N, P] per head, starts at zero
    y <- y silu(z)
    out = W_o ( y / sqrt(mean(y^2) + eps) * gain )     mean over each of ``norm_groups`` equal runs of all heads' columns

Head h uses group h // (heads / groups).  Per sequence the state is S of every
head and the convolution's last projected rows, float32, in the cache's state
area.  The projection leaves float32 rows, and everything from there to the
norm is float32 whatever the compute dtype (csrc/state_space.cu).
"""

from __future__ import annotations

import torch

from .. import kernels
from ..cache import StateNeed
from ..errors import Unsupported
from .linear import Linear
from .registry import register_mixer


@register_mixer("state_space")
class StateSpace:
    def __init__(self, spec, position, weights: dict, rt):
        self.rt = rt
        self.H, self.P, self.N, self.G = spec["n_heads"], spec["v_head_dim"], spec["state_size"], spec["n_groups"]
        self.taps, self.parts, self.eps = int(spec["conv_taps"]), int(spec["norm_groups"]), float(spec["eps"])
        if self.H % self.G:
            raise Unsupported(f"{self.H} heads are not a multiple of {self.G} groups")
        if self.P > 256 or self.N > 1024:
            raise Unsupported(f"head size {self.P}, state size {self.N}: the recurrence kernels take up to 256 and 1024")
        if not 1 <= self.taps <= kernels.SS_MAX_TAPS:
            raise Unsupported(f"{self.taps} taps: the recurrence kernels take 1 to {kernels.SS_MAX_TAPS}")
        self.inner = self.H * self.P
        if self.inner % self.parts:
            raise Unsupported(f"{self.inner} columns do not fall into {self.parts} equal parts")
        if position is not None and position.rotary_tables() is not None:
            raise Unsupported("a rotation inside the state-space recurrence is not built")
        t = spec.tensors
        self.proj = Linear(weights.pop(t["in"].name), rt)
        self.o = Linear(weights.pop(t["o"].name), rt)
        vec = lambda r: weights.pop(t[r].name).to(torch.float32).contiguous()
        # [channels, taps] -> tap-major [taps, channels]: neighbouring threads read neighbouring channels
        self.conv_w = vec("conv").t().contiguous()
        self.conv_b = vec("conv_bias") if "conv_bias" in t else None
        self.a_log, self.dt_bias, self.skip, self.gain = vec("a_log"), vec("dt_bias"), vec("skip"), vec("norm")
        self.ring_off = (self.H * self.N * self.P + 3) // 4 * 4
        self.state_floats = (self.ring_off + self.taps * self.conv_w.shape[1] + 3) // 4 * 4

    def cache_need(self):
        return None, StateNeed((self.state_floats,))

    def libraries(self) -> set:
        return {"state_space"} | self.proj.libraries() | self.o.libraries()

    adds_to_residual = True      # forward() takes ``residual`` and may return None: "already added"

    def forward(self, x, ctx, view, writes_cache=True, residual=None):
        if not writes_cache:
            raise Unsupported("a recurrent state has one writer: the layer that owns it")
        T = x.shape[0]
        proj = self.proj(x, out_dtype=torch.float32, splits_ok=True)
        y = torch.empty((T, self.inner), dtype=torch.float32, device=x.device)
        scan = kernels.ss_decode if ctx.is_decode else kernels.ss_prompt
        scan(proj, self.conv_w, self.conv_b, self.a_log, self.dt_bias, self.skip, view.state, self.ring_off, y, ctx, self.H,
             self.G, self.N, self.P)
        out = torch.empty((T, self.inner), dtype=self.rt.act_dtype, device=x.device)
        kernels.ss_norm(y, self.gain, self.eps, self.parts, out)
        if residual is not None and self.o.add_into(out, residual):
            return None
        return self.o(out, splits_ok=True)
