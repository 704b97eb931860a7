"""Attention whose queries, keys and values come through low-rank latents.

For the mixer's input x (one row per token), H heads, per head D unrotated and
R rotated query/key dimensions and values of size Dv:

    cq = rms(W_dq x) * g_q                     the query latent (rank ``q_rank``)
    q  = W_uq cq                               per head [D unrotated | R rotated]
    [c_raw | kr] = W_dkv x                     ``kv_rank`` + R rows
    c  = rms(c_raw) * g_kv                     the key/value latent
    k_h = [W_uk c (head h, D) | rot(kr)]       kr is one rotated part that all heads share
    v_h = W_uv c (head h, Dv)
    s   = (q_plain . k_plain + rot(q_rot) . rot(kr)) * scale, softmax over the window's keys
    out = W_o concat_h( sigmoid(W_g x)_h * sum_j w_j v_j )      (``out_gate`` "sigmoid"; None: no gate)

``q_rank`` 0: queries come straight from the input, q = W_q x (tensor ``q`` in
place of ``dq``, ``dq_norm``, ``uq``).  Tensor ``sink`` [H]: exp(sink_h) joins
head h's softmax denominator, a learned score without key and value that is
not scaled.

rms is x / sqrt(mean(x^2) + eps) in float32.  The rotation is the position
part's (any table of ``rot_dim`` dimensions: scaled frequencies, an amplitude).

What is cached.  The latent c and the rotated part kr are all that later
tokens need.  ``cache`` "heads" (the default) keeps every head's assembled key
[rot(kr) | k_plain] and value, H heads of R + D and Dv: for a design that
attends under a window the cache holds at most the window's tokens per sequence
whatever the context's length, and assembled keys run on every attention kernel
of this package (tensor cores for prompts and decode at R + D = Dv in {64,
128}) without a product per cached token in every step.  Within a head the
rotated part is stored first, which no scalar product notices as queries are
laid out alike.

``cache`` "latent" keeps the row [c | rot(kr)] alone, kv_rank + R numbers per
position for all heads together (built without a window, without an output
gate, with queries straight from the input).  Three ways to attend over it, all
the same sums:
  * few new tokens (decode steps, short portions), bfloat16: the query goes
    through W_uk first, so that the cached rows are keys and values of every
    head as they are (``kernels.latent_decode``), and the sum of latents goes
    through W_uv behind it;
  * prompts at R + D = Dv in {64, 128}, bfloat16: the latents of the step's
    sequences are gathered, one product [W_uk; W_uv] c makes every head's keys
    and values for them, these are laid out in scratch pages, and the tiled
    prompt attention reads those like a cache;
  * everything else (float32, other sizes): absorbed like the first, in float32
    arithmetic (``kernels.latent_paged``).

Products: W_dq, W_dkv and W_g read the same rows and are one fused product
(float32 out, so the norms and the gate see unrounded sums); W_uk and W_uv are
one product over c.  Two small kernels sit between them (``csrc/latent_attention.cu``):
the two latents' norms, and rotation + key assembly + cache write.
"""

from __future__ import annotations

import torch

from .. import kernels
from ..cache import KVNeed
from ..errors import Unsupported
from .linear import Linear
from .position import halves_order
from .registry import register_mixer


# Steps of single tokens, and others of up to this many, attend over the latents as they are; longer ones expand them
# first (see above).
ABSORB_MAX_TOKENS = 64


@register_mixer("latent_attention")
class LatentAttention:
    def __init__(self, spec, position, weights: dict, rt):
        self.rt = rt
        self.H, self.D, self.R, self.Dv = spec["n_heads"], spec["head_dim"], spec["rot_dim"], spec["v_head_dim"]
        self.Rq, self.Rkv = spec["q_rank"], spec["kv_rank"]
        self.eps, self.scale = float(spec["eps"]), float(spec["scale"])
        self.window = spec.get("window")
        self.gate = spec.get("out_gate")
        if self.gate not in (None, "sigmoid"):
            raise Unsupported(f"out_gate {self.gate!r}: 'sigmoid' or none")
        if position is None or position.rotary_tables() is None or position.n_rot != self.R:
            raise Unsupported("latent attention rotates exactly its rot_dim dimensions: the position part must say so")
        self.position = position
        self.E = self.R + self.D                      # an assembled key, a query head
        self.latent_cache = spec.get("cache", "heads") == "latent"
        if max(self.E, self.Dv) > 256 and not self.latent_cache:
            raise Unsupported(f"head sizes {self.E}/{self.Dv}: the attention kernels take sizes up to 256")
        H, D, R, Dv = self.H, self.D, self.R, self.Dv
        t = spec.tensors
        wdkv = weights.pop(t["dkv"].name)
        # the shared rotated part's rows in the order the kernels pair them
        wdkv = torch.cat([wdkv[: self.Rkv], halves_order(position, wdkv[self.Rkv :], 1, R)], dim=0)
        if self.latent_cache:
            self._init_latent_cache(wdkv, weights, t)
            return
        rows = ([weights.pop(t["dq"].name)] if self.Rq else []) + [wdkv] + ([weights.pop(t["g"].name)] if self.gate else [])
        if len({w.dtype for w in rows}) > 1:
            rows = [w.float() for w in rows]
        self.down = Linear(torch.cat(rows, dim=0).contiguous(), rt)
        self.k_rot_off, self.gate_off = self.Rq + self.Rkv, self.Rq + self.Rkv + R
        self.uq = Linear(self._query_rows(weights.pop(t["uq" if self.Rq else "q"].name)), rt)
        wuk, wuv = weights.pop(t["uk"].name), weights.pop(t["uv"].name)
        if wuk.dtype != wuv.dtype:
            wuk, wuv = wuk.float(), wuv.float()
        self.ukv = Linear(torch.cat([wuk, wuv], dim=0).contiguous(), rt)
        self.q_gain = weights.pop(t["dq_norm"].name).to(torch.float32).contiguous() if self.Rq else None
        self.sinks = weights.pop(t["sink"].name).to(torch.float32).contiguous() if "sink" in t else None
        self.kv_gain = weights.pop(t["dkv_norm"].name).to(torch.float32).contiguous()
        self.o = Linear(weights.pop(t["o"].name), rt)
        self.out_bias, self.defer_out_bias = None, False
        # the shape the tiled kernels are written for
        self.plain = self.E == Dv and self.E % 16 == 0

    def _query_rows(self, w):
        """Every head's rows of a query projection become [rotated (paired as the kernels pair) | unrotated]."""
        H, D, R = self.H, self.D, self.R
        w = halves_order(self.position, w, H, D + R, first=D)
        index = torch.tensor([h * (D + R) + i for h in range(H) for i in list(range(D, D + R)) + list(range(D))],
                             device=w.device)
        return w.index_select(0, index).contiguous()

    def _init_latent_cache(self, wdkv, weights, t):
        if self.Rq or self.gate or self.window:
            raise Unsupported("a cache of latents is built without a query latent, an output gate and a window")
        H, D, Dv, rank, rt = self.H, self.D, self.Dv, self.Rkv, self.rt
        wq = self._query_rows(weights.pop(t["q"].name))
        if wq.dtype != wdkv.dtype:
            wq, wdkv = wq.float(), wdkv.float()
        fused = torch.cat([wdkv, wq], dim=0).contiguous()
        n = rank + self.R
        # one product for both in steps of few tokens; in prompts the latent's rows leave it in float32, the query's in
        # the compute dtype
        self.down_q, self.down, self.q_proj = Linear(fused, rt), Linear(fused[:n], rt), Linear(fused[n:], rt)
        wuk, wuv = weights.pop(t["uk"].name), weights.pop(t["uv"].name)
        if wuk.dtype != wuv.dtype:
            wuk, wuv = wuk.float(), wuv.float()
        # keys into the query: W_uk,h^T as [H, rank, D]; values out of the sum of latents: W_uv,h as [H, Dv, rank]
        self.absorb_w = wuk.view(H, D, rank).transpose(1, 2).contiguous()
        ukv = torch.cat([wuk, wuv], dim=0).contiguous()
        self.expand_w = ukv[H * D :].view(H, Dv, rank)
        self.ukv = Linear(ukv, rt)
        self.kv_gain = weights.pop(t["dkv_norm"].name).to(torch.float32).contiguous()
        self.sinks = weights.pop(t["sink"].name).to(torch.float32).contiguous() if "sink" in t else None
        self.o = Linear(weights.pop(t["o"].name), rt)
        self.out_bias, self.defer_out_bias = None, False
        bf16 = rt.dtype == "bfloat16" and rt.tensor_cores and ukv.dtype == torch.bfloat16 and self.scale > 0
        self.fast_absorbed = bf16 and kernels.latent_decode_supports(rank, self.R) and D % 8 == 0
        self.fast_expanded = bf16 and self.E == Dv and self.E in (64, 128)

    def cache_need(self):
        if self.latent_cache:
            return KVNeed(1, self.Rkv + self.R, None, v_head_dim=0), None
        return KVNeed(self.H, self.E, self.window, v_head_dim=None if self.Dv == self.E else self.Dv), None

    def libraries(self) -> set:
        if self.latent_cache:
            libs = {"latent_cache", "elementwise"} | self.down_q.libraries() | self.ukv.libraries() | self.o.libraries()
            if self.fast_expanded:
                libs.add("attention_prefill_tc" if self.E == 128 else "attention_prefill")
            return libs
        libs = {"latent_attention", "elementwise"} | self.down.libraries() | self.uq.libraries() | self.o.libraries()
        if self.plain and self.rt.dtype == "bfloat16" and self.rt.tensor_cores:
            libs |= {kernels.capped_library("attention_decode", self.sinks is not None),
                     "attention_prefill_tc" if self.E == 128 else "attention_prefill" if self.E == 64 else "attention"}
        else:
            libs.add("attention")
        return libs

    def forward(self, x, ctx, view, writes_cache=True):
        if not writes_cache:
            raise Unsupported("a latent attention layer owns its cache entry")
        if self.latent_cache:
            return self.o(self._attend_latents(x, ctx, view), splits_ok=True)
        H, D, R, Dv, E = self.H, self.D, self.R, self.Dv, self.E
        T, dev, act = x.shape[0], x.device, self.rt.act_dtype
        down = self.down(x, out_dtype=torch.float32)                         # [T, Rq + Rkv + R (+ H)]
        cq = torch.empty((T, self.Rq), dtype=act, device=dev) if self.Rq else None
        c = torch.empty((T, self.Rkv), dtype=act, device=dev)
        kernels.latent_norms(down, self.q_gain, self.kv_gain, self.eps, cq, c, self.Rq, self.Rkv)
        q_up = self.uq(cq if self.Rq else x)
        kv_up = self.ukv(c)
        cos, sin, _ = self.position.rotary_tables()
        block_table = ctx.block_tables[view.group]
        q = torch.empty((T, H * E), dtype=act, device=dev)
        kernels.latent_rope_cache(q_up, kv_up, down, self.k_rot_off, q, view.k, view.v, block_table, ctx, cos, sin,
                                  H, D, R, Dv)
        gate = down[:, self.gate_off :] if self.gate else None               # the heads' gate logits, a view
        out = torch.empty((T, H * Dv), dtype=act, device=dev)
        self.attend(q, out, view, block_table, ctx, gate)
        return self.o(out, splits_ok=True)

    def _attend_latents(self, x, ctx, view):
        H, D, R, Dv, E, rank = self.H, self.D, self.R, self.Dv, self.E, self.Rkv
        T, dev, act = x.shape[0], x.device, self.rt.act_dtype
        cos, sin, _ = self.position.rotary_tables()
        block_table = ctx.block_tables[view.group]
        new = lambda *shape, dtype=act: torch.empty(shape, dtype=dtype, device=dev)
        if T <= ABSORB_MAX_TOKENS:
            both = self.down_q(x, out_dtype=torch.float32, splits_ok=True)
            down, q = both, both[..., rank + R :]
        else:
            down, q = self.down(x, out_dtype=torch.float32, splits_ok=True), self.q_proj(x)
        prep = lambda rot, plain: kernels.latent_prep(down, q, self.kv_gain, self.eps, view.k, rot, plain, block_table, ctx,
                                                      cos, sin, H, D, R, rank)
        out = new(T, H, Dv)
        if self.fast_expanded and T > ABSORB_MAX_TOKENS and not ctx.is_decode:
            qa = new(T, H, E)
            prep(qa[:, :, :R], qa[:, :, R:])
            n = ctx.ctx_pages
            table, c = torch.empty_like(block_table), new(kernels.PAGE * n, rank)
            kernels.latent_gather(view.k, block_table, ctx, table, c, rank)
            kv = self.ukv(c)
            keys, values = new(n, H, kernels.PAGE, E), new(n, H, kernels.PAGE, Dv)
            kernels.latent_assemble(kv, view.k, block_table, ctx, keys, values, H, D, R, Dv, rank)
            prompt = kernels.attention_prefill_tc if E == 128 else kernels.attention_prefill
            prompt(qa.view(T, H * E), out.view(T, H * Dv), keys, values, table, ctx.seq_start, ctx.seq_past, ctx.n_seqs,
                   ctx.max_new, H, H, E, None, self.scale, sinks=self.sinks)
            return out.view(T, H * Dv)
        # absorbed: [W_uk^T q_plain | rot(q_rot)] against the cached rows, then W_uv
        dtype = act if self.fast_absorbed else torch.float32
        qa, plain, lat = new(T, H, rank + R, dtype=dtype), new(T, H, D, dtype=dtype), new(T, H, rank, dtype=dtype)
        prep(qa[:, :, rank:], plain)
        kernels.head_product(plain, self.absorb_w, qa[:, :, :rank])
        if self.fast_absorbed:
            kernels.latent_decode(qa, lat, view.k, block_table, ctx, self.sinks, self.scale, rank)
        else:
            kernels.latent_paged(qa, lat, view.k, block_table, ctx, self.sinks, self.scale, rank)
        kernels.head_product(lat, self.expand_w, out)
        return out.view(T, H * Dv)

    def attend(self, q, out, view, block_table, ctx, gate):
        """The general kernel applies the heads' gates itself; the tiled bfloat16 kernels (decode, and prompts at
        head sizes 64 and 128) are followed by the gate's own small kernel."""
        H, E = self.H, self.E
        fast = (self.plain and q.dtype == torch.bfloat16 and view.k.dtype == torch.bfloat16
                and self.rt.tensor_cores and self.scale > 0)
        if fast and ctx.is_decode:
            kernels.attention_decode(q, out, view.k, view.v, block_table, ctx.seq_past, H, H, E, self.window, self.scale,
                                     sinks=self.sinks)
        elif fast and E == 128:
            kernels.attention_prefill_tc(q, out, view.k, view.v, block_table, ctx.seq_start, ctx.seq_past,
                                         ctx.n_seqs, ctx.max_new, H, H, E, self.window, self.scale, sinks=self.sinks)
        elif fast and kernels.attention_prefill_supports(q, view.k, E):
            kernels.attention_prefill(q, out, view.k, view.v, block_table, ctx.seq_start, ctx.seq_past,
                                      ctx.n_seqs, ctx.max_new, H, H, E, self.window, self.scale, sinks=self.sinks)
        else:
            kernels.attention_paged(q, out, view.k, view.v, block_table, ctx.token_seq, ctx.token_pos,
                                    H, H, E, self.window, self.scale, v_head_dim=self.Dv, gate=gate, sinks=self.sinks)
            return
        if gate is not None:
            kernels.head_gate(out, gate, H, self.Dv)
