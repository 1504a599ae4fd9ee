"""Retention: a linear recurrence whose heads fade at constant rates (a mixer).

In this file's notation, for the mixer's input h_t, with H heads of key size D and value size P:

    q, k, v = Wq h, Wk h, Wv h                       no bias
    q, k   <- turn(q), turn(k) * D^-1/2              the first ``position.dim`` dims of each head, by position
    S_t     = g_i S_(t-1) + k_t v_t^T                S: [D, P] per head, g_i the head's decay, a constant
    y_t     = S_t^T q_t
    o_t     = y_t / sqrt(mean(y_t^2) + eps) * silu(Wg h_t)      the mean per head
    out     = Wo o_t

The rotation, the recurrence, the norm and the gate run in 32-bit.  Per-sequence state: S, in 32-bit, zero at a sequence's
start.  Portions of more than a few tokens run in chunks side by side (the same sums in another order).

Alone (``forward``) or as a branch of a parallel mixer (``in_weight`` / ``out_weight`` / ``inner`` / ``mix``).
"""

from __future__ import annotations

import torch

from ..cache.spec import CacheNeed
from ..weights.loader import TensorDecl
from .base import MIXERS, POSITIONS, Mixer


@MIXERS.register("retention")
class Retention(Mixer):
    accepts_residual = True
    same_bits_across_steps = False      # long portions run in chunks

    @classmethod
    def declare(cls, spec, prefix):
        s, nm = spec, spec.names
        qk, v = s.heads * s.key_dim, s.heads * s.value_dim
        return [TensorDecl(prefix + n, (r, s.hidden)) for n, r in ((nm.q, qk), (nm.k, qk), (nm.v, v), (nm.gate, v))] + [
            TensorDecl(prefix + nm.o, (s.hidden, v))]

    @classmethod
    def cache_need(cls, spec) -> CacheNeed:
        return CacheNeed(kind="none", state_shape=(spec.heads * spec.key_dim * spec.value_dim,))

    def __init__(self, spec, weights, prefix, rt):
        s, nm = spec, spec.names
        if len(s.decay) != s.heads:
            raise ValueError(f"retention: {len(s.decay)} decays for {s.heads} heads")
        self.spec, self.rt = spec, rt
        self.in_weight = torch.cat([weights[prefix + n].to(rt.dtype) for n in (nm.q, nm.k, nm.v, nm.gate)], dim=0).contiguous()
        self.out_weight = weights[prefix + nm.o].to(rt.dtype).contiguous()
        self.decay = torch.tensor([float(g) for g in s.decay], dtype=torch.float32, device=rt.device)
        self.inner = s.heads * s.value_dim
        self.position = None
        if s.position is not None:
            variant = getattr(s.position, "variant", None)
            if variant not in ("half_partial", "half_whole_head") or s.position.dim > s.key_dim or s.position.dim % 2 \
                    or getattr(s.position, "scaling", None) is not None:
                raise ValueError(f"retention: position encoding variant {variant!r} over {s.position.dim} of {s.key_dim} dims is "
                                 f"not built; the kernels turn dim i with dim i + dim / 2 over the first `dim` dims of a head "
                                 f"('half_partial'), without a scaling")
            self.position = POSITIONS.get(s.position.kind)(s.position, weights, prefix, rt)

    # -- as a branch: columns [col0, col0 + in_weight rows) of `proj` are this mixer's projections of the step
    def mix(self, proj, col0, ctx, kv, state, out, out_col, out_scale):
        s, K = self.spec, self.rt.kernels
        cs = self.position.tables(ctx) if self.position is not None else None
        qk = s.heads * s.key_dim
        cols = (col0, col0 + qk, col0 + 2 * qk)
        y = K.retention(proj, cols, cs, s.key_dim ** -0.5, self.decay, state, ctx, s.heads, s.key_dim, s.value_dim)
        K.delta_out(y, None, s.eps, proj, col0 + 2 * qk + self.inner, out_scale, out, out_col, s.heads, s.value_dim, gate_act=1)

    def forward(self, x, ctx, kv, state, writes_cache: bool, residual=None):
        """Returns the delta ``[1, N, hidden]``, or None after adding it into ``residual`` in place."""
        K = self.rt.kernels
        proj = K.gemm_store(x, self.in_weight, pad=True)
        out = torch.empty((x.shape[0], self.inner), dtype=self.rt.dtype, device=x.device)
        self.mix(proj, 0, ctx, None, state, out, 0, 1.0)
        if residual is not None and getattr(K, "fused", False) and self.inner % 8 == 0:
            K.gemm_residual(out, self.out_weight, residual)
            return None
        return K.gemm(out, self.out_weight, pad=True)
