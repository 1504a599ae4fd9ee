"""Differential attention: a head subtracts a multiple of one softmax of its keys from another (a mixer).

In this file's notation, for the mixer's input h of one sequence (positions t = 0 .. T-1), with heads i and maps m = 1, 2:

    q, k, v   = filter(Wq h), filter(Wk h), filter(Wv h)     per channel, ``conv_taps`` taps, causal, zeros before t = 0
    q_m, k_m <- turn(q_m), turn(k_m)                         the first ``position.dim`` dims of each map, by position
    a_m       = softmax_j(scale * q_m,t . k_m,j) v_j         (j <= t)  q-head i reads kv-head i // (heads / kv_heads)
    lambda    = exp(lq1 . lk1) - exp(lq2 . lk2) + diff       one number for the layer
    o_t       = a_1 - lambda a_2
    o_t      <- o_t / sqrt(mean(o_t^2) + eps) * (1 - diff) * sigmoid(Wg h_t)_i
    out       = Wo o

A token's key row in the cache is a head's two maps side by side, ``[k_1 | k_2]``, as the projection makes them, and one value
row per head.  A query goes out as two rows, ``[q_1 | 0]`` and ``[0 | q_2]``: against the same key rows they score their maps
alone, so both maps are ordinary attention of twice as many query heads over one set of keys and values, which any of the
attention kernels runs and which reads the cache once.  Filters, rotation, scores, softmax, the combination, its norm and
the gate run in 32-bit.  A filter's last ``conv_taps - 1`` inputs are per-sequence state.

Alone (``forward``) or as a branch of a parallel mixer (``in_weight`` / ``out_weight`` / ``inner`` / ``mix``).
"""

from __future__ import annotations

import torch

from ..cache.spec import CacheNeed
from ..weights.loader import TensorDecl
from .base import MIXERS, POSITIONS, Mixer

MAPS = 2


@MIXERS.register("differential_attention")
class DifferentialAttention(Mixer):
    accepts_residual = True

    @staticmethod
    def _channels(s):
        """Filtered channels: q, k, v."""
        return (s.n_heads + s.n_kv_heads) * MAPS * s.key_dim + s.n_kv_heads * s.value_dim

    @classmethod
    def declare(cls, spec, prefix):
        s, nm = spec, spec.names
        rows = [(nm.q, s.n_heads * MAPS * s.key_dim), (nm.k, s.n_kv_heads * MAPS * s.key_dim), (nm.v, s.n_kv_heads * s.value_dim)]
        d = [TensorDecl(prefix + n, (r, s.hidden)) for n, r in rows]
        if s.conv_taps:
            d += [TensorDecl(prefix + n + nm.conv, (r, s.conv_taps), init="filter") for n, r in rows]
        d += [TensorDecl(prefix + n, (s.key_dim,)) for n in (nm.lambda_q1, nm.lambda_k1, nm.lambda_q2, nm.lambda_k2)]
        if s.head_gate:
            d.append(TensorDecl(prefix + nm.gate, (s.n_heads, s.hidden)))
        d.append(TensorDecl(prefix + nm.o, (s.hidden, s.n_heads * s.value_dim)))
        return d

    @classmethod
    def cache_need(cls, spec) -> CacheNeed:
        s = spec
        taps = s.conv_taps or 1
        return CacheNeed(kind="full", n_kv_heads=s.n_kv_heads, head_dim=MAPS * s.key_dim,
                         k_row=(s.n_kv_heads, MAPS * s.key_dim), v_row=(s.n_kv_heads, s.value_dim),
                         state_shape=((taps - 1) * cls._channels(s),) if taps > 1 else None)

    def __init__(self, spec, weights, prefix, rt):
        s, nm = spec, spec.names
        if s.n_heads % s.n_kv_heads:
            raise ValueError("n_heads must be a multiple of n_kv_heads")
        self.spec, self.rt = spec, rt
        mats = [weights[prefix + n] for n in (nm.q, nm.k, nm.v)] + ([weights[prefix + nm.gate]] if s.head_gate else [])
        self.in_weight = torch.cat([m.to(rt.dtype) for m in mats], dim=0).contiguous()
        self.out_weight = weights[prefix + nm.o].to(rt.dtype).contiguous()
        self.inner = s.n_heads * s.value_dim
        self.channels = self._channels(s)
        self.taps = s.conv_taps or 1
        if s.conv_taps:
            self.w_conv = torch.cat([weights[prefix + n + nm.conv].to(torch.float32) for n in (nm.q, nm.k, nm.v)], dim=0).contiguous()
        else:
            self.w_conv = torch.ones((self.channels, 1), dtype=torch.float32, device=rt.device)
        f64 = lambda n: weights[prefix + n].to(torch.float64)
        one, two = (torch.exp((f64(a) * f64(b)).sum()) for a, b in ((nm.lambda_q1, nm.lambda_k1), (nm.lambda_q2, nm.lambda_k2)))
        self.lam = float((one - two).item()) + float(s.diff)            # one number for the layer, made once at load
        self.position = None
        if s.position is not None:
            variant = getattr(s.position, "variant", None)
            if variant not in ("half_partial", "half_whole_head") or s.position.dim > s.key_dim or s.position.dim % 2 \
                    or getattr(s.position, "scaling", None) is not None:
                raise ValueError(f"differential attention: position encoding variant {variant!r} over {s.position.dim} of "
                                 f"{s.key_dim} dims is not built; the kernels turn dim i with dim i + dim / 2 over the first "
                                 f"`dim` dims of a map ('half_partial'), without a scaling")
            self.position = POSITIONS.get(s.position.kind)(s.position, weights, prefix, rt)

    # -- as a branch: columns [col0, col0 + in_weight rows) of `proj` are this mixer's projections of the step
    def mix(self, proj, col0, ctx, kv, state, out, out_col, out_scale):
        s, K = self.spec, self.rt.kernels
        cs = self.position.tables(ctx) if self.position is not None else None
        dk, dv = MAPS * s.key_dim, s.value_dim
        q = K.conv_qkv_cache(proj, col0, self.w_conv, state, s.n_heads, s.n_kv_heads, dk, dv, cs, kv, ctx, maps=MAPS)
        if self.taps > 1 and not ctx.single_token:
            K.conv_state_update(proj, col0, self.channels, self.taps, state, ctx)
        if K.attention_tc_fits(kv, dk, dv) and s.softmax_scale > 0:
            o = K.attention_tc(q, kv, ctx, s.softmax_scale)
        else:
            o = torch.empty((proj.shape[0], MAPS * self.inner), dtype=self.rt.dtype, device=proj.device)
            K.attention_biased(q, kv, ctx, s.softmax_scale, o, 0)
        gate = proj[:, col0 + self.channels:] if s.head_gate else None
        K.diff_combine(o, self.lam, s.eps, (1.0 - s.diff) * out_scale, gate, proj.shape[1], out, out_col, s.n_heads, dv)

    def forward(self, x, ctx, kv, state, writes_cache: bool, residual=None):
        """Returns the delta ``[1, N, hidden]``, or None after adding it into ``residual`` in place."""
        if not writes_cache:
            raise ValueError("this mixer writes its own keys and values")
        K = self.rt.kernels
        proj = K.gemm_store(x, self.in_weight, pad=True)
        out = torch.empty((x.shape[0], self.inner), dtype=self.rt.dtype, device=x.device)
        self.mix(proj, 0, ctx, kv, state, out, 0, 1.0)
        if residual is not None and getattr(K, "fused", False) and self.inner % 8 == 0:
            K.gemm_residual(out, self.out_weight, residual)
            return None
        return K.gemm(out, self.out_weight, pad=True)
