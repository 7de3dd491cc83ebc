"""Attentions with something on the way into or out of an ordinary paged softmax: short convolutions on queries,
keys and values in front of a sliding window that keeps the first tokens visible, and two maps per head over
the same values whose outputs are combined.

Both are ``ProjectedMixer``s and share ``PagedSoftmax``, which picks the attention kernel for a step.
"""

from __future__ import annotations

import torch

from ..csrc import ops
from .base import KVNeed, ParamDecl, PlanNeeds, StateNeed, register_mixer
from .builtin import _as_compute
from .mixers import ProjectedMixer, _f32, _half_rotation


class PagedSoftmax(ProjectedMixer):
    """Softmax attention over the paged cache for subclasses that prepare queries, keys and values themselves:
    ``_softmax_sizes`` fixes heads, row sizes and what a position sees, ``_attend`` runs the step.

    ``window``: position ``i`` sees ``j`` with ``0 <= i - j < window`` (None: the whole past), and with
    ``keep_first`` also ``j < keep_first``.  ``softcap`` > 0: a scaled score ``s`` becomes ``softcap tanh(s /
    softcap)``.  Scores, weights and sums are fp32 for either dtype."""

    def _softmax_sizes(self, nq: int, nkv: int, d: int, dv: int, scale: float, window: int | None, keep_first: int,
                       softcap: float) -> None:
        if nq % nkv:
            raise ValueError(f"{nq} query heads cannot share {nkv} key/value heads")
        if not (0 < d <= 1024 and 0 < dv <= 512):
            raise ValueError(f"head sizes {d} (keys, up to 1024) and {dv} (values, up to 512)")
        if keep_first < 0 or (keep_first and not window):
            raise ValueError("first tokens are kept visible beside a window")
        if softcap < 0:
            raise ValueError(f"a cap on scores is positive, got {softcap}")
        self.s_nq, self.s_nkv, self.s_d, self.s_dv, self.s_scale = nq, nkv, d, dv, scale
        self.s_window, self.s_keep, self.s_cap = window, keep_first, softcap

    def _tensor_core_sizes(self) -> bool:
        """Sizes the balanced decode kernel and the prefill kernels take: keys and values of one size, a multiple of 16."""
        return self.s_d == self.s_dv and self.s_d % 16 == 0 and 16 <= self.s_d <= 256 and self.s_scale > 0

    def cache_need(self):
        return KVNeed(self.s_nkv, self.s_d, self.s_window, None if self.s_dv == self.s_d else self.s_dv,
                      keep_first=self.s_keep)

    def plan_needs(self):
        tiles = {ops.ATTENTION_TILE_TOKENS}
        tiles |= ops.rows_attention_tile_sizes(self.s_nq, self.s_nkv, self.s_d, self.s_dv, False)
        if self._tensor_core_sizes():
            tiles |= set(ops.attention_tile_sizes(self.s_nq // self.s_nkv))
        return PlanNeeds(frozenset(tiles))

    def _attend(self, q, out, cache, ctx) -> None:
        """``q [M, nq * d]`` contiguous, ``out [M, nq * dv]``.  bfloat16 with sizes the tensor-core kernels take:
        those kernels (balanced decode, tcgen05 or mma.sync for prompt portions); else the kernel for keys and
        values of two sizes or the CUDA-core kernel."""
        args = dict(window=self.s_window or 0, keep_first=self.s_keep, softcap=self.s_cap)
        if q.dtype == torch.bfloat16 and self._tensor_core_sizes() and out.is_contiguous():
            ops.attention(q, q.stride(0), out, cache, ctx, self.s_nq, self.s_nkv, self.s_d, self.s_scale, **args)
        else:
            ops.attention_ext(q, out, cache, ctx, self.s_nq, self.s_nkv, self.s_d, self.s_dv, self.s_scale, **args)

    def _stack_in(self, tensors, names, dtype) -> torch.Tensor:
        """The named matrices on top of one another, padded with rows of zeros to a multiple of 8 (aligned rows of
        the product)."""
        rows = [_as_compute(tensors[n], dtype) for n in names]
        pad = self.in_width - sum(r.shape[0] for r in rows)
        if pad:
            rows.append(torch.zeros((pad, rows[0].shape[1]), dtype=dtype, device=rows[0].device))
        return torch.cat(rows, dim=0).contiguous()


class ConvAttention(PagedSoftmax):
    """Grouped attention (``num_heads`` query heads over ``num_kv_heads`` key/value heads, keys of ``head_dim``,
    values of ``value_dim``) whose projected queries, keys and values each pass a causal convolution per channel
    over ``conv_taps`` tokens (the last tap meets the current token; zeros before the start), and whose queries
    and keys are then rotated (a ``RotaryPosition``, half layout, or none).  ``window`` and ``keep_first`` as in
    ``PagedSoftmax``; the score is ``q . k * scale``.  The state (fp32, per request) is the last ``conv_taps - 1``
    projected rows of q, k and v, oldest first.

    params: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``scale``, ``conv_taps`` (1 to 16);
    optional ``value_dim`` (default ``head_dim``), ``window``, ``keep_first``, ``softcap``.
    tensors: ``q``, ``k``, ``v``, ``q.conv``, ``k.conv``, ``v.conv`` (``[channels, conv_taps]``), ``o``.
    """

    def __init__(self, spec):
        super().__init__(spec)
        g = self.spec.params.get
        self.hidden = int(self.param("hidden_size"))
        self.nq, self.nkv, self.d = (int(self.param(n)) for n in ("num_heads", "num_kv_heads", "head_dim"))
        self.dv = int(g("value_dim") or self.d)
        self.taps = int(self.param("conv_taps"))
        if not 1 <= self.taps <= ops.CONV_STORE_MAX_TAPS:
            raise ValueError(f"{self.taps} convolution taps (1 to {ops.CONV_STORE_MAX_TAPS} are taken)")
        self._softmax_sizes(self.nq, self.nkv, self.d, self.dv, float(self.param("scale")),
                            int(g("window")) if g("window") else None, int(g("keep_first") or 0),
                            float(g("softcap") or 0.0))
        self.channels = (self.nq + self.nkv) * self.d + self.nkv * self.dv
        self.in_width = -(-self.channels // 8) * 8
        self.out_width = self.nq * self.dv

    def param_decls(self):
        H, rows = self.hidden, {"q": self.nq * self.d, "k": self.nkv * self.d, "v": self.nkv * self.dv}
        decls = {n: ParamDecl((r, H)) for n, r in rows.items()}
        decls.update({n + ".conv": ParamDecl((r, self.taps), "table") for n, r in rows.items()})
        decls["o"] = ParamDecl((H, self.nq * self.dv))
        return decls

    def state_need(self):
        return StateNeed(((self.taps - 1) * self.channels,), torch.float32) if self.taps > 1 else None

    def bind(self, tensors, dtype, device):
        self.w_in = self._stack_in(tensors, ("q", "k", "v"), dtype)
        self.w_out = _as_compute(tensors["o"], dtype).contiguous()
        self.conv_w = torch.cat([_f32(tensors[n]) for n in ("q.conv", "k.conv", "v.conv")], dim=0).t().contiguous()
        self.finish_bind()

    def mix(self, proj, out, out_scale, ctx, cache, position):
        rot, _ = _half_rotation(position, self.d)
        q = torch.empty((ctx.n_tokens, self.nq * self.d), dtype=proj.dtype, device=proj.device)
        ops.conv_rope_store(proj, q, self.conv_w, cache.state, ctx, self.nq, self.nkv, self.d, self.dv, rot=rot,
                            angles=position.step_angles(ctx) if rot else None,
                            slots=ctx.groups[cache.group].slots, kcache=cache.k, vcache=cache.v)
        heads = out
        if out_scale != 1.0:
            heads = torch.empty((ctx.n_tokens, self.out_width), dtype=proj.dtype, device=proj.device)
        self._attend(q, heads, cache, ctx)
        if heads is not out:
            ops.gate_mul(heads, None, out, None, out_scale)


class DifferentialAttention(PagedSoftmax):
    """Two attentions per head over the same values, the second taken off the first.  ``W_q`` has ``num_heads * 2 *
    head_dim`` rows and ``W_k`` ``num_kv_heads * 2 * head_dim``, head by head the first map, then the second; with
    ``temp_coef`` the queries of position ``p`` are multiplied by ``1 + temp_coef ln(floor((p + 1) / temp_every) +
    1)``.  Each map is a causal softmax of its own (``scale``, ``softcap``, optional ``window`` and ``keep_first``, see
    ``PagedSoftmax``).  With ``lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff`` a head's output is ``a1 - lam a2``,
    divided by its root mean square over ``value_dim``, times ``1 - diff`` and, with ``head_gate``, times
    ``sigmoid(W_g h)``, one number per head.

    Both maps of a key lie in one cache row, ``[k1, k2]`` (zeros up to a multiple of 16), and a query of the first
    map is stored as ``[q1, 0]``, of the second as ``[0, q2]``: the attention kernels see ``2 num_heads`` ordinary
    query heads, keys and values are read once for both maps, and the zeros change no score.

    params: ``hidden_size``, ``num_heads``, ``num_kv_heads``, ``head_dim``, ``scale``, ``diff``, ``eps``; optional
    ``value_dim`` (default ``2 head_dim``), ``softcap``, ``temp_coef``, ``temp_every``, ``window``, ``keep_first``,
    ``head_gate`` (default False).
    tensors: ``q``, ``k``, ``v``, ``o``, ``lq1``, ``lk1``, ``lq2``, ``lk2`` and, with the gate, ``g``.
    """

    def __init__(self, spec):
        super().__init__(spec)
        g = self.spec.params.get
        self.hidden = int(self.param("hidden_size"))
        self.nq, self.nkv, self.d = (int(self.param(n)) for n in ("num_heads", "num_kv_heads", "head_dim"))
        self.dv = int(g("value_dim") or 2 * self.d)
        self.diff, self.eps = float(self.param("diff")), float(self.param("eps"))
        self.temp_coef, self.temp_every = float(g("temp_coef") or 0.0), int(g("temp_every") or 1)
        self.head_gate = bool(g("head_gate", False))
        if self.nq % self.nkv:
            raise ValueError(f"{self.nq} query heads cannot share {self.nkv} key/value heads")
        self.row = -(-2 * self.d // 16) * 16        # a key's two maps in the cache
        self._softmax_sizes(2 * self.nq, self.nkv, self.row, self.dv, float(self.param("scale")),
                            int(g("window")) if g("window") else None, int(g("keep_first") or 0),
                            float(g("softcap") or 0.0))
        self.k_off = 2 * self.nq * self.d
        self.v_off = self.k_off + 2 * self.nkv * self.d
        self.g_off = self.v_off + self.nkv * self.dv
        self.in_width = -(-(self.g_off + (self.nq if self.head_gate else 0)) // 8) * 8
        self.out_width = self.nq * self.dv

    def param_decls(self):
        H, d = self.hidden, self.d
        decls = {"q": ParamDecl((2 * self.nq * d, H)), "k": ParamDecl((2 * self.nkv * d, H)),
                 "v": ParamDecl((self.nkv * self.dv, H)), "o": ParamDecl((H, self.nq * self.dv))}
        decls.update({n: ParamDecl((d,), "table") for n in ("lq1", "lk1", "lq2", "lk2")})
        if self.head_gate:
            decls["g"] = ParamDecl((self.nq, H))
        return decls

    def bind(self, tensors, dtype, device):
        self.w_in = self._stack_in(tensors, ["q", "k", "v"] + (["g"] if self.head_gate else []), dtype)
        self.w_out = _as_compute(tensors["o"], dtype).contiguous()
        a, b, c, d = (tensors[n].to(torch.float64) for n in ("lq1", "lk1", "lq2", "lk2"))
        self.lam = float(torch.exp((a * b).sum()) - torch.exp((c * d).sum()) + self.diff)
        self.finish_bind()

    def mix(self, proj, out, out_scale, ctx, cache, position):
        if position is not None:
            raise ValueError("this mixer takes no position part")
        M, nq = ctx.n_tokens, self.nq
        q = torch.empty((M, 2 * nq * self.row), dtype=proj.dtype, device=proj.device)
        ops.split_maps_store(proj, q, self.k_off, self.v_off, nq, self.nkv, self.d, self.row, self.dv,
                             positions=ctx.positions, temp_coef=self.temp_coef, temp_every=self.temp_every,
                             slots=ctx.groups[cache.group].slots, kcache=cache.k, vcache=cache.v)
        heads = torch.empty((M, 2 * nq * self.dv), dtype=proj.dtype, device=proj.device)
        self._attend(q, heads, cache, ctx)
        gate = proj[:, self.g_off:self.g_off + nq] if self.head_gate else None
        ops.combine_maps(heads, gate, out, nq, self.dv, self.lam, self.eps, (1.0 - self.diff) * out_scale)


register_mixer("conv_attention", ConvAttention, replace=True)
register_mixer("differential_attention", DifferentialAttention, replace=True)
