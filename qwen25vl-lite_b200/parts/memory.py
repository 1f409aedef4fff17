"""Mixers that keep a matrix memory per head, with gates that depend on the token.

The first two read ``q = Wq h * dim^(-1/2)``, ``k = Wk h`` (heads x dim), ``v = Wv h`` (heads x value_dim) and carry, per head
and request, a float32 state ``S`` [dim, value_dim] from token to token: ``S_t = diag(a_t) S_(t-1) + b_t k_t v_t^T``,
``o_t = S_t^T q_t``.

* ``gated_linear_attention`` (Yang, Wang, Shen, Panda, Kim, "Gated Linear Attention Transformers with
  Hardware-Efficient Training"): a decay per key channel from a low-rank projection,
  ``a_t = sigmoid(Wa2 (Wa1 h) + ba2) ** (1 / tau)``, ``b_t = 1``.  Each head's ``o`` is RMS-normed over its
  ``value_dim`` channels with one weight shared by the heads, the heads are concatenated, multiplied by
  ``silu(Wg h)`` and projected by ``Wo``.
* ``mlstm`` (Beck, Poeppel, Spanring, Auer, Prudnikova, Kopp, Klambauer, Brandstetter, Hochreiter, "xLSTM: Extended
  Long Short-Term Memory"): per head the logarithm of an input gate ``i = cap tanh((Wi h + bi) / cap)`` and of a
  forget gate ``f = log sigmoid(cap tanh((Wf h + bf) / cap))``; with a running maximum ``m_t = max(f + m_(t-1), i)``
  (``m_0 = 0``), ``a_t = exp(f + m_(t-1) - m_t)``, ``b_t = exp(i - m_t)``; a normaliser ``n_t = a_t n_(t-1) + b_t k_t``;
  ``o_t`` is divided by ``max(|n_t . q_t|, exp(-m_t)) + 1e-6``, then by its root mean square per head, the heads are
  concatenated, multiplied by a weight over all heads' channels and by ``sigmoid(Wg h)``, and projected by ``Wo``.
* ``mamba2`` (Dao, Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space
  Duality"): ``[z | x | B | C | d] = Wi h``; x, B and C pass a causal convolution per channel with bias and silu; per head
  a step ``d_t = softplus(d + bias)``, ``a_t = exp(-exp(A_log) d_t)`` for every channel, ``b_t = d_t``, k = B and q = C
  shared by groups of consecutive heads, v = x; ``y_t = o_t + D x_t``, the heads are concatenated, multiplied by
  ``silu(z)``, RMS-normed in equal parts with a weight over all channels, and projected by ``Wo``.  The state keeps the
  convolution's last inputs beside S.
* ``gated_delta_rule`` (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"): q, k and v pass
  a short causal convolution and silu, q and k become unit vectors per head; per head a decay
  ``a_t = exp(-exp(A_log) softplus(Wa h + dt_bias))`` and a write strength ``beta_t = sigmoid(Wb h)``; the memory is told the
  difference between a value and what it would answer, ``S <- a_t S``, ``S <- S + k_t (beta_t (v_t - S^T k_t))^T``,
  ``o_t = S^T q_t``; each head's o is RMS-normed with one weight shared by the heads, multiplied by ``silu(Wg h)`` and
  projected by ``Wo``.

Float32 in both dtypes: the decays and gates from their pre-activations on (the gate rows of ``mlstm`` and the second
factor of the decay's projection are float32 products in a fixed order; the steps of ``mamba2`` leave their product in
float32), S, n, m, o and the norms.  The state is zero
at admission, so a run of tokens may be cut anywhere.  Single tokens and short runs are walked token by token; a
long run is cut into chunks that are walked in parallel, twice, with a fold over the chunks' sums in between
(``plan_step``).  Kernels: ``csrc/gated_memory.cu``.
"""

from __future__ import annotations

import numpy as np
import torch

from ..ops import delta_rule, kernels, state_space
from ..ops.linear import DeferredNorm, Linear
from .base import Mixer, StateNeed, TensorSpec, register_mixer


class _MatrixMemory(Mixer):
    graph_safe = True                # forward is a fixed sequence of this engine's kernels
    accepts_residual = True          # the output projection can add into the residual stream itself

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, norm_eps: float, position=None):
        self.hidden_size, self.num_heads, self.head_dim, self.value_dim = int(hidden_size), int(num_heads), int(head_dim), int(value_dim)
        if not 0 < self.head_dim <= 512:
            raise ValueError(f"a memory's key size is 1 to 512, got {head_dim}")
        self.norm_eps = float(norm_eps)
        self.in_proj = self.o_proj = self.norm_weight = None

    def _sizes(self):
        return self.hidden_size, self.num_heads * self.head_dim, self.num_heads * self.value_dim

    def plan_key(self):
        return ("matrix_memory",)             # the chunks of a step's long runs do not depend on a layer's sizes

    def plan_step(self, host):
        first, runs, second = kernels.plan_memory(host.q_lens)
        return {name: np.asarray(a, dtype=np.int32).reshape(-1) for name, a in (("first", first), ("runs", runs), ("second", second))}

    def _scan(self, ctx, x, decay, gates, cap, stop, o_raw, m_exp):
        H, D, Dv = self.num_heads, self.head_dim, self.value_dim
        plan = ctx.plan(self)
        if plan.get("first") is None:
            kernels.memory_scan(x, 0, H * D, 2 * H * D, decay, gates, cap, float(D) ** -0.5, stop.state, ctx.cu_q, ctx.slot_ids, o_raw, m_exp,
                                ctx.n_seqs, H, D, Dv)
        else:
            kernels.memory_scan_chunked(x, 0, H * D, 2 * H * D, decay, gates, cap, float(D) ** -0.5, stop.state, ctx.slot_ids, o_raw, m_exp,
                                        plan["first"], plan["runs"], plan["second"], H, D, Dv)

    def _common_specs(self):
        h, qk, v = self._sizes()
        return [TensorSpec("q", (qk, h)), TensorSpec("k", (qk, h)), TensorSpec("v", (v, h)), TensorSpec("g", (v, h)),
                TensorSpec("o", (h, v))]

    def _load_common(self, tensors, device, dtype, more=()):
        w = torch.cat([tensors["q"], tensors["k"], tensors["v"], tensors["g"], *more], dim=0)
        self.in_proj = Linear(w.to(device=device, dtype=dtype).contiguous())
        self.o_proj = Linear(tensors["o"].to(device=device, dtype=dtype).contiguous())


@register_mixer("gated_linear_attention")
class GatedLinearAttention(_MatrixMemory):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, tau: float, norm_eps: float,
                 decay_rank: int = None, position=None):
        """``decay_rank``: the inner size of the decay's two factors; None: whatever the checkpoint's ``a1`` has."""
        super().__init__(hidden_size, num_heads, head_dim, value_dim, norm_eps)
        self.decay_rank, self.tau = -1 if decay_rank is None else int(decay_rank), float(tau)
        if self.decay_rank == 0 or self.decay_rank < -1 or not self.tau > 0.0:
            raise ValueError(f"the decay's projection has a rank of at least 1 and tau is positive, got {decay_rank} and {tau}")

    def tensor_specs(self):
        h, qk, _ = self._sizes()
        return tuple(self._common_specs() + [TensorSpec("norm", (self.value_dim,), "norm"), TensorSpec("a1", (self.decay_rank, h), "matrix_wide"),
                                             TensorSpec("a2", (qk, self.decay_rank), "matrix_wide"), TensorSpec("a2.b", (qk,), "bias")])

    def state_need(self):
        return StateNeed((self.num_heads, self.head_dim, self.value_dim), "float32")

    def load(self, tensors, device, dtype):
        self.decay_rank = int(tensors["a1"].shape[0])
        if tensors["a2"].shape[1] != self.decay_rank:
            raise ValueError(f"the decay's factors do not fit: a1 has {self.decay_rank} rows, a2 {tensors['a2'].shape[1]} columns")
        self._load_common(tensors, device, dtype, (tensors["a1"],))
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        self.a2t = f32(tensors["a2"].t())                                  # [rank, heads * dim]
        self.a2_bias = f32(tensors["a2.b"])
        self.norm_weight = f32(tensors["norm"]).repeat(self.num_heads).contiguous()      # the same for every head

    def forward(self, ctx, h, stop, residual=None):
        H, D, Dv = self.num_heads, self.head_dim, self.value_dim
        n = h.shape[0]
        x = self.in_proj(h)                                             # [N, q | k | v | g | low]
        decay = torch.empty((n, H * D), dtype=torch.float32, device=x.device)
        kernels.gla_decay(x, 2 * H * D + 2 * H * Dv, self.decay_rank, self.a2t, self.a2_bias, self.tau, decay)
        o_raw = torch.empty((n, H, Dv), dtype=torch.float32, device=x.device)
        self._scan(ctx, x, decay, None, 0.0, stop, o_raw, None)
        out = torch.empty((n, H * Dv), dtype=x.dtype, device=x.device)
        kernels.memory_output(o_raw, None, x, 2 * H * D + H * Dv, self.norm_weight, self.norm_eps, "silu", out, H, Dv)
        return self.o_proj(out, residual=residual)


@register_mixer("mlstm")
class MLSTM(_MatrixMemory):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, gate_cap: float, norm_eps: float, position=None):
        super().__init__(hidden_size, num_heads, head_dim, value_dim, norm_eps)
        self.gate_cap = float(gate_cap or 0.0)
        if self.num_heads > 128:
            raise ValueError(f"the gates' kernel takes up to 128 heads, got {num_heads}")

    def tensor_specs(self):
        h, _, v = self._sizes()
        H = self.num_heads
        return tuple(self._common_specs() + [TensorSpec("norm", (v,), "norm"), TensorSpec("i", (H, h), "matrix_wide"), TensorSpec("i.b", (H,), "bias"),
                                             TensorSpec("f", (H, h), "matrix_wide"), TensorSpec("f.b", (H,), "bias")])

    def state_need(self):
        # one more column (the normaliser) and one more row (the running maximum, a copy in every column)
        return StateNeed((self.num_heads, self.head_dim + 1, self.value_dim + 1), "float32")

    def load(self, tensors, device, dtype):
        self._load_common(tensors, device, dtype)
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        self.gate_rows = f32(torch.cat([tensors["i"], tensors["f"]], dim=0))       # [2 heads, hidden]
        self.gate_bias = f32(torch.cat([tensors["i.b"], tensors["f.b"]], dim=0))
        self.norm_weight = f32(tensors["norm"])

    def forward(self, ctx, h, stop, residual=None):
        H, D, Dv = self.num_heads, self.head_dim, self.value_dim
        n = h.shape[0]
        x = self.in_proj(h)                                             # [N, q | k | v | g]
        gates = torch.empty((n, 2 * H), dtype=torch.float32, device=x.device)
        kernels.row_dots(h, self.gate_rows, self.gate_bias, gates)
        o_raw = torch.empty((n, H, Dv + 1), dtype=torch.float32, device=x.device)
        m_exp = torch.empty((n, H), dtype=torch.float32, device=x.device)
        self._scan(ctx, x, None, gates, self.gate_cap, stop, o_raw, m_exp)
        out = torch.empty((n, H * Dv), dtype=x.dtype, device=x.device)
        kernels.memory_output(o_raw, m_exp, x, 2 * H * D + H * Dv, self.norm_weight, self.norm_eps, "sigmoid", out, H, Dv)
        return self.o_proj(out, residual=residual)


@register_mixer("mamba2")
class Mamba2(Mixer):
    graph_safe = True                # forward is a fixed sequence of this engine's kernels
    accepts_residual = True          # the output projection can add into the residual stream itself

    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state_dim: int, groups: int, conv: int, norm_groups: int,
                 norm_eps: float, position=None):
        self.hidden_size, self.num_heads, self.value_dim, self.state_dim = int(hidden_size), int(num_heads), int(value_dim), int(state_dim)
        self.groups, self.conv, self.norm_groups, self.norm_eps = int(groups), int(conv), int(norm_groups), float(norm_eps)
        self.inner = self.num_heads * self.value_dim
        self.channels = self.inner + 2 * self.groups * self.state_dim      # what the convolution runs over: x | B | C
        if self.groups < 1 or self.num_heads % self.groups:
            raise ValueError(f"{num_heads} heads cannot share {groups} groups of B and C")
        if self.norm_groups < 1 or self.inner % self.norm_groups:
            raise ValueError(f"a norm over {self.inner} channels cannot be cut into {norm_groups} equal parts")
        if not 0 < self.state_dim <= 512:
            raise ValueError(f"a state has 1 to 512 rows, got {state_dim}")
        if not 1 <= self.conv <= 16:
            raise ValueError(f"the convolution takes 1 to 16 taps, got {conv}")
        self.in_proj = self.step_proj = self.out_proj = None

    def tensor_specs(self):
        h, H, c = self.hidden_size, self.num_heads, self.channels
        return (TensorSpec("in", (self.inner + c + H, h)), TensorSpec("conv", (c, self.conv), "matrix_wide"), TensorSpec("conv.b", (c,), "bias"),
                TensorSpec("dt_bias", (H,), "bias"), TensorSpec("A_log", (H,), "bias"), TensorSpec("D", (H,), "norm"),
                TensorSpec("norm", (self.inner,), "norm"), TensorSpec("o", (h, self.inner)))

    @property
    def _memory_floats(self) -> int:
        return self.num_heads * self.state_dim * self.value_dim

    def state_need(self):
        # S [heads, state, value_dim], then the last conv - 1 inputs of the convolution [conv - 1, channels]
        return StateNeed((self._memory_floats + (self.conv - 1) * self.channels,), "float32")

    @property
    def _tensor_cores(self) -> bool:
        """Whether this mixer's runs of tokens can go to the tensor-core kernel."""
        return self.out_proj is not None and kernels.state_space_mma_supports(self.out_proj.weight.dtype, self.num_heads, self.groups, self.state_dim,
                                                                              self.value_dim)

    def plan_key(self):
        return ("state_space",) if self._tensor_cores else ("matrix_memory",)

    def plan_step(self, host):
        return state_space.plan(host.q_lens, self._tensor_cores)

    def load(self, tensors, device, dtype):
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        w = tensors["in"]
        rows = self.inner + self.channels
        # the steps' rows are a product of their own, whose result stays in float32
        self.in_proj = Linear(w[:rows].to(device=device, dtype=dtype).contiguous())
        self.step_proj = Linear(w[rows:].to(device=device, dtype=dtype).contiguous())
        self.out_proj = Linear(tensors["o"].to(device=device, dtype=dtype).contiguous())
        self.conv_w, self.conv_b = f32(tensors["conv"].t()), f32(tensors["conv.b"])            # [taps, channels]
        self.step_bias, self.rate_log, self.skip, self.norm_weight = (f32(tensors[n]) for n in ("dt_bias", "A_log", "D", "norm"))

    def forward(self, ctx, h, stop, residual=None):
        n, inner, ch = h.shape[0], self.inner, self.channels
        zx = self.in_proj(h)                                            # [N, z | x | B | C]
        steps = self.step_proj(h, out_dtype=torch.float32)              # [N, heads]
        xbc = torch.empty((n, ch), dtype=zx.dtype, device=zx.device)
        kernels.causal_conv(zx[:, inner:], self.conv_w, self.conv_b, stop.state, self._memory_floats, ctx.cu_q, ctx.slot_ids, xbc, ctx.n_seqs,
                            ctx.max_q_len, silu=True)
        o_raw = torch.empty((n, inner), dtype=torch.float32, device=zx.device)
        state_space.run(ctx.plan(self), ctx, xbc, inner + self.groups * self.state_dim, inner, 0, steps, self.step_bias, self.rate_log, stop.state,
                        o_raw, self.num_heads, self.groups, self.state_dim, self.value_dim)
        out = torch.empty((n, inner), dtype=zx.dtype, device=zx.device)
        kernels.ssd_output(o_raw, xbc[:, :inner], zx[:, :inner], self.skip, self.norm_weight, self.norm_groups, self.norm_eps, out, self.value_dim)
        return self.out_proj(out, residual=residual)


@register_mixer("gated_delta_rule")
class GatedDeltaRule(Mixer):
    """``num_heads`` heads of ``value_dim`` channels over ``num_kv_heads`` query and key heads of ``head_dim`` (head h reads
    number ``h // (num_heads / num_kv_heads)``); ``conv`` taps.  Tensors: ``q``, ``k``, ``v`` with ``.conv`` (no biases), ``a``,
    ``dt_bias``, ``A_log``, ``b``, ``g``, ``norm``, ``o``.  The rows of a and b are a product of their own, whose result stays in
    float32.  A slot's state: S [heads, head_dim, value_dim], then the convolution's last inputs over q | k | v."""

    graph_safe = True                # forward is a fixed sequence of this engine's kernels
    accepts_residual = True          # the output projection can add into the residual stream itself
    accepts_scaled_residual = True
    accepts_deferred_norm = True
    UNIT_EPS = 1e-6                  # inside the root when q and k become unit vectors

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int, conv: int, norm_eps: float, position=None):
        self.hidden_size, self.num_heads, self.num_kv_heads = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.head_dim, self.value_dim, self.conv, self.norm_eps = int(head_dim), int(value_dim), int(conv), float(norm_eps)
        if self.num_kv_heads < 1 or self.num_heads % self.num_kv_heads:
            raise ValueError(f"{num_heads} heads cannot share {num_kv_heads} query and key heads")
        if not 0 < self.head_dim <= 512:
            raise ValueError(f"a memory's key size is 1 to 512, got {head_dim}")
        if not 1 <= self.conv <= 16:
            raise ValueError(f"the convolution takes 1 to 16 taps, got {conv}")
        self.channels = 2 * self.num_kv_heads * self.head_dim + self.num_heads * self.value_dim
        self.in_proj = self.o_proj = self.gate_proj = None

    def tensor_specs(self):
        h, H, qk, v = self.hidden_size, self.num_heads, self.num_kv_heads * self.head_dim, self.num_heads * self.value_dim
        return (TensorSpec("q", (qk, h)), TensorSpec("q.conv", (qk, self.conv), "matrix_wide"), TensorSpec("k", (qk, h)),
                TensorSpec("k.conv", (qk, self.conv), "matrix_wide"), TensorSpec("v", (v, h)), TensorSpec("v.conv", (v, self.conv), "matrix_wide"),
                TensorSpec("b", (H, h), "matrix_wide"), TensorSpec("A_log", (H,), "bias"), TensorSpec("norm", (self.value_dim,), "norm"),
                TensorSpec("a", (H, h), "matrix_wide"), TensorSpec("dt_bias", (H,), "bias"), TensorSpec("g", (v, h)), TensorSpec("o", (h, v)))

    @property
    def _memory_floats(self) -> int:
        return self.num_heads * self.head_dim * self.value_dim

    def state_need(self):
        floats = self._memory_floats + (self.conv - 1) * self.channels
        return StateNeed((-(-floats // 4) * 4,), "float32")              # every slot starts on a 16-byte boundary

    def load(self, tensors, device, dtype):
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        rows = lambda *names: torch.cat([tensors[n] for n in names], dim=0).to(device=device, dtype=dtype).contiguous()
        self.dtype = dtype
        self.in_proj = Linear(rows("q", "k", "v", "g"))
        self.gate_proj = Linear(rows("a", "b"))
        self.o_proj = Linear(rows("o"))
        self.conv_w = f32(torch.cat([tensors[n] for n in ("q.conv", "k.conv", "v.conv")], dim=0).t())              # [taps, channels]
        self.conv_b = torch.zeros(self.channels, dtype=torch.float32, device=device)
        self.rate_log, self.step_bias = f32(tensors["A_log"]), f32(tensors["dt_bias"])
        self.norm_weight = f32(tensors["norm"]).repeat(self.num_heads).contiguous()                               # the same for every head

    def products(self):
        return self.in_proj, self.o_proj

    def drop_products(self):
        self.in_proj = self.o_proj = None

    def scale_heads(self, factor: float):
        """The heads times a constant: it rides in the output norm's float32 weight."""
        self.norm_weight = (self.norm_weight * factor).contiguous()

    @property
    def _tensor_cores(self) -> bool:
        """Whether this mixer's runs of tokens can go to the tensor-core kernels."""
        return kernels.delta_mma_supports(getattr(self, "dtype", torch.float32), self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim)

    def plan_key(self):
        return ("delta_rule", self._tensor_cores)

    def plan_step(self, host):
        return delta_rule.plan(host.q_lens, self._tensor_cores)

    def side_products(self, ctx, h):
        return self.gate_proj(h, out_dtype=torch.float32)               # [N, a of every head | b of every head]

    def between(self, ctx, x, stop, side=None, out=None):
        """``x``: rows q | k | v | g as projected."""
        H, G, D, Dv, n = self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim, x.shape[0]
        state = stop.state
        qkv = torch.empty((n, self.channels), dtype=x.dtype, device=x.device)
        kernels.causal_conv(x[:, :self.channels], self.conv_w, self.conv_b, state, self._memory_floats, ctx.cu_q, ctx.slot_ids, qkv, ctx.n_seqs,
                            ctx.max_q_len, silu=True)
        if out is None:
            out = torch.empty((n, H * Dv), dtype=x.dtype, device=x.device)
        delta_rule.run(ctx.plan(self), ctx, qkv, side, self.step_bias, self.rate_log, state, x[:, self.channels:], self.norm_weight, self.norm_eps, out,
                       H, G, D, Dv, float(D) ** -0.5, self.UNIT_EPS)
        return out

    def forward(self, ctx, h, stop, residual=None, residual_scale=None):
        if isinstance(h, DeferredNorm) and not kernels.gemm_skinny_norm_supports(h.x, self.in_proj.weight):
            h = h.materialize()
        x = self.in_proj(h)
        return self.o_proj(self.between(ctx, x, stop, side=self.side_products(ctx, h)), residual=residual, residual_scale=residual_scale)
