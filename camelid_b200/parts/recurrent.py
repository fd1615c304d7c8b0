"""Mixers that keep a matrix state S [key_dim, value_dim] per head and sequence instead of keys
and values. The state is float32, starts at zero and is carried from token to token; gates,
decays, unit norms and the read-out norm are float32 as well.

``matrix_memory``: per head, with q = x Wq^T / sqrt(key_dim), k, v and capped log gates
i = cap tanh((x Wi^T + bi) / cap), f = logsigmoid(cap tanh((x Wf^T + bf) / cap)):

    m' = max(f + m, i)          (m starts at 0)
    S' = e^(f + m - m') S + e^(i - m') k v^T,   n' likewise with k alone
    o  = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6)

then o / rms(o) per head, times ``norm`` (all heads' size), times sigmoid(x Wg^T), then Wo.
Tensors: ``q k v g o i i.b f f.b norm``.

``channel_delta``: the gated delta rule with a decay per head and key channel. q, k
(``num_qk_heads`` heads, shared by groups of value heads) and v pass a short causal
convolution per channel (``<name>.conv`` [channels, taps], the last tap the current token's)
and SiLU; q and k become unit vectors (x / sqrt(sum x^2 + 1e-6)), q also times
1 / sqrt(key_dim); beta = sigmoid(x Wb^T); g = exp(-exp(A_log[head]) softplus(Wa2 (Wa1 x) + dt_bias)):

    S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

then o / rms(o) per head times ``norm`` (value_dim, shared), times sigmoid(Wg2 (Wg1 x)), then
Wo. The last taps - 1 inputs of the convolution are state too. Tensors:
``q q.conv k k.conv v v.conv b A_log dt_bias a1 a2 g1 g2 norm o``; the width of the two
low-rank pairs is the stored tensors' own.

``gated_delta``: the same rule with one decay per head, g = exp(-exp(A_log[head]) softplus(Wa x + dt_bias[head])) (S <- g S),
the decay's and the gate's inputs straight from the mixer's input (``a`` [heads, hidden], ``g`` [heads x value_dim, hidden])
and a SiLU gate on the read-out. Both are one part with three options: ``decay`` "channel" | "head", ``low_rank`` (the
pairs a1/a2, g1/g2 or the plain matrices a, g) and ``gate`` "sigmoid" | "silu".
"""
from __future__ import annotations

import math

import torch

from ..cache.book import StateSpec
from ..config.plan import PartSpec
from ..csrc import ops
from ..errors import ConfigError, WeightsError
from . import linear
from .base import Part, TensorSpec, build_part, register_part, to_device


def _check_dims(key_dim: int, value_dim: int):
    if not 1 <= key_dim <= 256:
        raise ConfigError("key_dim", f"the scan kernels take key sizes 1..256, got {key_dim}")
    if value_dim < 1:
        raise ConfigError("value_dim", f"must be greater than zero, got {value_dim}")


@register_part("mixer", "matrix_memory")
class MatrixMemory(Part):
    graph_safe = True
    graph_safe_any_step = True

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden_size = int(params["hidden_size"])
        self.eps = float(params.get("eps", 1e-6))
        self.num_heads = int(params["num_heads"])
        self.key_dim = int(params["key_dim"])
        self.value_dim = int(params["value_dim"])
        self.gate_cap = float(params["gate_cap"])
        _check_dims(self.key_dim, self.value_dim)
        self.qk_width = self.num_heads * self.key_dim
        self.v_width = self.num_heads * self.value_dim
        # columns of the stacked input projection: q, k, v, output gate, input gate, forget gate
        self.cols = (0, self.qk_width, 2 * self.qk_width, 2 * self.qk_width + 2 * self.v_width,
                     2 * self.qk_width + 2 * self.v_width + self.num_heads)
        self.gate_col = 2 * self.qk_width + self.v_width
        self.w_in = self.w_o = self.i_bias = self.f_bias = self.norm_w = None

    def tensor_specs(self):
        p, hid, h = self.prefix, self.hidden_size, self.num_heads
        return {p + "q": TensorSpec((self.qk_width, hid)), p + "k": TensorSpec((self.qk_width, hid)),
                p + "v": TensorSpec((self.v_width, hid)), p + "g": TensorSpec((self.v_width, hid)),
                p + "o": TensorSpec((hid, self.v_width)), p + "norm": TensorSpec((self.v_width,), "norm"),
                p + "i": TensorSpec((h, hid)), p + "i.b": TensorSpec((h,), "input_bias"),
                p + "f": TensorSpec((h, hid)), p + "f.b": TensorSpec((h,), "forget_bias")}

    def load(self, tensors, device, dtype):
        p = self.prefix
        self.w_in = torch.cat([to_device(tensors[p + n], device, dtype) for n in ("q", "k", "v", "g", "i", "f")], 0).contiguous()
        self.w_o = to_device(tensors[p + "o"], device, dtype)
        f32 = lambda n: tensors[p + n].to(device=device, dtype=torch.float32).contiguous()      # noqa: E731
        self.i_bias, self.f_bias, self.norm_w = f32("i.b"), f32("f.b"), f32("norm")

    def cache_spec(self):
        # S column by column with n as one more column; the running maximum, one copy per column
        return [StateSpec((self.num_heads, self.value_dim + 1, self.key_dim), "float32", "memory"),
                StateSpec((self.num_heads, self.value_dim + 1), "float32", "maximum")]

    def read_out(self, ctx, x, proj=None):
        n = ctx.n_rows
        if proj is None:
            proj = linear.product_rows_f32(ctx, x, self.w_in, "mm_proj")
        raw = ctx.buffer("mm_raw", (n, self.num_heads, self.value_dim + 2), torch.float32)
        ops.memory_scan(proj, self.cols, self.i_bias, self.f_bias, self.gate_cap, self.key_dim ** -0.5, ctx.state("memory"),
                        ctx.state("maximum"), ctx.seq_row0, ctx.seq_new, ctx.seq_start, ctx.seq_slot, raw, ctx.n_seqs, self.num_heads,
                        self.key_dim, self.value_dim)
        out = ctx.buffer("mm_out", (n, self.v_width))
        ops.head_norm_gate(raw, True, self.norm_w, True, proj, self.gate_col, out, self.num_heads, self.value_dim, self.eps)
        return out

    def forward(self, ctx, x, residual):
        linear.add_into_residual(ctx, self.read_out(ctx, x), self.w_o, residual, "o_partial")

    def branch_output(self, ctx, x, name: str, proj=None):
        return linear.product_f32(ctx, self.read_out(ctx, x, proj), self.w_o, name)


@register_part("mixer", "channel_delta")
class ChannelDelta(Part):
    graph_safe = True
    graph_safe_any_step = True
    default_decay, default_gate, default_low_rank = "channel", "sigmoid", True

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden_size = int(params["hidden_size"])
        self.eps = float(params.get("eps", 1e-6))
        self.num_heads = int(params["num_heads"])
        self.num_qk_heads = int(params.get("num_qk_heads") or self.num_heads)
        self.key_dim = int(params["key_dim"])
        self.value_dim = int(params["value_dim"])
        self.taps = int(params["conv_taps"])
        _check_dims(self.key_dim, self.value_dim)
        if self.num_qk_heads <= 0 or self.num_heads % self.num_qk_heads:
            raise ConfigError("num_qk_heads", f"{self.num_qk_heads} q/k heads do not divide {self.num_heads} heads")
        if self.taps < 1:
            raise ConfigError("conv_taps", f"must be at least 1, got {self.taps}")
        self.decay = params.get("decay") or self.default_decay
        self.gate = params.get("gate") or self.default_gate
        self.low_rank = bool(params["low_rank"]) if params.get("low_rank") is not None else self.default_low_rank
        if self.decay not in ("channel", "head"):
            raise ConfigError("decay", f"one decay per key 'channel' or per 'head', got {self.decay!r}")
        if self.gate not in ("sigmoid", "silu"):
            raise ConfigError("gate", f"unknown read-out gate {self.gate!r}; known: sigmoid, silu")
        # the low-rank width is the stored tensors' own; this one is for random weights
        self.rank = int(params.get("rank") or max(8, self.hidden_size // 8 // 8 * 8))
        self.qk_width = self.num_qk_heads * self.key_dim
        self.v_width = self.num_heads * self.value_dim
        self.decay_width = self.num_heads * (self.key_dim if self.decay == "channel" else 1)
        self.channels = 2 * self.qk_width + self.v_width
        self.w_in = self.w_low = self.w_high = self.w_o = None
        self.conv_w = self.a_log = self.dt_bias = self.norm_w = None

    def tensor_specs(self):
        p, hid, r = self.prefix, self.hidden_size, self.rank
        specs = {p + "q": TensorSpec((self.qk_width, hid)), p + "q.conv": TensorSpec((self.qk_width, self.taps), "conv"),
                 p + "k": TensorSpec((self.qk_width, hid)), p + "k.conv": TensorSpec((self.qk_width, self.taps), "conv"),
                 p + "v": TensorSpec((self.v_width, hid)), p + "v.conv": TensorSpec((self.v_width, self.taps), "conv"),
                 p + "b": TensorSpec((self.num_heads, hid)), p + "A_log": TensorSpec((self.num_heads,), "log_rate"),
                 p + "dt_bias": TensorSpec((self.decay_width,), "log_rate"), p + "norm": TensorSpec((self.value_dim,), "norm"),
                 p + "o": TensorSpec((hid, self.v_width))}
        if self.low_rank:
            specs.update({p + "a1": TensorSpec((r, hid), "linear", (0,)), p + "a2": TensorSpec((self.decay_width, r), "low_rank", (1,)),
                          p + "g1": TensorSpec((r, hid), "linear", (0,)), p + "g2": TensorSpec((self.v_width, r), "low_rank", (1,))})
        else:
            specs.update({p + "a": TensorSpec((self.decay_width, hid)), p + "g": TensorSpec((self.v_width, hid))})
        return specs

    def load(self, tensors, device, dtype):
        p = self.prefix
        dev = lambda n: to_device(tensors[p + n], device, dtype)                                  # noqa: E731
        f32 = lambda n: tensors[p + n].to(device=device, dtype=torch.float32).contiguous()      # noqa: E731
        self.w_o = dev("o")
        self.conv_w = torch.cat([f32("q.conv"), f32("k.conv"), f32("v.conv")], 0).contiguous()
        self.a_log, self.dt_bias, self.norm_w = f32("A_log"), f32("dt_bias"), f32("norm")
        if not self.low_rank:           # the decays' and the gate's inputs are columns of the one input product
            self.w_in = torch.cat([dev(n) for n in ("q", "k", "v", "b", "a", "g")], 0).contiguous()
            return
        self.w_in = torch.cat([dev(n) for n in ("q", "k", "v", "b")], 0).contiguous()
        a1, a2, g1, g2 = dev("a1"), dev("a2"), dev("g1"), dev("g2")
        wrong = [(p + n, exp, tuple(t.shape)) for n, t, exp in (("a2", a2, (self.decay_width, a1.shape[0])),
                                                                ("g2", g2, (self.v_width, g1.shape[0]))) if tuple(t.shape) != exp]
        if wrong:
            raise WeightsError(wrong_shape=wrong)
        ra, rg = a1.shape[0], g1.shape[0]
        # both low-rank pairs as two products: [a1; g1] x, then a block-diagonal [a2 0; 0 g2]; the inner
        # width is padded with zeros to a multiple of 8 (what the tensor-core product takes)
        inner = (ra + rg + 7) // 8 * 8
        self.w_low = torch.zeros((inner, self.hidden_size), dtype=a1.dtype, device=a1.device)
        self.w_low[:ra], self.w_low[ra:ra + rg] = a1, g1
        self.w_high = torch.zeros((self.decay_width + self.v_width, inner), dtype=a1.dtype, device=a1.device)
        self.w_high[:self.decay_width, :ra] = a2
        self.w_high[self.decay_width:, ra:ra + rg] = g2

    def cache_spec(self):
        return [StateSpec((self.num_heads, self.value_dim, self.key_dim), "float32", "memory"),
                StateSpec((max(self.taps - 1, 1), self.channels), "float32", "conv")]

    def read_out(self, ctx, x):
        n = ctx.n_rows
        proj = linear.product_rows_f32(ctx, x, self.w_in, "cd_proj")
        if self.low_rank:
            low = ctx.buffer("cd_low", (n, self.w_low.shape[0]))
            linear.product_act(ctx, x, self.w_low, low, "cd_low_partial", gelu=False)
            high = linear.product_rows_f32(ctx, low, self.w_high, "cd_high")      # decay inputs, then gate inputs
        else:
            high = proj[:, self.channels + self.num_heads:]                        # the same two, behind q, k, v and beta
        conv_state = ctx.state("conv")
        qkv = ctx.buffer("cd_qkv", (n, self.channels), torch.float32)
        decays = ctx.buffer("cd_decay", (n, self.decay_width), torch.float32)
        ops.conv_unit(proj, self.conv_w, conv_state, ctx.row_seq, ctx.row_pos, ctx.seq_row0, ctx.seq_slot, qkv,
                      self.num_qk_heads, self.num_heads, self.key_dim, self.value_dim, self.key_dim ** -0.5,
                      update_state=ctx.decode, decay=(high[:, :self.decay_width], self.a_log, self.dt_bias, decays))
        if self.taps > 1 and not ctx.decode:
            ops.keep_last_rows(proj, 0, self.channels, conv_state, ctx.seq_row0, ctx.seq_new, ctx.seq_start, ctx.seq_slot,
                               ctx.n_seqs)
        raw = ctx.buffer("cd_raw", (n, self.v_width), torch.float32)
        ops.delta_scan(qkv, proj, self.channels, decays, self.a_log, self.dt_bias, ctx.state("memory"),
                       ctx.seq_row0, ctx.seq_new, ctx.seq_start, ctx.seq_slot, raw, ctx.n_seqs, self.num_heads,
                       self.num_qk_heads, self.key_dim, self.value_dim, decay_ready=True)
        out = ctx.buffer("cd_out", (n, self.v_width))
        ops.head_norm_gate(raw, False, self.norm_w, False, high, self.decay_width, out, self.num_heads, self.value_dim, self.eps,
                           gate_silu=self.gate == "silu")
        return out

    def forward(self, ctx, x, residual):
        linear.add_into_residual(ctx, self.read_out(ctx, x), self.w_o, residual, "o_partial")

    def branch_output(self, ctx, x, name: str, proj=None):
        return linear.product_f32(ctx, self.read_out(ctx, x), self.w_o, name)


@register_part("mixer", "gated_delta")
class GatedDelta(ChannelDelta):
    """The gated delta rule with one decay per head, plain matrices for the decay's and the gate's inputs and a SiLU
    gate on the read-out (each still an option of its own)."""
    default_decay, default_gate, default_low_rank = "head", "silu", False


@register_part("mixer", "retention")
class Retention(Part):
    """Linear attention with a fixed decay per head and no softmax or denominator. q, k (``num_heads`` x ``key_dim``) and v
    (``num_heads`` x ``value_dim``) are plain projections; the first channels of every q and k head are turned by the
    position (``position``: a rotary part), k is then multiplied by key_dim^-1/2;

        S_t = decay[head] S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t

    o is divided by its root mean square per head (no weight), the heads side by side are multiplied by silu(Wg x) (a
    number per channel) and projected by Wo. S is float32 per sequence and head, zero at the start; rotation, scaling,
    the scan and the norm are float32. ``decay``: one number per head. Tensors ``q k v g o``."""
    graph_safe = True
    graph_safe_any_step = True

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden_size = int(params["hidden_size"])
        self.eps = float(params.get("eps", 1e-6))
        self.num_heads = int(params["num_heads"])
        self.key_dim = int(params["key_dim"])
        self.value_dim = int(params["value_dim"])
        _check_dims(self.key_dim, self.value_dim)
        self.decay = tuple(float(d) for d in params["decay"])
        if len(self.decay) != self.num_heads:
            raise ConfigError("decay", f"one decay per head: {self.num_heads} heads, {len(self.decay)} decays")
        self.position = build_part("position", params.get("position") or PartSpec("none"))
        if self.position.rotary_dim > self.key_dim:
            raise ConfigError("rotary_dim", f"{self.position.rotary_dim} exceeds the head size {self.key_dim}")
        self.qk_width = self.num_heads * self.key_dim
        self.v_width = self.num_heads * self.value_dim
        self.cols = (0, self.qk_width, 2 * self.qk_width)            # q, k, v in the stacked product; the gate behind them
        self.gate_col = 2 * self.qk_width + self.v_width
        self.w_in = self.w_o = self.decay_w = None

    def tensor_specs(self):
        p, hid = self.prefix, self.hidden_size
        return {p + "q": TensorSpec((self.qk_width, hid)), p + "k": TensorSpec((self.qk_width, hid)),
                p + "v": TensorSpec((self.v_width, hid)), p + "g": TensorSpec((self.v_width, hid)),
                p + "o": TensorSpec((hid, self.v_width))}

    def load(self, tensors, device, dtype):
        p = self.prefix
        self.w_in = torch.cat([to_device(tensors[p + n], device, dtype) for n in ("q", "k", "v", "g")], 0).contiguous()
        self.w_o = to_device(tensors[p + "o"], device, dtype)
        self.decay_w = torch.tensor(self.decay, dtype=torch.float64).to(torch.float32).to(device)
        self.position.load(tensors, device, dtype)

    def cache_spec(self):
        return StateSpec((self.num_heads, self.value_dim, self.key_dim), "float32", "retention")

    def read_out(self, ctx, x):
        n, pos = ctx.n_rows, self.position
        proj = linear.product_rows_f32(ctx, x, self.w_in, "rt_proj")
        # q and k heads stand side by side: one pass turns both and scales the k heads
        ops.rotate_rows_(proj, 0, 2 * self.num_heads, self.key_dim, pos.rotary_dim, pos.pairing == "interleaved", pos.inv_freq,
                         pos.amplitude, ctx.row_pos, self.num_heads, self.key_dim ** -0.5)
        raw = ctx.buffer("rt_raw", (n, self.v_width), torch.float32)
        ops.retention_scan(proj, self.cols, self.decay_w, ctx.state("retention"), ctx.seq_row0, ctx.seq_new, ctx.seq_start,
                           ctx.seq_slot, raw, ctx.n_seqs, self.num_heads, self.key_dim, self.value_dim)
        out = ctx.buffer("rt_out", (n, self.v_width))
        ops.head_norm_gate(raw, False, None, False, proj, self.gate_col, out, self.num_heads, self.value_dim, self.eps, gate_silu=True)
        return out

    def forward(self, ctx, x, residual):
        linear.add_into_residual(ctx, self.read_out(ctx, x), self.w_o, residual, "o_partial")

    def branch_output(self, ctx, x, name: str, proj=None):
        return linear.product_f32(ctx, self.read_out(ctx, x), self.w_o, name)


@register_part("mixer", "state_space")
class StateSpace(Part):
    """The state-space recurrence with one decay per head and token (Mamba-2). One input product gives, in this order, z (``inner`` =
    ``num_heads`` x ``value_dim``), x (``inner``), B and C (``groups`` x ``state_size`` each) and one step-size input per head. x, B and C
    together pass a short causal convolution per channel (``conv`` [channels, taps], the last tap the current token's, bias
    ``conv.b``) and SiLU; dt = softplus(input + ``dt_bias``). Per head (which shares B and C with the others of its group)

        S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t

    y times silu(z), the row's ``norm_groups`` equal parts each divided by its own root mean square, times ``norm``, is projected by
    ``o``. S (float32, zero at the start) and the convolution's last taps - 1 inputs are the sequence's state; steps, decays,
    the recurrence and the norm are float32. Tensors ``in conv conv.b dt_bias A_log D norm o``."""
    graph_safe = True
    graph_safe_any_step = True
    takes_split_rows = True                 # the input product's rows may come as split sums
    CHUNKED_FROM = 32                       # a step whose longest portion has as many tokens runs the recurrence by chunks

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden_size = int(params["hidden_size"])
        self.eps = float(params.get("eps", 1e-6))
        self.num_heads = int(params["num_heads"])
        self.value_dim = int(params["value_dim"])
        self.state_size = int(params["state_size"])
        self.groups = int(params.get("groups") or 1)
        self.norm_groups = int(params.get("norm_groups") or 1)
        self.taps = int(params["conv_taps"])
        if not 1 <= self.state_size <= 256:
            raise ConfigError("state_size", f"the scan kernels take states of 1..256 channels, got {self.state_size}")
        _check_dims(self.state_size, self.value_dim)
        self.inner = self.num_heads * self.value_dim
        if self.groups <= 0 or self.num_heads % self.groups:
            raise ConfigError("groups", f"{self.groups} groups do not divide {self.num_heads} heads")
        if self.norm_groups <= 0 or self.inner % self.norm_groups:
            raise ConfigError("norm_groups", f"{self.norm_groups} parts do not divide {self.inner} channels")
        if self.taps < 1:
            raise ConfigError("conv_taps", f"must be at least 1, got {self.taps}")
        self.channels = self.inner + 2 * self.groups * self.state_size         # x, B, C
        self.cols = (0, self.inner, self.inner + self.groups * self.state_size)
        self.in_width = self.inner + self.channels + self.num_heads
        self.w_in = self.w_o = self.conv_w = self.conv_b = self.dt_bias = self.a_log = self.d_skip = self.norm_w = None

    def tensor_specs(self):
        p, hid, h = self.prefix, self.hidden_size, self.num_heads
        return {p + "in": TensorSpec((self.in_width, hid)), p + "conv": TensorSpec((self.channels, self.taps), "conv"),
                p + "conv.b": TensorSpec((self.channels,), "input_bias"), p + "dt_bias": TensorSpec((h,), "log_rate"),
                p + "A_log": TensorSpec((h,), "log_rate"), p + "D": TensorSpec((h,), "norm"), p + "norm": TensorSpec((self.inner,), "norm"),
                p + "o": TensorSpec((hid, self.inner))}

    def load(self, tensors, device, dtype):
        p = self.prefix
        f32 = lambda n: tensors[p + n].to(device=device, dtype=torch.float32).contiguous()      # noqa: E731
        w = to_device(tensors[p + "in"], device, dtype)
        pad = -w.shape[0] % 8                       # rows of zeros, so that the product's float rows start on 16 bytes
        self.w_in = torch.cat([w, w.new_zeros((pad, w.shape[1]))], 0).contiguous() if pad else w
        self.w_o = to_device(tensors[p + "o"], device, dtype)
        self.conv_w = f32("conv").t().contiguous()  # tap by tap: the channels of a tap side by side
        self.conv_b, self.dt_bias, self.a_log, self.d_skip, self.norm_w = f32("conv.b"), f32("dt_bias"), f32("A_log"), f32("D"), f32("norm")

    def cache_spec(self):
        return [StateSpec((self.num_heads, self.value_dim, self.state_size), "float32", "ssm"),
                StateSpec((max(self.taps - 1, 1), self.channels), "float32", "ssm_conv")]

    @property
    def _chunks(self) -> bool:
        return ops.ssm_chunks_usable(self.state_size, self.value_dim)

    def query_tile_sizes(self):
        return [ops.SSM_CHUNK] if self._chunks else []

    def workspace_per_row(self):
        # the float32 rows of the input product, the convolved channels, the gates and the read-out, and the chunks' scratch
        per_chunk = (self.groups * ops.SSM_CHUNK ** 2 + self.num_heads * (self.value_dim * self.state_size + 3 * ops.SSM_CHUNK)) if self._chunks else 0
        return 4 * (self.in_width + self.channels + 2 * self.num_heads + self.inner + per_chunk // ops.SSM_CHUNK)

    def read_out(self, ctx, x, out=None, proj=None):
        n, H = ctx.n_rows, self.num_heads
        if proj is None:                            # (the kept inputs of a step of several rows per sequence are read from complete rows)
            proj = (linear.product_f32 if ctx.decode else linear.product_rows_f32)(ctx, x, self.w_in, "ss_proj")
        z = ctx.buffer("ss_z", (n, self.inner), torch.float32) if proj.dim() == 3 else None
        rows = ctx.buffer("ss_rows", (n, self.channels), torch.float32)
        gates = ctx.buffer("ss_gates", (n, 2 * H), torch.float32)
        conv_state = ctx.state("ssm_conv")
        ops.ssm_inputs(proj, self.conv_w, self.conv_b, self.dt_bias, self.a_log, conv_state, ctx.row_seq, ctx.row_pos, ctx.seq_row0,
                       ctx.seq_slot, rows, gates, self.inner, z, update_state=ctx.decode)
        if self.taps > 1 and not ctx.decode:
            ops.keep_last_rows(proj, self.inner, self.channels, conv_state, ctx.seq_row0, ctx.seq_new, ctx.seq_start, ctx.seq_slot,
                               ctx.n_seqs)
        y = ctx.buffer("ss_y", (n, self.inner), torch.float32)
        if self._chunks and not ctx.decode and ctx.max_new >= self.CHUNKED_FROM:
            # prompts: chunks of 64 tokens side by side, between them a walk over the chunks' states
            tile_seq, tile_q0, n_tiles = ctx.query_tiles(ops.SSM_CHUNK)
            scores = ctx.buffer("ss_scores", (n_tiles, self.groups, ops.SSM_CHUNK, ops.SSM_CHUNK), torch.float32)
            steps = ctx.buffer("ss_steps", (n_tiles, H, 3, ops.SSM_CHUNK), torch.float32)
            prev = ctx.buffer("ss_prev", (n_tiles, H, self.value_dim, self.state_size), torch.float32)
            ops.ssm_chunks(rows, self.cols, gates, self.a_log, self.d_skip, tile_seq, tile_q0, n_tiles, ctx.seq_row0, ctx.seq_new,
                           ctx.seq_start, ctx.seq_slot, ctx.state("ssm"), scores, steps, prev, y, ctx.n_seqs, H, self.groups, self.state_size,
                           self.value_dim)
        else:
            ops.ssm_scan(rows, self.cols, gates, self.d_skip, ctx.state("ssm"), ctx.seq_row0, ctx.seq_new, ctx.seq_start, ctx.seq_slot, y,
                         ctx.n_seqs, H, self.groups, self.state_size, self.value_dim)
        if out is None:
            out = ctx.buffer("ss_out", (n, self.inner))
        ops.gated_group_norm(y, z if z is not None else proj[:, :self.inner], self.norm_w, self.norm_groups, self.eps, out)
        return out

    def forward(self, ctx, x, residual):
        linear.add_into_residual(ctx, self.read_out(ctx, x), self.w_o, residual, "o_partial")

    def branch_output(self, ctx, x, name: str, proj=None):
        return linear.product_f32(ctx, self.read_out(ctx, x, None, proj), self.w_o, name)

    # a parent may put the rows that go into ``o`` beside others', with a factor of its own, and run one product for all
    def output_weight(self):
        return self.w_o

    def set_output_weight(self, w):
        self.w_o = w

    def output_rows(self, ctx, x, out, proj=None):
        self.read_out(ctx, x, out, proj)

    def scale_output(self, factor: float):
        self.norm_w = self.norm_w * float(factor)


@register_part("mixer", "general_delta")
class GeneralDelta(Part):
    """The delta rule with a decay w and a removal rate a per key channel. r, k (``num_heads`` x ``key_dim``) and v
    (``num_heads`` x ``value_dim``) are plain projections, u = k / sqrt(sum k^2 + 1e-6) per head,

        w = exp(-rate * sigmoid(W2 tanh(W1 x) + w0)),   a = sigmoid(Wa x + ba),
        S_t = diag(w) S_(t-1) - (a * u) (u^T S_(t-1)) + k v^T,   o_t = S_t^T r

    both terms of the write on the old state. o is divided by its root mean square per head; the heads side by side are
    multiplied by ``norm`` (all heads' size) and sigmoid(Wg x) and projected by Wo. S is float32 per sequence and head, zero at
    the start; decays, rates, unit keys, the scan and the norm are float32. ``decay_rate``: the factor of the decay's exponent
    (default exp(-1/2)). The width of the decays' narrow input is the stored tensors' own. Tensors ``r k v a a.b g w1 w2 w0
    norm o``."""
    graph_safe = True
    graph_safe_any_step = True
    FEW_ROWS = 32                   # up to here a step makes W2 tanh(.) in the kernel that prepares the scan's rows

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden_size = int(params["hidden_size"])
        self.eps = float(params.get("eps", 1e-6))
        self.num_heads = int(params["num_heads"])
        self.key_dim = int(params["key_dim"])
        self.value_dim = int(params.get("value_dim") or self.key_dim)
        self.decay_rate = float(params["decay_rate"]) if params.get("decay_rate") is not None else math.exp(-0.5)
        _check_dims(self.key_dim, self.value_dim)
        self.rank = int(params.get("rank") or max(8, self.hidden_size // 16 // 8 * 8))      # for random weights
        self.k_width = self.num_heads * self.key_dim
        self.v_width = self.num_heads * self.value_dim
        self.gate_col = 3 * self.k_width + self.v_width               # columns of the input product: r, k, v, a, g, w1
        self.narrow_col = self.gate_col + self.v_width
        self.w_in = self.w2 = self.w_o = self.a_bias = self.w0 = self.norm_w = None

    def tensor_specs(self):
        p, hid, K, V = self.prefix, self.hidden_size, self.k_width, self.v_width
        return {p + "r": TensorSpec((K, hid)), p + "k": TensorSpec((K, hid)), p + "v": TensorSpec((V, hid)),
                p + "a": TensorSpec((K, hid)), p + "a.b": TensorSpec((K,), "input_bias"), p + "g": TensorSpec((V, hid)),
                p + "w1": TensorSpec((self.rank, hid), "linear", (0,)), p + "w2": TensorSpec((K, self.rank), "low_rank", (1,)),
                p + "w0": TensorSpec((K,), "log_rate"), p + "norm": TensorSpec((V,), "norm"), p + "o": TensorSpec((hid, V))}

    def load(self, tensors, device, dtype):
        p = self.prefix
        dev = lambda n: to_device(tensors[p + n], device, dtype)                                  # noqa: E731
        f32 = lambda n: tensors[p + n].to(device=device, dtype=torch.float32).contiguous()      # noqa: E731
        w1, w2 = dev("w1"), dev("w2")
        if w2.shape[1] != w1.shape[0]:
            raise WeightsError(wrong_shape=[(p + "w2", (self.k_width, w1.shape[0]), tuple(w2.shape))])
        pad = -w1.shape[0] % 8                      # zeros: what the tensor-core product takes is a multiple of 8
        if pad:
            w1 = torch.cat([w1, w1.new_zeros((pad, w1.shape[1]))], 0)
            w2 = torch.cat([w2, w2.new_zeros((w2.shape[0], pad))], 1)
        self.w_in = torch.cat([dev(n) for n in ("r", "k", "v", "a", "g")] + [w1], 0).contiguous()
        self.w2, self.w_o = w2.contiguous(), dev("o")
        self.a_bias, self.w0, self.norm_w = f32("a.b"), f32("w0"), f32("norm")

    def cache_spec(self):
        return StateSpec((self.num_heads, self.value_dim, self.key_dim), "float32", "delta")

    def query_tile_sizes(self):
        return [ops.DELTA_CHUNK]

    def workspace_per_row(self):
        # the float32 input product and decays' inputs, and the chunks' matrices
        D, V = self.key_dim, self.value_dim
        return 4 * (self.narrow_col + self.k_width + self.num_heads * (ops.delta_chunk_floats(D, V) // ops.DELTA_CHUNK + 1))

    def read_out(self, ctx, x, out=None):
        n, H, D, V = ctx.n_rows, self.num_heads, self.key_dim, self.value_dim
        sums = linear.product_f32(ctx, x, self.w_in, "gd_proj")            # split sums where the step is small: added below
        split = sums.dim() == 3
        gate, gate_col, high = sums, self.gate_col, None
        if split:
            gate, gate_col = ctx.buffer("gd_gate", (n, self.v_width), torch.float32), 0
        if n > self.FEW_ROWS:
            low = ctx.buffer("gd_low", (n, self.w2.shape[1]))
            ops.tanh_columns(sums, self.narrow_col, low)
            high = linear.product_f32(ctx, low, self.w2, "gd_high")
        raw = ctx.buffer("gd_raw", (n, self.v_width), torch.float32)
        if high is not None and ctx.max_new >= ops.DELTA_CHUNK and ops.delta_chunks_usable(D, V, self.decay_rate):
            # prompts: chunks of 16 tokens side by side, then a walk over the chunks
            tile_seq, tile_q0, n_tiles = ctx.query_tiles(ops.DELTA_CHUNK)
            chunks = ctx.buffer("gd_chunks", (n_tiles, H, ops.delta_chunk_floats(D, V)), torch.float32)
            ops.delta_chunks(sums, high, self.a_bias, self.w0, self.decay_rate, tile_seq, tile_q0, n_tiles, ctx.seq_row0, ctx.seq_new,
                             chunks, H, D, V, gate if split else None)
            ops.delta_chunk_scan(chunks, ctx.state("delta"), ctx.seq_row0, ctx.seq_new, ctx.seq_start, ctx.seq_slot, raw, ctx.n_seqs, H, D, V)
        else:
            packed = ctx.buffer("gd_packed", (n, H, 4 * D + V), torch.float32)
            scal = ctx.buffer("gd_scalars", (n, H, 4), torch.float32)
            ops.delta_inputs(sums, self.a_bias, self.w0, self.decay_rate, packed, scal, H, D, V, high, None if high is not None else self.w2,
                             gate if split else None)
            ops.general_delta_scan(packed, scal, ctx.state("delta"), ctx.seq_row0, ctx.seq_new, ctx.seq_start, ctx.seq_slot, raw,
                                   ctx.n_seqs, H, D, V)
        if out is None:
            out = ctx.buffer("gd_out", (n, self.v_width))
        ops.head_norm_gate(raw, False, self.norm_w, True, gate, gate_col, out, H, V, self.eps)
        return out

    def forward(self, ctx, x, residual):
        linear.add_into_residual(ctx, self.read_out(ctx, x), self.w_o, residual, "o_partial")

    def branch_output(self, ctx, x, name: str, proj=None):
        return linear.product_f32(ctx, self.read_out(ctx, x), self.w_o, name)

    # a block may put the rows that go into ``o`` beside a feed-forward's and run one product for both
    def output_weight(self):
        return self.w_o

    def set_output_weight(self, w):
        self.w_o = w

    def output_rows(self, ctx, x, out):
        self.read_out(ctx, x, out)
