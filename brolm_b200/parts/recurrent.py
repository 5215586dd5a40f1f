"""Mixers that carry a state of fixed size from token to token: a gated diagonal recurrence,
a selective state space and a gated delta rule, each behind a short causal convolution, and linear attention
with a fixed decay.

All keep, per sequence, one float32 row of a state group: the recurrence's state first, then the
convolution's last ``taps - 1`` inputs (zeros before the sequence's start).  The row is zero when a slot is
taken, read at the start of a sequence's tokens in a step and written at their end; the same kernels serve
a prompt and a decode step, and nothing is read back to the host.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from ..cache import StateSpec
from .base import ParamSpec, Part, register_part
from .linear import linear


def _f32(t: torch.Tensor) -> torch.Tensor:
    return t.float().contiguous()


class GatedRecurrence(Part):
    """The recurrent block of Griffin (De et al., "Griffin: Mixing Gated Linear Recurrences with Local
    Attention for Efficient Language Models") with its real-gated linear recurrent unit.

    Two branches of ``width`` channels: g = gelu_tanh(W_y x + b_y) and u = conv(W_x x + b_x), a causal
    convolution per channel with ``taps`` taps, a bias and no activation.  u is cut into ``blocks`` equal
    parts; in each, r = sigmoid(Ra u + ra) and i = sigmoid(Ri u + ri) with square matrices of the part's
    size.  Per channel: a = exp(-decay_scale * r * softplus(lam)), S <- a S + sqrt(1 - a^2) (i u), and the
    result is W_o (S g).  S, the gates, the decay and the convolution are float32 in every mode; the block
    products run over float32 rows of u (for a prompt of a bfloat16 step: over u in two bfloat16 halves, which
    keep 16 bits of it, with float sums).
    """

    kind = "mixer"
    graph_safe = True
    SPLIT_ROWS = 64          # from this many tokens on a bfloat16 step's gate products run on the tensor cores

    def __init__(self, hidden: int, width: int, blocks: int, taps: int, decay_scale: float = 8.0):
        if width % blocks:
            raise ValueError("gated recurrence: width must be a multiple of blocks")
        if taps < 1:
            raise ValueError("gated recurrence: the convolution needs at least one tap")
        self.hidden, self.width, self.blocks, self.taps = hidden, width, blocks, taps
        self.bs = width // blocks
        self.decay_scale = float(decay_scale)
        self.tail_off = width

    def param_specs(self):
        W, nb, bs = self.width, self.blocks, self.bs
        return {"y": ParamSpec((W, self.hidden)), "y_bias": ParamSpec((W,), "vector"),
                "x": ParamSpec((W, self.hidden)), "x_bias": ParamSpec((W,), "vector"),
                "conv": ParamSpec((W, self.taps), "vector"), "conv_bias": ParamSpec((W,), "vector"),
                "ra": ParamSpec((nb, bs, bs)), "ra_bias": ParamSpec((nb, bs), "vector"),
                "ri": ParamSpec((nb, bs, bs)), "ri_bias": ParamSpec((nb, bs), "vector"),
                "lam": ParamSpec((W,), "vector"), "o": ParamSpec((self.hidden, W))}

    def bind(self, params):
        kinds = {params[n].dtype for n in ("y", "x")}
        dt = torch.float32 if (len(kinds) > 1 or torch.float32 in kinds) else next(iter(kinds))
        # one product for both branches: rows [Wy; Wx]
        self.w_in = torch.cat([params["y"].to(dt), params["x"].to(dt)], dim=0).contiguous()
        self.w_o = params["o"]
        # per block the rows [Ra; Ri], as float32: the gates' products take float32 rows of u
        self.w_gates = torch.cat([params["ra"].float(), params["ri"].float()], dim=1).contiguous()
        # the same rows as stored, when stored in bfloat16: a prompt's gate products run on the tensor cores over u in
        # two bfloat16 halves (16 bits of u; the products with bfloat16 matrices are exact in float)
        self.w_gates_bf16 = None
        if params["ra"].dtype == torch.bfloat16 and params["ri"].dtype == torch.bfloat16 and self.bs % 8 == 0:
            self.w_gates_bf16 = torch.cat([params["ra"], params["ri"]], dim=1).contiguous()
        self.y_bias, self.x_bias = _f32(params["y_bias"]), _f32(params["x_bias"])
        self.conv, self.conv_bias = _f32(params["conv"]), _f32(params["conv_bias"])
        self.r_bias, self.i_bias = _f32(params["ra_bias"]).view(-1), _f32(params["ri_bias"]).view(-1)
        self.lam = _f32(params["lam"])
        self.params = {}

    def cache_spec(self):
        return StateSpec((self.width * self.taps,), torch.float32)          # S, then taps - 1 rows of inputs

    def forward(self, x: torch.Tensor, ctx, entry, writes_cache: bool = True) -> torch.Tensor:
        """x (tokens, hidden) -> (tokens, hidden) float32, or partial sums [parts, tokens, hidden]."""
        if not writes_cache:
            raise NotImplementedError("a mixer with a state cannot run on another layer's state")
        T, W = x.shape[0], self.width
        state = ctx.state(entry)
        seq = (ctx.cu_q, ctx.kv_len, ctx.slots_dev, state)
        proj = linear(x, self.w_in, out_dtype=torch.float32)              # [ y_raw | x_raw ]
        x_raw = proj[:, W:]
        u = torch.empty((T, W), dtype=torch.float32, device=x.device)
        kernels.causal_conv(x_raw, self.x_bias, self.conv, self.conv_bias, "none", ctx.tok_seq, ctx.positions, *seq,
                            self.tail_off, u)
        pre_lo = None
        if kernels.block_matvec_ok(T, self.bs):
            pre = torch.empty((T, 2 * W), dtype=torch.float32, device=x.device)
            kernels.block_matvec_f32(u, self.bs, self.w_gates, pre, 2 * self.bs)       # a handful of tokens: a stream of the matrices
        elif ctx.dtype == torch.bfloat16 and self.w_gates_bf16 is not None and T >= self.SPLIT_ROWS:
            halves = torch.empty((2 * T, W), dtype=torch.bfloat16, device=x.device)
            kernels.split_halves(u, halves)
            both = torch.empty((2 * T, 2 * W), dtype=torch.float32, device=x.device)
            kernels.heads_linear(halves, self.bs, self.w_gates_bf16, both, 2 * self.bs)
            pre, pre_lo = both[:T], both[T:]
        else:
            pre = torch.empty((T, 2 * W), dtype=torch.float32, device=x.device)
            kernels.heads_linear(u, self.bs, self.w_gates, pre, 2 * self.bs)
        out = torch.empty((T, W), dtype=ctx.dtype, device=x.device)
        kernels.gated_scan(pre, u, proj[:, :W], self.y_bias, self.r_bias, self.i_bias, self.lam, self.decay_scale,
                           self.bs, ctx.positions, *seq, out, ctx.batch, ctx.max_q_len, pre_lo=pre_lo)
        kernels.conv_tail(x_raw, self.x_bias, self.taps, *seq, self.tail_off, ctx.batch)
        return linear(out, self.w_o, out_dtype=torch.float32, parts_ok=True)


register_part("mixer", "gated_recurrence", GatedRecurrence)


class StateSpace(Part):
    """The Mamba-2 mixer (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms
    Through Structured State Space Duality").

    W_in x is laid out as [z: inner | x: inner | B: groups*N | C: groups*N | dt: heads], inner = heads * P.
    x, B and C pass a causal convolution per channel (``taps`` taps, bias) and silu.  Per head h of group
    h // (heads / groups): dt = softplus(dt + dt_bias), S <- exp(-exp(A_log) dt) S + dt B x^T (S is N x P),
    y = S^T C + D x.  Then y * silu(z), an RMS norm over each of ``norm_groups`` equal parts with a gain, and
    W_o.  S, dt, the decay and the norm are float32 in every mode.
    """

    kind = "mixer"
    graph_safe = True

    def __init__(self, hidden: int, heads: int, head_size: int, state: int, groups: int, norm_groups: int, taps: int,
                 eps: float):
        if heads % groups:
            raise ValueError("state space: heads must be a multiple of groups")
        if (heads * head_size) % norm_groups:
            raise ValueError("state space: heads * head_size must be a multiple of norm_groups")
        if state > 256:
            raise ValueError("state space: a state of more than 256 numbers per channel is beyond the kernel")
        self.hidden, self.heads, self.P, self.N, self.groups = hidden, heads, head_size, state, groups
        self.norm_groups, self.taps, self.eps = norm_groups, taps, float(eps)
        self.inner = heads * head_size
        self.conv_cols = self.inner + 2 * groups * state
        self.in_cols = 2 * self.inner + 2 * groups * state + heads
        self.tail_off = heads * head_size * state

    def param_specs(self):
        return {"in": ParamSpec((self.in_cols, self.hidden)), "conv": ParamSpec((self.conv_cols, self.taps), "vector"),
                "conv_bias": ParamSpec((self.conv_cols,), "vector"), "dt_bias": ParamSpec((self.heads,), "vector"),
                "A_log": ParamSpec((self.heads,), "vector"), "D": ParamSpec((self.heads,), "vector"),
                "norm": ParamSpec((self.inner,), "vector"), "o": ParamSpec((self.hidden, self.inner))}

    def bind(self, params):
        self.w_in, self.w_o = params["in"], params["o"]
        self.conv, self.conv_bias = _f32(params["conv"]), _f32(params["conv_bias"])
        self.dt_bias, self.a_log, self.d = _f32(params["dt_bias"]), _f32(params["A_log"]), _f32(params["D"])
        self.gain = params["norm"].contiguous()
        self.params = {}

    def cache_spec(self):
        return StateSpec((self.tail_off + (self.taps - 1) * self.conv_cols,), torch.float32)

    def forward(self, x: torch.Tensor, ctx, entry, writes_cache: bool = True) -> torch.Tensor:
        if not writes_cache:
            raise NotImplementedError("a mixer with a state cannot run on another layer's state")
        T, inner = x.shape[0], self.inner
        state = ctx.state(entry)
        seq = (ctx.cu_q, ctx.kv_len, ctx.slots_dev, state)
        proj = linear(x, self.w_in, out_dtype=torch.float32)
        raw = proj[:, inner:inner + self.conv_cols]
        xbc = torch.empty((T, self.conv_cols), dtype=torch.float32, device=x.device)
        kernels.causal_conv(raw, None, self.conv, self.conv_bias, "silu", ctx.tok_seq, ctx.positions, *seq,
                            self.tail_off, xbc)
        y = torch.empty((T, inner), dtype=torch.float32, device=x.device)
        kernels.ssm_scan(xbc, proj[:, inner + self.conv_cols:], self.dt_bias, self.a_log, self.d, self.heads, self.groups,
                         self.P, self.N, *seq, y, ctx.batch, ctx.max_q_len)
        kernels.conv_tail(raw, None, self.taps, *seq, self.tail_off, ctx.batch)
        out = torch.empty((T, inner), dtype=ctx.dtype, device=x.device)
        kernels.gate_group_norm(y, proj[:, :inner], self.gain, self.eps, self.norm_groups, out)
        return linear(out, self.w_o, out_dtype=torch.float32, parts_ok=True)


register_part("mixer", "state_space", StateSpace)


class DecayLinearAttention(Part):
    """Linear attention with one fixed decay per head ("lightning" attention).

    q = act(W_q x), k = act(W_k x) (``heads`` x ``dim``) and v = act(W_v x) (``heads`` x ``v_dim``), laid out head by
    head; per head S <- decay_h S + k v^T and o = S^T q, with no other scale.  The heads' results together pass an
    RMS norm over the whole row with a gain (``norm``), are multiplied by sigmoid(W_g x) (``gate``) and go through
    W_o.  ``decay``: one number per head.  The projection's sums, the activation, S and the norm are float32 in
    every mode; S is a state row per sequence, zero at the sequence's start.

    Options: ``position`` rotates the first entries of every q and k head by the token's position, ``k_scale``
    multiplies k after that (retention: Sun et al., "Retentive Network: A Successor to Transformer for Large Language
    Models"); both act on the projection's float sums.  ``norm="head"``: every head's result is divided by its own
    root mean square, without a gain.  ``gate="silu"``: the results are multiplied by silu(W_g x)."""

    kind = "mixer"
    graph_safe = True

    def __init__(self, hidden: int, heads: int, dim: int, v_dim: int, decay, eps: float, activation: str = "silu",
                 norm=True, gate=True, position: Optional[Part] = None, k_scale: float = 1.0):
        decay = [float(d) for d in decay]
        if len(decay) != heads:
            raise ValueError(f"decay attention: {len(decay)} decays for {heads} heads")
        if any(not 0.0 <= d <= 1.0 for d in decay):
            raise ValueError("decay attention: every decay lies between 0 and 1")
        if activation not in kernels.SCAN_ACTS:
            raise ValueError(f"decay attention: unknown activation '{activation}'")
        if dim > 512:
            raise ValueError("decay attention: more than 512 query/key entries per head are beyond the kernel")
        if norm not in (True, False, "head") or gate not in (True, False, "sigmoid", "silu"):
            raise ValueError(f"decay attention: unknown norm '{norm}' or gate '{gate}'")
        if norm == "head" and not gate:
            raise ValueError("decay attention: a norm per head without a gate is not built")
        if norm != "head" and gate == "silu":
            raise ValueError("decay attention: a silu gate goes with the norm per head")
        if position is not None and (position.pairing != "half" or position.rotary_dim > dim):
            raise ValueError("decay attention: the rotation pairs entries i and i + r/2 of a head's first r")
        self.position, self.k_scale = position, float(k_scale)
        self.head_norm, self.gate_act = norm == "head", "silu" if gate == "silu" else "sigmoid"
        self.hidden, self.heads, self.dim, self.v_dim, self.decay = hidden, heads, dim, v_dim, decay
        self.eps, self.activation, self.has_norm, self.has_gate = float(eps), activation, norm is True, bool(gate)
        self.qk_cols, self.v_cols = heads * dim, heads * v_dim

    def param_specs(self):
        specs = {"q": ParamSpec((self.qk_cols, self.hidden)), "k": ParamSpec((self.qk_cols, self.hidden)),
                 "v": ParamSpec((self.v_cols, self.hidden)), "o": ParamSpec((self.hidden, self.v_cols))}
        if self.has_gate:
            specs["g"] = ParamSpec((self.v_cols, self.hidden))
        if self.has_norm:
            specs["norm"] = ParamSpec((self.v_cols,), "vector")
        return specs

    def bind(self, params):
        names = ("q", "k", "v") + (("g",) if self.has_gate else ())
        kinds = {params[n].dtype for n in names}
        dt = torch.float32 if (len(kinds) > 1 or torch.float32 in kinds) else next(iter(kinds))
        # one product for q, k, v and the gate's logits: rows [Wq; Wk; Wv; Wg]
        self.w_in = torch.cat([params[n].to(dt) for n in names], dim=0).contiguous()
        self.w_o = params["o"]
        self.gain = params["norm"].contiguous() if self.has_norm else None
        # decay - 1, taken in double: what a float keeps of it is far finer than what it keeps of the decay itself
        self.decay_m1 = torch.tensor([d - 1.0 for d in self.decay], dtype=torch.float64).to(torch.float32) \
            .to(self.w_in.device)
        self.params = {}

    def cache_spec(self):
        return StateSpec((kernels.decay_state_size(self.heads, self.dim, self.v_dim),), torch.float32)

    def prepare(self, max_positions, device):
        if self.position is not None:
            self.position.prepare(max_positions, device)

    def forward(self, x: torch.Tensor, ctx, entry, writes_cache: bool = True) -> torch.Tensor:
        """x (tokens, hidden) -> (tokens, hidden) float32, or partial sums [parts, tokens, hidden]."""
        if not writes_cache:
            raise NotImplementedError("a mixer with a state cannot run on another layer's state")
        T = x.shape[0]
        proj = linear(x, self.w_in, out_dtype=torch.float32)              # [ q | k | v | gate logits ]
        y = torch.empty((T, self.v_cols), dtype=torch.float32, device=x.device)
        act = self.activation
        if act != "none" and ctx.max_q_len > 1:
            # a prompt: every block of a head's scan would apply the activation to the head's q and k anew, so it
            # is applied once, in place, by a pass of its own; a step of single tokens leaves it to the scan
            qkv = proj[:, :2 * self.qk_cols + self.v_cols]
            kernels.bias_act(qkv, None, act, qkv)
            act = "none"
        table, k_scale = self.position.table if self.position is not None else None, self.k_scale
        if (table is not None or k_scale != 1.0) and ctx.max_q_len > 1:
            # the same for the rotation and k's scale (after the activation, as in the scan)
            kernels.rotate_heads(proj, 0, self.qk_cols, self.heads, self.dim, ctx.positions, table, k_scale)
            table, k_scale = None, 1.0
        kernels.decay_scan(proj, 0, self.qk_cols, 2 * self.qk_cols, self.heads, self.dim, self.v_dim, act,
                           self.decay_m1, ctx.cu_q, ctx.kv_len, ctx.slots_dev, ctx.state(entry), y, ctx.batch, ctx.max_q_len,
                           cos_sin=table, k_scale=k_scale)
        if self.head_norm:
            out = torch.empty((T, self.v_cols), dtype=ctx.dtype, device=x.device)
            kernels.head_norm_gate(y, proj[:, 2 * self.qk_cols + self.v_cols:], None, self.eps, self.heads, self.gate_act, out)
        elif self.has_norm or self.has_gate:
            out = torch.empty((T, self.v_cols), dtype=ctx.dtype, device=x.device)
            if self.has_gate:
                kernels.norm_sigmoid_gate(y, proj[:, 2 * self.qk_cols + self.v_cols:], self.gain, self.eps, out)
            else:
                kernels.rmsnorm(y, self.gain, self.eps, 0.0, out)
        else:
            out = y if ctx.dtype == torch.float32 else y.to(ctx.dtype)
        return linear(out, self.w_o, out_dtype=torch.float32, parts_ok=True)


register_part("mixer", "decay_attention", DecayLinearAttention)


class GatedDeltaRule(Part):
    """The gated delta rule (Yang et al., "Gated Delta Networks: Improving Mamba2 with Delta Rule").

    q = W_q x and k = W_k x (``kv_heads`` x ``dim``), v = W_v x (``heads`` x ``v_dim``), each through a causal
    convolution per channel over time (``taps`` taps, no bias) and silu; q and k are made unit vectors per head and q is
    multiplied by dim^(-1/2); value head h works with q/k head h // (heads / kv_heads).  Per head, with
    beta = sigmoid(W_b x) and g = exp(-exp(A_log) softplus(W_a x + dt_bias)):

        S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

    Every head's o is divided by its own root mean square, times a gain of ``v_dim`` numbers for all heads (``norm``),
    times silu(W_g x), then W_o.  The projection's sums and everything up to the last product's input are float32 in
    every mode; S and the convolutions' newest inputs are a state row per sequence, zero at the sequence's start.  A
    step of single tokens is one kernel from the projection to o; a prompt runs the recurrence sixteen tokens at a time."""

    kind = "mixer"
    graph_safe = True

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, v_dim: int, taps: int, eps: float):
        if heads % kv_heads:
            raise ValueError("delta rule: heads must be a multiple of kv_heads")
        if taps < 1:
            raise ValueError("delta rule: the convolution needs at least one tap")
        if dim > 512:
            raise ValueError("delta rule: more than 512 query/key entries per head are beyond the kernel")
        self.hidden, self.heads, self.kv_heads, self.dim, self.v_dim = hidden, heads, kv_heads, dim, v_dim
        self.taps, self.eps = taps, float(eps)
        self.qk_cols, self.v_cols = kv_heads * dim, heads * v_dim
        self.conv_cols = 2 * self.qk_cols + self.v_cols
        # the gate's columns of the projection start at a multiple of four, so that its rows can be read four at a time
        self.gate_from = (self.conv_cols + 2 * heads + 3) // 4 * 4
        self.tail_off = kernels.decay_state_size(heads, dim, v_dim)

    def param_specs(self):
        W, K = self.hidden, self.taps
        return {"q": ParamSpec((self.qk_cols, W)), "q_conv": ParamSpec((self.qk_cols, K), "vector"),
                "k": ParamSpec((self.qk_cols, W)), "k_conv": ParamSpec((self.qk_cols, K), "vector"),
                "v": ParamSpec((self.v_cols, W)), "v_conv": ParamSpec((self.v_cols, K), "vector"),
                "b": ParamSpec((self.heads, W)), "a": ParamSpec((self.heads, W)), "A_log": ParamSpec((self.heads,), "vector"),
                "dt_bias": ParamSpec((self.heads,), "vector"), "g": ParamSpec((self.v_cols, W)),
                "norm": ParamSpec((self.v_dim,), "vector"), "o": ParamSpec((W, self.v_cols))}

    def bind(self, params):
        names = ("q", "k", "v", "b", "a", "g")
        kinds = {params[n].dtype for n in names}
        dt = torch.float32 if (len(kinds) > 1 or torch.float32 in kinds) else next(iter(kinds))
        # one product: rows [Wq; Wk; Wv; Wb; Wa; (rows of zeros up to a multiple of four); Wg]
        rows = [params[n].to(dt) for n in names]
        pad = self.gate_from - self.conv_cols - 2 * self.heads
        if pad:
            rows.insert(5, torch.zeros((pad, self.hidden), dtype=dt, device=rows[0].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_o = params["o"]
        # tap by tap, so that neighbouring channels lie next to one another
        self.conv = torch.cat([params[n + "_conv"].float() for n in ("q", "k", "v")], dim=0).t().contiguous()
        self.a_log, self.dt_bias = _f32(params["A_log"]), _f32(params["dt_bias"])
        self.gain = _f32(params["norm"]).repeat(self.heads).contiguous()
        self.params = {}

    def cache_spec(self):
        # S, then a ring of inputs; a row of the state group is a whole number of 16-byte pieces
        n = self.tail_off + (self.taps if self.taps > 1 else 0) * self.conv_cols
        return StateSpec(((n + 3) // 4 * 4,), torch.float32)

    def forward(self, x: torch.Tensor, ctx, entry, writes_cache: bool = True) -> torch.Tensor:
        """x (tokens, hidden) -> (tokens, hidden) float32, or partial sums [parts, tokens, hidden]."""
        if not writes_cache:
            raise NotImplementedError("a mixer with a state cannot run on another layer's state")
        T = x.shape[0]
        seq = (ctx.cu_q, ctx.kv_len, ctx.slots_dev, ctx.state(entry), self.tail_off)
        sizes = (self.kv_heads, self.dim, self.heads, self.v_dim, self.a_log, self.dt_bias)
        proj = linear(x, self.w_in, out_dtype=torch.float32)              # [ q | k | v | b | a | gate logits ]
        y = torch.empty((T, self.v_cols), dtype=torch.float32, device=x.device)
        if ctx.max_q_len == 1:
            kernels.delta_step(proj, self.conv, *sizes, *seq, y, ctx.batch)
        else:
            kernels.delta_prompt(proj, self.conv, *sizes, ctx.tok_seq, ctx.positions, *seq, y, ctx.batch, ctx.max_q_len)
        out = torch.empty((T, self.v_cols), dtype=ctx.dtype, device=x.device)
        kernels.head_norm_gate(y, proj[:, self.gate_from:], self.gain, self.eps, self.heads, "silu", out)
        return linear(out, self.w_o, out_dtype=torch.float32, parts_ok=True)


register_part("mixer", "gated_delta_rule", GatedDeltaRule)


class SideBySide(Part):
    """Two mixers that read the same input; the result is left_scale * left + right_scale * right.
    Each keeps what it keeps: the pair's cache spec is the tuple of both."""

    kind = "mixer"

    def __init__(self, left: Part, right: Part, left_scale: float = 1.0, right_scale: float = 1.0):
        self.left, self.right = left, right
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)

    @property
    def graph_safe(self) -> bool:
        return self.left.graph_safe and self.right.graph_safe

    def cache_spec(self):
        return (self.left.cache_spec(), self.right.cache_spec())

    def prepare(self, max_positions, device):
        self.left.prepare(max_positions, device)
        self.right.prepare(max_positions, device)

    def forward(self, x: torch.Tensor, ctx, entry, writes_cache: bool = True) -> torch.Tensor:
        a = self.left.forward(x, ctx, entry.parts[0], writes_cache)
        b = self.right.forward(x, ctx, entry.parts[1], writes_cache)
        out = torch.empty(a.shape[-2:], dtype=torch.float32, device=x.device)
        kernels.scaled_sum(a, self.left_scale, b, self.right_scale, out)
        return out


register_part("mixer", "side_by_side", SideBySide)
