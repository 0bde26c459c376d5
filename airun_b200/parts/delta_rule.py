"""Gated delta rule: a recurrent mixer whose state is a matrix per head that is corrected, not only added to.

With h the mixer's input, per head of D key channels and Dv value channels (q and k have ``num_kv_heads`` heads,
head i of the state reads q/k head i // (heads / kv_heads)):

    q, k, v = silu(conv(Wq h)), silu(conv(Wk h)), silu(conv(Wv h))      a causal convolution over time per channel
    q <- q / |q| * D^-1/2,  k <- k / |k|                               per head, |x| = sqrt(sum x^2 + 1e-6)
    beta = sigmoid(Wb h)                                               one number per head
    g = exp(-exp(A_log[head]) * softplus(Wa2 (Wa1 h) + dt_bias))       a decay per head and key channel
                                                                       or, with ``decay="head"``, one per head:
    g = exp(-exp(A_log[head]) * softplus(Wa h + dt_bias))
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q  (token by token; S starts at zero)
    out = Wo concat_heads( o / rms(o) * w_norm * sigmoid(Wg2 (Wg1 h)) )   or, with ``gate="silu"``, * silu(Wg h)

The state, the decays, beta, the unit vectors, the norm and the gate are float32.  The matrix state of a request
and the last ``taps - 1`` inputs of the convolution live side by side in its slot of the cache manager's state
tensor (one flat float32 row), so prompts cut anywhere, single tokens and whole prompts run the same recurrence.
The six input projections run as one product over [Wq; Wk; Wv; Wb; Wa1; Wg1], with a silu gate [Wq; Wk; Wv; Wg; Wb; ...].
A decay per head is worked out inside the recurrence's kernel, from its projection.  The part has the split form
(parts/base.py): ``forward_core`` leaves the gated heads, times ``out_scale``, in a buffer, and can be handed the columns
of a product that an arrangement has run over several parts' stacked input matrices (``proj``).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from ..weights.loader import WeightSpec
from .base import Mixer, StateSpec, register_part
from .linear import linear


class GatedDeltaRule(Mixer):
    device_driven = True

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int,
                 conv_taps: int, norm_eps: float, decay_rank: int = 0, gate_rank: int = 0, decay: str = "channel",
                 gate: str = "lowrank_sigmoid", unit_eps: float = 1e-6, q_scale: Optional[float] = None,
                 out_scale: float = 1.0, dtype: torch.dtype = torch.bfloat16, device=None,
                 names: Optional[Dict[str, str]] = None):
        self.prefix, self.H = prefix, int(hidden_size)
        self.nh, self.nkv, self.D, self.Dv = int(num_heads), int(num_kv_heads), int(key_dim), int(value_dim)
        if decay not in ("channel", "head") or gate not in ("lowrank_sigmoid", "silu"):
            raise ValueError("decay is 'channel' (a low-rank pair) or 'head'; gate is 'lowrank_sigmoid' or 'silu'")
        self.head_decay, self.silu_gate = decay == "head", gate == "silu"
        # columns of the input product that lead to the decay and to the gate
        self.taps, self.rank_a, self.rank_g = int(conv_taps), int(decay_rank), int(gate_rank)
        if self.head_decay:
            self.rank_a = self.nh
        if self.silu_gate:
            self.rank_g = self.nh * self.Dv
        if min(self.nh, self.nkv, self.D, self.Dv, self.taps, self.rank_a, self.rank_g) <= 0:
            raise ValueError("heads, sizes, taps and ranks must be positive")
        if self.nh % self.nkv:
            raise ValueError(f"heads ({num_heads}) must be a multiple of kv_heads ({num_kv_heads})")
        if self.D > 256:
            raise ValueError(f"{self.D} key channels a head are above the recurrence kernel's limit of 256")
        self.eps, self.unit_eps, self.out_scale = float(norm_eps), float(unit_eps), float(out_scale)
        self.q_scale = float(q_scale) if q_scale is not None else self.D ** -0.5
        self.dtype, self.device = dtype, device
        n = dict(q="q", k="k", v="v", q_conv="q.conv", k_conv="k.conv", v_conv="v.conv", beta="b", a_log="A_log", norm="norm",
                 decay_in="a" if self.head_decay else "a1", decay_out="a2", decay_bias="dt_bias",
                 gate_in="g" if self.silu_gate else "g1", gate_out="g2", o="o")
        n.update(names or {})
        self.names = {k: f"{prefix}.{v}" for k, v in n.items()}
        self.kd, self.vd = self.nkv * self.D, self.nh * self.Dv
        self.core_width = self.vd
        self.C = 2 * self.kd + self.vd                       # channels that pass the convolution
        self.state_matrix = self.nh * self.D * self.Dv       # the flat state: the matrices, then the convolution's tail
        self.w_in = self.w_out = self.conv_w = self.w_a2 = self.w_g2 = self.dt_bias = self.a_log = self.norm_w = None

    # ---- weights ----
    def weight_specs(self) -> List[WeightSpec]:
        nm, H = self.names, self.H
        specs = [WeightSpec(nm["q"], (self.kd, H)), WeightSpec(nm["k"], (self.kd, H)), WeightSpec(nm["v"], (self.vd, H)),
                WeightSpec(nm["q_conv"], (self.kd, self.taps), storage="float32"),
                WeightSpec(nm["k_conv"], (self.kd, self.taps), storage="float32"),
                WeightSpec(nm["v_conv"], (self.vd, self.taps), storage="float32"),
                WeightSpec(nm["beta"], (self.nh, H)), WeightSpec(nm["a_log"], (self.nh,), storage="float32"),
                WeightSpec(nm["norm"], (self.Dv,), storage="float32", init="norm"),
                WeightSpec(nm["decay_in"], (self.rank_a, H)),
                WeightSpec(nm["decay_bias"], (self.nh if self.head_decay else self.nh * self.D,), storage="float32"),
                WeightSpec(nm["gate_in"], (self.rank_g, H)), WeightSpec(nm["o"], (H, self.vd))]
        if not self.head_decay:
            specs.append(WeightSpec(nm["decay_out"], (self.nh * self.D, self.rank_a)))
        if not self.silu_gate:
            specs.append(WeightSpec(nm["gate_out"], (self.vd, self.rank_g)))
        return specs

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        nm = self.names
        # a whole gate comes right behind q, k and v: its rows then begin on the boundary that vector loads want
        order = ("q", "k", "v", "gate_in", "beta", "decay_in") if self.silu_gate else ("q", "k", "v", "beta", "decay_in", "gate_in")
        self.w_in = torch.cat([tensors.pop(nm[k]) for k in order], dim=0).contiguous()
        self.conv_w = torch.cat([tensors.pop(nm[k]) for k in ("q_conv", "k_conv", "v_conv")], dim=0).contiguous()
        self.w_a2 = None if self.head_decay else tensors.pop(nm["decay_out"])
        self.w_g2 = None if self.silu_gate else tensors.pop(nm["gate_out"])
        self.w_out = tensors.pop(nm["o"])
        self.dt_bias, self.a_log, self.norm_w = tensors[nm["decay_bias"]], tensors[nm["a_log"]], tensors[nm["norm"]]
        if self.out_scale != 1.0:           # the norm's weight is the last factor of the heads
            self.norm_w = self.norm_w * self.out_scale

    def adopt_w_out(self, view: torch.Tensor) -> None:
        self.w_out = view

    # ---- cache ----
    def cache_spec(self):
        return StateSpec((self.state_matrix + (self.taps - 1) * self.C,), torch.float32)

    # ---- compute ----
    def forward_core(self, ctx, h: torch.Tensor, act: torch.Tensor, cache, proj: Optional[torch.Tensor] = None) -> None:
        """Writes out_scale * the normed, gated heads into ``act`` ([T, heads * value_dim], rows may be strided)."""
        T, ws, C, nh = act.shape[0], ctx.ws, self.C, self.nh
        if proj is None:
            proj = ws.alloc((T, C + nh + self.rank_a + self.rank_g), torch.float32)
            linear(ctx, h, self.w_in, proj)
        at = C + (self.rank_g if self.silu_gate else 0)
        qkv, beta, low_a = proj[:, :C], proj[:, at:at + nh], proj[:, at + nh:at + nh + self.rank_a]
        low_g = proj[:, C:at] if self.silu_gate else proj[:, at + nh + self.rank_a:]
        conv = ws.alloc((T, C), torch.float32)
        ops.short_conv(qkv, self.conv_w, cache.state, self.state_matrix, ctx, conv, n_unit_heads=2 * self.nkv,
                       q_heads=self.nkv, unit_dim=self.D, unit_eps=self.unit_eps, q_scale=self.q_scale)
        if self.head_decay:
            decay, per_head = low_a, dict(a_log=self.a_log, dt_bias=self.dt_bias)
        else:
            decay, per_head = ws.alloc((T, nh * self.D), torch.float32), {}
            ops.lowrank_act(low_a, self.w_a2, self.dt_bias, decay, ctx.req_of_token, ops.LOWRANK_EXP_SOFTPLUS,
                            group_param=self.a_log, group=self.D)
        gate = low_g
        if not self.silu_gate:
            gate = ws.alloc((T, self.vd), torch.float32)
            ops.lowrank_act(low_g, self.w_g2, None, gate, ctx.req_of_token, ops.LOWRANK_SIGMOID)
        o = ws.alloc((T, self.vd), torch.float32)
        ops.recurrent_state(ops.RECURRENCE_DELTA_HEAD if self.head_decay else ops.RECURRENCE_DELTA, conv[:, :self.kd],
                            conv[:, self.kd:2 * self.kd], conv[:, 2 * self.kd:], decay,
                            cache.state, ctx, o, nh, nh // self.nkv, self.D, self.Dv, beta=beta, tail_src=qkv,
                            tail_off=self.state_matrix, tail_rows=self.taps - 1, **per_head)
        ops.gla_out_gate(o, gate, self.norm_w, self.eps, act, nh, self.Dv, ctx.req_of_token,
                         gate_act=ops.GATE_SILU if self.silu_gate else ops.GATE_AS_IS)

    def forward(self, ctx, h: torch.Tensor, cache, sink=None):
        T = h.shape[0]
        act = ctx.ws.alloc((T, self.vd), self.dtype)
        self.forward_core(ctx, h, act, cache)
        delta = ctx.ws.alloc((T, self.H), torch.float32)
        linear(ctx, act, self.w_out, delta)
        return delta


register_part("mixer", "gated_delta_rule", GatedDeltaRule)
