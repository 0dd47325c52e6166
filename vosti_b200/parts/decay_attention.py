"""Linear attention with one fixed decay per head: a recurrent mixer. Per request and head it keeps a
float32 matrix S [head_dim, v_head_dim] and per token does

    S <- decay_h S + k v^T;   o = S^T q

with no softmax and no denominator. Parameters: num_heads, head_dim, v_head_dim, `decay` (one constant
in (0, 1] per head), and what surrounds the recurrence:

* `activation` "silu": q, k and v pass SiLU (lightning attention);
* `position`: the `PartSpec` of a rotation (kind "rope", halves paired) of q and k (retention); the
  angles are formed in float32 in the kernels, so positions have no limit;
* `key_scale`: a constant on k (default 1);
* `out_norm` "head": each head's o is divided by its own root mean square (no weight); "all": the
  concatenated heads are normed together, with a plain weight `norm` [num_heads * v_head_dim];
  `eps` inside the root either way;
* `gate_activation` "silu" or "sigmoid" of W_g h multiplies the result, which W_o projects.

One product makes q | k | v | g. The recurrence, rotations, norms and gates are float32 in both serving
types. The state slot of a request holds S for every head; the scheduler hands it out zeroed. Steps of few
tokens a request run token by token, long portions in bfloat16 as chunks side by side
(`ops.decay_attention`). `partial_out`: the output product may stay unsummed for the kernel after it.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch

from .. import ops
from ..config.schema import ConfigError, PartSpec
from ..weights.loader import WeightSpec
from .base import Mixer, PositionEncoding, StateSpec, build_position, register_part, register_step_layout
from .linear import linear, prepare_weight


class DecayAttention(Mixer):
    def __init__(self, spec: PartSpec, hidden_size: int, position: Optional[PositionEncoding]):
        super().__init__(spec, hidden_size, position)
        if position is not None:
            raise ConfigError("decay_attention: the rotation is named by the mixer's own `position` parameter")
        self.heads, self.dk, self.dv = int(spec["num_heads"]), int(spec["head_dim"]), int(spec["v_head_dim"])
        self.decays = tuple(float(d) for d in spec["decay"])
        self.eps, self.key_scale = float(spec["eps"]), float(spec.get("key_scale", 1.0))
        activation, norm, gate = spec.get("activation"), spec.get("out_norm", "head"), spec.get("gate_activation", "sigmoid")
        if activation not in (None, "silu") or norm not in ("head", "all") or gate not in ("silu", "sigmoid"):
            raise ConfigError("decay_attention: activation is 'silu' or none, out_norm 'head' or 'all', gate_activation 'silu' or 'sigmoid'")
        self.silu, self.joint, self.gate_silu = activation == "silu", norm == "all", gate == "silu"
        self.partial_out, self.out_scratch = bool(spec.get("partial_out", False)), "split_k"
        self.rotation = build_position(spec.get("position"), hidden_size, self.dk)
        if self.heads <= 0 or not 0 < self.dk <= 256 or self.dv <= 0:
            raise ConfigError("decay_attention: num_heads and v_head_dim must be positive, head_dim between 1 and 256")
        if len(self.decays) != self.heads or any(not 0.0 < d <= 1.0 for d in self.decays):
            raise ConfigError("decay_attention: one decay in (0, 1] per head")
        if self.rotation is not None and (self.silu or self.rotation.interleaved or not hasattr(self.rotation, "frequencies")):
            raise ConfigError("decay_attention: a rotation pairs halves, gives frequencies and does not go with an activation")
        cq, cv = self.heads * self.dk, self.heads * self.dv
        self.offsets = {"q": 0, "k": cq, "v": 2 * cq, "g": 2 * cq + cv}
        self.w_in = self.w_o = self.norm = self.freq = self.decay = self.log2_decay = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        h, cq, cv = self.hidden_size, self.heads * self.dk, self.heads * self.dv
        specs = {"q": WeightSpec((cq, h)), "k": WeightSpec((cq, h)), "v": WeightSpec((cv, h)), "g": WeightSpec((cv, h)),
                 "o": WeightSpec((h, cv))}
        if self.joint:
            specs["norm"] = WeightSpec((cv,), init="norm", std=0.1)
        return specs

    def load(self, tensors, dtype):
        parts = [tensors[n] for n in ("q", "k", "v", "g")]
        common = torch.float32 if any(p.dtype == torch.float32 for p in parts) else parts[0].dtype
        self.w_in = prepare_weight(torch.cat([p.to(common) for p in parts], dim=0).contiguous(), dtype)
        self.w_o = prepare_weight(tensors["o"], dtype)
        self.norm = tensors["norm"].contiguous() if self.joint else None

    def setup(self, device, dtype):
        self.decay = torch.tensor(self.decays, dtype=torch.float64).to(torch.float32).to(device)
        self.log2_decay = torch.tensor([math.log2(d) for d in self.decays], dtype=torch.float64).to(torch.float32).to(device)
        if self.rotation is not None:
            self.freq = self.rotation.frequencies().to(device=device, dtype=torch.float32).contiguous()

    def first_weight(self):
        return self.w_in

    def state_spec(self) -> StateSpec:
        return StateSpec(((self.heads * self.dk * self.dv + 3) // 4 * 4,), torch.float32)     # slots start on 16-byte boundaries

    def forward(self, ctx, x, cache, writes_cache: bool = True):
        if not writes_cache:
            raise ConfigError("decay_attention: a recurrent state cannot be shared between layer runs")
        # the K splits of a short step's product are added by the kernels that read it
        proj = linear(ctx, x, self.w_in, allow_partial=True)
        if isinstance(proj, ops.PartialSum) and proj.dtype == torch.float32:
            proj = proj.materialize()
        y = ops.decay_attention(proj, self.offsets, cache.state, ctx, heads=self.heads, dk=self.dk, dv=self.dv, decay=self.decay,
                                log2_decay=self.log2_decay, silu=self.silu, key_scale=self.key_scale, freq=self.freq,
                                finish=ops.DecayOut(self.offsets["g"], self.eps, self.norm, self.gate_silu, ctx.dtype))
        return linear(ctx, y, self.w_o, out_dtype=torch.float32, allow_partial=self.partial_out, scratch=self.out_scratch)


register_part("mixer", "decay_attention", DecayAttention, replace=True)
register_step_layout("decay", ops.decay_step_layout)
