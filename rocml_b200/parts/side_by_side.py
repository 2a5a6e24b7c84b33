"""Two mixers side by side: both read the same input, result = left_scale * left + right_scale * right, or, with ``out_norms``,
result = out_factor * (rms(left) * w_left + rms(right) * w_right): each side normalised over the model width with a weight of its own.

With ``out_norms`` the sides keep output products of their own, and the two norms and the sum are left to the consumer, which may do
them in its own kernel (``NormedPair``).  Otherwise both products are shared.  The two share one input product (their column blocks lie behind one another) and one output product: the rows that
each mixer's output product would read lie side by side in one row, and the output weight is [Wo_left | Wo_right],
so that the sum over the inner size adds the two results.  The constants: right_scale / left_scale rides on the right
mixer's last 32-bit factor (``result_factor``), left_scale on the whole result, which a consumer may apply itself
(``ScaledDelta``); no weight is rounded again.

A mixer can stand on a side when it shows its input product's column blocks (``in_stems``, ``in_outs``), makes the output
product's rows from such columns (``mix_rows``, ``out_width``) and names its other tensors and accounts (``declare_inner``,
``load_inner``, ``inner_bytes``, ``inner_workspace``, ``inner_cost``); the right one needs ``result_factor`` as well.  What
the two keep per sequence becomes one bundle: the left one's requirement, and the right one's fixed-size states under the
names ``right_<name>``."""
from __future__ import annotations

from typing import Dict, List

import torch

from .. import kernels
from ..cache.requirements import BundleRequirement, StateRequirement
from ..cache.sequence_cache import CacheView
from ..config.specs import MixerSpec
from ..errors import ConfigError
from ..profile import scope
from ..weights.decl import TensorDecl
from .base import BuildEnv, DeferredNorm, Mixer, NormedPair, ScaledDelta, build_mixer, register_mixer
from .linear import Linear

SIDES = ("left", "right")


@register_mixer("side_by_side")
class SideBySide(Mixer):
    scales_later = True         # forward() accepts scale_later=True and may then return a ScaledDelta
    norms_later = True          # ... and norm_later=True, and may then return a NormedPair

    def __init__(self, spec: MixerSpec, hidden: int, env: BuildEnv):
        p = spec.params
        self.env = env
        self.hidden = hidden
        self.prefixes = {s: dict(p.get("prefixes") or ()).get(s, f"{s}.") for s in SIDES}
        self.scales = (float(p.get("left_scale", 1.0)), float(p.get("right_scale", 1.0)))
        self.left = build_mixer(p["left"], hidden, env)
        self.right = build_mixer(p["right"], hidden, env)
        self.out_norms = bool(p.get("out_norms", False))
        self.out_norm_eps = float(p.get("out_norm_eps", 1e-6))
        self.out_factor = float(p.get("out_factor", 0.5))
        if self.out_norms and self.scales != (1.0, 1.0):
            raise ConfigError("side_by_side: a side's scale is lost in the norm that follows it")
        for side, m in zip(SIDES, (self.left, self.right)):
            if not hasattr(m, "mix_rows") or (side == "right" and not self.out_norms and not hasattr(m, "result_factor")):
                raise ConfigError(f"side_by_side: the {side} mixer cannot stand on that side")
        states = self.right.cache_requirement()
        main = states.main if isinstance(states, BundleRequirement) else states
        if not isinstance(main, StateRequirement):
            raise ConfigError("side_by_side: the right mixer must keep states of fixed size")
        # left_scale multiplies the whole result, the right side's share of it is right_scale / left_scale
        left, right = self.scales
        self.factor = left if left != 0.0 else 1.0
        if not self.out_norms:
            self.right.result_factor = right / left if left != 0.0 else right
            if self.left.o.has_bias or self.right.o.has_bias:
                raise ConfigError("side_by_side: biases on the output products need out_norms (each side's product on its own)")
        self.split = sum(self.left.in_outs)
        stems = [f"{self.prefixes[s]}{n}" for s, m in zip(SIDES, (self.left, self.right)) for n in m.in_stems]
        biased = [f"{self.prefixes[s]}{n}" for s, m in zip(SIDES, (self.left, self.right)) for n in getattr(m, "in_biased", ())]
        self.proj = Linear(stems, list(self.left.in_outs) + list(self.right.in_outs), hidden, biased, env)
        self.o = Linear(["o"], [hidden], self.left.out_width + self.right.out_width, False, env)      # (not used with out_norms)
        self.o.label = "o"
        self.out_stem = (p.get("out_stem") or "out")
        self.out_w = {}

    @property
    def graph_safe(self) -> bool:
        return self.left.graph_safe and self.right.graph_safe

    def cache_requirement(self):
        req = self.right.cache_requirement()
        main, extras = (req.main, dict(req.extras)) if isinstance(req, BundleRequirement) else (req, {})
        return BundleRequirement.of(self.left.cache_requirement(), right_state=main, **{f"right_{k}": v for k, v in extras.items()})

    def declare(self, prefix: str) -> List[TensorDecl]:
        out = self.proj.declare(prefix)
        for s, m in zip(SIDES, (self.left, self.right)):
            out += m.o.declare(prefix + self.prefixes[s]) + m.declare_inner(prefix + self.prefixes[s])
            if self.out_norms:
                out.append(TensorDecl(f"{prefix}{self.prefixes[s]}{self.out_stem}.weight", (self.hidden,), "norm"))
        return out

    def load(self, tensors: Dict[str, torch.Tensor], prefix: str) -> None:
        self.proj.load(tensors, prefix)
        self.proj.pad_rows(8)
        outs = []
        for s, m in zip(SIDES, (self.left, self.right)):
            m.load_inner(tensors, prefix + self.prefixes[s])
            if self.out_norms:
                m.o.load(tensors, prefix + self.prefixes[s])
                self.out_w[s] = tensors[f"{prefix}{self.prefixes[s]}{self.out_stem}.weight"].float().contiguous()
                continue
            outs.append(tensors[f"{prefix}{self.prefixes[s]}{m.o.names[0]}.weight"])
        if self.out_norms:
            return
        if self.scales[0] == 0.0:
            outs[0] = torch.zeros_like(outs[0])
        if outs[0].dtype != outs[1].dtype:
            outs = [w.float() for w in outs]
        self.o.weight = torch.cat(outs, dim=1).contiguous()

    def weight_bytes(self) -> int:
        o = self.left.o.weight_bytes() + self.right.o.weight_bytes() if self.out_norms else self.o.weight_bytes()
        return self.proj.weight_bytes() + o + self.left.inner_bytes() + self.right.inner_bytes()

    def workspace_bytes(self, n_tokens: int) -> int:
        esz = 4 if self.env.mode == "float32" else 2
        parts = 8 if n_tokens <= 128 else 1
        return n_tokens * (self.proj.n * max(esz, 4 * parts if parts > 1 else esz) + self.hidden * 4 * parts * (2 if self.out_norms else 1) + self.o.k * esz) + \
            self.left.inner_workspace(n_tokens) + self.right.inner_workspace(n_tokens)

    def cost(self, q_lens, kv_lens):
        T = sum(q_lens)
        parts = [self.proj.cost(T), self.o.cost(T), self.left.inner_cost(q_lens, kv_lens), self.right.inner_cost(q_lens, kv_lens)]
        return sum(p[0] for p in parts), sum(p[1] for p in parts)

    def forward(self, xn, batch, view, scale_later=False, norm_later=False):
        T = batch.n_tokens
        if isinstance(xn, DeferredNorm):
            xn = xn.materialize()
        proj = self.proj.forward_auto(xn, T)
        state = view.extras["right_state"]
        right_view = CacheView("state", state.group, state.index, view.writes,
                               {n[len("right_"):]: v for n, v in view.extras.items() if n.startswith("right_") and n != "right_state"})
        if self.out_norms:
            left = self.left.o.forward_delta(self.left.mix_rows(proj[..., :self.split], batch, view), T)
            right = self.right.o.forward_delta(self.right.mix_rows(proj[..., self.split:], batch, right_view), T)
            pair = NormedPair(left, right, self.out_w["left"], self.out_w["right"], self.out_norm_eps, self.out_factor)
            return pair if norm_later else pair.materialize()
        rows = torch.empty((T, self.o.k), dtype=self.env.act_dtype, device=self.env.device)
        self.left.mix_rows(proj[..., :self.split], batch, view, rows[:, :self.left.out_width])
        self.right.mix_rows(proj[..., self.split:], batch, right_view, rows[:, self.left.out_width:])
        delta = self.o.forward_delta(rows, T)
        if self.factor == 1.0:
            return delta
        if scale_later:
            return ScaledDelta(delta, self.factor)
        with scope(op="scale"):
            kernels.scale_(delta, self.factor)
        return delta
