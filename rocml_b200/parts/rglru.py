"""A recurrent block around a real-gated linear recurrent unit (Griffin's): one state number a channel.

    y = gelu_tanh(Wy h + by)                                  the branch that multiplies the result
    u = causal convolution(Wx h + bx) + bc                    per channel over the last ``conv_taps`` tokens
    r = sigmoid(Ra u + ba),  i = sigmoid(Ri u + bi)           block-diagonal: ``blocks`` square matrices over equal parts of u
    log a = -DECAY_RATE * r * softplus(lam)
    S_t = a S_(t-1) + sqrt(1 - a^2) i u                       zero when the sequence starts
    out = Wo (S * y)

What a sequence keeps, whatever its length: S and the convolution's last inputs, both 32-bit.  One stacked product makes both branches;
one kernel convolves; prompts then take one kernel for the gates and one that scans (runs of tokens side by side), single tokens one
kernel for everything.  From the projections on everything is 32-bit, the block products too."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels
from ..cache.requirements import BundleRequirement, StateRequirement
from ..config.specs import MixerSpec, tensor_names
from ..errors import ConfigError
from ..profile import scope
from ..weights.decl import TensorDecl
from .base import BuildEnv, DeferredNorm, Mixer, register_mixer
from .linear import Linear

DECAY_RATE = 8.0

TENSOR_NAMES = {"y": "y_proj", "x": "x_proj", "conv": "conv", "ra": "r_gate", "ri": "i_gate", "lam": "lambda", "o": "o_proj"}


@register_mixer("rg_lru")
class RealGatedLRU(Mixer):
    graph_safe = True

    def __init__(self, spec: MixerSpec, hidden: int, env: BuildEnv):
        p = spec.params
        self.env = env
        self.hidden = hidden
        self.width = int(p["width"])
        self.blocks = int(p.get("blocks", 1))
        self.taps = int(p.get("conv_taps", 1))
        self.rate_scale = float(p.get("decay_rate", DECAY_RATE))
        if min(self.width, self.blocks) <= 0 or self.width % self.blocks:
            raise ConfigError(f"rg_lru: {self.width} channels do not split in {self.blocks} equal parts")
        if not 1 <= self.taps <= kernels.CONV_MAX_TAPS:
            raise ConfigError(f"rg_lru: a convolution of {self.taps} taps is not built (1 to {kernels.CONV_MAX_TAPS})")
        if spec.position.kind != "none":
            raise ConfigError("rg_lru: a position encoding inside the mixer is not part of it")
        self.part = self.width // self.blocks
        try:
            self.names = n = tensor_names(p, TENSOR_NAMES)
        except ValueError as e:
            raise ConfigError(f"rg_lru: {e}") from None
        self.in_stems, self.in_outs, self.out_width = [n["y"], n["x"]], [self.width, self.width], self.width
        self.in_biased = list(self.in_stems)
        self.proj = Linear(self.in_stems, self.in_outs, hidden, True, env)
        self.o = Linear([n["o"]], [hidden], self.width, False, env)
        self.conv_w = self.conv_b = self.ra = self.ri = self.ra_b = self.ri_b = None
        self.rate: Optional[torch.Tensor] = None          # float32 [width]: -DECAY_RATE * softplus(lam)
        self.result_factor = 1.0

    def cache_requirement(self):
        main = StateRequirement((self.width,), torch.float32)
        if self.taps == 1:
            return main
        return BundleRequirement.of(main, conv=StateRequirement((self.taps - 1, self.width), torch.float32))

    # ---- tensors ------------------------------------------------------------------------------------
    def _small(self, prefix: str):
        n, w, square = self.names, (self.width,), (self.blocks, self.part, self.part)
        return [("conv_w", f"{prefix}{n['conv']}.weight", (self.width, self.taps), "matrix"), ("conv_b", f"{prefix}{n['conv']}.bias", w, "bias"),
                ("ra", f"{prefix}{n['ra']}.weight", square, "matrix"), ("ra_b", f"{prefix}{n['ra']}.bias", square[:2], "bias"),
                ("ri", f"{prefix}{n['ri']}.weight", square, "matrix"), ("ri_b", f"{prefix}{n['ri']}.bias", square[:2], "bias"),
                ("lam", f"{prefix}{n['lam']}.weight", w, "norm")]

    def declare_inner(self, prefix: str) -> List[TensorDecl]:
        """The tensors beside the input and the output product."""
        return [TensorDecl(name, shape, role) for _, name, shape, role in self._small(prefix)]

    def declare(self, prefix: str) -> List[TensorDecl]:
        return self.proj.declare(prefix) + self.o.declare(prefix) + self.declare_inner(prefix)

    def load_inner(self, tensors: Dict[str, torch.Tensor], prefix: str) -> None:
        t = {attr: tensors[name] for attr, name, _, _ in self._small(prefix)}
        self.conv_w, self.conv_b = t["conv_w"].float().contiguous(), t["conv_b"].float().contiguous()
        self.ra, self.ri = t["ra"], t["ri"]
        if self.ra.dtype != self.ri.dtype:
            self.ra, self.ri = self.ra.float(), self.ri.float()
        self.ra, self.ri = self.ra.contiguous(), self.ri.contiguous()
        self.ra_b, self.ri_b = t["ra_b"].float().reshape(-1).contiguous(), t["ri_b"].float().reshape(-1).contiguous()
        self.rate = (-self.rate_scale * torch.nn.functional.softplus(t["lam"].double())).float().contiguous()

    def load(self, tensors: Dict[str, torch.Tensor], prefix: str) -> None:
        self.proj.load(tensors, prefix)
        self.proj.pad_rows(8)
        self.o.load(tensors, prefix)
        self.load_inner(tensors, prefix)

    # ---- accounts -------------------------------------------------------------------------------------
    def inner_bytes(self) -> int:
        esz = self.ra.element_size() if self.ra is not None else (4 if self.env.mode == "float32" else 2)
        return 2 * self.width * self.part * esz + 4 * self.width * (self.taps + 4)

    def weight_bytes(self) -> int:
        return self.proj.weight_bytes() + self.o.weight_bytes() + self.inner_bytes()

    def inner_workspace(self, n_tokens: int) -> int:
        return n_tokens * self.width * (12 + (4 if self.env.mode == "float32" else 2))

    def workspace_bytes(self, n_tokens: int) -> int:
        esz = 4 if self.env.mode == "float32" else 2
        parts = 8 if n_tokens <= 128 else 1
        return n_tokens * (self.proj.n * max(esz, 4 * parts if parts > 1 else esz) + self.hidden * 4 * parts) + self.inner_workspace(n_tokens)

    def inner_cost(self, q_lens, kv_lens):
        T = sum(q_lens)
        live = sum(1 for n in q_lens if n > 0)
        return self.inner_bytes() + T * self.width * 16 + 8 * live * self.width, T * self.width * (4 * self.part + 2 * self.taps + 30)

    def cost(self, q_lens, kv_lens):
        T = sum(q_lens)
        parts = [self.proj.cost(T), self.o.cost(T), self.inner_cost(q_lens, kv_lens)]
        return sum(p[0] for p in parts), sum(p[1] for p in parts)

    # ---- the pass -------------------------------------------------------------------------------------
    def mix_rows(self, proj, batch, view, out=None):
        """The rows that the output product reads, from the layer's projection rows ([T, >= 2 * width], or float32 partial sums
        [S, T, ..]).  ``out`` [T, width] (any row stride) receives them if given."""
        T = batch.n_tokens
        dev = self.env.device
        u = torch.empty((T, self.width), dtype=torch.float32, device=dev)
        with scope(op="causal_conv"):
            kernels.causal_conv(proj, T, self.width, self.width, self.taps, self.conv_w, self.conv_b, "none",
                                view.extras["conv"].state if self.taps > 1 else None, batch.seq_slot, batch.cu_q, batch.n_seqs,
                                batch.max_q_len, u)
        if out is None:
            out = torch.empty((T, self.width), dtype=self.env.act_dtype, device=dev)
        weights = (self.ra, self.ri, self.ra_b, self.ri_b, self.rate)
        if batch.is_decode:
            with scope(op="rglru_step"):
                kernels.rglru_step(u, T, *weights, proj[..., :self.width], self.result_factor, view.state, batch.slot_of_token, out)
            return out
        ax = torch.empty((T, self.width, 2), dtype=torch.float32, device=dev)
        with scope(op="rglru_gates"):
            kernels.rglru_gates(u, T, *weights, ax)
        with scope(op="rglru_scan"):
            kernels.rglru_scan(ax, T, proj[..., :self.width], self.result_factor, view.state, batch.seq_slot, batch.cu_q, batch.n_seqs, out)
        return out

    def forward(self, xn, batch, view):
        T = batch.n_tokens
        if isinstance(xn, DeferredNorm):
            xn = xn.materialize()
        return self.o.forward_delta(self.mix_rows(self.proj.forward_auto(xn, T), batch, view), T)
