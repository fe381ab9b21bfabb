"""Mupulorn: multi-head latent attention and PolyNorm feed-forwards between two norms, a short causal convolution in front of
every sublayer, layers that share weights.

Data flow of one layer (the residual and all norms in fp32, activations between the launches in the model's dtype):

  sandwich launch  norm of the previous sublayer's output, residual sum, norm1, convolution
  mixer            [query latent | latent | rotated key part | gate] projection, norms + rotation + cache, query projection,
                   attention (expanded or absorbed) with a sink and the output gate, output projection
  sandwich launch  the same for the mixer's output, with norm2
  feed-forward     up projection, PolyNorm, down projection

A layer may use another layer's weights; every layer has its own cache and convolution state.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch
from torch import nn

from ..layers.activation import PolyNorm
from ..layers.embed_head import PaddedLMHead, PaddedTable
from ..layers.latent_attention import LatentAttention, PagedLatent
from ..layers.linear import MergeHeadsLinear, _tp_rank_world, pad8
from ..layers.sandwich import CausalConv, GainNorm, first_input, next_input
from ..layers.state import SlotState
from ..utils.loader import load_exactly


@dataclass
class MupulornConfig:
    vocab_size: int
    width: int
    layers: list[dict]
    taps: int
    norm_eps: float
    logit_scale: float
    logit_softcap: float
    eos_token_id: int | None = None
    architecture: str = field(default="Mupulorn", init=False)

    @classmethod
    def from_dict(cls, d: dict) -> "MupulornConfig":
        cfg = cls(vocab_size=d["vocab"], width=d["width"], layers=d["layers"], taps=d["canon"]["taps"], norm_eps=d["norm"]["eps"],
                  logit_scale=d["logit_scale"], logit_softcap=d["logit_softcap"], eos_token_id=d.get("eos_token_id"))
        if cfg.taps < 1:
            raise ValueError(f"a convolution of {cfg.taps} taps")
        for i, l in enumerate(cfg.layers):
            if l["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
            if l.get("mlp") is not None and l["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {l['mlp']['kind']!r}")
            cfg.owner(i)
        return cfg

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = [i]
        while self.layers[seen[-1]].get("weights_of") is not None:
            j = self.layers[seen[-1]]["weights_of"]
            if j in seen or not 0 <= j < len(self.layers):
                raise ValueError(f"layer {i}: no weights at the end of {seen + [j]}")
            seen.append(j)
        return seen[-1]

    @property
    def hidden_size(self) -> int:
        """Stored row length of the model's activations."""
        return pad8(self.width)

    @property
    def logits_size(self) -> int:
        """Stored row length of the logits."""
        return pad8(self.vocab_size)

    def widest(self) -> int:
        """Elements per token of the widest activation, in bf16 units (the fp32 residual counts twice)."""
        w = [2 * self.hidden_size]
        for l in self.layers:
            m = l["mixer"]
            w.append(pad8(m["q_rank"]) + pad8(m["kv_rank"]) + pad8(m["rot_dim"]) + m["heads"] * pad8(m["vdim"]))
            w.append(m["heads"] * max(pad8(m["dim"]) + max(pad8(m["rot_dim"]), pad8(m["vdim"])), pad8(m["kv_rank"]) + pad8(m["rot_dim"])))
            if l.get("mlp") is not None:
                w.append(pad8(l["mlp"]["ff"]))
        return max(w)


class MupulornMLP(nn.Module):

    def __init__(self, width: int, ff: int, eps: float) -> None:
        super().__init__()
        self.up_proj = MergeHeadsLinear(1, width, ff)
        self.act = PolyNorm(ff, eps)
        self.down_proj = MergeHeadsLinear(1, ff, width)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return self.down_proj(self.act(self.up_proj(x)))


class MupulornLayer(nn.Module):
    """The weights of a layer (and of those that share them)."""

    def __init__(self, config: MupulornConfig, spec: dict) -> None:
        super().__init__()
        c, m = config, spec["mixer"]
        self.mixer = LatentAttention(c.width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], m["rot"]["dims"],
                                     m["rot"]["base"], c.norm_eps)
        self.mlp = MupulornMLP(c.width, spec["mlp"]["ff"], c.norm_eps) if spec.get("mlp") is not None else None
        for n in ("1", "2") if self.mlp is not None else ("1",):
            setattr(self, "norm" + n, GainNorm(c.width, c.norm_eps))
            setattr(self, "norm" + n + "b", GainNorm(c.width, c.norm_eps))
            setattr(self, "canon" + n, CausalConv(c.width, c.taps))


@dataclass
class Sublayer:
    """One step of the model: norm and convolution of the residual, the call, the norm of its output."""
    norm: GainNorm
    conv: CausalConv
    state: SlotState
    call: object
    post: GainNorm
    ends_layer: bool


class MupulornForCausalLM(nn.Module):
    runs_in_fp32 = True
    paged_prefill = True  # a portion of a prompt reads its earlier tokens from the cache

    def __init__(self, config: MupulornConfig) -> None:
        super().__init__()
        if _tp_rank_world()[1] != 1:
            raise ValueError("Mupulorn runs on one GPU: its latents and PolyNorm rows are not sharded")
        self.config = config
        self.embed = PaddedTable(config.vocab_size, config.width)
        self.head = PaddedLMHead(config.vocab_size, config.width, config.logit_scale, config.logit_softcap)
        self.layers = nn.ModuleDict({str(i): MupulornLayer(config, spec) for i, spec in enumerate(config.layers) if config.owner(i) == i})
        self.final_norm = GainNorm(config.width, config.norm_eps)
        self.caches: list[PagedLatent] = []
        self.program: list[Sublayer] = []
        for i in range(len(config.layers)):
            layer = self.layers[str(config.owner(i))]
            cache = layer.mixer.new_cache()
            self.caches.append(cache)
            self.program.append(Sublayer(layer.norm1, layer.canon1, layer.canon1.new_state(), lambda h, pos, f=layer.mixer, c=cache: f(h, pos, c),
                                         layer.norm1b, layer.mlp is None))
            if layer.mlp is not None:
                self.program.append(Sublayer(layer.norm2, layer.canon2, layer.canon2.new_state(), lambda h, pos, f=layer.mlp: f(h), layer.norm2b, True))
        self.run_hook = None  # called with the residual [tokens, width] after every layer (inspection only)

    # ---- what the runner binds ----------------------------------------------
    def kv_layers(self) -> list[PagedLatent]:
        return self.caches

    def state_layers(self) -> list[SlotState]:
        return [s.state for s in self.program]

    def activation_width(self) -> int:
        return self.config.widest()

    def bind_positions(self, positions: int) -> None:
        for layer in self.layers.values():
            layer.mixer.rotation.bind(positions, self.embed.weight.device)

    @property
    def fused_sampling(self) -> bool:
        return self.head.fused_sampling

    # ---- forward ----------------------------------------------------------------
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        c, prog = self.config, self.program
        x, h = first_input(input_ids, self.embed.weight, prog[0].norm, prog[0].conv, prog[0].state)
        for i, sub in enumerate(prog):
            y = sub.call(h, positions)
            if i + 1 == len(prog):
                x, h = next_input(x, y, sub.post, self.final_norm, None, None, store=self.run_hook is not None)
            else:
                nxt = prog[i + 1]
                x, h = next_input(x, y, sub.post, nxt.norm, nxt.conv, nxt.state)
            if self.run_hook is not None and sub.ends_layer:
                self.run_hook(x[:, :c.width])
        return h

    def compute_logits(self, hidden_states: torch.Tensor) -> torch.Tensor:
        return self.head.head(hidden_states)

    def logits_of_rows(self, hidden_states: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
        return self.head.logits(hidden_states, rows)

    def sample_tokens(self, hidden_states: torch.Tensor, temperatures: torch.Tensor | None, seed: int, out: torch.Tensor | None = None):
        return self.head.head_sample(hidden_states, temperatures, seed, out)

    # ---- weights ------------------------------------------------------------------
    def weight_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of a checkpoint of this configuration, by name."""
        c = self.config
        out = {"embed": (c.vocab_size, c.width), "final.norm": (), "head": (c.vocab_size, c.width)}
        for i, layer in self.layers.items():
            p = f"l{i}."
            for n in ("1", "2") if layer.mlp is not None else ("1",):
                out.update({p + "norm" + n: (), p + "norm" + n + "b": (), p + "canon" + n: (c.width, c.taps)})
            out.update({p + "mix." + name: shape for name, shape in layer.mixer.weight_shapes(c.width).items()})
            if layer.mlp is not None:
                ff = layer.mlp.act.dim
                out.update({p + "mlp.up": (ff, c.width), p + "mlp.down": (c.width, ff), p + "mlp.act": (4,)})
        return out

    def load_weight(self, name: str, w: torch.Tensor) -> None:
        """One checkpoint tensor into the parameter it belongs to."""
        def put(param):
            loader = getattr(param, "weight_loader", None)
            w_dev = w.to(param.device)
            loader(param, w_dev) if loader is not None else param.data.copy_(w_dev)

        top = {"embed": self.embed, "head": self.head, "final.norm": self.final_norm}
        if name in top:
            return put(top[name].weight)
        head, rest = name.split(".", 1)
        layer = self.layers[head[1:]]
        part, _, leaf = rest.partition(".")
        if part == "mix":
            return layer.mixer.load_weight(leaf, w)
        if part == "mlp":
            return put({"up": layer.mlp.up_proj.weight, "down": layer.mlp.down_proj.weight, "act": layer.mlp.act.coef}[leaf])
        return put(getattr(layer, part).weight)

    def load_full_weights(self, weights) -> None:
        load_exactly(self, weights)

    def random_init_(self, seed: int) -> None:
        """Seeded weights generated on the device: N(0, 0.02) matrices, unit norms, a mild convolution."""
        g = torch.Generator(device="cuda").manual_seed(seed * 1000)
        for name, shape in self.weight_shapes().items():
            if "norm" in name:
                w = torch.ones(shape, device="cuda")
            elif name.endswith("act"):
                w = torch.tensor([0.5, 0.5, 0.5, 0.0], device="cuda")
            elif name.endswith("sink"):
                w = torch.zeros(shape, device="cuda")
            else:
                w = torch.empty(shape, dtype=torch.float32, device="cuda").normal_(0, 0.1 if ".canon" in name else 0.02, generator=g)
            self.load_weight(name, w)
