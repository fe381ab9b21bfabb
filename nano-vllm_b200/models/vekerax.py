"""Vekerax: windowed softmax attention and decayed linear attention layers over hyper-connected residual streams.

Data flow of one layer (all residual arithmetic in fp32, activations between the launches in the model's dtype):

  stream launch   mix streams, add the previous sublayer's output, combine, norm1
  mixer           attention: qkv projection with q/k head norm and K/V scatter, window attention, o projection
                  lightning: q/k/v/gate projection with SiLU in the epilogue, linear attention, gated norm, o projection
  stream launch   the same for the mixer's output, with norm2
  feed-forward    gate/up projection with relu(gate) * up in the epilogue, down projection

A range of layers may run several times with the same weights; every run has its own cache or state.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch
from torch import nn

from .. import _abi, ops
from ..layers.attention import PagedKV, WindowAttention
from ..layers.embed_head import TiedEmbedding
from ..layers.linear import MergedColumnParallelLinear, MergeHeadsLinear, _tp_rank_world, pad8
from ..layers.linear_attention import DecayedLinearAttention, RecurrentState
from ..layers.streams import StreamConnection, StreamNorm
from ..utils.loader import load_exactly


@dataclass
class VekeraxConfig:
    vocab_size: int
    width: int
    streams: int
    layers: list[dict]
    norm_eps: float
    residual_mult: float
    embedding_scale: float
    loop: dict | None = None
    eos_token_id: int | None = None
    architecture: str = field(default="Vekerax", init=False)

    @classmethod
    def from_dict(cls, d: dict) -> "VekeraxConfig":
        cfg = cls(vocab_size=d["vocab"], width=d["width"], streams=d["streams"], layers=d["layers"], norm_eps=d["norm"]["eps"],
                  residual_mult=d["residual_mult"], embedding_scale=d["embedding"]["scale"], loop=d.get("loop"), eos_token_id=d.get("eos_token_id"))
        for i, l in enumerate(cfg.layers):
            if l["type"] not in ("attention", "lightning"):
                raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
            if l.get("mlp") is not None and l["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {l['mlp']['kind']!r}")
        return cfg

    @property
    def hidden_size(self) -> int:
        """Stored row length of the model's activations."""
        return pad8(self.width)

    @property
    def logits_size(self) -> int:
        """Stored row length of the logits."""
        return pad8(self.vocab_size)

    def layer_runs(self) -> list[int]:
        """Layer numbers in the order they run."""
        n = len(self.layers)
        if not self.loop:
            return list(range(n))
        start, stop, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def widest(self) -> int:
        """Elements per token of the widest activation, in bf16 units (the fp32 streams count twice)."""
        w = [2 * self.streams * self.hidden_size]
        for l in self.layers:
            m = l["mixer"]
            if l["type"] == "attention":
                w.append((m["heads"] + m["kv_heads"]) * pad8(m["dim"]) + m["kv_heads"] * pad8(m["vdim"]))
            else:
                w.append(2 * m["heads"] * (pad8(m["dim"]) + pad8(m["vdim"])))
            if l.get("mlp") is not None:
                w.append(2 * pad8(l["mlp"]["ff"]))
        return max(w)


class VekeraxMLP(nn.Module):

    def __init__(self, width: int, ff: int) -> None:
        super().__init__()
        self.width, self.ff = width, ff
        self.gate_up_proj = MergedColumnParallelLinear(pad8(width), [pad8(ff)] * 2, bias=False).pair_rows()
        self.gate_up_proj.weight.data.zero_()
        self.down_proj = MergeHeadsLinear(1, ff, width)

    def load_gate_up(self, shard_id: int, w: torch.Tensor) -> None:
        full = torch.zeros(pad8(self.ff), pad8(self.width), dtype=w.dtype, device=w.device)
        full[:self.ff, :self.width] = w
        self.gate_up_proj.weight_loader(self.gate_up_proj.weight, full, shard_id)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return self.down_proj(ops.gemm_act_mul(x, self.gate_up_proj.paired_weight(), _abi.ACT_RELU))


class VekeraxLayer(nn.Module):

    def __init__(self, config: VekeraxConfig, spec: dict) -> None:
        super().__init__()
        c, m = config, spec["mixer"]
        self.kind = spec["type"]
        if self.kind == "attention":
            self.mixer = WindowAttention(c.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["softcap"], m["mask"]["size"],
                                         m["mask"]["keep_first"], c.norm_eps)
        else:
            self.mixer = DecayedLinearAttention(c.width, m["heads"], m["dim"], m["vdim"], m["decay"], c.norm_eps)
        self.mlp = VekeraxMLP(c.width, spec["mlp"]["ff"]) if spec.get("mlp") is not None else None
        self.norm1 = StreamNorm(c.width, c.hidden_size, c.norm_eps)
        self.hc1 = StreamConnection(c.streams)
        if self.mlp is not None:
            self.norm2 = StreamNorm(c.width, c.hidden_size, c.norm_eps)
            self.hc2 = StreamConnection(c.streams)

    def new_cache(self) -> PagedKV | RecurrentState:
        """Cache or state of one run of this layer."""
        x = self.mixer
        return PagedKV(x.num_kv_heads, x.qk_pad, x.v_pad) if self.kind == "attention" else RecurrentState(x.heads, x.qk_pad, x.v_pad)


class VekeraxForCausalLM(nn.Module):
    runs_in_fp32 = True
    paged_prefill = True  # attention reads K and V from the cache in every step

    def __init__(self, config: VekeraxConfig) -> None:
        super().__init__()
        if _tp_rank_world()[1] != 1:
            raise ValueError("Vekerax runs on one GPU: the norm over its concatenated linear-attention heads is not sharded")
        self.config = config
        self.embed = TiedEmbedding(config.vocab_size, config.width)
        self.layers = nn.ModuleList([VekeraxLayer(config, spec) for spec in config.layers])
        self.final_norm = StreamNorm(config.width, config.hidden_size, config.norm_eps)
        self.runs = [(self.layers[i], self.layers[i].new_cache()) for i in config.layer_runs()]
        # sublayers in the order they run: (connection, norm, call, ends a layer run)
        self.program = []
        for layer, cache in self.runs:
            mixer = layer.mixer
            self.program.append((layer.hc1, layer.norm1, lambda h, f=mixer, c=cache: f(h, c), layer.mlp is None))
            if layer.mlp is not None:
                self.program.append((layer.hc2, layer.norm2, layer.mlp, True))
        self.run_hook = None  # called with the summed streams [tokens, width] after every layer run (inspection only)

    # ---- what the runner binds ----------------------------------------------
    def kv_layers(self) -> list[PagedKV]:
        return [c for _, c in self.runs if isinstance(c, PagedKV)]

    def state_layers(self) -> list[RecurrentState]:
        return [c for _, c in self.runs if isinstance(c, RecurrentState)]

    def activation_width(self) -> int:
        return self.config.widest()

    @property
    def fused_sampling(self) -> bool:
        return self.embed.fused_sampling

    # ---- forward ----------------------------------------------------------------
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        c, prog = self.config, self.program
        conn, norm, call, ends = prog[0]
        x, h = norm.start(input_ids, self.embed.weight, c.embedding_scale, c.streams, conn)
        for i in range(len(prog)):
            conn, _, call, ends = prog[i]
            y = call(h)
            last = i + 1 == len(prog)
            nxt_norm, w_in = (self.final_norm, None) if last else (prog[i + 1][1], prog[i + 1][0].w_in)
            h = nxt_norm.step(x, y, conn, c.residual_mult, w_in, store=not last or self.run_hook is not None)
            if self.run_hook is not None and ends:
                self.run_hook(x.sum(1)[:, :c.width])
        return h

    def compute_logits(self, hidden_states: torch.Tensor) -> torch.Tensor:
        return self.embed.head(hidden_states)

    def logits_of_rows(self, hidden_states: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
        return self.embed.logits(hidden_states, rows)

    def sample_tokens(self, hidden_states: torch.Tensor, temperatures: torch.Tensor | None, seed: int, out: torch.Tensor | None = None):
        return self.embed.head_sample(hidden_states, temperatures, seed, out)

    # ---- weights ------------------------------------------------------------------
    def weight_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of a checkpoint of this configuration, by name."""
        c, s = self.config, self.config.streams
        out = {"embed": (c.vocab_size, c.width), "final.norm": (c.width,)}
        for i, l in enumerate(c.layers):
            m, p = l["mixer"], f"l{i}."
            subs = [("hc1", "norm1")] + ([("hc2", "norm2")] if l.get("mlp") is not None else [])
            for hc, norm in subs:
                out.update({p + norm: (c.width,), p + hc + ".in": (s,), p + hc + ".out": (s,), p + hc + ".mix": (s, s)})
            h, d, v = m["heads"], m["dim"], m["vdim"]
            g = h if l["type"] == "lightning" else m["kv_heads"]
            out.update({p + "mix.q": (h * d, c.width), p + "mix.k": (g * d, c.width), p + "mix.v": (g * v, c.width), p + "mix.o": (c.width, h * v)})
            if l["type"] == "lightning":
                out.update({p + "mix.g": (h * v, c.width), p + "mix.norm": (h * v,)})
            else:
                out.update({p + "mix.q.norm": (d,), p + "mix.k.norm": (d,), p + "mix.sink": (h,)})
            if l.get("mlp") is not None:
                ff = l["mlp"]["ff"]
                out.update({p + "mlp.gate": (ff, c.width), p + "mlp.up": (ff, c.width), p + "mlp.down": (c.width, ff)})
        return out

    def load_weight(self, name: str, w: torch.Tensor) -> None:
        """One checkpoint tensor into the parameter it belongs to."""
        def put(param, *shard):
            loader = getattr(param, "weight_loader", None)
            w_dev = w.to(param.device)
            loader(param, w_dev, *shard) if loader is not None else param.data.copy_(w_dev)

        if name == "embed":
            return put(self.embed.weight)
        if name == "final.norm":
            return put(self.final_norm.weight)
        head, rest = name.split(".", 1)
        layer = self.layers[int(head[1:])]
        if rest in ("norm1", "norm2"):
            return put(getattr(layer, rest).weight)
        part, leaf = rest.split(".", 1)
        if part in ("hc1", "hc2"):
            return put(getattr(getattr(layer, part), {"in": "w_in", "out": "w_out", "mix": "mix"}[leaf]))
        if part == "mlp":
            if leaf == "down":
                return put(layer.mlp.down_proj.weight)
            return layer.mlp.load_gate_up({"gate": 0, "up": 1}[leaf], w.to(layer.mlp.gate_up_proj.weight.device))
        mixer = layer.mixer
        if leaf == "o":
            return put(mixer.o_proj.weight)
        if layer.kind == "attention":
            if leaf in "qkv":
                return put(mixer.qkv_proj.weight, "qkv".index(leaf))
            return put({"q.norm": mixer.q_norm, "k.norm": mixer.k_norm, "sink": mixer.sink}[leaf])
        return put(mixer.norm_weight) if leaf == "norm" else put(mixer.in_proj.weight, "qkvg".index(leaf))

    def load_full_weights(self, weights) -> None:
        load_exactly(self, weights)

    def random_init_(self, seed: int) -> None:
        """Seeded weights generated on the device: N(0, 0.02) matrices, unit norms, streams that stay alike in size."""
        g = torch.Generator(device="cuda").manual_seed(seed * 1000)
        s = self.config.streams
        for name, shape in self.weight_shapes().items():
            if "norm" in name:
                w = torch.ones(shape, device="cuda")
            elif name.endswith((".in", ".mix")) and ".hc" in name:
                w = torch.full(shape, 1.0 / s, device="cuda")
            elif name.endswith(".out"):
                w = torch.ones(shape, device="cuda")
            elif name.endswith("sink"):
                w = torch.zeros(shape, device="cuda")
            else:
                w = torch.empty(shape, dtype=torch.float32, device="cuda").normal_(0, 0.02, generator=g)
            self.load_weight(name, w)
