"""Subivik: a decoder with an fp32 residual stream, an element-wise norm (Dynamic Tanh) in front of every sublayer, and layers
that take either capped attention with heads mixed after the softmax beside RWKV time mixing, or differential attention in
chunks of the sequence, perhaps over an earlier layer's keys and values; feed-forwards are dense (xIELU), a mixture of experts
(silu), or absent.

    x = embed[token] + sinusoids of the position
    x += mixer(norm1(x));  x += feed_forward(norm2(x))
    logits = embed final_norm(x)

Every size and constant is read from the configuration or a tensor's shape.  The mixers and feed-forwards are the modules of
layers/; the addition of a sublayer's result and the norm in front of the next are one launch.
"""
from dataclasses import dataclass

import torch
import torch.nn as nn
import torch.nn.functional as F

from ..layers.diff_attention import DifferentialAttention
from ..layers.mlp import XieluMLP
from ..layers.moe import MixtureOfExperts
from ..layers.parallel import ScaledMixers
from ..layers.talk_attention import TalkingAttention
from ..layers.tanh_norm import TanhEntry, position_frequencies, tanh_embed, tanh_step
from ..layers.time_mix import TimeMixing
from ..utils.context import get_context
from .weights import RandomWeights

MIXERS = ("parallel", "attention")
FEED_FORWARDS = {
    "dense": XieluMLP,
    "moe": lambda spec, width, load: MixtureOfExperts(spec, width, load, router_bias=False, over_all=True),
}

# spread of seeded weights: vectors whose natural centre is not zero
_VECTOR_INIT = {"norm": (1.0, 0.1), "norm1": (1.0, 0.1), "norm2": (1.0, 0.1), ".alpha": (0.7, 0.1), ".r1": (0.5, 0.1),
                ".r2": (0.5, 0.1), "mu.r": (0.5, 0.1), "mu.k": (0.5, 0.1), "mu.v": (0.5, 0.1), "mu.g": (0.5, 0.1),
                "mu.w": (0.5, 0.1), ".w0": (-3.0, 1.5), ".act": (0.5, 0.2)}


@dataclass
class SubivikConfig:
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    max_position: int = 4096

    @staticmethod
    def from_dict(c):
        layers = c["layers"]
        for i, l in enumerate(layers):
            if l["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer '{l['type']}' (known: {', '.join(MIXERS)})")
            if l.get("mlp") and l["mlp"].get("kind") not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward '{l['mlp'].get('kind')}'")
            j = l["mixer"].get("kv_from")
            if j is not None and not (0 <= j < i and layers[j]["type"] == "attention"):
                raise ValueError(f"layer {i}: kv_from {j} names no attention layer before it")
        return SubivikConfig(vocab_size=c["vocab"], hidden_size=c["width"], layers=layers, norm_eps=c["norm"]["eps"],
                             max_position=c.get("max_position", c.get("max_model_length", 4096)))

    @property
    def num_layers(self):
        return len(self.layers)

    def widest_activation(self):
        """Elements per token of the widest stage of a layer, for the activation reserve of the cache pool."""
        wide, lent = 0, {l["mixer"]["kv_from"] for l in self.layers if l["mixer"].get("kv_from") is not None}
        for l in self.layers:
            m, e = l["mixer"], l.get("mlp")
            if l["type"] == "parallel":
                a, b = m["left"], m["right"]
                n = a["heads"] * (a["dim"] + (a["kv_heads"] + 1) * a["vdim"]) + 3 * a["kv_heads"] * (a["dim"] + a["vdim"]) + \
                    10 * b["heads"] * b["dim"] + 5 * self.hidden_size
            else:
                n = m["heads"] * (2 * m["dim"] + 2 * m["vdim"]) + 2 * m["kv_heads"] * (2 * m["dim"] + m["vdim"])
            if e and e["kind"] == "dense":
                n = max(n, 2 * e["ff"])
            elif e:
                n = max(n, e["router"]["top"] * (2 * self.hidden_size + e["expert"]["ff"]))
            wide = max(wide, n)
        kept = sum(m["kv_heads"] * (2 * m["dim"] + m["vdim"]) for m in (self.layers[j]["mixer"] for j in lent))
        return wide + kept + 8 * self.hidden_size


class SubivikLayer(nn.Module):
    """`before`: the layers in front of this one."""

    def __init__(self, cfg, index, load, before):
        super().__init__()
        spec, W = cfg.layers[index], cfg.hidden_size
        m, mix = spec["mixer"], load.scoped("mix.")
        if spec["type"] == "parallel":
            self.mixer = ScaledMixers(m, W, cfg.norm_eps, mix, left=TalkingAttention, right=TimeMixing)
        else:
            source = before[m["kv_from"]].mixer if m.get("kv_from") is not None else None
            self.mixer = DifferentialAttention(m, W, cfg.norm_eps, mix, source)
        self.entry1 = tanh_entry(load, "norm1", W, self.mixer.shift)
        self.mlp = self.entry2 = None
        if spec.get("mlp"):
            self.entry2 = tanh_entry(load, "norm2", W)
            self.mlp = FEED_FORWARDS[spec["mlp"]["kind"]](spec["mlp"], W, load.scoped("mlp."))

    def forward(self, inputs, x, after):
        """inputs: what this layer's entry gave, x: the fp32 stream, after: entry of what follows.  Returns the new stream and
        what `after` gives."""
        x, h = tanh_step(x, self.mixer(inputs), after if self.mlp is None else self.entry2)
        if self.mlp is not None:
            x, h = tanh_step(x, self.mlp.routed(h) if isinstance(self.mlp, MixtureOfExperts) else self.mlp(h), after)
        return x, h


def tanh_entry(load, name, width, shift=None):
    return TanhEntry(load(name + ".alpha", ()), load(name, (width,)), load(name + ".b", (width,)), shift)


class SubivikForCausalLM(nn.Module):
    mixed_steps = True       # every prefill step goes through the paged cache and the state slots
    tensor_parallel = False

    def __init__(self, cfg: SubivikConfig, tp_rank=0, tp_size=1, dtype=torch.bfloat16, device="cuda", seed=0,
                 weights=None):
        super().__init__()
        if tp_size != 1:
            raise ValueError("Subivik runs on one GPU")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Subivik runs in bfloat16 or float32")
        w = weights if weights is not None else RandomWeights(seed, dtype, device, _VECTOR_INIT)
        self.cfg, self.dtype, self.comm = cfg, dtype, None
        V, W = cfg.vocab_size, cfg.hidden_size
        self.embed = nn.Parameter(w("embed", (V, W)), requires_grad=False)
        self.lm_head = self.embed        # tied
        self.inv_freq = position_frequencies(W, self.embed.device)
        self.head_entry = tanh_entry(w, "final.norm", W)
        self.layers = nn.ModuleList()
        for i in range(cfg.num_layers):
            self.layers.append(SubivikLayer(cfg, i, w.scoped(f"l{i}."), list(self.layers)))
        w.check_all_used()
        self.layer_probe = None      # tests: called with (layer index, residual stream) after every layer

    def forward(self, input_ids):
        """input_ids (tokens,) int64 -> hidden (tokens, width); positions, slots and tables come from the Context."""
        if get_context().positions is None:
            raise ValueError("Context.positions must be set before the model runs")
        entries = [l.entry1 for l in self.layers] + [self.head_entry]
        x, h = tanh_embed(input_ids, self.embed, entries[0], self.inv_freq)
        for i, layer in enumerate(self.layers):
            x, h = layer(h, x, entries[i + 1])
            if self.layer_probe is not None:
                self.layer_probe(i, x)
        return h

    def compute_logits(self, hidden, vocab_shard=None):
        """Rows named by Context.last_token_index when it is set, all rows otherwise."""
        ctx = get_context()
        if ctx.last_token_index is not None:
            hidden = hidden[ctx.last_token_index]
        if vocab_shard is not None:
            raise ValueError("Subivik's head is not sharded")
        return F.linear(hidden, self.lm_head)
