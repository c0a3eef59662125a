"""Dafotar: a decoder with several residual streams (hyper-connections), layer norms, a convolution over time in front of
every mixer, and layers that take either windowed attention with rotated values, perhaps over an earlier layer's keys and
values, or a matrix memory (mLSTM), with or without a dense feed-forward.

    u = sum_s in[s] x_s;  h = norm1(u);  y = mixer(h + conv(h));  x_t = sum_s mix[s, t] x_s + out[t] y
    the same with norm2 and the feed-forward, without the convolution
    logits = embed final_norm(sum_s x_s)

Every size and constant is read from the configuration.  The mixers, the feed-forward and the streams are modules of
layers/; the update behind a sublayer and the sum and norm in front of the next are one launch.
"""
from dataclasses import dataclass

import torch
import torch.nn as nn
import torch.nn.functional as F

from ..layers.mlp import GatedMLP
from ..layers.mlstm import MatrixMemory
from ..layers.rotary_attention import RotaryWindowAttention
from ..layers.streams import InputConvolution, StreamEntry, stream_embed, stream_step
from ..utils.context import get_context
from .weights import RandomWeights

MIXERS = ("attention", "mlstm")
FEED_FORWARDS = {"dense": lambda spec, width, load: GatedMLP(spec, width, load, act="relu")}

# spread of seeded weights: vectors whose natural centre is not zero
_VECTOR_INIT = {"norm": (1.0, 0.1), "norm1": (1.0, 0.1), "norm2": (1.0, 0.1), "temp": (1.0, 0.1), "f.b": (3.0, 1.0),
                ".in": (0.5, 0.1), ".out": (0.5, 0.1)}


@dataclass
class DafotarConfig:
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    streams: int
    taps: int
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
        if c["streams"] < 1 or c["canon"]["taps"] < 1:
            raise ValueError("streams and canon.taps must be at least 1")
        return DafotarConfig(vocab_size=c["vocab"], hidden_size=c["width"], layers=layers, norm_eps=c["norm"]["eps"],
                             streams=c["streams"], taps=c["canon"]["taps"],
                             max_position=c.get("max_position", c.get("max_model_length", 4096)))

    @property
    def num_layers(self):
        return len(self.layers)

    def widest_activation(self):
        """Elements per token of the widest stage of a layer, for the activation reserve of the cache pool."""
        wide, lent = 0, {l["mixer"]["kv_from"] for l in self.layers if l["mixer"].get("kv_from") is not None}
        for l in self.layers:
            m = l["mixer"]
            if l["type"] == "mlstm":
                n = m["heads"] * (2 * m["dim"] + 6 * m["vdim"])
            else:
                n = m["heads"] * (m["dim"] + m["vdim"]) + 3 * m["kv_heads"] * (m["dim"] + m["vdim"])
            wide = max(wide, n, 3 * l["mlp"]["ff"] if l.get("mlp") else 0)
        kept = sum(m["kv_heads"] * (m["dim"] + m["vdim"]) for m in (self.layers[j]["mixer"] for j in lent))
        return wide + kept + (2 * self.streams + 6) * self.hidden_size


class DafotarLayer(nn.Module):
    """`before`: the layers in front of this one."""

    def __init__(self, cfg, index, load, before):
        super().__init__()
        spec, W, S = cfg.layers[index], cfg.hidden_size, cfg.streams
        m, eps = spec["mixer"], cfg.norm_eps
        param = lambda t: nn.Parameter(t, requires_grad=False)
        conv = InputConvolution(load("canon1", (W, cfg.taps)))
        entry = lambda q, conv=None: StreamEntry(load(f"hc{q}.in", (S,)), load(f"norm{q}", (W,)), load(f"norm{q}.b", (W,)), eps, conv)
        self.entry1, self.mix1, self.out1 = entry(1, conv), param(load("hc1.mix", (S, S))), param(load("hc1.out", (S,)))
        if spec["type"] == "mlstm":
            self.mixer = MatrixMemory(m, W, eps, load.scoped("mix."))
        else:
            source = before[m["kv_from"]].mixer if m.get("kv_from") is not None else None
            self.mixer = RotaryWindowAttention(m, W, eps, load.scoped("mix."), cfg.max_position, source)
        self.mlp = self.entry2 = None
        if spec.get("mlp"):
            self.entry2, self.mix2, self.out2 = entry(2), param(load("hc2.mix", (S, S))), param(load("hc2.out", (S,)))
            self.mlp = FEED_FORWARDS[spec["mlp"]["kind"]](spec["mlp"], W, load.scoped("mlp."))

    def forward(self, h, x, after):
        """h: this layer's input, x: the streams, updated in place, after: entry of what follows.  Returns its input."""
        h = stream_step(x, self.mixer(h), self.mix1, self.out1, after if self.mlp is None else self.entry2)
        if self.mlp is not None:
            h = stream_step(x, self.mlp(h), self.mix2, self.out2, after)
        return h


class DafotarForCausalLM(nn.Module):
    mixed_steps = True       # every prefill step goes through the paged cache and the state slots
    tensor_parallel = False

    def __init__(self, cfg: DafotarConfig, tp_rank=0, tp_size=1, dtype=torch.bfloat16, device="cuda", seed=0,
                 weights=None):
        super().__init__()
        if tp_size != 1:
            raise ValueError("Dafotar runs on one GPU")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Dafotar runs in bfloat16 or float32")
        w = weights if weights is not None else RandomWeights(seed, dtype, device, _VECTOR_INIT)
        self.cfg, self.dtype, self.comm = cfg, dtype, None
        V, W = cfg.vocab_size, cfg.hidden_size
        self.embed = nn.Parameter(w("embed", (V, W)), requires_grad=False)
        self.lm_head = self.embed        # tied
        self.head_entry = StreamEntry(None, w("final.norm", (W,)), w("final.norm.b", (W,)), cfg.norm_eps)
        self.layers = nn.ModuleList()
        for i in range(cfg.num_layers):
            self.layers.append(DafotarLayer(cfg, i, w.scoped(f"l{i}."), list(self.layers)))
        w.check_all_used()
        self.layer_probe = None      # tests: called with (layer index, sum of the streams) after every layer

    def forward(self, input_ids):
        """input_ids (tokens,) int64 -> hidden (tokens, width); positions, slots and tables come from the Context."""
        if get_context().positions is None:
            raise ValueError("Context.positions must be set before the model runs")
        entries = [l.entry1 for l in self.layers] + [self.head_entry]
        x, h = stream_embed(input_ids, self.embed, self.cfg.streams, entries[0])
        for i, layer in enumerate(self.layers):
            h = layer(h, x, entries[i + 1])
            if self.layer_probe is not None:
                self.layer_probe(i, x.sum(1))
        return h

    def compute_logits(self, hidden, vocab_shard=None):
        """Rows named by Context.last_token_index when it is set, all rows otherwise."""
        ctx = get_context()
        if ctx.last_token_index is not None:
            hidden = hidden[ctx.last_token_index]
        if vocab_shard is not None:
            raise ValueError("Dafotar's head is not sharded")
        return F.linear(hidden, self.lm_head)
