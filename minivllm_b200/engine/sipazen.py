"""Sipazen: a decoder whose layers each take one of several mixers (latent attention or a Mamba-2 state space) and a
mixture-of-experts feed-forward, with a grouped RMS norm before and after every sublayer, an element-wise sigmoid
gate on every sublayer's result, and an fp32 residual stream that results enter with a constant factor.

    h = norm1(x);  x += m * norm1b(mixer(h) * sigmoid(W1 h + b1))
    h = norm2(x);  x += m * norm2b(experts(h) * sigmoid(W2 h + b2))
    logits = head final_norm(x)

Every size and constant is read from the configuration.  The mixers and the feed-forward are the modules of
layers/; a layer's norm, gate and residual step is one launch that also writes the next sublayer's input.
"""
from dataclasses import dataclass

import torch
import torch.nn as nn
import torch.nn.functional as F

from ..layers.group_norm import embed_norm, gated_residual_norm
from ..layers.latent_attention import LatentAttention
from ..layers.mamba2 import Mamba2
from ..layers.moe import MixtureOfExperts
from ..utils.context import get_context
from .weights import RandomWeights

MIXERS = {"latent_attention": LatentAttention, "mamba2": Mamba2}
FEED_FORWARDS = {"moe": MixtureOfExperts}

# spread of seeded weights: vectors whose natural centre is not zero
_VECTOR_INIT = {"norm1": (1.0, 0.1), "norm2": (1.0, 0.1), "norm1b": (1.0, 0.1), "norm2b": (1.0, 0.1),
                "norm": (1.0, 0.1), "A_log": (0.0, 1.0), "dt_bias": (-3.0, 1.0), ".D": (1.0, 0.2), "sink": (0.0, 1.0)}


@dataclass
class SipazenConfig:
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float
    norm_groups: int
    residual_mult: float
    max_position: int = 4096

    @staticmethod
    def from_dict(c):
        layers = c["layers"]
        for i, l in enumerate(layers):
            if l["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer '{l['type']}' (known: {', '.join(sorted(MIXERS))})")
            kind = (l.get("mlp") or {}).get("kind", "moe")
            if kind not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward '{kind}'")
        if c["width"] % c["norm"]["groups"]:
            raise ValueError("norm.groups must divide width")
        return SipazenConfig(vocab_size=c["vocab"], hidden_size=c["width"], layers=layers, norm_eps=c["norm"]["eps"],
                             norm_groups=c["norm"]["groups"], residual_mult=c["residual_mult"],
                             max_position=c.get("max_position", c.get("max_model_length", 4096)))

    @property
    def num_layers(self):
        return len(self.layers)

    def widest_activation(self):
        """Elements per token of the widest stage of a layer, for the activation reserve of the cache pool."""
        wide = 0
        for l in self.layers:
            m = l["mixer"]
            if l["type"] == "mamba2":
                n = 5 * m["heads"] * m["vdim"] + 4 * m["groups"] * m["state"]
            else:
                n = m["heads"] * (4 * m["dim"] + 3 * m["rot_dim"] + 4 * m["vdim"]) + 2 * m["kv_rank"]
            e = l.get("mlp")
            if e:
                n = max(n, e["router"]["top"] * (2 * self.hidden_size + e["expert"]["ff"]) +
                        3 * (e.get("shared") or {"ff": 0})["ff"])
            wide = max(wide, n)
        return wide + 8 * self.hidden_size


class SipazenLayer(nn.Module):
    def __init__(self, cfg, index, load):
        super().__init__()
        spec, W = cfg.layers[index], cfg.hidden_size
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.mult, self.groups, self.eps = cfg.residual_mult, cfg.norm_groups, cfg.norm_eps
        self.norm1, self.norm1b = param(load("norm1", (W,))), param(load("norm1b", (W,)))
        self.rg1_b = param(load("rg1.b", (W,)))
        extra = {"residual_gate": load("rg1", (W, W))}
        scoped = lambda p: (lambda name, shape: load(p + name, shape))
        kw = {"max_position": cfg.max_position} if spec["type"] == "latent_attention" else {}
        self.mixer = MIXERS[spec["type"]](spec["mixer"], W, self.eps, scoped("mix."), extra, **kw)
        self.mlp = None
        if spec.get("mlp"):
            self.norm2, self.norm2b = param(load("norm2", (W,))), param(load("norm2b", (W,)))
            self.rg2_b = param(load("rg2.b", (W,)))
            self.mlp = FEED_FORWARDS[spec["mlp"].get("kind", "moe")](
                spec["mlp"], W, scoped("mlp."), {"residual_gate": load("rg2", (W, W))})

    def forward(self, h, x, next_norm):
        """h: this layer's normalised input, x: residual stream, updated in place.  Returns the input of the layer
        (or head) whose norm weight is `next_norm`."""
        y, p = self.mixer(h)
        after = self.norm2 if self.mlp is not None else next_norm
        h = gated_residual_norm(x, y, p["residual_gate"], self.rg1_b, self.norm1b, after, self.mult, self.groups,
                                self.eps)
        if self.mlp is not None:
            h = self.mlp(h, x, self.rg2_b, self.norm2b, next_norm, self.mult, self.groups, self.eps)
        return h


class SipazenForCausalLM(nn.Module):
    mixed_steps = True       # every prefill step goes through the paged cache and the state slots
    tensor_parallel = False

    def __init__(self, cfg: SipazenConfig, tp_rank=0, tp_size=1, dtype=torch.bfloat16, device="cuda", seed=0,
                 weights=None):
        super().__init__()
        if tp_size != 1:
            raise ValueError("Sipazen runs on one GPU")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Sipazen runs in bfloat16 or float32")
        w = weights if weights is not None else RandomWeights(seed, dtype, device, _VECTOR_INIT)
        self.cfg, self.dtype, self.comm = cfg, dtype, None
        V, W = cfg.vocab_size, cfg.hidden_size
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.embed, self.lm_head = param(w("embed", (V, W))), param(w("head", (V, W)))
        self.final_norm = param(w("final.norm", (W,)))
        self.layers = nn.ModuleList(SipazenLayer(cfg, i, w.scoped(f"l{i}.")) for i in range(cfg.num_layers))
        w.check_all_used()
        self.layer_probe = None      # tests: called with (layer index, residual stream) after every layer

    def forward(self, input_ids):
        """input_ids (tokens,) int64 -> hidden (tokens, width); positions, slots and tables come from the Context."""
        if get_context().positions is None:
            raise ValueError("Context.positions must be set before the model runs")
        c = self.cfg
        norms = [l.norm1 for l in self.layers] + [self.final_norm]
        x, h = embed_norm(input_ids, self.embed, norms[0], c.norm_groups, c.norm_eps)
        for i, layer in enumerate(self.layers):
            h = layer(h, x, norms[i + 1])
            if self.layer_probe is not None:
                self.layer_probe(i, x)
        return h

    def compute_logits(self, hidden, vocab_shard=None):
        """Rows named by Context.last_token_index when it is set, all rows otherwise."""
        ctx = get_context()
        if ctx.last_token_index is not None:
            hidden = hidden[ctx.last_token_index]
        if vocab_shard is not None:
            raise ValueError("Sipazen's head is not sharded")
        return F.linear(hidden, self.lm_head)
