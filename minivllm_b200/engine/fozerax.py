"""Fozerax: a decoder whose layers each take gated linear attention, or windowed attention and a gated delta rule side by
side, and a dense or mixture-of-experts feed-forward.  Sublayers read the fp32 residual stream itself; only their results
are normed.

    x = norm_e(embed[token])
    x += norm1(mixer(x));  x += norm2(feed_forward(x))
    logits = head final_norm(x)

Every size and constant is read from the configuration or a tensor's shape.  The mixers and feed-forwards are the modules
of layers/; a sublayer's norm and its addition to the stream are one launch that also writes the next sublayer's input.
"""
from dataclasses import dataclass

import torch
import torch.nn as nn
import torch.nn.functional as F

from ..layers.gated_delta import GatedDeltaRule
from ..layers.gla import GatedLinearAttention
from ..layers.group_norm import embed_norm, gated_residual_norm, pair_residual_norm
from ..layers.mlp import GatedMLP
from ..layers.moe import MixtureOfExperts
from ..layers.parallel import ParallelMixers
from ..layers.window_attention import WindowAttention
from ..utils.context import get_context
from .weights import RandomWeights

MIXERS = {
    "gla": GatedLinearAttention,
    "parallel": lambda *a: ParallelMixers(*a, left=WindowAttention, right=GatedDeltaRule),
}
FEED_FORWARDS = {
    "dense": lambda spec, width, load: GatedMLP(spec, width, load, act="gelu_tanh"),
    "moe": lambda spec, width, load: MixtureOfExperts(spec, width, load, act="clamped", router_bias=False,
                                                      shared_gate=False),
}

# spread of seeded weights: vectors whose natural centre is not zero
_VECTOR_INIT = {"norm": (1.0, 0.1), "norm1": (1.0, 0.1), "norm2": (1.0, 0.1), ".out": (1.0, 0.1), "a2.b": (3.0, 1.0),
                "A_log": (0.0, 1.0), "dt_bias": (-3.0, 1.0), "sink": (0.0, 1.0)}


@dataclass
class FozeraxConfig:
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
                raise ValueError(f"layer {i}: unknown mixer '{l['type']}' (known: {', '.join(sorted(MIXERS))})")
            if l.get("mlp") and l["mlp"].get("kind") not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward '{l['mlp'].get('kind')}'")
        return FozeraxConfig(vocab_size=c["vocab"], hidden_size=c["width"], layers=layers, norm_eps=c["norm"]["eps"],
                             max_position=c.get("max_position", c.get("max_model_length", 4096)))

    @property
    def num_layers(self):
        return len(self.layers)

    def widest_activation(self):
        """Elements per token of the widest stage of a layer, for the activation reserve of the cache pool."""
        wide = 0
        for l in self.layers:
            m = l["mixer"]
            if l["type"] == "gla":
                n = m["heads"] * (3 * m["dim"] + 4 * m["vdim"])
            else:
                a, b = m["left"], m["right"]
                n = a["heads"] * (a["dim"] + a["vdim"]) + 3 * a["kv_heads"] * (a["dim"] + a["vdim"]) + \
                    4 * b["kv_heads"] * b["dim"] + 5 * b["heads"] * b["vdim"]
            e = l.get("mlp")
            if e and e["kind"] == "dense":
                n = max(n, 3 * e["ff"])
            elif e:
                n = max(n, e["router"]["top"] * (2 * self.hidden_size + e["expert"]["ff"]) +
                        3 * (e.get("shared") or {"ff": 0})["ff"])
            wide = max(wide, n)
        return wide + 8 * self.hidden_size


class FozeraxLayer(nn.Module):
    def __init__(self, cfg, index, load):
        super().__init__()
        spec, W = cfg.layers[index], cfg.hidden_size
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.eps = cfg.norm_eps
        self.norm1 = param(load("norm1", (W,)))
        self.mixer = MIXERS[spec["type"]](spec["mixer"], W, self.eps, load.scoped("mix."))
        self.mlp = None
        if spec.get("mlp"):
            self.norm2 = param(load("norm2", (W,)))
            self.mlp = FEED_FORWARDS[spec["mlp"]["kind"]](spec["mlp"], W, load.scoped("mlp."))

    def forward(self, h, x, next_norm):
        """h: the residual stream as the mixer reads it, x: the fp32 stream, updated in place.  Returns the input of the
        next layer (`next_norm` None: the stream again) or of the head."""
        after = None if self.mlp is not None else next_norm
        y = self.mixer(h)
        if isinstance(y, tuple):
            h = pair_residual_norm(x, y[0], self.mixer.left_out, y[1], self.mixer.right_out, self.norm1, after, 1.0, 1,
                                   self.eps)
        else:
            h = gated_residual_norm(x, y, None, None, self.norm1, after, 1.0, 1, self.eps)
        if isinstance(self.mlp, MixtureOfExperts):
            h = self.mlp(h, x, None, self.norm2, next_norm, 1.0, 1, self.eps)
        elif self.mlp is not None:
            h = gated_residual_norm(x, self.mlp(h), None, None, self.norm2, next_norm, 1.0, 1, self.eps)
        return h


class FozeraxForCausalLM(nn.Module):
    mixed_steps = True       # every prefill step goes through the paged cache and the state slots
    tensor_parallel = False

    def __init__(self, cfg: FozeraxConfig, tp_rank=0, tp_size=1, dtype=torch.bfloat16, device="cuda", seed=0,
                 weights=None):
        super().__init__()
        if tp_size != 1:
            raise ValueError("Fozerax runs on one GPU")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("Fozerax runs in bfloat16 or float32")
        w = weights if weights is not None else RandomWeights(seed, dtype, device, _VECTOR_INIT)
        self.cfg, self.dtype, self.comm = cfg, dtype, None
        V, W = cfg.vocab_size, cfg.hidden_size
        param = lambda t: nn.Parameter(t, requires_grad=False)
        self.embed, self.lm_head = param(w("embed", (V, W))), param(w("head", (V, W)))
        self.embed_norm, self.final_norm = param(w("embed.norm", (W,))), param(w("final.norm", (W,)))
        self.layers = nn.ModuleList(FozeraxLayer(cfg, i, w.scoped(f"l{i}.")) for i in range(cfg.num_layers))
        w.check_all_used()
        self.layer_probe = None      # tests: called with (layer index, residual stream) after every layer

    def forward(self, input_ids):
        """input_ids (tokens,) int64 -> hidden (tokens, width); positions, slots and tables come from the Context."""
        if get_context().positions is None:
            raise ValueError("Context.positions must be set before the model runs")
        c = self.cfg
        first = None if len(self.layers) else self.final_norm
        x, h = embed_norm(input_ids, self.embed, first, 1, c.norm_eps, w_post=self.embed_norm)
        for i, layer in enumerate(self.layers):
            h = layer(h, x, None if i + 1 < len(self.layers) else self.final_norm)
            if self.layer_probe is not None:
                self.layer_probe(i, x)
        return h

    def compute_logits(self, hidden, vocab_shard=None):
        """Rows named by Context.last_token_index when it is set, all rows otherwise."""
        ctx = get_context()
        if ctx.last_token_index is not None:
            hidden = hidden[ctx.last_token_index]
        if vocab_shard is not None:
            raise ValueError("Fozerax's head is not sharded")
        return F.linear(hidden, self.lm_head)
