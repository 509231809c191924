"""Ragilorn: a decoder whose layers are listed one by one in its configuration, on an fp32 residual whose branches are
gated element by element and whose layers hand on a weighted sum of everything before them:

    X_0 = x = scale E[token]
    x <- x + sigmoid(W_1 h + b_1) . mixer(h), h = N1(x);   x <- x + sigmoid(W_2 h + b_2) . ff(h), h = N2(x)
    X_(i+1) = x (the result of layer i);   x <- sum_(j <= i+1) a_i[j] X_j;   logits = c tanh(s head N(x) / c)

(N: RMS norm with a plain weight.) Each layer has one of two mixers and an optional feed-forward (dense with silu(gate) *
up, or a mixture of such experts behind a sigmoid router whose chosen scores, as they are, multiply what the experts READ):

  attention         q, k, v projections with biases -> short causal convolution over time on every channel -> rotary
                    positions on the first rot.dims columns of every q and k head (pairs (2i, 2i+1); frequencies stretched
                    band by band, layers.seq_mixers.BandScaledRotary) -> softmax attention inside chunks of the sequence
                    counted from position 0 -> W_o with a bias
  latent_attention  q projection; ONE cached row per token = [normed key/value latent | rotated shared key part] (the same
                    kind of rotation); causal softmax attention with the up-projections absorbed into the query and the
                    output; W_o

Launches per mixer sublayer: ONE GEMM in (every projection of the sublayer and the logits of its branch gate), the
convolution, rotation + K/V scatter (or latent norm + rotation + scatter), the attention, one GEMM out, and ONE kernel for
"gate the branch, add it, keep the layer's result, average over the depth, norm for the next sublayer". The history X_j
is one fp32 buffer per pass. What the design fixes is a constant here; every size and every constant that may differ
between models comes from the config.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from .. import ops
from ..layers.activation import GatedFeedForward
from ..layers.embed_head import ParallelLMHead, VocabParallelEmbedding
from ..layers.linear import PaddedMergedLinear, ReplicatedLinear, RowParallelLinear, tp_rank_size
from ..layers.moe import GroupedSigmoidMoe
from ..layers.seq_mixers import BandScaledRotary, LatentAttention, ShortConv, VarSizeAttention, small_param
from ..utils.context import get_context

FF_ACT = "silu"


@dataclass
class RagilornSpec:
    """What the runner asks of a model's spec."""
    vocab_size: int
    hidden_size: int
    num_layers: int
    rms_eps: float
    num_experts: int = 0
    tie_embeddings: bool = False


class BranchNorm(nn.Module):
    """Weight of one RMS norm of the residual path; the arithmetic runs fused with the residual update."""

    def __init__(self, size: int):
        super().__init__()
        self.weight = small_param(size, fill=1.0)


def _rotary(m: dict) -> BandScaledRotary:
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    return BandScaledRotary(rot["dims"], rot["base"], interleaved=True, scaling=rot.get("scaling"))


class ChunkedAttentionMixer(nn.Module):

    def __init__(self, width: int, m: dict, eps: float):
        super().__init__()
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.H, self.G, self.d, self.dv = H, G, d, dv
        self.sizes = [H * d, G * d, G * dv]                             # q | k | v
        self.proj = PaddedMergedLinear(width, [self.sizes, width], bias=True)            # q | k | v, then the branch gate
        taps = int(m.get("conv") or 0)
        self.conv = ShortConv(self.sizes, taps) if taps else None
        self.rot = _rotary(m)
        self.attn = VarSizeAttention(H, G, d, dv, float(m["scale"]), chunk=int((m.get("mask") or {}).get("size") or 0))
        self.o_proj = RowParallelLinear(H * dv, width, bias=True)

    def forward(self, positions, h):
        """-> (the mixer's result, the logits of its branch gate)."""
        p = self.proj(h)
        nq, nk, _ = self.sizes
        qkv = self.proj.part(p, 0)
        if self.conv is not None:
            qkv = self.conv(qkv)
        attn = self.attn
        ctx = get_context()
        have_cache = attn.k_cache.numel() > 0 and ctx.slot_mapping is not None
        ops.rope_mix_cache(qkv, self.rot.table(positions), self.H, self.G, self.d, self.dv, self.rot.dims,
                           self.rot.interleaved, k_cache=attn.k_cache if have_cache else None,
                           v_cache=attn.v_cache if have_cache else None, slots=ctx.slot_mapping if have_cache else None)
        q = qkv[:, :nq].unflatten(1, (self.H, self.d))
        k = qkv[:, nq:nq + nk].unflatten(1, (self.G, self.d))
        v = qkv[:, nq + nk:].unflatten(1, (self.G, self.dv))
        return self.o_proj(attn(q, k, v)), self.proj.part(p, 1)


class LatentAttentionMixer(nn.Module):

    def __init__(self, width: int, m: dict, eps: float):
        super().__init__()
        H, d, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
        self.H, self.d, self.dr, self.dv, self.eps = H, d, dr, dv, eps
        self.rank = m["kv_rank"]
        self.proj = PaddedMergedLinear(width, [H * (d + dr), self.rank + dr, width], bias=True)   # q | dkv | branch gate
        self.kv_norm = small_param(self.rank, fill=1.0)
        self.rot = _rotary(m)
        self.attn = LatentAttention(H, d, dr, dv, self.rank, float(m["scale"]))
        self.o_proj = RowParallelLinear(H * dv, width)

    def forward(self, positions, h):
        """-> (the mixer's result, the logits of its branch gate)."""
        p = self.proj(h)
        attn = self.attn
        ctx = get_context()
        have_cache = attn.k_cache.numel() > 0 and ctx.slot_mapping is not None
        _, kc = ops.latent_kv_prep(None, self.proj.part(p, 1), None, self.kv_norm, positions, self.rank, self.dr,
                                   self.rot.dims, 1.0, self.rot.interleaved, self.eps,
                                   cache=attn.k_cache if have_cache else None,
                                   slots=ctx.slot_mapping if have_cache else None, table=self.rot.table(positions))
        q = self.proj.part(p, 0).unflatten(1, (self.H, self.d + self.dr))
        o = attn(q[:, :, :self.d], lambda out: self.rot(q[:, :, self.d:], positions, out=out), kc)
        return self.o_proj(o), self.proj.part(p, 2)


MIXERS = {"attention": ChunkedAttentionMixer, "latent_attention": LatentAttentionMixer}


class GatedMoe(nn.Module):
    """The mixture of experts of one layer and the logits of its branch gate."""

    def __init__(self, width: int, mlp: dict):
        super().__init__()
        r = mlp["router"]
        self.moe = GroupedSigmoidMoe(width, mlp["expert"]["ff"], r["experts"], r["top"], correction=False, normalize=False,
                                     weigh="input")
        self.branch_gate = ReplicatedLinear(width, width, bias=True)

    def forward(self, h):
        return self.moe(h), self.branch_gate(h)


def build_feed_forward(width: int, mlp: dict) -> nn.Module:
    """A module whose forward gives (the feed-forward's result, the logits of its branch gate)."""
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return GatedFeedForward(width, mlp["ff"], FF_ACT, extra=width)
    if kind == "moe":
        return GatedMoe(width, mlp)
    raise ValueError(f"unknown feed-forward kind {kind!r}")


class RagilornLayer(nn.Module):

    def __init__(self, index: int, width: int, entry: dict, eps: float):
        super().__init__()
        if entry["type"] not in MIXERS:
            raise ValueError(f"unknown mixer {entry['type']!r}")
        self.mix = MIXERS[entry["type"]](width, entry["mixer"], eps)
        self.norm1 = BranchNorm(width)
        if entry.get("mlp"):
            self.mlp = build_feed_forward(width, entry["mlp"])
            self.norm2 = BranchNorm(width)
        else:
            self.mlp = None
        self.dwa = small_param(index + 2)              # weights of X_0 .. X_(index + 1)


class RagilornForCausalLM(nn.Module):
    supports_fp32 = True            # every kernel of this stack has a true 32-bit form
    prefix_caching = False          # the convolution tails at a prefix's end are not kept, so cached blocks are no use
    split_decode = False

    def __init__(self, config):
        super().__init__()
        if tp_rank_size()[1] != 1:
            raise ValueError("Ragilorn runs on one GPU per replica (no tensor-parallel sharding of its mixers)")
        c = config.to_dict() if hasattr(config, "to_dict") else dict(config)
        self.eps = float(c["norm"]["eps"])
        self.embed_scale = float((c.get("embedding") or {}).get("scale", 1.0))
        W = c["width"]
        n_exp = max([e["mlp"]["router"]["experts"] for e in c["layers"]
                     if e.get("mlp") and e["mlp"].get("kind") == "moe"] or [0])
        self.spec = RagilornSpec(c["vocab"], W, len(c["layers"]), self.eps, num_experts=n_exp)
        self.embed_tokens = VocabParallelEmbedding(c["vocab"], W)
        self.layers = nn.ModuleList([RagilornLayer(i, W, entry, self.eps) for i, entry in enumerate(c["layers"])])
        self.norm = BranchNorm(W)
        self.lm_head = ParallelLMHead(c["vocab"], W, scale=float(c.get("logit_scale", 1.0)),
                                      softcap=float(c.get("logit_softcap") or 0.0))
        self.trace_layers = None                       # a list: what every layer hands on is appended

    # ------------------------------------------------------------------ forward
    def forward(self, input_ids, positions):
        # what the layers share lives for ONE pass: a context may see several passes (an eager pass, then the capture
        # of a CUDA graph), and what an earlier pass computed is neither current nor part of the graph
        get_context().scratch.clear()
        table = self.embed_tokens.weight
        ids = input_ids.to(torch.int64).contiguous()
        L = len(self.layers)
        hist = torch.empty(max(L, 1), ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)   # X_0 .. X_(L-1)
        stream = torch.empty(hist.shape[1:], dtype=torch.float32, device=table.device)
        norm = lambda n: dict(w=n.weight, eps=self.eps, dtype=table.dtype)
        # the scaled embedding and the first norm in one launch
        h = ops.residual_gate_average(None, table, None, c=self.embed_scale, y_index=ids, keep=hist[0],
                                      **norm(self.layers[0].norm1 if L else self.norm))
        x = hist[0]
        for i, layer in enumerate(self.layers):
            y, gate = layer.mix(positions, h)
            if layer.mlp is not None:
                h = ops.residual_gate_average(x, y, gate, x_out=stream, **norm(layer.norm2))
                x = stream
                y, gate = layer.mlp(h)
            last = i + 1 == L
            traced = self.trace_layers is not None
            h = ops.residual_gate_average(x, y, gate, keep=None if last else hist[i + 1], hist=hist, n=i + 1, avg=layer.dwa,
                                          x_out=stream if not last or traced else None,
                                          **norm(self.norm if last else self.layers[i + 1].norm1))
            x = stream
            if traced:
                self.trace_layers.append(stream.clone())
        return h                                       # already through the final norm

    def compute_logits(self, hidden_states):
        return self.lm_head(hidden_states)

    # ------------------------------------------------------------------ weights
    def route_checkpoint_tensor(self, name: str):
        """Checkpoint tensor name -> (parameter name, shard id or None)."""
        top = {"embed": "embed_tokens.weight", "head": "lm_head.weight", "final.norm": "norm.weight"}
        if name in top:
            return top[name], None
        layer, _, rest = name.partition(".")
        i = int(layer[1:])
        base = f"layers.{i}."
        mix, mlp = self.layers[i].mix, self.layers[i].mlp
        if rest in ("norm1", "norm2"):
            return base + rest + ".weight", None
        if rest == "dwa":
            return base + "dwa", None
        kind = "bias" if rest.endswith(".b") else "weight"
        rest = rest[:-2] if kind == "bias" else rest
        if rest == "rg1":
            return base + "mix.proj." + kind, 1 if isinstance(mix, ChunkedAttentionMixer) else 2
        if rest == "rg2":
            if isinstance(mlp, GatedMoe):
                return base + "mlp.branch_gate." + kind, None
            return base + "mlp.gate_up_proj." + kind, 1
        part, _, key = rest.partition(".")
        if part == "mlp":
            if isinstance(mlp, GatedMoe):
                if key == "router":
                    return base + "mlp.moe.router", None
                e, which = key.split(".")
                e = int(e[1:])
                return {"gate": (base + "mlp.moe.w13", (e, 0)), "up": (base + "mlp.moe.w13", (e, 1)),
                        "down": (base + "mlp.moe.w2", e)}[which]
            return {"gate": (base + "mlp.gate_up_proj.weight", (0, 0)), "up": (base + "mlp.gate_up_proj.weight", (0, 1)),
                    "down": (base + "mlp.down_proj.weight", None)}[key]
        if part != "mix":
            raise KeyError(name)
        if key == "o":
            return base + "mix.o_proj." + kind, None
        if isinstance(mix, ChunkedAttentionMixer):
            if key.endswith(".conv"):
                return base + "mix.conv.weight", "qkv".index(key[:-5])
            return base + "mix.proj." + kind, (0, "qkv".index(key))
        return {"q": (base + "mix.proj.weight", 0), "dkv": (base + "mix.proj.weight", 1),
                "dkv.norm": (base + "mix.kv_norm", None), "uk": (base + "mix.attn.w_uk", None),
                "uv": (base + "mix.attn.w_uv", None)}[key]

    @torch.no_grad()
    def random_init(self, seed: int = 0, std: float | None = None) -> None:
        """Random weights for synthetic runs: matrices N(0, 1/fan_in), norm weights near one, biases small, taps of the
        order of one, every layer handing on mostly its own result."""
        g = torch.Generator().manual_seed(seed)
        for name, p in sorted(self.named_parameters()):
            if name.endswith("conv.weight"):
                v = 0.5 * torch.randn(p.shape, generator=g)
            elif name.endswith(".bias"):
                v = 0.2 * torch.randn(p.shape, generator=g)
            elif name.endswith(".dwa"):
                v = 0.1 * torch.randn(p.shape, generator=g)
                v[-1] += 1.0
            elif p.dim() == 1:
                v = 1 + 0.1 * torch.randn(p.shape, generator=g)
            elif name == "embed_tokens.weight":
                v = torch.randn(p.shape, generator=g) / self.embed_scale
            else:
                v = torch.randn(p.shape, generator=g) * (std if std is not None else p.shape[-1] ** -0.5)
            p.data.copy_(v.to(p.dtype))
        for m in self.modules():                       # padding of the fused projections stays zero
            if isinstance(m, PaddedMergedLinear):
                m.zero_padding()
        for layer in self.layers:                      # q and the latent have no bias
            if isinstance(layer.mix, LatentAttentionMixer):
                layer.mix.proj.bias.data[:sum(layer.mix.proj.padded_sizes[:2])].zero_()
