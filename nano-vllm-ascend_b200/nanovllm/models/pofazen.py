"""Pofazen: a decoder whose layers are listed one by one in its configuration, on an fp32 residual stream whose norm is
taken of the SUM -- what the norm gives is the new stream, and the sublayers read the stream itself:

    x <- N(E[token]);   x <- N1(alpha x + mixer(x));   x <- N2(alpha x + ff(x));   logits = head N(x)

(N: RMS norm with a plain weight.) Each layer has one of two mixers and an optional silu-gated feed-forward:

  parallel   two mixers side by side on the same input, left_scale * left + right_scale * right.
             left: q, k, v projections; q and k heads divided by their root mean square times a weight shared by the
             heads; rotary positions on the first rot.dims columns of a head (pairs (2i, 2i+1), frequencies stretched by
             wavelength); softmax attention in a sliding window whose first keep_first tokens stay visible; the heads
             times sigmoid(W_g x) element by element; W_o.
             right: q, k, v projections -> short causal convolution + silu; q, k unit vectors per head, q times dim^-1/2;
             beta = sigmoid(W_b x); one decay per head exp(-exp(A) softplus(W_a x + bias)); gated delta rule (fp32
             state); o / rms(o) per head times a weight shared by the heads, times silu(W_g x); W_o.
  wkv        r, k, v, g and the decay each read a mix of the token with the token before; decay
             exp(-exp(W_2 tanh(W_1 .) + w0)) per head and key channel; per head o = (S + diag(u) k v^T)^T r, then
             S <- diag(w) S + k v^T (fp32 state); o / rms(o) per head, times a weight, times silu(g); W_o.

Launches per sublayer. parallel: ONE GEMM in (the projections of both branches), norm + rotation + K/V scatter,
attention, gate; convolution, unit vectors + decays, delta rule, norm + gate; ONE GEMM out -- the branches' results lie
side by side in its input row, already multiplied by their scales, so that the sum of the branches is the GEMM's own
accumulation. wkv: the five mixes, one batched product for r, k, v, g, two small ones with a tanh between for the decay,
the recurrence's inputs, the recurrence, norm + gate, GEMM out. Then ONE kernel for "add to alpha times the stream, norm,
hand the stream on". What the design fixes is a constant here; every size and every constant that may differ between
models comes from the config.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from .. import ops
from ..layers.activation import GatedFeedForward
from ..layers.embed_head import ParallelLMHead, VocabParallelEmbedding
from ..layers.linear import (ConcatInputLinear, F32OutLinear, PaddedMergedLinear, ReplicatedLinear, RowParallelLinear,
                             StackedLinear, tp_rank_size)
from ..layers.seq_mixers import (DeltaRule, GatedNorm, ShortConv, TokenShift, VarSizeAttention, WavelengthScaledRotary,
                                 WkvRecurrence, small_param)
from ..utils.context import get_context

UNIT_EPS = 1e-6            # inside the root of the delta rule's unit vectors
FF_ACT = "silu"
SHIFTED = "rkvgw"          # what reads a mix of its own, in the order of TokenShift's rows


@dataclass
class PofazenSpec:
    """What the runner asks of a model's spec."""
    vocab_size: int
    hidden_size: int
    num_layers: int
    rms_eps: float
    num_experts: int = 0
    tie_embeddings: bool = False


class SumNorm(nn.Module):
    """Weight of one RMS norm of the residual path; the arithmetic runs fused with the residual update."""

    def __init__(self, size: int):
        super().__init__()
        self.weight = small_param(size, fill=1.0)


class ParallelMixer(nn.Module):

    def __init__(self, width: int, m: dict, eps: float):
        super().__init__()
        a, b = m["left"], m["right"]
        self.eps = eps
        self.left_scale, self.right_scale = float(m["left_scale"]), float(m["right_scale"])
        self.H, self.G, self.d, self.dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        H, G, d, dv = b["heads"], b["kv_heads"], b["dim"], b["vdim"]
        self.nqk = 2 * G * d
        self.left_sizes = [self.H * self.d, self.G * self.d, self.G * self.dv]           # q | k | v
        self.right_sizes = [G * d, G * d, H * dv]                                        # q | k | v (convolved)
        n_left, n_right = self.H * self.dv, H * dv
        # every projection of both branches: left qkv | left gate | right qkv | right gate | beta | decay
        self.proj = PaddedMergedLinear(width, [self.left_sizes, n_left, self.right_sizes, n_right, H, H])
        self.q_norm, self.k_norm = small_param(self.d, fill=1.0), small_param(self.d, fill=1.0)
        rot = a.get("rot") or {"dims": 0, "base": 1.0}
        self.rot = WavelengthScaledRotary(rot["dims"], rot["base"], interleaved=True, scaling=rot.get("scaling"))
        mask = a.get("mask") or {}
        self.attn = VarSizeAttention(self.H, self.G, self.d, self.dv, float(a["scale"]), window=int(mask.get("size") or 0),
                                     keep_first=int(mask.get("keep_first") or 0))
        self.left_gate = GatedNorm(n_left, eps, norm=False)
        self.conv = ShortConv(self.right_sizes, b["conv"], act="silu")
        self.rule = DeltaRule(H, G, d, dv, unit_eps=UNIT_EPS, per_head=True)
        self.right_norm = GatedNorm(n_right, eps, groups=H, gate_first=False, gate_act="silu")
        self.right_norm.weight.weight_loader = lambda p, w: p.data.copy_(w.repeat(H))    # one [vdim] weight for all heads
        self.o_proj = ConcatInputLinear([n_left, n_right], width)

    def forward(self, positions, h):
        p = self.proj(h)
        part = lambda i: self.proj.part(p, i)
        y = self.o_proj.empty_input(p.shape[0], p)
        self._attention(positions, part(0), part(1), self.o_proj.part(y, 0))
        qkv = self.conv(part(2))
        o = self.rule(qkv[:, :self.nqk], qkv[:, self.nqk:], part(5), part(4))
        self.right_norm(o, part(3), out=self.o_proj.part(y, 1), scale=self.right_scale)
        return self.o_proj(y)

    def _attention(self, positions, qkv, gate, out):
        attn = self.attn
        ctx = get_context()
        have_cache = attn.k_cache.numel() > 0 and ctx.slot_mapping is not None
        ops.norm_rope_cache(qkv, self.q_norm, self.k_norm, self.eps, self.rot.table(positions), self.H, self.G, self.d,
                            self.dv, self.rot.dims, self.rot.interleaved, attn.k_cache if have_cache else None,
                            attn.v_cache if have_cache else None, ctx.slot_mapping if have_cache else None)
        nq, nk, _ = self.left_sizes
        q = qkv[:, :nq].unflatten(1, (self.H, self.d))
        k = qkv[:, nq:nq + nk].unflatten(1, (self.G, self.d))
        v = qkv[:, nq + nk:].unflatten(1, (self.G, self.dv))
        self.left_gate(attn(q, k, v), gate, out=out, scale=self.left_scale)


class WkvMixer(nn.Module):

    def __init__(self, width: int, m: dict, eps: float, rank: int):
        super().__init__()
        H, d = m["heads"], m["dim"]
        n = H * d
        self.shift = TokenShift(width, len(SHIFTED))
        self.proj = StackedLinear(4, width, n)                                           # r, k, v, gate
        self.w1 = ReplicatedLinear(width, rank)
        self.w2 = F32OutLinear(rank, n)
        self.rec = WkvRecurrence(H, d)
        self.norm = GatedNorm(n, eps, groups=H, gate_first=False, gate_act="silu")
        self.o_proj = RowParallelLinear(n, width)

    def forward(self, positions, h):
        mixes = self.shift(h)
        r, k, v, gate = self.proj(mixes[:4])
        z = self.w2(ops.act_only(self.w1(mixes[4]), "tanh"))
        return self.o_proj(self.norm(self.rec(r, k, v, z), gate))


def build_feed_forward(width: int, mlp: dict) -> nn.Module:
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return GatedFeedForward(width, mlp["ff"], FF_ACT)
    raise ValueError(f"unknown feed-forward kind {kind!r}")


class PofazenLayer(nn.Module):

    def __init__(self, width: int, entry: dict, eps: float, rank: int):
        super().__init__()
        kind, m = entry["type"], entry["mixer"]
        if kind == "parallel":
            self.mix = ParallelMixer(width, m, eps)
        elif kind == "wkv":
            self.mix = WkvMixer(width, m, eps, rank)
        else:
            raise ValueError(f"unknown mixer {kind!r}")
        self.norm1 = SumNorm(width)
        if entry.get("mlp"):
            self.mlp = build_feed_forward(width, entry["mlp"])
            self.norm2 = SumNorm(width)
        else:
            self.mlp = None


class PofazenForCausalLM(nn.Module):
    supports_fp32 = True            # every kernel of this stack has a true 32-bit form
    reads_checkpoint_shapes = True  # the inner size of the wkv mixers' decay projection is the tensors' shape
    prefix_caching = False          # recurrent state at a prefix's end is not kept, so cached blocks are no use
    split_decode = False

    def __init__(self, config):
        super().__init__()
        if tp_rank_size()[1] != 1:
            raise ValueError("Pofazen runs on one GPU per replica (no tensor-parallel sharding of its mixers)")
        c = config.to_dict() if hasattr(config, "to_dict") else dict(config)
        self.eps = float(c["norm"]["eps"])
        self.alpha = float(c["postln_alpha"])
        W = c["width"]
        self.spec = PofazenSpec(c["vocab"], W, len(c["layers"]), self.eps)
        self.embed_tokens = VocabParallelEmbedding(c["vocab"], W)
        self.embed_norm = SumNorm(W)
        shapes = getattr(config, "checkpoint_shapes", None) or {}
        self.layers = nn.ModuleList([PofazenLayer(W, entry, self.eps, self._decay_rank(i, entry, shapes))
                                     for i, entry in enumerate(c["layers"])])
        self.norm = SumNorm(W)
        self.lm_head = ParallelLMHead(c["vocab"], W)
        self.trace_layers = None                       # a list: the residual stream after every layer is appended

    # ------------------------------------------------------------------ forward
    def _sublayers(self):
        """(callable, norm of the sum, closes a layer) in execution order."""
        out = []
        for layer in self.layers:
            out.append((layer.mix, layer.norm1, layer.mlp is None))
            if layer.mlp is not None:
                out.append((lambda pos, h, f=layer.mlp: f(h), layer.norm2, True))
        return out

    def forward(self, input_ids, positions):
        # what the layers share lives for ONE pass: a context may see several passes (an eager pass, then the capture
        # of a CUDA graph), and what an earlier pass computed is neither current nor part of the graph
        get_context().scratch.clear()
        table = self.embed_tokens.weight
        dtype = table.dtype
        ids = input_ids.to(torch.int64).contiguous()
        x = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)     # the residual stream
        norm = dict(b=None, eps=self.eps, dtype=dtype, kind="rms")
        h = ops.norm_residual_(x, table, self.embed_norm.weight, accumulate=False, y_index=ids, **norm)
        for fn, sum_norm, closes in self._sublayers():
            y = fn(positions, h).contiguous()
            h = ops.norm_residual_(x, y, sum_norm.weight, carry=self.alpha, **norm)
            if closes and self.trace_layers is not None:
                self.trace_layers.append(x.clone())
        return ops.residual_rmsnorm(x, self.norm.weight, self.eps, dtype, offset=0.0)

    def compute_logits(self, hidden_states):
        return self.lm_head(hidden_states)

    # ------------------------------------------------------------------ weights
    @staticmethod
    def _decay_rank(i: int, entry: dict, shapes: dict) -> int:
        """Inner size of layer i's low-rank decay projection: the checkpoint tensor's shape; a configuration without a
        checkpoint (synthetic weights) may give "decay_rank"."""
        if f"l{i}.mix.w1" in shapes:
            return shapes[f"l{i}.mix.w1"][0]
        return int(entry["mixer"].get("decay_rank", 64))

    def route_checkpoint_tensor(self, name: str):
        """Checkpoint tensor name -> (parameter name, shard id or None)."""
        top = {"embed": "embed_tokens.weight", "head": "lm_head.weight", "embed.norm": "embed_norm.weight",
               "final.norm": "norm.weight"}
        if name in top:
            return top[name], None
        layer, _, rest = name.partition(".")
        base = f"layers.{int(layer[1:])}."
        if rest in ("norm1", "norm2"):
            return base + rest + ".weight", None
        if rest.startswith("mlp."):
            return {"gate": (base + "mlp.gate_up_proj.weight", 0), "up": (base + "mlp.gate_up_proj.weight", 1),
                    "down": (base + "mlp.down_proj.weight", None)}[rest[4:]]
        key = rest[4:]                                  # after "mix."
        base += "mix."
        if key.startswith("left."):
            key = key[5:]
            return {"q": (base + "proj.weight", (0, 0)), "k": (base + "proj.weight", (0, 1)),
                    "v": (base + "proj.weight", (0, 2)), "g": (base + "proj.weight", 1), "q.norm": (base + "q_norm", None),
                    "k.norm": (base + "k_norm", None), "o": (base + "o_proj.weight", 0)}[key]
        if key.startswith("right."):
            key = key[6:]
            if key.endswith(".conv"):
                return base + "conv.weight", "qkv".index(key[0])
            return {"q": (base + "proj.weight", (2, 0)), "k": (base + "proj.weight", (2, 1)),
                    "v": (base + "proj.weight", (2, 2)), "g": (base + "proj.weight", 3), "b": (base + "proj.weight", 4),
                    "a": (base + "proj.weight", 5), "A_log": (base + "rule.A_log", None),
                    "dt_bias": (base + "rule.dt_bias", None), "norm": (base + "right_norm.weight", None),
                    "o": (base + "o_proj.weight", 1)}[key]
        if key.startswith("mu."):
            return base + "shift.mu", SHIFTED.index(key[3:])
        return {"r": (base + "proj.weight", 0), "k": (base + "proj.weight", 1), "v": (base + "proj.weight", 2),
                "g": (base + "proj.weight", 3), "w1": (base + "w1.weight", None), "w2": (base + "w2.weight", None),
                "w0": (base + "rec.w0", None), "u": (base + "rec.u", None), "norm": (base + "norm.weight", None),
                "o": (base + "o_proj.weight", None)}[key]

    @torch.no_grad()
    def random_init(self, seed: int = 0, std: float | None = None) -> None:
        """Random weights for synthetic runs: matrices N(0, 1/fan_in), norm weights near one, shift weights inside (0, 1),
        decay parameters in the range where the recurrences neither vanish nor blow up."""
        g = torch.Generator().manual_seed(seed)
        for name, p in sorted(self.named_parameters()):
            if name.endswith("A_log"):
                v = torch.rand(p.shape, generator=g) * 3 - 4
            elif name.endswith("rec.w0"):
                v = torch.rand(p.shape, generator=g) * 4 - 5
            elif name.endswith("dt_bias") or name.endswith("rec.u") or name.endswith("conv.weight"):
                v = 0.5 * torch.randn(p.shape, generator=g)
            elif name.endswith("shift.mu"):
                v = torch.rand(p.shape, generator=g)
            elif p.dim() == 1:
                v = 1 + 0.1 * torch.randn(p.shape, generator=g)
            elif name == "embed_tokens.weight":
                v = torch.randn(p.shape, generator=g)
            else:
                v = torch.randn(p.shape, generator=g) * (std if std is not None else p.shape[-1] ** -0.5)
            p.data.copy_(v.to(p.dtype))
        for layer in self.layers:
            mix = layer.mix
            if isinstance(mix, ParallelMixer):         # padding of the fused projections stays zero
                mix.proj.zero_padding()
                mix.o_proj.zero_padding()
                mix.right_norm.weight.data.copy_(mix.right_norm.weight.data[:mix.rule.vdim].repeat(mix.rule.num_heads))
