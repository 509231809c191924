"""A plain, slow restatement of the Pofazen decoder in float64, one function per mechanism, for the tests.

It shares no code with the package: every function works on whole sequences held in torch tensors on the CPU, token by
token where there is a state and query by query where there is a mask. Weights come as a dict {checkpoint tensor name:
tensor}; the configuration is the dict of config.json.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def rms_norm(x, w, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def post_norm(x, y, w, alpha: float, eps: float):
    """The residual rule: the norm is taken of alpha x + y, and what it gives IS the new stream."""
    return rms_norm(alpha * x + y, w, eps)


# ---------------------------------------------------------------------------------------------- attention branch
def frequencies(rot: dict):
    """Rotary frequencies [dims/2]: long wavelengths are divided by `factor`, short ones kept, a linear blend between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    sc = rot.get("scaling")
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wave = 2 * math.pi / f
            short, long = sc["original"] / sc["high"], sc["original"] / sc["low"]
            if wave > long:
                f = f / sc["factor"]
            elif wave >= short:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x, positions, rot: dict):
    """x [T, heads, dim]: pairs (2i, 2i+1) of the first rot.dims columns turned by position * frequency_i."""
    dims = int(rot["dims"])
    a = positions.to(F64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def visible(i: int, mask: dict | None):
    """Positions that position i sees."""
    if not mask:
        return list(range(i + 1))
    return [j for j in range(i + 1) if i - j < mask["size"] or j < mask.get("keep_first", 0)]


def window_attention(q, k, v, scale: float, mask: dict | None, first_pos: int = 0):
    """q [Tq, H, d]; k [Tk, G, d], v [Tk, G, dv] hold positions 0..Tk-1; query t sits at first_pos + t."""
    Tq, H, d = q.shape
    G = k.shape[1]
    rep = H // G
    out = torch.zeros(Tq, H, v.shape[2], dtype=q.dtype)
    for t in range(Tq):
        see = visible(first_pos + t, mask)
        kk, vv = k[see], v[see]
        for h in range(H):
            p = torch.softmax((kk[:, h // rep] @ q[t, h]) * scale, 0)
            out[t, h] = p @ vv[:, h // rep]
    return out


def attention_branch(h, w, pre: str, m: dict, eps: float, past=None):
    """One branch of the 'parallel' mixer over tokens h [T, width]; past = (k, v) of the tokens before (rotated keys).
    Returns (output, (k, v) of all tokens)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, d)
    k = (h @ w[pre + "k"].T).view(T, G, d)
    v = (h @ w[pre + "v"].T).view(T, G, dv)
    q, k = rms_norm(q, w[pre + "q.norm"], eps), rms_norm(k, w[pre + "k.norm"], eps)
    at = 0 if past is None else past[0].shape[0]
    if m.get("rot"):
        pos = torch.arange(at, at + T)
        q, k = rotate(q, pos, m["rot"]), rotate(k, pos, m["rot"])
    if past is not None:
        k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    o = window_attention(q, k, v, m["scale"], m.get("mask"), at).reshape(T, H * dv)
    o = o * torch.sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T, (k, v)


# ---------------------------------------------------------------------------------------------- delta-rule branch
def short_conv(u, w, tail=None):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros (or `tail`, the taps-1 inputs before u)
    ahead of the sequence. Returns (y, the last taps-1 inputs)."""
    taps = w.shape[1]
    T, C = u.shape
    if tail is None:
        tail = torch.zeros(taps - 1, C, dtype=u.dtype)
    full = torch.cat([tail, u], 0)
    y = torch.zeros(T, C, dtype=u.dtype)
    for j in range(taps):
        y += full[j:j + T] * w[:, j]
    return y, full[full.shape[0] - (taps - 1):]


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def softplus(z):
    return torch.where(z > 0, z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def delta_rule(q, k, v, g, beta, S):
    """q, k [T, G, d]; v [T, H, dv]; g, beta [T, H]; S [H, d, dv]. Returns (o [T, H, dv], S after the last token)."""
    T, H, dv = v.shape
    rep = H // q.shape[1]
    S = S.clone()
    out = torch.zeros(T, H, dv, dtype=v.dtype)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // rep], q[t, h // rep]
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] = S[h] + torch.outer(kk, u)
            out[t, h] = S[h].T @ qq
    return out, S


def delta_branch(h, w, pre: str, m: dict, eps: float, past=None):
    """past = (S, tails of q, k, v). Returns (output, state after the last token)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    S, tq, tk, tv = past if past is not None else (torch.zeros(H, d, dv, dtype=h.dtype), None, None, None)
    q, tq = short_conv(h @ w[pre + "q"].T, w[pre + "q.conv"], tq)
    k, tk = short_conv(h @ w[pre + "k"].T, w[pre + "k.conv"], tk)
    v, tv = short_conv(h @ w[pre + "v"].T, w[pre + "v.conv"], tv)
    q, k, v = silu(q).view(T, G, d), silu(k).view(T, G, d), silu(v).view(T, H, dv)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    g = torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(h @ w[pre + "a"].T + w[pre + "dt_bias"]))
    o, S = delta_rule(q, k, v, g, beta, S)
    o = rms_norm(o, w[pre + "norm"], eps).reshape(T, H * dv) * silu(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T, (S, tq, tk, tv)


# ---------------------------------------------------------------------------------------------- wkv mixer
def token_shift(h, mu, last=None):
    """h + (previous h - h) mu; `last` is the token before h[0] (zeros at a sequence's start)."""
    prev = torch.cat([torch.zeros_like(h[:1]) if last is None else last[None], h[:-1]])
    return h + (prev - h) * mu


def wkv_recurrence(r, k, v, decay, u, S):
    """r, k, decay [T, H, d]; v [T, H, d]; u [H, d]; S [H, d, d] (key rows). The bonus counts only at the current token."""
    T, H, d = r.shape
    S = S.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=r.dtype)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = decay[t, h][:, None] * S[h] + kv
    return out, S


def wkv_mixer(h, w, pre: str, m: dict, eps: float, past=None):
    """past = (S, last h). Returns (output, state after the last token)."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    S, last = past if past is not None else (torch.zeros(H, d, d, dtype=h.dtype), None)
    mix = {s: token_shift(h, w[pre + "mu." + s], last) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[pre + s].T).view(T, H, d) for s in "rkv")
    gate = silu(mix["g"] @ w[pre + "g"].T)
    z = torch.tanh(mix["w"] @ w[pre + "w1"].T) @ w[pre + "w2"].T + w[pre + "w0"]
    decay = torch.exp(-torch.exp(z)).view(T, H, d)
    o, S = wkv_recurrence(r, k, v, decay, w[pre + "u"], S)
    o = rms_norm(o, 1.0, eps).reshape(T, H * d) * w[pre + "norm"] * gate
    return o @ w[pre + "o"].T, (S, h[-1])


# ---------------------------------------------------------------------------------------------- the model
def dense_ff(h, w, pre: str):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def parallel_mixer(h, w, pre: str, m: dict, eps: float, past=None):
    pl, pr = past if past is not None else (None, None)
    left, pl = attention_branch(h, w, pre + "left.", m["left"], eps, pl)
    right, pr = delta_branch(h, w, pre + "right.", m["right"], eps, pr)
    return m["left_scale"] * left + m["right_scale"] * right, (pl, pr)


MIXERS = {"parallel": parallel_mixer, "wkv": wkv_mixer}


def forward(tokens, w, cfg: dict, past=None, layers=None):
    """Logits [T, vocab] of `tokens`; past: the list of per-layer states that an earlier call returned (tokens then
    continue that sequence). Returns (logits, states). `layers`: a list that receives the stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = rms_norm(w["embed"][tokens], w["embed.norm"], eps)
    states = []
    for i, entry in enumerate(cfg["layers"]):
        pre = f"l{i}."
        y, st = MIXERS[entry["type"]](x, w, pre + "mix.", entry["mixer"], eps, None if past is None else past[i])
        states.append(st)
        x = post_norm(x, y, w[pre + "norm1"], alpha, eps)
        if entry.get("mlp"):
            x = post_norm(x, dense_ff(x, w, pre + "mlp."), w[pre + "norm2"], alpha, eps)
        if layers is not None:
            layers.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T, states


def to64(tensors: dict):
    return {k: v.to(F64) for k, v in tensors.items()}


def tensor_shapes(cfg: dict):
    """{checkpoint tensor name: shape} of a configuration; a wkv mixer's decay rank is its "decay_rank" (default 8)."""
    V, W = cfg["vocab"], cfg["width"]
    s = {"embed": (V, W), "embed.norm": (W,), "final.norm": (W,), "head": (V, W)}
    for i, entry in enumerate(cfg["layers"]):
        m, pre = entry["mixer"], f"l{i}.mix."
        s[f"l{i}.norm1"] = (W,)
        if entry["type"] == "wkv":
            n, rank = m["heads"] * m["dim"], m.get("decay_rank", 8)
            for c in "rkvgw":
                s[pre + "mu." + c] = (W,)
            for c in "rkvg":
                s[pre + c] = (n, W)
            s.update({pre + "w1": (rank, W), pre + "w2": (n, rank), pre + "w0": (n,), pre + "u": (m["heads"], m["dim"]),
                      pre + "norm": (n,), pre + "o": (W, n)})
        else:
            a, b = m["left"], m["right"]
            pl, pr = pre + "left.", pre + "right."
            nq, nk, nv, no = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"], a["heads"] * a["vdim"]
            s.update({pl + "q": (nq, W), pl + "k": (nk, W), pl + "v": (nv, W), pl + "q.norm": (a["dim"],),
                      pl + "k.norm": (a["dim"],), pl + "g": (no, W), pl + "o": (W, no)})
            nqk, nv = b["kv_heads"] * b["dim"], b["heads"] * b["vdim"]
            for c, n in (("q", nqk), ("k", nqk), ("v", nv)):
                s[pr + c], s[pr + c + ".conv"] = (n, W), (n, b["conv"])
            s.update({pr + "b": (b["heads"], W), pr + "a": (b["heads"], W), pr + "A_log": (b["heads"],),
                      pr + "dt_bias": (b["heads"],), pr + "norm": (b["vdim"],), pr + "g": (nv, W), pr + "o": (W, nv)})
        if entry.get("mlp"):
            ff = entry["mlp"]["ff"]
            s[f"l{i}.norm2"] = (W,)
            s.update({f"l{i}.mlp.gate": (ff, W), f"l{i}.mlp.up": (ff, W), f"l{i}.mlp.down": (W, ff)})
    return s


def random_weights(cfg: dict, seed: int = 0):
    """bf16 tensors for every name: matrices N(0, 1/fan_in) (queries a bit larger, so that the attention is not flat),
    norm weights near one, decays spread so that states neither vanish at once nor never."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = torch.randn(shape, generator=g)
        tail = name.split(".")[-1]
        if tail in ("norm", "norm1", "norm2"):
            z = 1 + 0.2 * z
            if name.endswith("left.q.norm"):
                z = z * 2
        elif ".mu." in name:
            z = torch.rand(shape, generator=g)
        elif tail == "conv":
            z = 0.6 * z
        elif tail == "A_log":
            z = torch.rand(shape, generator=g) * 3 - 4
        elif tail == "dt_bias":
            z = 0.5 * z
        elif tail == "w0":
            z = torch.rand(shape, generator=g) * 4 - 5
        elif tail == "u":
            z = 0.7 * z
        elif name == "embed":
            pass
        else:
            z = z * shape[-1] ** -0.5
        out[name] = z.to(torch.bfloat16)
    return out
