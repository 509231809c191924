"""A plain, slow restatement of the Ragilorn decoder in float64, one function per mechanism, for the tests.

It shares no code with the package: every function works on whole sequences held in torch tensors on the CPU. Weights
come as a dict {checkpoint tensor name: tensor}; the configuration is the dict of config.json.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def to64(tensors: dict) -> dict:
    return {k: v.to(F64) for k, v in tensors.items()}


def sub(tensors: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def rms_norm(x, w, eps: float):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ----------------------------------------------------------------------------- positions
def yarn_table(rot: dict):
    """(frequency of every pair, factor on cos and sin)."""
    n, base = int(rot["dims"]), float(rot["base"])
    freqs, mag = [base ** (-2.0 * i / n) for i in range(n // 2)], 1.0
    if rot.get("scaling"):
        s = rot["scaling"]

        def pair_with(turns):                    # the (fractional) pair that turns `turns` times over the original length
            return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

        first = max(math.floor(pair_with(s["fast"])), 0)
        last = min(math.ceil(pair_with(s["slow"])), n - 1)
        for i in range(n // 2):
            ramp = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
            freqs[i] = freqs[i] / s["factor"] * ramp + freqs[i] * (1.0 - ramp)
        mag = 0.1 * math.log(s["factor"]) + 1.0
    return freqs, mag


def rotate(x, positions, rot: dict):
    """x [T, heads, dim]: neighbouring pairs of the first rot.dims columns turned by position times frequency."""
    freqs, mag = yarn_table(rot)
    out = x.clone()
    for i, f in enumerate(freqs):
        a = positions.to(F64) * f
        c, s = (torch.cos(a) * mag)[:, None], (torch.sin(a) * mag)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


# ----------------------------------------------------------------------------- sequence mixers
def short_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                y[t] += w[:, j] * u[src]
    return y


def visible_from(pos: int, chunk: int) -> int:
    """First position that `pos` sees: the start of its chunk (chunks counted from position 0), or 0."""
    return pos // chunk * chunk if chunk else 0


def attention(q, k, v, scale: float, chunk: int = 0, first_pos: int = 0):
    """q [Tq, H, d] at positions first_pos ..; k [Tk, G, d], v [Tk, G, dv] of positions 0 .. Tk - 1; causal, inside the
    query's chunk. -> [Tq, H, dv]"""
    Tq, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(Tq, H, v.shape[2], dtype=q.dtype)
    for t in range(Tq):
        pos = first_pos + t
        lo = visible_from(pos, chunk)
        for h in range(H):
            p = torch.softmax((k[lo:pos + 1, h // rep] @ q[t, h]) * scale, 0)
            out[t, h] = p @ v[lo:pos + 1, h // rep]
    return out


def attention_mixer(h, P, m, positions, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = {}
    for n in "qkv":
        u = h @ P[n].T + P[n + ".b"]
        proj[n] = short_conv(u, P[n + ".conv"]) if n + ".conv" in P else u
    q = rotate(proj["q"].reshape(T, H, d), positions, m["rot"])
    k = rotate(proj["k"].reshape(T, G, d), positions, m["rot"])
    o = attention(q, k, proj["v"].reshape(T, G, dv), m["scale"], int((m.get("mask") or {}).get("size", 0)))
    return o.reshape(T, H * dv) @ P["o"].T + P["o.b"]


def latent_rows(h, P, m, positions, eps):
    """What a token leaves in the cache: (normed latent [T, kv_rank], rotated key part [T, rot_dim])."""
    both = h @ P["dkv"].T
    c = rms_norm(both[:, :m["kv_rank"]], P["dkv.norm"], eps)
    return c, rotate(both[:, None, m["kv_rank"]:], positions, m["rot"])[:, 0]


def latent_attention_mixer(h, P, m, positions, eps):
    """Keys and values up-projected explicitly from the latent."""
    T = h.shape[0]
    H, d, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ P["q"].T).reshape(T, H, d + dr)
    q_rot = rotate(q[:, :, d:], positions, m["rot"])
    c, kr = latent_rows(h, P, m, positions, eps)
    k = (c @ P["uk"].T).reshape(T, H, d)
    v = (c @ P["uv"].T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        for n in range(H):
            s = (k[:t + 1, n] @ q[t, n, :d] + kr[:t + 1] @ q_rot[t, n]) * m["scale"]
            out[t, n] = torch.softmax(s, 0) @ v[:t + 1, n]
    return out.reshape(T, H * dv) @ P["o"].T


MIXERS = {"attention": attention_mixer, "latent_attention": latent_attention_mixer}


# ----------------------------------------------------------------------------- feed-forward
def gated_ff(u, P, prefix=""):
    return (silu(u @ P[prefix + "gate"].T) * (u @ P[prefix + "up"].T)) @ P[prefix + "down"].T


def route(z, top: int):
    """z [T, E] -> (chosen [T, top], their sigmoid scores, not normalised)."""
    s = sigmoid(z)
    w, ids = s.topk(top, -1)
    return ids, w


def moe_ff(u, P, top: int):
    """Every chosen expert reads its weight times the token; the outputs are added as they are."""
    ids, w = route(u @ P["router"].T, top)
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(top):
            out[t] += gated_ff(w[t, j] * u[t], P, f"e{int(ids[t, j])}.")
    return out


def feed_forward(u, P, mlp: dict):
    return gated_ff(u, P) if mlp["kind"] == "dense" else moe_ff(u, P, mlp["router"]["top"])


# ----------------------------------------------------------------------------- the residual
def gated_branch(x, y, h, W, b):
    """x + y times the gate that the sublayer's input h opens, element by element."""
    return x + y * sigmoid(h @ W.T + b)


def depth_average(outputs: list, weights):
    """sum_j weights[j] outputs[j]: the embedding output and every layer's result so far."""
    assert len(outputs) == len(weights)
    total = torch.zeros_like(outputs[0])
    for wj, xj in zip(weights, outputs):
        total = total + wj * xj
    return total


def cap_logits(z, scale: float, cap: float):
    z = z * scale
    return cap * torch.tanh(z / cap) if cap else z


def forward(cfg: dict, weights: dict, tokens, layers_out: list | None = None):
    """Logits [T, vocab] of a whole sequence; layers_out receives the stream that every layer hands on."""
    w = to64(weights)
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    positions = torch.arange(x.shape[0])
    outputs = [x]
    for i, entry in enumerate(cfg["layers"]):
        P = sub(w, f"l{i}.")
        h = rms_norm(x, P["norm1"], eps)
        y = MIXERS[entry["type"]](h, sub(P, "mix."), entry["mixer"], positions, eps)
        x = gated_branch(x, y, h, P["rg1"], P["rg1.b"])
        if entry.get("mlp"):
            h = rms_norm(x, P["norm2"], eps)
            x = gated_branch(x, feed_forward(h, sub(P, "mlp."), entry["mlp"]), h, P["rg2"], P["rg2.b"])
        outputs.append(x)
        x = depth_average(outputs, P["dwa"])
        if layers_out is not None:
            layers_out.append(x)
    z = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    return cap_logits(z, float(cfg.get("logit_scale", 1.0)), float(cfg.get("logit_softcap") or 0.0))


# ----------------------------------------------------------------------------- random weights
def random_weights(cfg: dict, seed: int = 0, dtype=torch.bfloat16) -> dict:
    """Random weights for a configuration, rounded to `dtype` (the values every implementation then starts from)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}

    def mat(name, o, i, std=None):
        out[name] = torch.randn(o, i, generator=g) * (std if std is not None else i ** -0.5)

    def vec(name, n, mean=0.0, std=0.1):
        out[name] = mean + std * torch.randn(n, generator=g)

    out["embed"] = torch.randn(cfg["vocab"], W, generator=g) / float(cfg["embedding"]["scale"])
    mat("head", cfg["vocab"], W, 3.0 * W ** -0.5)
    vec("final.norm", W, 1.0)
    for i, entry in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", entry["mixer"], entry.get("mlp")
        for n in ("1", "2") if mlp else ("1",):
            vec(p + "norm" + n, W, 1.0)
            mat(p + "rg" + n, W, W)
            vec(p + f"rg{n}.b", W, 0.5, 0.5)
        out[p + "dwa"] = 0.15 * torch.randn(i + 2, generator=g)
        out[p + "dwa"][-1] += 1.0
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if entry["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                mat(p + "mix." + n, rows, W)
                vec(p + f"mix.{n}.b", rows, 0.0, 0.5)
                if m.get("conv"):
                    out[p + f"mix.{n}.conv"] = 0.5 * torch.randn(rows, m["conv"], generator=g)
            vec(p + "mix.o.b", W, 0.0, 0.3)
        else:
            R, dr = m["kv_rank"], m["rot_dim"]
            mat(p + "mix.q", H * (d + dr), W)
            mat(p + "mix.dkv", R + dr, W)
            vec(p + "mix.dkv.norm", R, 1.0)
            mat(p + "mix.uk", H * d, R)
            mat(p + "mix.uv", H * dv, R)
        mat(p + "mix.o", W, H * dv)
        if mlp and mlp["kind"] == "dense":
            mat(p + "mlp.gate", mlp["ff"], W, 2.0 * W ** -0.5)
            mat(p + "mlp.up", mlp["ff"], W, 2.0 * W ** -0.5)
            mat(p + "mlp.down", W, mlp["ff"])
        elif mlp:
            ff = mlp["expert"]["ff"]
            mat(p + "mlp.router", mlp["router"]["experts"], W, 2.0 * W ** -0.5)
            for e in range(mlp["router"]["experts"]):
                mat(p + f"mlp.e{e}.gate", ff, W, 2.0 * W ** -0.5)
                mat(p + f"mlp.e{e}.up", ff, W, 2.0 * W ** -0.5)
                mat(p + f"mlp.e{e}.down", W, ff, 2.0 * ff ** -0.5)
    return {k: v.to(dtype) for k, v in out.items()}
