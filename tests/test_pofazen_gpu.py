"""-m gpu: the Pofazen decoder (windowed softmax attention with kept first tokens and an element-wise gate beside a gated
delta rule with one decay per head in one mixer; wkv recurrences that read mixes of a token with the token before; a
residual whose RMS norm is taken of the sum; silu-gated feed-forwards) against tests/pofazen_oracle.py, a plain float64
restatement.

Every test makes its own small configuration and random weights. Models run in true fp32 (the sharp comparison: relative
error of every row of logits below 2e-4) and in bf16 (the serving precision). The schedules are fed through
LLMEngine.step_given -- the scheduler's block manager, the runner's step and the model's kernels -- so what is compared
is the engine, not a forward function. Where random weights would hide a fault (a key just outside the window, a kept
first token, a block border) the mechanism tests scale one query and key so that one score takes the whole softmax.
"""
import json
import os
import random

import pytest
import torch

import pofazen_oracle as O

pytestmark = pytest.mark.gpu
F64 = torch.float64


def rot(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def dense(ff):
    return {"kind": "dense", "ff": ff}


def wkv(heads, dim, rank, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}, "mlp": mlp}


def parallel(left, right, scales=(1.0, 1.0), mlp=None):
    """left: (heads, kv_heads, dim, vdim, scale, window, keep_first, rot); right: (heads, kv_heads, dim, vdim, conv)."""
    h, g, d, dv, scale, size, keep, r = left
    lm = {"heads": h, "kv_heads": g, "dim": d, "vdim": dv, "scale": scale, "rot": r}
    if size:
        lm["mask"] = {"size": size, "keep_first": keep}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": lm, "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right)),
                      "left_scale": scales[0], "right_scale": scales[1]}}


def config_a():
    """Odd sizes: 6 query heads over 2 key/value heads with key size 24 and value size 20, a window of 13 with three kept
    tokens, 16 rotated columns of which some keep their frequency, some are divided and some lie between; delta heads of
    24 x 12 in pairs; a layer whose attention has no window and no stretch, with other sizes everywhere; wkv heads of 20
    with a decay rank of 7; layers with and without feed-forward, a wkv layer first and a parallel layer last."""
    r = rot(16, 700.0, (6.0, 1.5, 5.0, 90))
    return {"architecture": "Pofazen", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "postln_alpha": 1.7,
            "layers": [wkv(3, 20, 7),
                       parallel((6, 2, 24, 20, 0.3, 13, 3, r), (4, 2, 24, 12, 4), (1.3, 0.6), dense(72)),
                       wkv(2, 36, 12, dense(40)),
                       parallel((4, 4, 12, 28, 0.4, 0, 0, rot(12, 300.0)), (3, 1, 40, 16, 2), (0.7, 1.1))]}


def config_b():
    """Values that are 1 or equal: as many key/value heads as heads, key size = value size, every column rotated, the
    window as wide as a block of the cache, one kept token, unit scales and alpha, a factor of one, one delta head."""
    r = rot(32, 10000.0, (1.0, 1.0, 4.0, 64))
    return {"architecture": "Pofazen", "vocab": 320, "width": 128, "norm": {"eps": 1e-6}, "postln_alpha": 1.0,
            "layers": [parallel((4, 4, 32, 32, 0.18, 16, 1, r), (1, 1, 32, 32, 3), (1.0, 1.0), dense(128)),
                       wkv(4, 32, 16, dense(128)),
                       parallel((2, 1, 32, 32, 0.18, 32, 0, r), (2, 2, 16, 64, 3), (1.0, 1.0), dense(64))]}


def config_c():
    """The head sizes that 16-bit models run on the tensor cores, key size unlike value size both ways."""
    r = rot(48, 5e5, (4.0, 1.0, 3.0, 200))
    return {"architecture": "Pofazen", "vocab": 410, "width": 256, "norm": {"eps": 1e-5}, "postln_alpha": 2.2,
            "layers": [parallel((6, 2, 64, 128, 0.12, 40, 5, r), (4, 1, 64, 64, 4), (0.8, 1.2), dense(192)),
                       wkv(4, 64, 32, dense(96)),
                       parallel((4, 1, 128, 64, 0.1, 21, 0, r), (2, 2, 128, 64, 3), (1.1, 0.9), dense(192))]}


def config_d():
    """Nothing is a multiple of 8, and more tokens are kept than the window is wide."""
    r = rot(6, 50.0, (3.0, 1.0, 6.0, 30))
    return {"architecture": "Pofazen", "vocab": 97, "width": 50, "norm": {"eps": 1e-4}, "postln_alpha": 0.6,
            "layers": [parallel((3, 1, 10, 6, 0.4, 5, 9, r), (5, 5, 6, 9, 3), (0.5, 1.4), dense(30)),
                       wkv(5, 9, 3, dense(21)),
                       parallel((3, 3, 7, 5, 0.5, 3, 2, rot(4, 20.0)), (2, 1, 11, 3, 5), (1.0, 0.3))]}


CONFIGS = {"a": config_a, "b": config_b, "c": config_c, "d": config_d}
# bf16 models: (root mean square over the rows, largest row) of the relative error, about three times what rounding the
# oracle's matrix products to bf16 alone causes -- a small alpha lets the norm of the sum amplify it
BF16_LIMITS = {"a": (0.02, 0.05), "b": (0.04, 0.12), "c": (0.015, 0.03), "d": (0.1, 0.4)}
_MODELS, _ENGINES = {}, {}


def reference(cfg, w64, toks, layers=None):
    return O.forward(torch.tensor(toks), w64, cfg, layers=layers)[0]


def model_dir(tmp_path_factory, name):
    """(folder with config.json + model.safetensors, config, fp64 weights) of a named test model, made once."""
    if name not in _MODELS:
        from safetensors.torch import save_file
        cfg = CONFIGS[name]()
        tensors = O.random_weights(cfg, seed=ord(name))
        d = tmp_path_factory.mktemp("pofazen_" + name)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
        save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(d, "model.safetensors"))
        _MODELS[name] = (str(d), cfg, O.to64(tensors))
    return _MODELS[name]


def engine(tmp_path_factory, name, dtype, eager=False, blocks=24, block_size=16):
    key = (name, dtype, eager, blocks, block_size)
    if key not in _ENGINES:
        from nanovllm.engine.llm_engine import LLMEngine
        path = model_dir(tmp_path_factory, name)[0]
        _ENGINES[key] = LLMEngine(path, dtype=dtype, kvcache_block_size=block_size, num_kvcache_blocks=blocks + 1,
                                  max_num_seqs=4, max_model_len=blocks * block_size,
                                  max_num_batched_tokens=4 * blocks * block_size, return_logits=True,
                                  enforce_eager=eager, chunked_prefill=True)
    return _ENGINES[key], _MODELS[name][1], _MODELS[name][2]


def row_err(got, want):
    """Per row: root mean square of the difference (row means removed) over that of the reference."""
    d = got.to(F64).cpu() - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()


def close(got, want, dtype, name):
    e = row_err(got, want)
    if dtype == "float32":
        return bool((e < 2e-4).all())
    rms, worst = BF16_LIMITS[name]
    return float(e.pow(2).mean().sqrt()) < rms and float(e.max()) < worst


def tokens_of(cfg, n, seed):
    g = random.Random(seed)
    return [g.randrange(cfg["vocab"]) for _ in range(n)]


def feed(eng, rid, toks, cuts):
    """One request alone, cut at `cuts`; returns logits of every position."""
    outs, lo = [], 0
    for hi in list(cuts) + [len(toks)]:
        if hi <= lo:
            continue
        outs.append(eng.step_given([(rid, toks[lo:hi], list(range(hi - lo)))], [rid] if hi == len(toks) else []))
        lo = hi
    return torch.cat(outs)


CASES = [(n, dt) for n in "abcd" for dt in ("float32", "bfloat16")]


# ------------------------------------------------------------------ whole prompts, decoding, portions
@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_prompt_and_layers(tmp_path_factory, name, dtype):
    eng, cfg, w = engine(tmp_path_factory, name, dtype)
    toks = tokens_of(cfg, 75, 1)
    layers = []
    want = reference(cfg, w, toks, layers)
    model = eng.model_runner.model
    model.trace_layers = []
    try:
        got = feed(eng, "w", toks, [])
        seen = [x.cpu() for x in model.trace_layers]
    finally:
        model.trace_layers = None
    assert len(seen) == len(cfg["layers"]) and all(x.dtype == torch.float32 for x in seen)
    if dtype == "float32":
        for i, x in enumerate(seen):                  # the residual stream after every layer
            assert float((x.to(F64) - layers[i]).abs().max() / layers[i].abs().max()) < 1e-4, i
    assert close(got, want, dtype, name), float(row_err(got, want).max())


@pytest.mark.parametrize("name,dtype", CASES)
@pytest.mark.parametrize("eager", [False, True])
def test_prefill_then_token_by_token(tmp_path_factory, name, dtype, eager):
    """Most of a prompt in one step, the rest one token a step (CUDA-graph decode and eager decode): decoded positions
    cross block borders and window edges, states, convolution tails and shifted rows are carried token by token; a
    one-token prompt starts from the first token, which has no token before it."""
    eng, cfg, w = engine(tmp_path_factory, name, dtype, eager)
    toks = tokens_of(cfg, 70, 2)
    want = reference(cfg, w, toks)
    for first in (1, 2, 29):
        got = feed(eng, "d", toks, range(first, len(toks)))
        assert close(got, want, dtype, name), (first, float(row_err(got, want).max()))


@pytest.mark.parametrize("name,dtype", CASES)
def test_portions_of_every_size(tmp_path_factory, name, dtype):
    eng, cfg, w = engine(tmp_path_factory, name, dtype)
    toks = tokens_of(cfg, 90, 3)
    want = reference(cfg, w, toks)
    for size in (2, 3, 7, 16, 19, 33):
        got = feed(eng, "p", toks, range(size, len(toks), size))
        assert close(got, want, dtype, name), (size, float(row_err(got, want).max()))
    g = random.Random(5)
    cuts, at = [], 0
    while at < len(toks):
        at += g.choice([1, 1, 2, 2, 3, 5, 16, 21])
        cuts.append(at)
    got = feed(eng, "p", toks, [c for c in cuts if c < len(toks)])
    assert close(got, want, dtype, name)


@pytest.mark.parametrize("name,dtype", CASES)
def test_unequal_batches_and_reused_slots(tmp_path_factory, name, dtype):
    """Up to four live requests, portions of some beside single tokens of others, requests that sit out a step;
    every request ends at its own time and later ones take over its blocks and state slot (the pool has 12 blocks,
    the seven requests need 23); each must match its own run alone."""
    pool = 12
    eng, cfg, w = engine(tmp_path_factory, name, dtype, blocks=pool)
    g = random.Random(7)
    lens = [37, 90, 5, 64, 51, 33, 18]
    reqs = {f"r{i}": tokens_of(cfg, n, 10 + i) for i, n in enumerate(lens)}
    want = {k: reference(cfg, w, v) for k, v in reqs.items()}
    at = {k: 0 for k in reqs}
    got = {k: [] for k in reqs}
    waiting, live = list(reqs), []
    bm = eng.scheduler.block_manager
    blocks_of = lambda k: -(-len(reqs[k]) // bm.block_size)
    slots, tables = {}, {}
    while waiting or live:
        while waiting and len(live) < 4 and sum(map(blocks_of, live)) + blocks_of(waiting[0]) <= pool:
            live.append(waiting.pop(0))
        entries, end = [], []
        for k in live:
            if at[k] > 0 and g.random() < 0.15:
                continue                                   # left out of this step, goes on later
            n = min(len(reqs[k]) - at[k], g.choice([1, 1, 1, 2, 3, 11, 24]))
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(reqs[k]):
                end.append(k)
        if not entries:
            continue
        out = eng.step_given(entries, end)
        row = 0
        for k, t, places in entries:
            got[k].append(out[row:row + len(places)])
            row += len(places)
            if k in eng.scheduler.given:
                slots[k] = eng.scheduler.given[k].state_slot
                tables[k] = list(eng.scheduler.given[k].block_table)
        live = [k for k in live if k not in end]
    assert len(set(slots.values())) <= 4 < len(slots)                            # slots were used again
    assert sum(len(t) for t in tables.values()) > pool                           # and so were blocks
    assert len(bm.free_block_ids) == pool and len(bm.free_state_slots) == 4      # everything was given back
    for k in reqs:
        assert close(torch.cat(got[k]), want[k], dtype, name), (k, float(row_err(torch.cat(got[k]), want[k]).max()))


@pytest.mark.parametrize("name,dtype,n", [("a", "float32", 303), ("c", "bfloat16", 370)])
def test_long_decoding(tmp_path_factory, name, dtype, n):
    """Hundreds of tokens one by one after a short prompt: states are carried all along, the window passes over decoded
    tokens and over every tile of keys in between, positions go past the stretch's original length."""
    eng, cfg, w = engine(tmp_path_factory, name, dtype)
    toks = tokens_of(cfg, n, 4)
    want = reference(cfg, w, toks)
    got = feed(eng, "l", toks, range(3, len(toks)))
    assert close(got, want, dtype, name), float(row_err(got, want).max())


def test_greedy_generation_through_the_scheduler(tmp_path_factory):
    """LLM.generate (waiting/running queues, prefill steps, graph decode steps, sampling) in fp32 against the
    oracle's greedy continuation, for three prompts of unequal length at once."""
    from nanovllm import LLM, SamplingParams
    path, cfg, w = model_dir(tmp_path_factory, "b")
    llm = LLM(path, dtype="float32", kvcache_block_size=16, num_kvcache_blocks=40, max_num_seqs=4, max_model_len=128,
              max_num_batched_tokens=512)
    prompts = [tokens_of(cfg, n, 20 + n) for n in (9, 30, 17)]
    outs = llm.generate(prompts, SamplingParams(temperature=1.0, max_tokens=10, ignore_eos=True, greedy=True),
                        use_tqdm=False)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for tok in o["token_ids"]:
            logits = reference(cfg, w, seq)[-1]
            top = torch.topk(logits, 2).values
            # sampling reads bf16 logits: two entries closer than that rounding may change places
            if float(top[0] - top[1]) > 1e-2 * float(logits.abs().max()):
                assert tok == int(logits.argmax()), (len(seq), tok)
            seq.append(tok)
    llm.exit()


# ------------------------------------------------------------------ mechanisms alone
def _dev(x, dtype=torch.float32):
    return x.to(dtype).cuda().contiguous()


def _cu(lens):
    return torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32).cuda()


def _spans(q_lens, k_lens):
    from nanovllm import ops
    return ops.StepSpans(_cu(q_lens), _cu(k_lens), None, max(q_lens))


def _decode_spans(ctx_lens):
    from nanovllm import ops
    return ops.StepSpans(None, None, torch.tensor(ctx_lens, dtype=torch.int32).cuda())


def _slots(*ids):
    return torch.tensor(ids, dtype=torch.int32).cuda()


@pytest.mark.parametrize("W", [37, 50, 96, 512, 2048])
def test_norm_of_the_sum(W):
    """x <- N(alpha x + y) and the stream in the model dtype, for widths that take the 16-byte form and widths that do
    not; the first norm straight from the embedding table; two branches in one launch."""
    from nanovllm import ops
    g = torch.Generator().manual_seed(W)
    rows, eps, alpha = 9, 1e-3, 1.8
    x0, y, y2 = (torch.randn(rows, W, generator=g, dtype=F64) * s for s in (2.0, 3.0, 1.0))
    w = 1 + 0.2 * torch.randn(W, generator=g, dtype=F64)
    want = O.post_norm(x0, y, w, alpha, eps)
    assert float((want - (x0 + O.rms_norm(y, w, eps))).abs().max()) > 0.5          # not "add the norm of the branch"
    for dtype in (torch.float32, torch.bfloat16):
        yy = y.to(dtype)
        want = O.post_norm(x0, yy.to(F64), w, alpha, eps)
        x = _dev(x0)
        h = ops.norm_residual_(x, yy.cuda(), _dev(w), None, eps, dtype, kind="rms", carry=alpha)
        assert float((x.cpu().to(F64) - want).abs().max()) < 2e-6 and x.dtype == torch.float32
        assert torch.equal(h, x.to(dtype))
    x = _dev(x0)
    ops.norm_residual_(x, _dev(y), _dev(w), None, eps, torch.float32, kind="rms", carry=alpha, y2=_dev(y2))
    assert float((x.cpu().to(F64) - O.post_norm(x0, y + y2, w, alpha, eps)).abs().max()) < 2e-6
    table = torch.randn(20, W, generator=g, dtype=F64)
    idx = torch.tensor([3, 19, 0, 7, 7, 12, 1, 5, 18])
    x = torch.full((rows, W), float("nan"), device="cuda")
    ops.norm_residual_(x, _dev(table), _dev(w), None, eps, torch.float32, kind="rms", accumulate=False,
                       y_index=idx.cuda())
    assert float((x.cpu().to(F64) - O.rms_norm(table[idx], w, eps)).abs().max()) < 2e-6


@pytest.mark.parametrize("scaling", [None, (8.0, 1.0, 4.0, 100), (3.0, 2.0, 2.0, 500), (2.0, 0.5, 8.0, 20000)])
@pytest.mark.parametrize("H,G,d,dv,dims", [(3, 1, 10, 5, 6), (4, 2, 24, 20, 16), (6, 2, 64, 128, 48), (2, 2, 128, 64, 128),
                                           (2, 1, 16, 8, 0)])
def test_head_norm_rotation_and_cache_rows(H, G, d, dv, dims, scaling):
    """Per-head norm with a shared weight, rotation of the first columns at positions up to a million (fp64 angles), k and
    v at their slots (flat, and (block, offset) pairs; a negative slot writes nothing), for sizes of the scalar and of
    the 16-byte form, in a slice of a wider row, fp32 and bf16."""
    from nanovllm import ops
    from nanovllm.layers.seq_mixers import WavelengthScaledRotary
    g = torch.Generator().manual_seed(dims + d)
    pos, eps, bs = torch.tensor([0, 1, 2, 63, 4097, 1000003]), 1e-3, 4
    T, nq, nk, nv = 6, H * d, G * d, G * dv
    r = rot(dims, 500.0, scaling)
    wr = WavelengthScaledRotary(dims, 500.0, True, r.get("scaling"))
    wq, wk = (1 + 0.3 * torch.randn(d, generator=g, dtype=F64) for _ in range(2))
    table = ops.rotary_table(pos.cuda(), wr.freq.cuda()) if dims else None
    slots = torch.tensor([5, 2, -1, 11, 0, 7], dtype=torch.int32)
    for dtype in (torch.float32, torch.bfloat16):
        wide = torch.randn(T, nq + nk + nv + 16, generator=g, dtype=F64).to(dtype)
        src = wide[:, :nq + nk + nv].to(F64)
        q = O.rms_norm(src[:, :nq].reshape(T, H, d), wq, eps)
        k = O.rms_norm(src[:, nq:nq + nk].reshape(T, G, d), wk, eps)
        if dims:
            q, k = O.rotate(q, pos, r), O.rotate(k, pos, r)
        tol = 3e-6 if dtype == torch.float32 else 3e-2
        for paired in (False, True):
            kc = torch.zeros(3, bs, nk, dtype=dtype, device="cuda")
            vc = torch.zeros(3, bs, nv, dtype=dtype, device="cuda")
            sl = slots.clone()
            if paired:
                sl = torch.stack([slots // bs, slots % bs], 1)
                sl[2] = torch.tensor([-1, 0])
            x = wide.cuda()
            ops.norm_rope_cache(x[:, :nq + nk + nv], _dev(wq), _dev(wk), eps, table, H, G, d, dv, dims, True, kc, vc,
                                sl.contiguous().cuda())
            got = x.cpu().to(F64)
            assert float((got[:, :nq].reshape(T, H, d) - q).abs().max()) < tol * 4
            assert float((got[:, nq:nq + nk].reshape(T, G, d) - k).abs().max()) < tol * 4
            assert torch.equal(x[:, nq + nk:], wide[:, nq + nk:].cuda())                      # values and what lies behind
            for t, s in enumerate(slots.tolist()):
                if s >= 0:
                    assert torch.equal(kc.view(-1, nk)[s], x[t, nq:nq + nk])
                    assert torch.equal(vc.view(-1, nv)[s], x[t, nq + nk:nq + nk + nv])
            assert int((kc.view(-1, nk).abs().sum(1) > 0).sum()) == 5                          # the negative slot wrote nothing


# ---- attention in a window with kept first tokens
def _attn_case(n, H, G, d, dv, seed, dtype=torch.float32, star=None, gain=7.0):
    """Random q, k, v of one sequence; `star` = (query position, key position, head): that query's head and that key
    are made parallel and long, so that the key takes the softmax wherever it is visible; its value is 5."""
    g = torch.Generator().manual_seed(seed)
    q = torch.randn(n, H, d, generator=g, dtype=F64)
    k = torch.randn(n, G, d, generator=g, dtype=F64)
    v = torch.randn(n, G, dv, generator=g, dtype=F64)
    if star is not None:
        i, j, h = star
        k[j, h // (H // G)] = gain * q[i, h] / q[i, h].norm()
        q[i, h] = gain * q[i, h] / q[i, h].norm()
        v[j, h // (H // G)] = 5.0
    rd = lambda x: x.to(dtype).to(F64)
    return rd(q), rd(k), rd(v)


def _paged(k, v, bs, order):
    """Caches whose blocks are in `order`; returns (k_cache, v_cache, block table [1, n])."""
    n, G, d = k.shape
    dv = v.shape[-1]
    nb = -(-n // bs)
    kc = torch.zeros(max(order) + 2, bs, G * d, dtype=k.dtype)
    vc = torch.zeros(max(order) + 2, bs, G * dv, dtype=v.dtype)
    for b in range(nb):
        rows = slice(b * bs, min(n, (b + 1) * bs))
        kc[order[b], :rows.stop - rows.start] = k[rows].reshape(-1, G * d)
        vc[order[b], :rows.stop - rows.start] = v[rows].reshape(-1, G * dv)
    return kc, vc, torch.tensor([order[:nb]], dtype=torch.int32)


def _module(H, G, d, dv, scale, mask, dtype, kc=None, vc=None, generic=False):
    from nanovllm.layers.seq_mixers import VarSizeAttention
    m = VarSizeAttention(H, G, d, dv, scale, window=mask["size"] if mask else 0,
                         keep_first=mask["keep_first"] if mask else 0).cuda()
    m.force_generic = generic
    if kc is not None:
        m.k_cache, m.v_cache = kc.to(dtype).cuda(), vc.to(dtype).cuda()
    return m


def _run(m, q, k, v, dtype, q_lens=None, k_lens=None, ctx_lens=None, table=None, bs=16):
    """The attention block as a layer calls it, under a step context made by hand."""
    from nanovllm.utils.context import reset_context, set_context
    if ctx_lens is None:
        spans, at = [], 0
        for ql, kl in zip(q_lens, k_lens):
            spans.append((at, ql, kl))
            at += ql
        set_context(True, _cu(q_lens), _cu(k_lens), max(q_lens), max(k_lens), block_tables=table, block_size=bs,
                    host_spans=spans)
    else:
        set_context(False, context_lens=torch.tensor(ctx_lens, dtype=torch.int32).cuda(), block_tables=table, block_size=bs)
    try:
        return m(_dev(q, dtype), _dev(k, dtype), _dev(v, dtype)).cpu().to(F64)
    finally:
        reset_context()


SHAPES = [(6, 2, 24, 20), (3, 1, 10, 6), (4, 2, 64, 64), (6, 2, 64, 128), (4, 1, 128, 64), (8, 1, 128, 128)]


@pytest.mark.parametrize("H,G,d,dv", SHAPES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("size,keep", [(20, 3), (16, 0), (7, 16), (1, 1), (33, 40)])
def test_window_with_kept_tokens(H, G, d, dv, dtype, size, keep):
    """A whole prompt from this step's rows, the same prompt as portions over a shuffled block table beside a second
    sequence, and decode rows beside a padded row, for windows narrower and wider than a block and than what is kept."""
    n, bs, scale = 83, 16, 0.35
    mask = {"size": size, "keep_first": keep}
    q, k, v = _attn_case(n, H, G, d, dv, 3, dtype)
    want = O.window_attention(q, k, v, scale, mask)
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    got = _run(_module(H, G, d, dv, scale, mask, dtype), q, k, v, dtype, [n], [n])
    assert float((got.view(n, H, dv) - want).abs().max()) < tol
    kc, vc, table = _paged(k, v, bs, [5, 0, 3, 1, 4, 2])
    m = _module(H, G, d, dv, scale, mask, dtype, kc, vc)
    table2, at = torch.cat([table, table], 0).cuda(), 0
    for ql in (2, 19, 30, 32):                                         # portions start inside blocks; a neighbour rides along
        qq = torch.cat([q[at:at + ql], q[:5]])
        got = _run(m, qq, qq[:, :G], v[:ql + 5], dtype, [ql, 5], [at + ql, 5], table=table2)
        assert float((got[:ql].view(ql, H, dv) - want[at:at + ql]).abs().max()) < tol, at
        assert float((got[ql:].view(5, H, dv) - want[:5]).abs().max()) < tol
        at += ql
    table3 = torch.cat([table, table, table], 0).cuda()
    for pos in (0, 1, keep, size - 1, size, size + 1, 47, 48, 82):     # decode rows: first tokens, edges, block borders
        pos = min(pos, n - 1)
        got = _run(m, q[[pos, 0, 31]], k[[pos, 0, 31]], v[[pos, 0, 31]], dtype, ctx_lens=[pos + 1, 0, 32], table=table3)
        assert float((got[0].view(H, dv) - want[pos]).abs().max()) < tol, pos
        assert float((got[2].view(H, dv) - want[31]).abs().max()) < tol


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 20), (6, 2, 64, 128), (4, 1, 128, 64)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_keys_just_inside_and_outside(H, G, d, dv, dtype):
    """One key takes the whole softmax of one head where it is visible: the oldest key of the window and the one before
    it, the last kept token and the first that is not, keys at block borders -- in a prompt, in a portion over cached
    keys and for a decoded token, 500 tokens on, so that whole tiles of keys lie between the kept ones and the window."""
    n, bs, scale, size, keep, i = 600, 16, 1.0, 150, 6, 590
    mask = {"size": size, "keep_first": keep}
    order = list(range(37, -1, -1))
    tol = 1e-4 if dtype == torch.float32 else 6e-2
    for j, seen in ((i - size + 1, True), (i - size, False), (keep - 1, True), (keep, False), (0, True), (300, False),
                    (i - 15, True), (i, True), (447, True), (448, True)):
        q, k, v = _attn_case(n, H, G, d, dv, 5 + j, dtype, star=(i, j, 1))
        want = O.window_attention(q[i:i + 1], k[:i + 1], v[:i + 1], scale, mask, first_pos=i)
        assert (float(want[0, 1].min()) > 4.4) == seen, j              # the oracle agrees on who is visible
        got = _run(_module(H, G, d, dv, scale, mask, dtype), q, k, v, dtype, [n], [n])
        assert float((got[i].view(H, dv) - want[0]).abs().max()) < tol, j
        kc, vc, table = _paged(k, v, bs, order)
        m = _module(H, G, d, dv, scale, mask, dtype, kc, vc)
        got = _run(m, q[i - 9:i + 1], k[:10], v[:10], dtype, [10], [i + 1], table=table.cuda())
        assert float((got[9].view(H, dv) - want[0]).abs().max()) < tol, j
        got = _run(m, q[i:i + 1], k[:1], v[:1], dtype, ctx_lens=[i + 1], table=table.cuda())
        assert float((got.view(1, H, dv) - want).abs().max()) < tol, j


@pytest.mark.parametrize("H,G,D,DV", [(4, 2, 64, 64), (4, 2, 64, 128), (4, 1, 128, 64), (8, 1, 128, 128), (8, 8, 64, 128)])
@pytest.mark.parametrize("size,keep", [(300, 5), (1024, 0), (50, 200), (129, 128)])
def test_window_on_the_tensor_core_kernels(H, G, D, DV, size, keep):
    """The tcgen05 prompt kernel in both CTA layouts and the paged decode kernel against the generic kernel: long prompts,
    short portions over thousands of cached keys (split along the keys), a long and short sequences in one launch,
    decode rows whose keys are split over CTAs beside short ones; with a sink too, which must join once."""
    from nanovllm import _C, ops
    g = torch.Generator().manual_seed(D + H + size)
    n, bs, scale = 2900, 64, D ** -0.5 * 2.0
    q = torch.randn(n, H, D, generator=g).bfloat16().cuda()
    k = torch.randn(n, G, D, generator=g).bfloat16().cuda()
    v = torch.randn(n, G, DV, generator=g).bfloat16().cuda()
    sink = torch.tensor([0.0, 1.5, -2.0, 0.3] * (H // 4), dtype=torch.float32).cuda()
    nb = -(-n // bs)
    order = torch.randperm(nb, generator=g)
    pad = nb * bs - n
    kc = torch.zeros(nb + 1, bs, G * D, dtype=torch.bfloat16, device="cuda")
    vc = torch.zeros(nb + 1, bs, G * DV, dtype=torch.bfloat16, device="cuda")
    kc[order.cuda()] = torch.nn.functional.pad(k.view(n, -1), (0, 0, 0, pad)).view(nb, bs, -1)
    vc[order.cuda()] = torch.nn.functional.pad(v.view(n, -1), (0, 0, 0, pad)).view(nb, bs, -1)
    table = order.to(torch.int32).cuda()[None, :].contiguous()
    win = dict(window=size, keep_first=keep)
    for s in (None, sink):
        ref = ops.attn_generic(q, k, v, ops.StepSpans(_cu([n]), _cu([n]), None, n), scale, G, DV, sink=s, **win).float()
        for layout in (1, 2, 0):
            _C.check(_C.load().b200_prefill_set_query_tiles(layout), "b200_prefill_set_query_tiles")
            try:
                got = ops.prefill_varlen_attn(q, k, v, _cu([n]), _cu([n]), n, n, scale, G, vdim=DV, sink=s, **win).float()
                assert float((got - ref).abs().max()) < 3e-2, layout
                for ql in (128, 40, 3):                                # few queries over many keys
                    got = ops.prefill_varlen_attn(q[n - ql:], kc, vc, _cu([ql]), _cu([n]), ql, n, scale, G, vdim=DV,
                                                  block_tables=table, sink=s, **win).float()
                    assert float((got - ref[n - ql:]).abs().max()) < 3e-2, (layout, ql)
                # one long sequence, one that ends inside the first tile, one whose window has just begun to move
                lens, starts = [40, 9, 30], [n - 40, 3, size]
                rows = torch.cat([torch.arange(a, a + b) for a, b in zip(starts, lens)]).cuda()
                got = ops.prefill_varlen_attn(q[rows], kc, vc, _cu(lens), _cu([a + b for a, b in zip(starts, lens)]), 40, n,
                                              scale, G, vdim=DV, block_tables=table.repeat(3, 1).contiguous(), sink=s,
                                              **win).float()
                assert float((got - ref[rows]).abs().max()) < 3e-2, layout
            finally:
                _C.load().b200_prefill_set_query_tiles(0)
        rows = [n - 1, 16, size - 1, size, 0, size + keep, n - 200]
        tables = table.repeat(len(rows) + 1, 1).contiguous()
        ctx_lens = torch.tensor([r + 1 for r in rows] + [0], dtype=torch.int32).cuda()
        for ctas in (0, 3):
            got = ops.paged_decode_attn(torch.cat([q[rows], q[:1]]), kc, vc, tables, ctx_lens, scale, G, vdim=DV, sink=s,
                                        num_ctas=ctas, **win).float()
            assert float((got[:-1] - ref[rows]).abs().max()) < 3e-2, ctas
            assert not bool(got[-1].any())                             # the padded row
        one = ops.paged_decode_attn(q[n - 1:], kc, vc, table, ctx_lens[:1], scale, G, vdim=DV, sink=s, **win).float()
        assert float((one - ref[n - 1:]).abs().max()) < 3e-2
    # the window matters on this input, and so do the kept tokens
    full = ops.attn_generic(q[-8:], kc, vc, ops.StepSpans(_cu([8]), _cu([n]), None, 8), scale, G, DV, block_tables=table)
    ref = ops.attn_generic(q[-8:], kc, vc, ops.StepSpans(_cu([8]), _cu([n]), None, 8), scale, G, DV, block_tables=table, **win)
    assert float((full.float() - ref.float()).abs().max()) > 0.05


def test_sink_joins_for_short_sequences_beside_a_long_one():
    """Keys split over CTAs: a sequence with fewer key tiles than there are splits leaves the first splits empty, and its
    sink still joins the denominator once."""
    from nanovllm import ops
    H, G, D, n, bs = 4, 1, 64, 3000, 64
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(n, h, D, generator=g).bfloat16().cuda() for h in (H, G, G))
    sink = torch.full((H,), 3.0).cuda()
    nb = -(-n // bs)
    pad = nb * bs - n
    kc = torch.nn.functional.pad(k.view(n, -1), (0, 0, 0, pad)).view(nb, bs, -1).contiguous()
    vc = torch.nn.functional.pad(v.view(n, -1), (0, 0, 0, pad)).view(nb, bs, -1).contiguous()
    table = torch.arange(nb, dtype=torch.int32).cuda()[None, :].repeat(2, 1).contiguous()
    rows = torch.cat([torch.arange(n - 20, n), torch.arange(0, 12)]).cuda()
    spans = ops.StepSpans(_cu([20, 12]), _cu([n, 12]), None, 20)
    want = ops.attn_generic(q[rows], kc, vc, spans, 0.2, G, D, block_tables=table, sink=sink).float()
    got = ops.prefill_varlen_attn(q[rows], kc, vc, _cu([20, 12]), _cu([n, 12]), 20, n, 0.2, G, block_tables=table,
                                  sink=sink).float()
    assert float((got - want).abs().max()) < 2e-2


# ---- what surrounds the branches
@pytest.mark.parametrize("n,groups,offset", [(48, 1, 8), (60, 5, 3), (256, 4, 16), (96, 3, 0)])
def test_gates_write_scaled_slices_of_a_wider_row(n, groups, offset):
    """The element-wise sigmoid gate and the per-head norm with its silu gate, times a branch's scale, written into a
    slice of a wider row (what lies beside it is left alone)."""
    from nanovllm import ops
    g = torch.Generator().manual_seed(n)
    rows, eps = 7, 1e-4
    y, gate = (torch.randn(rows, n, generator=g, dtype=F64) for _ in range(2))
    w = 1 + 0.3 * torch.randn(n, generator=g, dtype=F64)
    for dtype in (torch.float32, torch.bfloat16):
        gt = gate.to(dtype)
        wide = torch.full((rows, n + offset + 8), 7.0, dtype=dtype, device="cuda")
        out = wide[:, offset:offset + n]
        ops.gated_norm(_dev(y, dtype), gt.cuda(), None, eps, out=out, scale=1.3)
        want = 1.3 * y.to(dtype).to(F64) * torch.sigmoid(gt.to(F64))
        assert float((out.cpu().to(F64) - want).abs().max()) < (1e-5 if dtype == torch.float32 else 3e-2)
        ops.gated_norm(_dev(y), gt.cuda(), _dev(w), eps, groups=groups, gate_act="silu", out=out, scale=0.4)
        normed = O.rms_norm(y.reshape(rows, groups, n // groups), 1.0, eps).reshape(rows, n) * w
        want = 0.4 * normed * O.silu(gt.to(F64))
        assert float((out.cpu().to(F64) - want).abs().max()) < (1e-5 if dtype == torch.float32 else 3e-2)
        assert bool((wide[:, :offset] == 7).all()) and bool((wide[:, offset + n:] == 7).all())


def test_two_branches_in_one_product():
    """The sum of two output projections as one product over the branches' rows side by side, padded and not."""
    from nanovllm.layers.linear import ConcatInputLinear
    g = torch.Generator().manual_seed(1)
    for sizes in ((20, 12), (16, 24)):
        m = ConcatInputLinear(sizes, 18).cuda()
        ws = [torch.randn(18, s, generator=g) for s in sizes]
        for i, wi in enumerate(ws):
            m.weight.weight_loader(m.weight, wi, i)
        xs = [torch.randn(5, s, generator=g) for s in sizes]
        x = m.empty_input(5, m.weight)
        for i, xi in enumerate(xs):
            m.part(x, i).copy_(xi)
        want = sum(xi.to(F64) @ wi.to(F64).T for xi, wi in zip(xs, ws))
        assert float((m(x).cpu().to(F64) - want).abs().max()) < 1e-4


# ---- the delta rule with one decay per head
def test_delta_inputs_with_one_decay_per_head():
    from nanovllm import ops
    g = torch.Generator().manual_seed(2)
    T, H, G, d = 11, 40, 4, 20                                          # more heads than a warp has lanes
    qk, a, b = (torch.randn(T, s, generator=g, dtype=F64) * 2 for s in (2 * G * d, H, H))
    dt_bias, a_log = torch.randn(H, generator=g, dtype=F64), torch.rand(H, generator=g, dtype=F64) * 3 - 4
    a[0, 0], a[0, 1] = 60.0, -60.0                                      # both ends of softplus
    qk32, dec, beta = ops.delta_prep(_dev(qk), _dev(a), _dev(b), _dev(dt_bias), _dev(a_log), H, G, d, O.UNIT_EPS, d ** -0.5,
                                     per_head=True)
    want = O.unit(qk.reshape(T, 2 * G, d))
    want[:, :G] *= d ** -0.5
    assert float((qk32.cpu().to(F64).reshape(T, 2 * G, d) - want).abs().max()) < 1e-6
    assert dec.shape == (T, H)
    assert float((dec.cpu().to(F64) - torch.exp(-torch.exp(a_log) * O.softplus(a + dt_bias))).abs().max()) < 1e-6
    assert float((beta.cpu().to(F64) - torch.sigmoid(b)).abs().max()) < 1e-6
    zero = ops.delta_prep(torch.zeros(1, 2 * d).cuda(), *(torch.zeros(1, 1).cuda() for _ in range(2)),
                          torch.zeros(1).cuda(), torch.zeros(1).cuda(), 1, 1, d, O.UNIT_EPS, 1.0, per_head=True)[0]
    assert not bool(zero.any())                                         # a zero vector stays zero, not NaN


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 12), (1, 1, 32, 32), (5, 5, 6, 9), (4, 1, 64, 64), (2, 2, 128, 64),
                                      (3, 1, 200, 40), (2, 1, 72, 130)])
@pytest.mark.parametrize("vdtype", [torch.float32, torch.bfloat16])
def test_delta_rule_with_one_decay_per_head(H, G, d, dv, vdtype):
    """Two sequences in portions of several sizes (single tokens as decode rows beside a padded row) whose slots hold
    leftovers, against the restatement token by token."""
    from nanovllm import ops
    g = torch.Generator().manual_seed(d + dv)
    n = [31, 18]
    seqs, want = [], []
    for m in n:
        q, k = (O.unit(torch.randn(m, G, d, generator=g, dtype=F64)) for _ in range(2))
        v = torch.randn(m, H, dv, generator=g, dtype=F64).to(vdtype).to(F64)
        dec, beta = (torch.rand(m, H, generator=g, dtype=F64) for _ in range(2))
        seqs.append([q.reshape(m, -1), k.reshape(m, -1), v.reshape(m, -1), 0.5 + dec / 2, beta])
        want.append(O.delta_rule(q, k, v, 0.5 + dec / 2, beta, torch.zeros(H, d, dv, dtype=F64))[0].reshape(m, -1))
    state = torch.full((3, H, d, dv), 9.0, device="cuda")
    at, got = [0, 0], [[], []]
    for step in ((13, 5), (2, 1), (1, 1), (1, 1), (7, 10), (7, 0)):
        live = [s for s in (0, 1) if step[s]]
        pick = lambda c, dt=torch.float32: torch.cat([seqs[s][c][at[s]:at[s] + step[s]] for s in live]).to(dt).cuda()
        ql, kl = [step[s] for s in live], [at[s] + step[s] for s in live]
        ins = [pick(0), pick(1), pick(2, vdtype), pick(3), pick(4)]
        if ql == [1, 1]:                                                # decode rows, the second one padded
            ins = [torch.cat([x[:1], x[:1], x[1:]]).contiguous() for x in ins]
            out = ops.delta_rule(*ins, _decode_spans([kl[0], 0, kl[1]]), H, G, d, dv, state, _slots(2, 1, 0))[[0, 2]]
        else:
            out = ops.delta_rule(*ins, _spans(ql, kl), H, G, d, dv, state, _slots(*[(2, 0)[s] for s in live]))
        for s, o in zip(live, out.split(ql)):
            got[s].append(o)
            at[s] += step[s]
    for s in (0, 1):
        assert at[s] == n[s]
        assert float((torch.cat(got[s]).cpu().to(F64) - want[s]).abs().max()) < 2e-5
    assert bool((state[1] == 9.0).all())                                # the padded row's slot was left alone


# ---- wkv
@pytest.mark.parametrize("H,d", [(3, 20), (5, 9), (4, 32), (4, 64), (2, 128), (1, 200), (3, 72)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_wkv_in_portions(H, d, dtype):
    """Inputs (fp32 receptance and key, double-exponential decay, the current token's coefficient) and recurrence: two
    sequences in portions of several sizes and as decode rows, slots that hold leftovers."""
    from nanovllm import ops
    g = torch.Generator().manual_seed(d)
    n, nd = [29, 17], H * d
    w0 = torch.rand(nd, generator=g, dtype=F64) * 4 - 4
    u = torch.randn(nd, generator=g, dtype=F64)
    seqs, want = [], []
    for m in n:
        r, k, v = (torch.randn(m, nd, generator=g, dtype=F64).to(dtype).to(F64) for _ in range(3))
        z = torch.randn(m, nd, generator=g, dtype=F64)
        dec = torch.exp(-torch.exp(z + w0))
        sh = lambda x: x.reshape(m, H, d)
        seqs.append([r, k, v, z])
        want.append(O.wkv_recurrence(sh(r), sh(k), sh(v), sh(dec), u.reshape(H, d), torch.zeros(H, d, d, dtype=F64))[0]
                    .reshape(m, nd))
    r32, k32, dec, bonus = ops.wkv_prep(_dev(seqs[0][0], dtype), _dev(seqs[0][1], dtype), _dev(seqs[0][3]), _dev(w0), _dev(u),
                                        H, d)
    assert float((dec.cpu().to(F64) - torch.exp(-torch.exp(seqs[0][3] + w0))).abs().max()) < 1e-6
    assert float((bonus.cpu().to(F64) - (seqs[0][0] * u * seqs[0][1]).reshape(-1, H, d).sum(-1)).abs().max()) < 1e-4
    assert torch.equal(r32.cpu().to(F64), seqs[0][0]) and torch.equal(k32.cpu().to(F64), seqs[0][1])
    state = torch.full((3, H, d, d), -5.0, device="cuda")
    at, got = [0, 0], [[], []]
    for step in ((12, 4), (2, 1), (1, 1), (1, 1), (6, 10), (7, 0)):
        live = [s for s in (0, 1) if step[s]]
        pick = lambda c, dt: torch.cat([seqs[s][c][at[s]:at[s] + step[s]] for s in live]).to(dt).cuda()
        ql, kl = [step[s] for s in live], [at[s] + step[s] for s in live]
        r32, k32, dec, bonus = ops.wkv_prep(pick(0, dtype), pick(1, dtype), pick(3, torch.float32), _dev(w0), _dev(u), H, d)
        ins = [r32, k32, pick(2, dtype), dec, bonus]
        if ql == [1, 1]:
            ins = [torch.cat([x[:1], x[:1], x[1:]]).contiguous() for x in ins]
            out = ops.wkv(*ins, _decode_spans([kl[0], 0, kl[1]]), H, d, d, state, _slots(2, 1, 0))[[0, 2]]
        else:
            out = ops.wkv(*ins, _spans(ql, kl), H, d, d, state, _slots(*[(2, 0)[s] for s in live]))
        for s, o in zip(live, out.split(ql)):
            got[s].append(o)
            at[s] += step[s]
    for s in (0, 1):
        err = (torch.cat(got[s]).cpu().to(F64) - want[s]).abs().max() / want[s].abs().max()
        assert at[s] == n[s] and float(err) < 5e-6
    assert bool((state[1] == -5.0).all())


def test_wkv_reads_before_it_writes():
    """Without a bonus the first token returns zero and the second reads the first token's value; with a decay of one a
    value comes back hundreds of tokens later, and the bonus counts at its own token only."""
    from nanovllm import ops
    d, n = 8, 400
    r = torch.zeros(n, d)
    k = torch.zeros(n, d)
    r[:, 0], k[0, 0] = 1.0, 1.0                                         # only the first token writes
    v = torch.randn(n, d, generator=torch.Generator().manual_seed(0))
    one, zero = torch.ones(n, d).cuda(), torch.zeros(n, 1).cuda()
    out = ops.wkv(r.cuda(), k.cuda(), v.cuda(), one, zero, _spans([n], [n]), 1, d, d).cpu()
    assert not bool(out[0].any()) and float((out[1:] - v[0]).abs().max()) < 1e-6
    bonus = torch.zeros(n, 1)
    bonus[5] = 2.0
    out2 = ops.wkv(r.cuda(), k.cuda(), v.cuda(), one, bonus.cuda(), _spans([n], [n]), 1, d, d).cpu()
    assert float((out2[5] - out[5] - 2.0 * v[5]).abs().max()) < 1e-5 and torch.equal(out2[6:], out[6:])


@pytest.mark.parametrize("W,M", [(50, 5), (96, 5), (256, 3), (37, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_shift_over_portions(W, M, dtype):
    """Mixes with the token before, in portions of 1 to 20 tokens of two sequences: the first token of a sequence sees
    zeros whatever its slot holds, a later portion sees the row that the step before left."""
    from nanovllm import ops
    g = torch.Generator().manual_seed(W)
    mu = torch.rand(M, W, generator=g, dtype=F64)
    n = [30, 26]
    h = [torch.randn(m, W, generator=g, dtype=F64).to(dtype).to(F64) for m in n]
    want = [torch.stack([O.token_shift(x, mu[i]) for i in range(M)]) for x in h]
    state = torch.full((3, W), 8.0, dtype=dtype, device="cuda")
    at, got = [0, 0], [[], []]
    tol = 1e-6 if dtype == torch.float32 else 2e-2
    for step in ((1, 3), (2, 1), (1, 1), (1, 1), (20, 9), (5, 11)):
        x = torch.cat([h[s][at[s]:at[s] + step[s]] for s in (0, 1)])
        kl = [at[s] + step[s] for s in (0, 1)]
        if step == (1, 1):
            x = torch.cat([x[:1], x[:1], x[1:]])
            out = ops.token_shift(_dev(x, dtype), _dev(mu), _decode_spans([kl[0], 0, kl[1]]), state, _slots(0, 1, 2))[:, [0, 2]]
        else:
            out = ops.token_shift(_dev(x, dtype), _dev(mu), _spans(list(step), kl), state, _slots(0, 2))
        for s, o in enumerate(out.split(list(step), 1)):
            got[s].append(o)
            at[s] += step[s]
        for s, slot in ((0, 0), (1, 2)):
            assert torch.equal(state[slot].cpu().to(F64), h[s][at[s] - 1])
    for s in (0, 1):
        assert at[s] == n[s]
        assert float((torch.cat(got[s], 1).cpu().to(F64) - want[s]).abs().max()) < tol
    assert bool((state[1] == 8.0).all())


def test_decay_projection_keeps_fp32():
    """The low-rank decay path of a 16-bit model leaves its second product in fp32."""
    from nanovllm import ops
    from nanovllm.layers.linear import F32OutLinear
    g = torch.Generator().manual_seed(6)
    m = F32OutLinear(24, 40).to(torch.bfloat16).cuda()
    m.weight.data.copy_(torch.randn(40, 24, generator=g))
    x = torch.randn(9, 24, generator=g).bfloat16().cuda() * 3
    t = ops.act_only(x, "tanh")
    assert float((t.float() - torch.tanh(x.float())).abs().max()) < 5e-3
    y = m(t)
    assert y.dtype == torch.float32
    want = t.cpu().to(F64) @ m.weight.data.cpu().to(F64).T
    assert float((y.cpu().to(F64) - want).abs().max()) < 1e-5
