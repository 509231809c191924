"""-m gpu: the Ragilorn decoder (attention inside chunks of the sequence behind short convolutions, latent attention, both with
rotary positions stretched band by band; branches gated element by element; every layer hands on a weighted sum of the
embedding and all layers so far; silu-gated feed-forwards, dense or a mixture whose sigmoid scores multiply what the experts
read; capped logits) against tests/ragilorn_oracle.py, a plain float64 restatement.

Every test makes its own small configuration and random weights. Models run in true fp32 (the sharp comparison:
relative error of every row of logits below 2e-4) and in bf16 (the serving precision). The schedules are fed through
LLMEngine.step_given -- the scheduler's block manager, the runner's step and the model's kernels -- so what is
compared is the engine, not a forward function. Where random weights would hide a fault (a key far back, a chunk's or
block's border, the first tokens) the mechanism tests scale one query and key so that one score stands out.
"""
import json
import os
import random

import pytest
import torch

import ragilorn_oracle as O

pytestmark = pytest.mark.gpu
F64 = torch.float64


def rot(dims, base=10000.0, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def attention(heads, kv, dim, vdim, rt, chunk=24, conv=3, scale=0.2, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": rt, "scale": scale}
    if conv:
        m["conv"] = conv
    if chunk:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def latent(heads, dim, rot_dim, vdim, rank, rt=None, scale=0.2, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
                      "rot": rt or rot(rot_dim, 2000.0, (3.0, 40, 5.0, 1.0))}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(vocab, width, layers, eps=1e-5, embed=2.5, scale=0.7, cap=6.0):
    return {"architecture": "Ragilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "logit_scale": scale, "logit_softcap": cap, "layers": layers}


def config_a():
    """Odd sizes everywhere: 6 query heads over 2 key/value heads with key size 24 and value size 20, 16 rotated columns
    stretched by 8 over a short original length, five taps, chunks of 20; a latent of 40 with 8 rotated columns; 7 experts
    of which 3; layers without feed-forward of both kinds; a latent layer first."""
    r = rot(16, 5000.0, (8.0, 48, 6.0, 1.5))
    return model(211, 96, [latent(3, 24, 8, 20, 40, mlp=moe(7, 3, 40)),
                           attention(6, 2, 24, 20, r, chunk=20, conv=5, mlp=dense(72)),
                           attention(6, 2, 24, 20, r, chunk=33, conv=2),
                           latent(5, 12, 16, 28, 24),
                           attention(4, 4, 12, 36, rot(8, 300.0), chunk=20, conv=4, mlp=moe(5, 2, 24))])


def config_b():
    """Values that are 1 or equal: one key/value head, one tap, every column rotated, no stretch, unit multipliers, one
    layer without chunks, no cap on the logits, every expert chosen (no discrete choice: the strict bf16 comparison),
    key size = value size = latent size."""
    r = rot(32, 10000.0)
    return model(320, 128, [attention(4, 1, 32, 32, r, chunk=16, conv=1, scale=0.18, mlp=dense(128)),
                            latent(4, 32, 32, 32, 32, r, scale=0.12, mlp=moe(2, 2, 64)),
                            attention(4, 1, 32, 32, r, chunk=0, conv=0, scale=0.18, mlp=dense(64))],
                 embed=1.0, scale=1.0, cap=0.0)


def config_c():
    """The sizes that 16-bit models run on the tensor cores: six heads of 64 over two key/value heads with values of 128 in
    chunks of 40; a latent of 72 with 48 + 16 key columns and values of 64; experts of 128 behind a router of 8."""
    r = rot(48, 5e5, (2.5, 300, 16.0, 2.0))
    return model(410, 384, [attention(6, 2, 64, 128, r, chunk=40, scale=0.11, mlp=dense(192)),
                            latent(4, 48, 16, 64, 72, scale=0.12, mlp=moe(8, 2, 128)),
                            attention(6, 2, 64, 64, r, chunk=25, scale=0.11, mlp=moe(4, 1, 64))])


def config_d():
    """Nothing is a multiple of 8: width 100, five heads of 10 (6 rotated) with values of 6 in chunks of 7, a latent of 30
    with 2 rotated columns, 50- and 18-wide feed-forwards, three experts of which one is chosen."""
    r = rot(6, 777.0, (3.0, 20, 4.0, 0.5))
    return model(97, 100, [attention(5, 5, 10, 6, r, chunk=7, conv=3, scale=0.4, mlp=dense(50)),
                           latent(3, 10, 2, 14, 30, rot(2, 50.0), scale=0.3, mlp=moe(3, 1, 18))], eps=1e-4, cap=3.0)


CONFIGS = {"a": config_a, "b": config_b, "c": config_c, "d": config_d}
STRICT_BF16 = {"a": False, "b": True, "c": False, "d": False}
_MODELS = {}


def model_dir(tmp_path_factory, name):
    """(folder with config.json + model.safetensors, config, tensors) of a named test model, made once."""
    if name not in _MODELS:
        from safetensors.torch import save_file
        cfg = CONFIGS[name]()
        tensors = O.random_weights(cfg, seed=len(name) + ord(name[0]))
        d = tmp_path_factory.mktemp("ragilorn_" + name)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
        save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(d, "model.safetensors"))
        _MODELS[name] = (str(d), cfg, tensors)
    return _MODELS[name]


_ENGINES = {}


def engine(tmp_path_factory, name, dtype, eager=False, blocks=24, block_size=16):
    key = (name, dtype, eager, blocks, block_size)
    if key not in _ENGINES:
        from nanovllm.engine.llm_engine import LLMEngine
        path, cfg, tensors = model_dir(tmp_path_factory, name)
        _ENGINES[key] = LLMEngine(path, dtype=dtype, kvcache_block_size=block_size, num_kvcache_blocks=blocks + 1,
                                  max_num_seqs=4, max_model_len=blocks * block_size,
                                  max_num_batched_tokens=4 * blocks * block_size, return_logits=True,
                                  enforce_eager=eager, chunked_prefill=True)
    return _ENGINES[key], _MODELS[name][1], _MODELS[name][2]


_LOGITS = {}


def oracle_logits(name, cfg, tensors, toks):
    """The oracle's logits of a whole sequence, computed once per (model, tokens)."""
    key = (name, tuple(toks))
    if key not in _LOGITS:
        _LOGITS[key] = O.forward(cfg, tensors, toks)
    return _LOGITS[key]


def row_err(got, want):
    """Per row: root mean square of the difference (row means removed) over that of the reference."""
    d = got.to(F64).cpu() - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()


def close(got, want, dtype, strict=True):
    e = row_err(got, want)
    if dtype == "float32":
        return bool((e < 2e-4).all())
    if strict:
        return float(e.pow(2).mean().sqrt()) < 3e-2 and float(e.max()) < 0.2
    # a model that chooses experts: bf16 rounding may flip a close choice for a token, so a few rows may differ
    return float(e.median()) < 3e-2 and float((e < 0.2).double().mean()) >= 0.9


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


CASES = [(n, d) for n in "abcd" for d in ("float32", "bfloat16")]


# ------------------------------------------------------------------ whole prompts, decoding, portions
@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_prompt_and_layers(tmp_path_factory, name, dtype):
    eng, cfg, tensors = engine(tmp_path_factory, name, dtype)
    toks = tokens_of(cfg, 75, 1)
    layers = []
    want = O.forward(cfg, tensors, toks, layers)
    mdl = eng.model_runner.model
    mdl.trace_layers = []
    try:
        got = feed(eng, "w", toks, [])
        seen = [x.cpu() for x in mdl.trace_layers]
    finally:
        mdl.trace_layers = None
    assert len(seen) == len(cfg["layers"])
    if dtype == "float32":
        for i, x in enumerate(seen):                  # what every layer hands on, after the average over the depth
            assert float((x.to(F64) - layers[i]).abs().max() / layers[i].abs().max()) < 2e-4, i
    assert close(got, want, dtype, STRICT_BF16[name])


@pytest.mark.parametrize("name,dtype", CASES)
@pytest.mark.parametrize("eager", [False, True])
def test_prefill_then_token_by_token(tmp_path_factory, name, dtype, eager):
    """Most of a prompt in one step, the rest one token a step (CUDA-graph decode and eager decode): decoded positions
    cross block and chunk borders, the convolution tails are carried token by token; a one-token prompt starts from the
    first token."""
    eng, cfg, tensors = engine(tmp_path_factory, name, dtype, eager)
    toks = tokens_of(cfg, 70, 2)
    want = oracle_logits(name, cfg, tensors, toks)
    for first in (1, 2, 29):
        got = feed(eng, "d", toks, range(first, len(toks)))
        assert close(got, want, dtype, STRICT_BF16[name]), first


@pytest.mark.parametrize("name,dtype", CASES)
def test_portions_of_every_size(tmp_path_factory, name, dtype):
    """Portions down to two tokens, cut in the middle of blocks and chunks; portions of 64 and more over a cached past (the
    up-projected prompt path of latent layers)."""
    eng, cfg, tensors = engine(tmp_path_factory, name, dtype)
    toks = tokens_of(cfg, 150, 3)
    want = oracle_logits(name, cfg, tensors, toks)
    for size in (2, 3, 7, 16, 19, 33, 70):
        got = feed(eng, "p", toks, range(size, len(toks), size))
        assert close(got, want, dtype, STRICT_BF16[name]), size
    g = random.Random(5)
    cuts, at = [], 0
    while at < len(toks):
        at += g.choice([1, 1, 2, 2, 3, 5, 16, 21])
        cuts.append(at)
    got = feed(eng, "p", toks, [c for c in cuts if c < len(toks)])
    assert close(got, want, dtype, STRICT_BF16[name])


@pytest.mark.parametrize("name,dtype", CASES)
def test_unequal_batches_and_reused_slots(tmp_path_factory, name, dtype):
    """Up to four live requests, portions of some beside single tokens of others, requests that sit out a step;
    every request ends at its own time and later ones take over its blocks and state slot (the pool has 12 blocks,
    the seven requests need 23); each must match its own run alone."""
    pool = 12
    eng, cfg, tensors = engine(tmp_path_factory, name, dtype, blocks=pool)
    g = random.Random(7)
    lens = [37, 90, 5, 64, 51, 33, 18]
    reqs = {f"r{i}": tokens_of(cfg, n, 10 + i) for i, n in enumerate(lens)}
    want = {k: oracle_logits(name, cfg, tensors, v) for k, v in reqs.items()}
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
        for k, t, w in entries:
            got[k].append(out[row:row + len(w)])
            row += len(w)
            if k in eng.scheduler.given:
                slots[k] = eng.scheduler.given[k].state_slot
                tables[k] = list(eng.scheduler.given[k].block_table)
        live = [k for k in live if k not in end]
    stateful = bool(eng.model_runner.state_modules)                              # config b carries nothing but its caches
    assert stateful == (name != "b") and (not stateful or len(set(slots.values())) <= 4 < len(slots))    # slots were used again
    assert sum(len(t) for t in tables.values()) > pool                           # and so were blocks
    assert len(bm.free_block_ids) == pool and len(bm.free_state_slots) == (4 if stateful else 0)         # all was given back
    for k in reqs:
        assert close(torch.cat(got[k]), want[k], dtype, STRICT_BF16[name]), \
            (k, float(row_err(torch.cat(got[k]), want[k]).max()))


def test_long_decoding(tmp_path_factory):
    """300 tokens one by one after a 3-token prompt in fp32: tails are carried 300 times, latent layers read 19 blocks
    through the table, chunks begin 15 times, the rotation reaches positions far past the original length."""
    eng, cfg, tensors = engine(tmp_path_factory, "a", "float32", blocks=20)
    toks = tokens_of(cfg, 303, 4)
    want = O.forward(cfg, tensors, toks)
    got = feed(eng, "l", toks, range(3, len(toks)))
    assert float(row_err(got, want).max()) < 2e-4


def test_greedy_generation_through_the_scheduler(tmp_path_factory):
    """LLM.generate (waiting/running queues, prefill steps, graph decode steps, sampling from fp32 logits) against the
    oracle's greedy continuation, for three prompts of unequal length at once."""
    from nanovllm import LLM, SamplingParams
    path, cfg, tensors = model_dir(tmp_path_factory, "a")
    llm = LLM(path, dtype="float32", kvcache_block_size=16, num_kvcache_blocks=40, max_num_seqs=4, max_model_len=128,
              max_num_batched_tokens=512)
    prompts = [tokens_of(cfg, n, 20 + n) for n in (9, 30, 17)]
    outs = llm.generate(prompts, SamplingParams(temperature=1.0, max_tokens=10, ignore_eos=True, greedy=True),
                        use_tqdm=False)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for tok in o["token_ids"]:
            logits = O.forward(cfg, tensors, seq)[-1]
            top = torch.topk(logits, 2).values
            if float(top[0] - top[1]) > 1e-4:
                assert tok == int(logits.argmax()), (len(seq), tok)
            seq.append(tok)
    llm.exit()


# ------------------------------------------------------------------ mechanisms alone
def _dev(x, dtype=torch.float32):
    return x.to(dtype).cuda().contiguous()


def _cu(v):
    return torch.tensor([0] + list(torch.tensor(v).cumsum(0)), dtype=torch.int32).cuda()


@pytest.mark.parametrize("W,n", [(37, 1), (96, 3), (64, 9), (512, 4), (4096, 6), (8192, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_branch_and_depth_average(W, n, dtype):
    """v = x + y sigmoid(gate), kept as an entry of the history; the weighted sum of n earlier entries and v; the norm of
    that -- for widths that take the 16-byte form and widths that do not; without average, without gate, and the scaled
    embedding by lookup."""
    from nanovllm import ops
    g = torch.Generator().manual_seed(W + n)
    rows, eps = 5, 1e-5
    rd = lambda x: x.to(dtype).to(F64)
    x = torch.randn(rows, W, generator=g, dtype=F64).float().to(F64)
    y = rd(torch.randn(rows, W, generator=g, dtype=F64) * 2)
    wide = rd(torch.randn(rows, W + 24, generator=g, dtype=F64) * 3)          # the gate's logits lie inside a wider row
    gate = wide[:, 16:16 + W]
    hist = torch.randn(n + 2, rows, W, generator=g, dtype=F64).float().to(F64)
    avg = torch.randn(n + 1, generator=g, dtype=F64).float().to(F64)
    w = (1 + 0.2 * torch.randn(W, generator=g, dtype=F64)).float().to(F64)
    v = x + y * O.sigmoid(gate)
    want_x = O.depth_average([hist[j] for j in range(n)] + [v], avg)
    hd, xd = _dev(hist), _dev(x)
    gd = wide.to(dtype).cuda()[:, 16:16 + W]
    h = ops.residual_gate_average(xd, _dev(y, dtype), gd, _dev(w), eps, dtype, x_out=xd, keep=hd[n], hist=hd, n=n, avg=_dev(avg))
    size = float(want_x.abs().max())
    assert h.dtype == dtype and xd.dtype == torch.float32
    assert float((xd.cpu().to(F64) - want_x).abs().max()) < 1e-5 * size
    assert float((hd[n].cpu().to(F64) - v).abs().max()) < 1e-5 * float(v.abs().max())
    assert torch.equal(hd[n + 1].cpu().to(F64), hist[n + 1]) and torch.equal(hd[:n].cpu().to(F64), hist[:n])
    tol = 1e-5 if dtype == torch.float32 else 4e-2
    assert float((h.cpu().to(F64) - O.rms_norm(want_x, w, eps)).abs().max()) < tol * 5
    # every weight and every entry matters on this input
    assert float((want_x - O.depth_average([hist[j] for j in range(n)] + [v], torch.cat([avg[:n], avg[n:] * 0]))).abs().max()) > 1e-2
    # in the middle of a layer: no average; the stream is written in place
    xd = _dev(x)
    h = ops.residual_gate_average(xd, _dev(y, dtype), gd, _dev(w), eps, dtype, x_out=xd)
    assert float((xd.cpu().to(F64) - v).abs().max()) < 1e-5 * float(v.abs().max())
    assert float((h.cpu().to(F64) - O.rms_norm(v, w, eps)).abs().max()) < tol * 5
    # the scaled embedding: a lookup, no earlier stream, no gate
    table = rd(torch.randn(20, W, generator=g, dtype=F64))
    idx = torch.tensor([3, 19, 0, 7, 7])
    out = torch.full((rows, W), float("nan"), device="cuda")
    h = ops.residual_gate_average(None, _dev(table, dtype), None, _dev(w), eps, dtype, c=1.7, y_index=idx.cuda(), keep=out)
    assert float((out.cpu().to(F64) - 1.7 * table[idx]).abs().max()) < 1e-5
    assert float((h.cpu().to(F64) - O.rms_norm(1.7 * table[idx], w, eps)).abs().max()) < tol * 5


@pytest.mark.parametrize("V", [7, 320, 4099])
def test_capped_logits(V):
    from nanovllm import ops
    z = torch.randn(3, V, generator=torch.Generator().manual_seed(V), dtype=F64) * 40
    for scale, cap in ((0.5, 7.0), (1.0, 30.0), (0.25, 0.0)):
        got = ops.logit_cap_(_dev(z), scale, cap).cpu().to(F64)
        assert float((got - O.cap_logits(z.float().to(F64), scale, cap)).abs().max()) < 2e-5, (scale, cap)


def test_sampling_from_fp32_logits():
    """Greedy choice on fp32 logits that 16 bits could not tell apart; ties go to the lower index; at a temperature the
    draws follow the softmax."""
    from nanovllm import ops
    z = torch.full((3, 1003), -5.0)
    z[0, 700], z[0, 300] = 11.0001, 11.0
    z[1, 5], z[1, 900] = 2.5, 2.5
    z[2, 1002] = 1.0
    assert ops.sample(z.cuda()).tolist() == [700, 5, 1002]
    assert ops.sample(torch.nn.functional.pad(z, (0, 1))[:, :1003].cuda()).tolist() == [700, 5, 1002]    # rows without 16-byte starts
    p = torch.tensor([0.5, 0.3, 0.2]).log().repeat(20000, 1).cuda()
    ids = ops.sample(p, torch.ones(20000, device="cuda"), seed=3)
    share = torch.bincount(ids.cpu(), minlength=3).double() / 20000
    assert float((share - torch.tensor([0.5, 0.3, 0.2], dtype=F64)).abs().max()) < 0.02


# ------------------------------------------------------------------ attention inside chunks
def _attn_case(n, H, G, d, dv, seed, dtype, star=None, gain=7.0):
    """Random q, k, v of one sequence; `star` = (query position, key position, head): that query's head and that key
    are made parallel and long, so that the key stands out wherever it is visible."""
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


def _paged(rows, bs, order):
    """A cache [nb, bs, row] whose blocks are in `order`, and the block table [1, n]."""
    n = rows.shape[0]
    nb = -(-n // bs)
    c = torch.zeros(max(order) + 2, bs, rows[0].numel(), dtype=rows.dtype)
    for b in range(nb):
        part = rows[b * bs:(b + 1) * bs].reshape(-1, rows[0].numel())
        c[order[b], :part.shape[0]] = part
    return c, torch.tensor([order[:nb]], dtype=torch.int32)


def _chunked_module(H, G, d, dv, scale, chunk, dtype, kc=None, vc=None):
    from nanovllm.layers.seq_mixers import VarSizeAttention
    m = VarSizeAttention(H, G, d, dv, scale, chunk=chunk).cuda()
    if kc is not None:
        m.k_cache, m.v_cache = kc.to(dtype).cuda(), vc.to(dtype).cuda()
    return m


def _in_context(fn, q_lens=None, k_lens=None, ctx_lens=None, table=None, bs=16):
    """fn() under a step context made by hand: packed spans, or decode rows."""
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
        with torch.no_grad():
            return fn().cpu().to(F64)
    finally:
        reset_context()


# sizes that run on the generic kernel, and (bf16) on the tcgen05 prompt kernel and the paged decode kernel
SHAPES = [(6, 2, 24, 20), (5, 5, 48, 32), (4, 2, 64, 64), (8, 1, 128, 128), (3, 1, 64, 128), (4, 4, 128, 64)]


@pytest.mark.parametrize("H,G,d,dv", SHAPES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunk", [1, 7, 16, 50, 200])
def test_attention_inside_chunks(H, G, d, dv, dtype, chunk):
    """Chunks of one token, smaller and larger than a block, larger than the sequence: a whole prompt from this step's
    rows, the same prompt as portions over a shuffled block table beside a second sequence, and decode rows at the last
    token of a chunk, the first of the next, and a padded row."""
    n, bs, scale = 131, 16, 0.35
    q, k, v = _attn_case(n, H, G, d, dv, 3, dtype)
    want = O.attention(q, k, v, scale, chunk)
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    dev = lambda x: _dev(x, dtype)
    m = _chunked_module(H, G, d, dv, scale, chunk, dtype)
    got = _in_context(lambda: m(dev(q), dev(k), dev(v)), [n], [n])
    assert float((got.view(n, H, dv) - want).abs().max()) < tol
    if chunk < n:
        assert float((O.attention(q, k, v, scale, 0) - want).abs().max()) > 0.2          # the chunks matter on this input
    order = [5, 0, 3, 1, 8, 4, 2, 7, 6]
    kc, table = _paged(k, bs, order)
    vc, _ = _paged(v, bs, order)
    m = _chunked_module(H, G, d, dv, scale, chunk, dtype, kc, vc)
    table2 = torch.cat([table, table], 0).cuda()
    at = 0
    for ql in (21, 2, 60, 48):                                          # portions start inside blocks and chunks
        qq = torch.cat([q[at:at + ql], q[:5]])
        got = _in_context(lambda: m(dev(qq), dev(qq[:, :G]), dev(v[:ql + 5])), [ql, 5], [at + ql, 5], table=table2)
        assert float((got[:ql].view(ql, H, dv) - want[at:at + ql]).abs().max()) < tol, at
        assert float((got[ql:].view(5, H, dv) - want[:5]).abs().max()) < tol
        at += ql
    last = (n - 1) // chunk * chunk
    for pos in sorted({0, 1, chunk - 1, chunk, chunk + 1, last - 1, last, 15, 16, n - 1} & set(range(n))):
        rows = [pos, 0, 31]
        got = _in_context(lambda: m(dev(q[rows]), dev(k[rows]), dev(v[rows])), ctx_lens=[pos + 1, 0, 32],
                          table=table.repeat(3, 1).contiguous().cuda())
        assert float((got[0].view(H, dv) - want[pos]).abs().max()) < tol, pos
        assert float((got[2].view(H, dv) - want[31]).abs().max()) < tol


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 20), (4, 2, 64, 64), (2, 1, 128, 64)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunk", [48, 150, 300])
def test_a_key_just_inside_and_just_outside_a_chunk(H, G, d, dv, dtype, chunk):
    """One key that would take the whole softmax of one query head, at the first place of the query's chunk (visible) and
    one place earlier (not visible): for the chunk's first, second and last token, in a prompt, in a portion that
    continues a cached past and for a decoded token."""
    bs, scale = 16, 1.0
    n = 2 * chunk + 5
    tol = 1e-4 if dtype == torch.float32 else 5e-2
    dev = lambda x: _dev(x, dtype)
    order = list(range(-(-n // bs) - 1, -1, -1))
    for i in (chunk, chunk + 1, 2 * chunk - 1, 2 * chunk):
        start = i // chunk * chunk
        for j in (start, start - 1):
            q, k, v = _attn_case(n, H, G, d, dv, 5 + j, dtype, star=(i, j, 1))
            want = O.attention(q[i:i + 1], k[:i + 1], v[:i + 1], scale, chunk, first_pos=i)[0]
            seen = float(want[1].min()) > 4.5                           # the far value (5.0) is what the head returns
            assert seen == (j == start), (i, j)
            m = _chunked_module(H, G, d, dv, scale, chunk, dtype)
            got = _in_context(lambda: m(dev(q), dev(k), dev(v)), [n], [n]).view(n, H, dv)
            assert float((got[i] - want).abs().max()) < tol, (i, j)
            kc, table = _paged(k, bs, order)
            vc, _ = _paged(v, bs, order)
            m = _chunked_module(H, G, d, dv, scale, chunk, dtype, kc, vc)
            lo = i - 9
            got = _in_context(lambda: m(dev(q[lo:i + 1]), dev(k[lo:i + 1]), dev(v[lo:i + 1])), [10], [i + 1], table=table.cuda())
            assert float((got[9].view(H, dv) - want).abs().max()) < tol, (i, j)
            got = _in_context(lambda: m(dev(q[i:i + 1]), dev(k[i:i + 1]), dev(v[i:i + 1])), ctx_lens=[i + 1], table=table.cuda())
            assert float((got[0].view(H, dv) - want).abs().max()) < tol, (i, j)


@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (8, 1, 128)])
def test_chunks_on_long_sequences(H, G, D):
    """The tcgen05 prompt kernel and the paged decode kernel with chunks of hundreds of tokens against the generic kernel:
    a long prompt (both CTA layouts), a short portion over thousands of cached keys (keys are split over CTAs), decode
    rows beside short ones."""
    from nanovllm import _C, ops
    g = torch.Generator().manual_seed(D + H)
    n, bs, scale, chunk = 3000, 64, D ** -0.5 * 2.0, 700
    q = torch.randn(n, H, D, generator=g).bfloat16().cuda()
    k = torch.randn(n, G, D, generator=g).bfloat16().cuda()
    v = torch.randn(n, G, D, generator=g).bfloat16().cuda()
    nb = -(-n // bs)
    order = torch.randperm(nb, generator=g).tolist()
    kc, table = _paged(k.cpu(), bs, order)
    vc, _ = _paged(v.cpu(), bs, order)
    kc, vc, table = kc.cuda(), vc.cuda(), table.cuda()
    cu = lambda *x: torch.tensor(x, dtype=torch.int32).cuda()
    ref = ops.attn_generic(q, k, v, ops.StepSpans(cu(0, n), cu(0, n), None, n), scale, G, D, chunk=chunk).float()
    for layout in (1, 2):
        _C.load().b200_prefill_set_query_tiles(layout)
        try:
            got = ops.prefill_varlen_attn(q, k, v, cu(0, n), cu(0, n), n, n, scale, G, chunk=chunk).float()
        finally:
            _C.load().b200_prefill_set_query_tiles(0)
        assert float((got - ref).abs().max()) < 3e-2, layout
    for ql in (300, 40):
        got = ops.prefill_varlen_attn(q[n - ql:], kc, vc, cu(0, ql), cu(0, n), ql, n, scale, G, block_tables=table,
                                      chunk=chunk).float()
        assert float((got - ref[n - ql:]).abs().max()) < 3e-2, ql
    rows = [n - 1, 16, 699, 700, 1399, 0]
    got = ops.paged_decode_attn(q[rows], kc, vc, table.repeat(len(rows), 1).contiguous(),
                                cu(*[r + 1 for r in rows]), scale, G, chunk=chunk).float()
    assert float((got - ref[rows]).abs().max()) < 3e-2


# ------------------------------------------------------------------ latent attention
def _latent_case(n, H, d, dr, dv, R, dtype, seed, star=None, gain=9.0):
    """(q [n, H, d + dr] with its rotated part already rotated, cached rows [n, R + dr], W_uk [H, d, R], W_uv [H, dv, R]).
    `star` = (query position, key position, head): the key's rotated part is made parallel to that query head's."""
    g = torch.Generator().manual_seed(seed)
    rd = lambda x: x.to(dtype).to(F64)
    q = torch.randn(n, H, d + dr, generator=g, dtype=F64)
    rows = torch.randn(n, R + dr, generator=g, dtype=F64)
    if star is not None:
        i, j, h = star
        q[i, h, d:] *= gain / q[i, h, d:].norm()
        rows[j, R:] = q[i, h, d:]
    wk = torch.randn(H, d, R, generator=g, dtype=F64) * R ** -0.5
    wv = torch.randn(H, dv, R, generator=g, dtype=F64) * R ** -0.5
    return rd(q), rd(rows), rd(wk), rd(wv)


def _latent_want(q, rows, wk, wv, scale, first_pos=0):
    Tq, H, _ = q.shape
    d, R = wk.shape[1:]
    out = torch.zeros(Tq, H, wv.shape[1], dtype=F64)
    for h in range(H):
        key = torch.cat([rows[:, :R] @ wk[h].T, rows[:, R:]], 1)
        s = (q[:, h] @ key.T) * scale
        hidden = torch.arange(rows.shape[0])[None, :] > first_pos + torch.arange(Tq)[:, None]
        out[:, h] = torch.softmax(s.masked_fill(hidden, float("-inf")), 1) @ (rows[:, :R] @ wv[h].T)
    return out


def _latent_module(H, d, dr, wk, wv, scale, dtype, cache=None):
    from nanovllm.layers.seq_mixers import LatentAttention
    torch.set_default_dtype(dtype)
    try:
        m = LatentAttention(H, d, dr, wv.shape[1], wk.shape[2], scale)
    finally:
        torch.set_default_dtype(torch.float32)
    m.w_uk.data.copy_(wk)
    m.w_uv.data.copy_(wv)
    m = m.cuda()
    if cache is not None:
        m.k_cache = cache.to(dtype).cuda()
    return m


def _run_latent(m, q, rows, d, dtype, **ctx):
    qd = _dev(q, dtype)
    return _in_context(lambda: m(qd[:, :, :d], lambda out: out.copy_(qd[:, :, d:]), _dev(rows, dtype)), **ctx)


# head sizes whose keys fill 64, 128 and 192 columns of the tcgen05 kernel or leave some of them, value sizes it does not
# take, sizes that no 16-bit kernel takes, more heads than a row tile holds
LATENT = [(4, 48, 16, 64, 72), (3, 40, 8, 64, 24), (2, 128, 64, 128, 512), (5, 12, 4, 20, 40), (3, 10, 2, 14, 30),
          (40, 32, 32, 64, 128), (8, 96, 32, 128, 264)]


@pytest.mark.parametrize("H,d,dr,dv,R", LATENT)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_attention_without_a_window(H, d, dr, dv, R, dtype):
    """Prompts from this step's rows (long: explicit keys and values; short: the latent kernel), portions of 2 to 90 tokens
    over a shuffled block table beside a second sequence, decode rows at block borders beside a padded row -- all against
    the restatement with explicit keys and values."""
    n, bs, scale = 171, 16, 1.5 * (d + dr) ** -0.5
    q, rows, wk, wv = _latent_case(n, H, d, dr, dv, R, dtype, 1)
    want = _latent_want(q, rows, wk, wv, scale)
    size = float(want.abs().max())
    tol = 2e-5 * size if dtype == torch.float32 else 2.5e-2 * size
    m = _latent_module(H, d, dr, wk, wv, scale, dtype)
    for ln in (n, 40, 1):
        got = _run_latent(m, q[:ln], rows[:ln], d, dtype, q_lens=[ln], k_lens=[ln])
        assert float((got.view(ln, H, dv) - want[:ln]).abs().max()) < tol, ln
    order = [5, 0, 3, 1, 8, 4, 2, 7, 6, 10, 9]
    cache, table = _paged(rows, bs, order)
    m = _latent_module(H, d, dr, wk, wv, scale, dtype, cache)
    table2 = torch.cat([table, table], 0).cuda()
    at = 0
    for ql in (30, 2, 90, 49):
        qq, rr = torch.cat([q[at:at + ql], q[:5]]), torch.cat([rows[at:at + ql], rows[:5]])
        got = _run_latent(m, qq, rr, d, dtype, q_lens=[ql, 5], k_lens=[at + ql, 5], table=table2)
        assert float((got[:ql].view(ql, H, dv) - want[at:at + ql]).abs().max()) < tol, at
        assert float((got[ql:].view(5, H, dv) - want[:5]).abs().max()) < tol
        at += ql
    for pos in (0, 15, 16, 63, 64, 130, n - 1):
        pick = [pos, 0, 31]
        got = _run_latent(m, q[pick], rows[pick], d, dtype, ctx_lens=[pos + 1, 0, 32],
                          table=table.repeat(3, 1).contiguous().cuda())
        assert float((got[0].view(H, dv) - want[pos]).abs().max()) < tol, pos
        assert float((got[2].view(H, dv) - want[31]).abs().max()) < tol


@pytest.mark.parametrize("H,d,dr,dv,R", [(4, 48, 16, 64, 72), (3, 10, 6, 14, 30), (2, 128, 64, 128, 512)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_far_latent_row_at_block_borders(H, d, dr, dv, R, dtype):
    """One cached row hundreds of tokens back, at a block's last and first place and at the very first, takes the whole
    softmax of one query head: in a prompt, in a portion over a cached past, for a decoded token."""
    n, bs, i, head = 500, 16, 499, 1
    order = list(range(31, -1, -1))
    for j in (0, 15, 16, 63, 64):
        q, rows, wk, wv = _latent_case(n, H, d, dr, dv, R, dtype, 7 + j, star=(i, j, head))
        want = _latent_want(q[i:], rows, wk, wv, 1.0, first_pos=i)[0]
        alone = rows[j, :R] @ wv[head].T
        assert float((want[head] - alone).abs().max()) < 0.05 * float(alone.abs().max())       # it is the far row's value
        tol = (1e-4 if dtype == torch.float32 else 3e-2) * float(want.abs().max())
        m = _latent_module(H, d, dr, wk, wv, 1.0, dtype)
        got = _run_latent(m, q, rows, d, dtype, q_lens=[n], k_lens=[n])
        assert float((got[i].view(H, dv) - want).abs().max()) < tol, j
        cache, table = _paged(rows, bs, order)
        m = _latent_module(H, d, dr, wk, wv, 1.0, dtype, cache)
        for ql in (3, 200):
            got = _run_latent(m, q[n - ql:], rows[n - ql:], d, dtype, q_lens=[ql], k_lens=[n], table=table.cuda())
            assert float((got[-1].view(H, dv) - want).abs().max()) < tol, (j, ql)
        got = _run_latent(m, q[i:], rows[i:], d, dtype, ctx_lens=[n], table=table.cuda())
        assert float((got[0].view(H, dv) - want).abs().max()) < tol, j


@pytest.mark.parametrize("H,D,R", [(4, 88, 72), (8, 576, 512), (40, 72, 64), (6, 288, 256), (17, 136, 128)])
@pytest.mark.parametrize("window", [0, 90])
def test_latent_kernel_splits_and_spans(H, D, R, window):
    """The 16-bit latent kernel alone against the generic kernel in fp32: packed rows, portions and decode rows of unequal
    sequences, any number of key splits (more than a short row has tiles), with and without a window."""
    from nanovllm import ops
    g = torch.Generator(device="cuda").manual_seed(D)
    kl, bs, scale = [300, 1, 77, 513], 64, D ** -0.5 * 1.5
    cache = torch.randn(40, bs, D, device="cuda", generator=g).bfloat16()
    table = torch.randperm(39, device="cuda", generator=g)[:36].view(4, 9).int().contiguous()
    for ql in ([300, 1, 77, 513], [33, 1, 77, 2], None):
        paged = ql != kl
        T = sum(ql) if ql else 4
        q = torch.randn(T, H, D, device="cuda", generator=g).bfloat16()
        spans = ops.StepSpans(_cu(ql), _cu(kl), None, max(ql)) if ql else \
            ops.StepSpans(None, None, torch.tensor(kl, dtype=torch.int32).cuda())
        rows = cache if paged else torch.randn(sum(kl), D, device="cuda", generator=g).bfloat16()
        ref = ops.attn_generic(q.float(), rows.float() if paged else rows.float().unsqueeze(1), None, spans, scale, 1, R,
                               block_tables=table if paged else None, window=window)
        for splits in (None, 1, 2, 5, 13):
            got = ops.latent_attn(q, rows, spans, scale, R, block_tables=table if paged else None, window=window, splits=splits)
            assert float((got.float() - ref).abs().max()) < 3e-2, (ql, splits)


def test_latent_rows_and_query_rotation_by_table():
    """The latent norm, the rotation of the shared key part and of the queries by a stretched table (magnitude included) at
    positions up to a million, and the cache rows (flat slots, pairs, a negative slot)."""
    from nanovllm import ops
    from nanovllm.layers.seq_mixers import BandScaledRotary
    R, dr, T, H, d, bs, eps = 20, 12, 6, 3, 8, 4, 1e-5
    r = rot(dr, 500.0, (4.0, 64, 8.0, 1.0))
    g = torch.Generator().manual_seed(5)
    both = torch.randn(T, R + dr + 7, generator=g, dtype=F64)[:, 7:]
    w = 1 + 0.2 * torch.randn(R, generator=g, dtype=F64)
    pos = torch.tensor([0, 1, 63, 64, 4097, 1000003])
    br = BandScaledRotary(dr, 500.0, True, r["scaling"])
    table = ops.rotary_table(pos.cuda(), br.freq.cuda(), br.magnitude)
    want = torch.cat([O.rms_norm(both[:, :R], w, eps), O.rotate(both[:, None, R:], pos, r)[:, 0]], 1)
    slots = torch.tensor([5, 2, -1, 11, 0, 7], dtype=torch.int32)
    for paired in (False, True):
        cache = torch.zeros(3, bs, R + dr, device="cuda")
        sl = torch.stack([slots // bs, slots % bs], 1).contiguous() if paired else slots.clone()
        if paired:
            sl[2] = torch.tensor([-1, 0])
        none, kc = ops.latent_kv_prep(None, both.float().cuda(), None, _dev(w), pos.cuda(), R, dr, dr, 1.0, True, eps,
                                      cache=cache, slots=sl.cuda(), table=table)
        assert none is None and float((kc.cpu().to(F64) - want).abs().max()) < 1e-5
        flat = cache.view(-1, R + dr)
        assert all(torch.equal(flat[int(s)], kc[t]) for t, s in enumerate(slots) if s >= 0)
        assert int((flat.abs().sum(1) > 0).sum()) == 5
    q = torch.randn(T, H, d + dr, generator=g, dtype=F64)
    out = torch.zeros(T, H, 30, device="cuda")
    ops.rotary_heads(q.float().cuda()[:, :, d:], pos.cuda(), H, dr, dr, 1.0, True, out=out[:, :, 18:], table=table)
    assert float((out[:, :, 18:].cpu().to(F64) - O.rotate(q[:, :, d:], pos, r)).abs().max()) < 1e-5
    assert float(out[:, :, :18].abs().max()) == 0.0


# ------------------------------------------------------------------ mixture of experts
@pytest.mark.parametrize("E,top", [(10, 3), (6, 6), (16, 1), (5, 2), (300, 9)])
def test_sigmoid_scores_as_they_are(E, top):
    from nanovllm import ops
    z = (torch.randn(50, E, generator=torch.Generator().manual_seed(E + top), dtype=F64) * 2).float().to(F64)
    ids, w = ops.moe_route_grouped(_dev(z), None, top, normalize=False)
    want_ids, want_w = O.route(z, top)
    assert torch.equal(ids.cpu().long().sort(1).values, want_ids.sort(1).values)
    full = lambda i, x: torch.zeros(50, E, dtype=F64).scatter_(1, i, x)
    assert float((full(ids.cpu().long(), w.cpu().to(F64)) - full(want_ids, want_w)).abs().max()) < 1e-6


@pytest.mark.parametrize("dtype,T,hidden,inter,E,top", [
    (torch.float32, 19, 40, 24, 4, 2), (torch.float32, 7, 128, 64, 8, 3), (torch.bfloat16, 33, 96, 40, 6, 3),
    (torch.bfloat16, 5, 128, 64, 8, 4), (torch.bfloat16, 1024, 128, 64, 4, 2), (torch.bfloat16, 600, 256, 128, 2, 2),
    (torch.bfloat16, 40, 128, 64, 12, 10)])
def test_experts_weighted_at_their_input(dtype, T, hidden, inter, E, top):
    """expert(w h) is not w expert(h): the mixture layer against the restatement -- fp32 and bf16, sizes only the generic
    kernels take, the weight-streaming kernels, prompt-sized batches on the grouped tcgen05 product, and more experts per
    token than the tensor-core kernels take."""
    from nanovllm.layers.moe import GroupedSigmoidMoe
    g = torch.Generator().manual_seed(T + hidden)
    w = {"router": torch.randn(E, hidden, generator=g) * 0.2}
    for e in range(E):
        w[f"e{e}.gate"] = torch.randn(inter, hidden, generator=g) * hidden ** -0.5 * 3
        w[f"e{e}.up"] = torch.randn(inter, hidden, generator=g) * hidden ** -0.5 * 3
        w[f"e{e}.down"] = torch.randn(hidden, inter, generator=g) * inter ** -0.5
    w = {k: v.to(dtype).to(F64) for k, v in w.items()}
    x = torch.randn(T, hidden, generator=g, dtype=F64).to(dtype).to(F64)
    torch.set_default_dtype(dtype)                                     # as the runner builds a model: the router stays fp32
    try:
        m = GroupedSigmoidMoe(hidden, inter, E, top, correction=False, normalize=False, weigh="input")
    finally:
        torch.set_default_dtype(torch.float32)
    assert m.router.dtype == torch.float32 and m.w13.dtype == dtype and m.correction is None
    m.router.data.copy_(w["router"])
    for e in range(E):
        m.w13.data[e, :inter].copy_(w[f"e{e}.gate"])
        m.w13.data[e, inter:].copy_(w[f"e{e}.up"])
        m.w2.data[e].copy_(w[f"e{e}.down"])
    m = m.cuda()
    with torch.no_grad():
        got = m(x.to(dtype).cuda()).cpu().to(F64)
    rows = slice(0, min(T, 64))
    want = O.moe_ff(x[rows], w, top)
    ids, sc = O.route(x[rows] @ w["router"].T, top)
    after = sum(sc[:, j:j + 1] * torch.stack([O.gated_ff(x[t:t + 1], w, f"e{int(ids[t, j])}.")[0] for t in range(want.shape[0])])
                for j in range(top))
    assert float((after - want).abs().max()) > 0.1 * float(want.abs().max())         # weighting the output is another result
    if dtype == torch.float32:
        assert float((got[rows] - want).abs().max()) < 1e-4
    else:
        err = (got[rows] - want).abs().max(1).values / want.abs().max()
        assert float(err.median()) < 2e-2 and float((err < 5e-2).double().mean()) > 0.9       # a close choice may flip
    if T > 64:                                                         # the tensor-core form against the generic one
        m.fast = False
        with torch.no_grad():
            slow = m(x.to(dtype).cuda()).cpu().to(F64)
        assert float((got - slow).abs().max() / slow.abs().max()) < 3e-2


def test_feed_forward_with_the_branch_gate_in_one_product():
    """gate | up | branch gate as one product with biases for the last part only; the activation reads a row-strided view."""
    from nanovllm.layers.activation import GatedFeedForward
    for width, ff in ((40, 24), (100, 50)):
        g = torch.Generator().manual_seed(width)
        P = {n: torch.randn(a, b, generator=g, dtype=F64) * b ** -0.5
             for n, (a, b) in {"gate": (ff, width), "up": (ff, width), "down": (width, ff), "rg": (width, width)}.items()}
        b = torch.randn(width, generator=g, dtype=F64)
        m = GatedFeedForward(width, ff, "silu", extra=width)
        load = m.gate_up_proj.weight_loader
        load(m.gate_up_proj.weight, P["gate"].float(), (0, 0))
        load(m.gate_up_proj.weight, P["up"].float(), (0, 1))
        load(m.gate_up_proj.weight, P["rg"].float(), 1)
        load(m.gate_up_proj.bias, b.float(), 1)
        m.down_proj.weight.data.copy_(P["down"])
        h = torch.randn(9, width, generator=g, dtype=F64)
        with torch.no_grad():
            y, gate = m.cuda()(_dev(h))
        assert float((y.cpu().to(F64) - O.gated_ff(h, P)).abs().max()) < 1e-5
        assert float((gate.cpu().to(F64) - (h @ P["rg"].T + b)).abs().max()) < 1e-5
