"""CPU: the host side of the Ragilorn decoder -- registry and native configuration, presets, checkpoint tensors routed
onto fused projections with biases and stacked experts, the matrix that turns cached rows into keys and values,
configurations that are refused, and the float64 oracle's own invariants (so that the GPU tests compare against something
sound)."""
import json

import pytest
import torch

import ragilorn_oracle as O
from test_ragilorn_gpu import (_latent_case, _latent_want, config_a, config_b, config_c, config_d, tokens_of)

F64 = torch.float64


def test_registry_native_config_and_presets(tmp_path):
    from nanovllm.config import Config, NativeConfig
    from nanovllm.models.models_map import model_dict
    from nanovllm.engine.model_runner import _resolve_dtype
    with open(tmp_path / "config.json", "w") as f:
        json.dump(config_a(), f)
    c = Config(str(tmp_path), max_model_len=4096, max_num_batched_tokens=4096, dtype="float32")
    assert isinstance(c.hf_config, NativeConfig) and c.hf_config.architectures == ["Ragilorn"]
    cls = model_dict["Ragilorn"]
    assert cls.supports_fp32 and not cls.prefix_caching
    assert _resolve_dtype(c.hf_config, "float32", cls) == torch.float32
    p = Config("tiny-ragilorn").hf_config.to_dict()
    assert [(l["type"], l["mlp"] and l["mlp"]["kind"]) for l in p["layers"]] == [
        ("attention", "dense"), ("latent_attention", "moe"), ("attention", None)]
    big = Config("ragilorn-1k").hf_config.to_dict()
    assert len(big["layers"]) == 28 and big["width"] == 1024
    assert sum(e["type"] == "latent_attention" for e in big["layers"]) == 12


@pytest.mark.parametrize("make", [config_a, config_b, config_c, config_d])
def test_checkpoint_tensors_route_onto_the_model(tmp_path, make):
    """Every tensor of a checkpoint lands somewhere, every parameter that has a tensor is covered, the fused projections hold
    their parts (and biases) in the order the mixers slice them, experts are stacked gate rows first."""
    from safetensors.torch import save_file
    from nanovllm.config import NativeConfig
    from nanovllm.models.models_map import model_dict
    from nanovllm.models.ragilorn import GatedMoe
    from nanovllm.utils.loader import load_model
    cfg = make()
    tensors = O.random_weights(cfg, seed=3)
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(tmp_path / "model.safetensors"))
    model = model_dict["Ragilorn"](NativeConfig(cfg))
    padded = {n for n, m in model.named_modules() if hasattr(m, "padded_sizes")}
    for n, p in model.named_parameters():
        if n.rsplit(".", 1)[0] not in padded:
            p.data.fill_(float("nan"))                                 # padding (zeros) is all that may stay as it was
    assert load_model(model, str(tmp_path)) == len(tensors)
    assert not any(torch.isnan(p).any() for p in model.parameters())
    assert model.lm_head.scale == cfg["logit_scale"] and model.lm_head.softcap == cfg["logit_softcap"]
    assert model.embed_scale == cfg["embedding"]["scale"] and model.eps == cfg["norm"]["eps"]
    assert torch.equal(model.norm.weight, tensors["final.norm"].float())
    for i, entry in enumerate(cfg["layers"]):
        lay, mix, m = model.layers[i], model.layers[i].mix, entry["mixer"]
        t = lambda n: tensors[f"l{i}.{n}"].float()
        part = lambda lin, j: (lin.part(lin.weight.float().T, j).T, lin.part(lin.bias.float()[None], j)[0])
        assert torch.equal(lay.norm1.weight, t("norm1"))
        assert lay.dwa.dtype == torch.float32 and torch.equal(lay.dwa, t("dwa")) and lay.dwa.numel() == i + 2
        if entry["type"] == "attention":
            w, b = part(mix.proj, 0)
            assert torch.equal(w, torch.cat([t("mix." + n) for n in "qkv"]))
            assert torch.equal(b, torch.cat([t(f"mix.{n}.b") for n in "qkv"]))
            gate = part(mix.proj, 1)
            assert torch.equal(mix.o_proj.bias.float(), t("mix.o.b"))
            assert mix.attn.chunk == (m.get("mask") or {"size": 0})["size"] and mix.attn.window == 0
            assert mix.attn.cache_rows() == (m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"])
            if m.get("conv"):
                assert torch.equal(mix.conv.weight, torch.cat([t(f"mix.{n}.conv") for n in "qkv"]))
                assert bool(mix.conv.state_shapes()) == (m["conv"] > 1)
            else:
                assert mix.conv is None
        else:
            (wq, bq), (wd, bd) = part(mix.proj, 0), part(mix.proj, 1)
            assert torch.equal(wq, t("mix.q")) and torch.equal(wd, t("mix.dkv"))
            assert float(bq.abs().max()) == 0.0 and float(bd.abs().max()) == 0.0
            gate = part(mix.proj, 2)
            assert torch.equal(mix.kv_norm, t("mix.dkv.norm"))
            assert torch.equal(mix.attn.w_uk.float().reshape(-1, m["kv_rank"]), t("mix.uk"))
            assert torch.equal(mix.attn.w_uv.float().reshape(-1, m["kv_rank"]), t("mix.uv"))
            assert mix.attn.cache_rows() == (m["kv_rank"] + m["rot_dim"], 0) and mix.attn.window == 0
            assert mix.o_proj.bias is None
        assert torch.equal(gate[0], t("rg1")) and torch.equal(gate[1], t("rg1.b"))
        assert mix.attn.scale == m["scale"] and mix.rot.interleaved and torch.equal(mix.o_proj.weight.float(), t("mix.o"))
        freqs, mag = O.yarn_table(m["rot"])
        assert mix.rot.freq.tolist() == pytest.approx(freqs, rel=1e-14) and mix.rot.magnitude == pytest.approx(mag)
        mlp = entry["mlp"]
        if mlp is None:
            assert lay.mlp is None and not hasattr(lay, "norm2")
            continue
        assert torch.equal(lay.norm2.weight, t("norm2"))
        if mlp["kind"] == "dense":
            w, b = part(lay.mlp.gate_up_proj, 0)
            assert torch.equal(w, torch.cat([t("mlp.gate"), t("mlp.up")])) and float(b.abs().max()) == 0.0
            w, b = part(lay.mlp.gate_up_proj, 1)
            assert torch.equal(w, t("rg2")) and torch.equal(b, t("rg2.b"))
        else:
            assert isinstance(lay.mlp, GatedMoe) and lay.mlp.moe.router.dtype == torch.float32
            assert torch.equal(lay.mlp.branch_gate.weight.float(), t("rg2"))
            assert torch.equal(lay.mlp.branch_gate.bias.float(), t("rg2.b"))
            ff, r, x = mlp["expert"]["ff"], mlp["router"], lay.mlp.moe
            assert x.top_k == r["top"] and x.weigh_input and not x.normalize and x.correction is None and x.groups == 1
            e = r["experts"] - 1
            assert torch.equal(x.w13.float()[e], torch.cat([t(f"mlp.e{e}.gate"), t(f"mlp.e{e}.up")]))
            assert torch.equal(x.w2.float()[e], t(f"mlp.e{e}.down"))


def test_synthetic_weights_keep_padding_and_missing_biases_zero():
    from nanovllm.config import NativeConfig
    from nanovllm.models.models_map import model_dict
    model = model_dict["Ragilorn"](NativeConfig(config_d()))
    model.random_init(0)
    mix = model.layers[1].mix                                          # latent: q | dkv | branch gate, padded to 8 rows each
    p = mix.proj
    assert p.padded_sizes != p.output_sizes
    off = 0
    for j, (n, pad) in enumerate(zip(p.output_sizes, p.padded_sizes)):
        assert float(p.weight[off + n:off + pad].abs().sum()) == 0.0 and float(p.bias[off + n:off + pad].abs().sum()) == 0.0
        assert (float(p.bias[off:off + n].abs().sum()) > 0) == (j == 2)
        off += pad
    assert all(bool(torch.isfinite(q).all()) for q in model.parameters())


@pytest.mark.parametrize("H,d,dr,dv,R", [(3, 40, 8, 64, 24), (2, 96, 64, 64, 40), (4, 48, 16, 128, 16)])
def test_one_product_gives_keys_and_values(H, d, dr, dv, R):
    """Cached rows times the module's matrix are every head's key (up-projected part, rotated part, zeros up to the
    kernel's width) and value: attention on them equals the restatement. It is made anew when a parameter changes."""
    from nanovllm.layers.seq_mixers import LatentAttention
    q, rows, wk, wv = _latent_case(9, H, d, dr, dv, R, torch.float32, 2)
    m = LatentAttention(H, d, dr, dv, R, 0.3)
    m.w_uk.data.copy_(wk)
    m.w_uv.data.copy_(wv)
    Kw = m._key_width()
    assert Kw % 64 == 0 and Kw >= d + dr > Kw - 64
    kv = rows @ m._up_matrix().to(F64).T
    k, v = kv[:, :H * Kw].reshape(9, H, Kw), kv[:, H * Kw:].reshape(9, H, dv)
    assert float(k[:, :, d + dr:].abs().sum()) == 0.0
    assert torch.equal(k[:, 1, d:d + dr], rows[:, R:])
    got = O.attention(q, k[:, :, :d + dr], v, 0.3)
    assert float((got - _latent_want(q, rows, wk, wv, 0.3)).abs().max()) < 1e-6
    first = m._up_matrix()
    assert m._up_matrix() is first
    with torch.no_grad():
        m.w_uv.mul_(2.0)
    assert torch.equal(m._up_matrix()[H * Kw:], 2 * first[H * Kw:])


def test_refused_configurations():
    from nanovllm.config import NativeConfig
    from nanovllm.layers.moe import GroupedSigmoidMoe
    from nanovllm.layers.seq_mixers import VarSizeAttention
    from nanovllm.models.models_map import model_dict
    cls = model_dict["Ragilorn"]
    cfg = config_b()
    cfg["layers"][0]["type"] = "recurrence"
    with pytest.raises(ValueError):
        cls(NativeConfig(cfg))
    cfg = config_b()
    cfg["layers"][1]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError):
        cls(NativeConfig(cfg))
    with pytest.raises(ValueError):
        VarSizeAttention(2, 1, 8, 8, 1.0, window=4, chunk=4)
    with pytest.raises(ValueError):
        GroupedSigmoidMoe(8, 8, 2, 1, weigh="both")


def test_key_splits_of_the_latent_kernel():
    """Few row tiles over many keys are split, a grid that fills the machine or short keys are not; a split keeps at least two
    64-key tiles."""
    from nanovllm import _C
    lib = _C.load()
    assert lib.b200_latent_attn_splits(1, 64) == 1 and lib.b200_latent_attn_splits(1, 127) == 1
    assert lib.b200_latent_attn_splits(1, 8192) > 8 and lib.b200_latent_attn_splits(16, 1024) > 1
    assert lib.b200_latent_attn_splits(4096, 1024) == 1
    for n in (128, 200, 1000):
        assert lib.b200_latent_attn_splits(1, n) <= n // 128
    one = __import__("ctypes").c_void_p(16)
    call = lambda dim, rank, splits, dtype: lib.b200_latent_attn(one, one, one, dim, None, 0, 0, one, one, None, 1, 1, 1, 2,
                                                                 dim, rank, 1.0, 0, splits, None, None, dtype, None)
    assert call(72, 64, 1, 2) < 0 and call(70, 64, 1, 0) == -3 and call(584, 512, 1, 0) == -3      # fp32, odd, too wide
    assert call(64, 72, 1, 0) == -2 and call(72, 64, 2, 0) == -1                                   # rank > dim; no workspace


# ------------------------------------------------------------------ the oracle's own invariants
def test_oracle_is_causal_and_chunks_hide():
    cfg = config_a()
    tensors = O.random_weights(cfg, seed=4)
    toks = tokens_of(cfg, 30, 9)
    a = O.forward(cfg, tensors, toks)
    other = list(toks)
    other[22] = (other[22] + 1) % cfg["vocab"]
    b = O.forward(cfg, tensors, other)
    assert torch.equal(a[:22], b[:22]) and not torch.equal(a[22:], b[22:])
    # with chunked layers only (no latent layer, no convolution), nothing crosses a chunk's border
    only = config_b()
    only["layers"] = [dict(only["layers"][0])]
    t = O.random_weights(only, seed=5)
    seq = tokens_of(only, 40, 3)
    whole = O.forward(only, t, seq)
    other = list(seq)
    other[15] = (other[15] + 1) % only["vocab"]                        # the last token of the first chunk of 16
    changed = O.forward(only, t, other)
    assert torch.equal(whole[16:], changed[16:]) and not torch.equal(whole[15], changed[15])
    other[16] = (other[16] + 1) % only["vocab"]
    assert not torch.equal(whole[31], O.forward(only, t, other)[31])   # the first token of a chunk is seen to its end


def test_oracle_mechanisms_on_small_inputs():
    assert [O.visible_from(p, 4) for p in (0, 3, 4, 7, 8)] == [0, 0, 4, 4, 8] and O.visible_from(9, 0) == 0
    x = [torch.full((2, 3), float(v), dtype=F64) for v in (1, 10, 100)]
    assert float(O.depth_average(x, [0.5, 2.0, -1.0])[0, 0]) == 0.5 + 20.0 - 100.0
    y, h = torch.ones(2, 3, dtype=F64), torch.zeros(2, 3, dtype=F64)
    b = torch.tensor([0.0, 50.0, -50.0], dtype=F64)
    got = O.gated_branch(x[0], y, h, torch.zeros(3, 3, dtype=F64), b)[0]
    assert got.tolist() == pytest.approx([1.5, 2.0, 1.0])
    ids, w = O.route(torch.tensor([[0.0, 3.0, -1.0]], dtype=F64), 2)
    assert ids[0].tolist() == [1, 0] and w[0].tolist() == pytest.approx([1 / (1 + 2.718281828459045 ** -3), 0.5])
    assert float(O.cap_logits(torch.tensor(1e9, dtype=F64), 0.5, 7.0)) == pytest.approx(7.0)
    assert float(O.cap_logits(torch.tensor(8.0, dtype=F64), 0.5, 0.0)) == 4.0
    u, cw = torch.randn(6, 3, dtype=F64), torch.randn(3, 4, dtype=F64)
    assert torch.allclose(O.short_conv(u, cw)[0], cw[:, 3] * u[0])
    f, mag = O.yarn_table({"dims": 8, "base": 100.0})
    assert mag == 1.0 and f[0] == 1.0 and f[1] == pytest.approx(100.0 ** -0.25)
