"""CPU: the host side of the Pofazen decoder -- registry and native configuration, presets, checkpoint tensors routed onto
fused, stacked and side-by-side parameters, the wavelength-scaled frequencies, configurations that are refused, and the
float64 oracle's own invariants (so that the GPU tests compare against something sound)."""
import json
import math

import pytest
import torch

import pofazen_oracle as O
from test_pofazen_gpu import config_a, config_b, config_c, config_d, reference, rot, tokens_of

F64 = torch.float64


def test_registry_native_config_and_presets(tmp_path):
    from nanovllm.config import Config, NativeConfig
    from nanovllm.models.models_map import model_dict
    from nanovllm.engine.model_runner import _resolve_dtype
    with open(tmp_path / "config.json", "w") as f:
        json.dump(config_a(), f)
    c = Config(str(tmp_path), max_model_len=4096, max_num_batched_tokens=4096, dtype="float32")
    assert isinstance(c.hf_config, NativeConfig) and c.hf_config.architectures == ["Pofazen"]
    cls = model_dict["Pofazen"]
    assert cls.supports_fp32 and cls.reads_checkpoint_shapes and not cls.prefix_caching
    assert _resolve_dtype(c.hf_config, "float32", cls) == torch.float32
    p = Config("tiny-pofazen").hf_config.to_dict()
    assert [e["type"] for e in p["layers"]] == ["parallel", "wkv", "wkv"] and p["layers"][2]["mlp"] is None
    for name, layers, width in (("pofazen-1k", 28, 1024), ("pofazen-2k", 16, 2048)):
        big = Config(name).hf_config.to_dict()
        assert len(big["layers"]) == layers and big["width"] == width


@pytest.mark.parametrize("make", [config_a, config_b, config_c, config_d])
def test_checkpoint_tensors_route_onto_the_model(tmp_path, make):
    """Every tensor of a checkpoint lands somewhere, every parameter is covered but for the padding (which stays zero),
    the fused projections hold their parts where the mixers slice them, the two output projections lie side by side, and
    the decay projection's inner size is the checkpoint's."""
    from safetensors.torch import save_file
    from nanovllm.config import NativeConfig
    from nanovllm.models.models_map import model_dict
    from nanovllm.utils.loader import checkpoint_shapes, load_model
    cfg = make()
    tensors = O.random_weights(cfg, seed=3)
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(tmp_path / "model.safetensors"))
    conf = NativeConfig(json.loads(json.dumps(cfg)))
    for e in conf.to_dict()["layers"]:
        e["mixer"].pop("decay_rank", None)              # a checkpoint's configuration does not give it
    conf.checkpoint_shapes = checkpoint_shapes(str(tmp_path))
    model = model_dict["Pofazen"](conf)
    padded = set()
    for name, p in model.named_parameters():
        if name.endswith("mix.proj.weight") and p.dim() == 2 or name.endswith("mix.o_proj.weight"):
            padded.add(name)
        else:
            p.data.fill_(float("nan"))
    assert load_model(model, str(tmp_path)) == len(tensors)
    assert not any(torch.isnan(p).any() for p in model.parameters())
    assert model.alpha == cfg["postln_alpha"] and model.eps == cfg["norm"]["eps"]
    assert torch.equal(model.embed_norm.weight, tensors["embed.norm"].float())
    assert torch.equal(model.norm.weight, tensors["final.norm"].float())
    for i, entry in enumerate(cfg["layers"]):
        lay, mix, m = model.layers[i], model.layers[i].mix, entry["mixer"]
        t = lambda n: tensors[f"l{i}.{n}"].float()
        assert torch.equal(lay.norm1.weight, t("norm1"))
        if entry["type"] == "wkv":
            assert mix.w1.weight.shape[0] == m["decay_rank"]
            for s, c in enumerate("rkvg"):
                assert torch.equal(mix.proj.weight[s].float(), t("mix." + c))
            for s, c in enumerate("rkvgw"):
                assert torch.equal(mix.shift.mu[s], t("mix.mu." + c))
            assert torch.equal(mix.w2.weight.float(), t("mix.w2")) and torch.equal(mix.rec.w0, t("mix.w0"))
            assert torch.equal(mix.rec.u, t("mix.u").reshape(-1)) and torch.equal(mix.norm.weight, t("mix.norm"))
            n = m["heads"] * m["dim"]
            assert mix.rec.state_shapes()["state"][0] == (m["heads"], m["dim"], m["dim"]) and mix.proj.weight.shape[1] == n
            assert mix.shift.state_shapes() == {"shift_state": ((cfg["width"],), None)}
        else:
            a, b = m["left"], m["right"]
            y = torch.arange(mix.proj.weight.shape[0])[None, :]
            pick = lambda part, lo=0, n=None: mix.proj.weight.float()[mix.proj.part(y, part)[0][lo:None if n is None else lo + n]]
            nq, nk = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            assert torch.equal(pick(0, 0, nq), t("mix.left.q")) and torch.equal(pick(0, nq, nk), t("mix.left.k"))
            assert torch.equal(pick(0, nq + nk), t("mix.left.v")) and torch.equal(pick(1), t("mix.left.g"))
            nqk = b["kv_heads"] * b["dim"]
            assert torch.equal(pick(2, 0, nqk), t("mix.right.q")) and torch.equal(pick(2, nqk, nqk), t("mix.right.k"))
            assert torch.equal(pick(2, 2 * nqk), t("mix.right.v")) and torch.equal(pick(3), t("mix.right.g"))
            assert torch.equal(pick(4), t("mix.right.b")) and torch.equal(pick(5), t("mix.right.a"))
            assert all(int(mix.proj.part(y, p)[0][0]) % 8 == 0 for p in range(6))          # 16-byte aligned parts
            used = sum(mix.proj.output_sizes)
            assert int((mix.proj.weight.abs().sum(1) == 0).sum()) == mix.proj.weight.shape[0] - used
            cw = mix.conv.weight
            assert torch.equal(cw[:nqk], t("mix.right.q.conv")) and torch.equal(cw[2 * nqk:], t("mix.right.v.conv"))
            assert torch.equal(mix.right_norm.weight, t("mix.right.norm").repeat(b["heads"]))
            x = torch.arange(mix.o_proj.weight.shape[1])[None, :]
            assert torch.equal(mix.o_proj.weight.float()[:, mix.o_proj.part(x, 0)[0]], t("mix.left.o"))
            assert torch.equal(mix.o_proj.weight.float()[:, mix.o_proj.part(x, 1)[0]], t("mix.right.o"))
            assert (mix.left_scale, mix.right_scale) == (m["left_scale"], m["right_scale"])
            mask = a.get("mask") or {"size": 0, "keep_first": 0}
            assert (mix.attn.window, mix.attn.keep_first, mix.attn.scale) == (mask["size"], mask["keep_first"], a["scale"])
            assert mix.attn.cache_rows() == (nk, a["kv_heads"] * a["vdim"])
            assert mix.rule.A_log.numel() == mix.rule.dt_bias.numel() == b["heads"]
        if entry["mlp"] is None:
            assert lay.mlp is None and not hasattr(lay, "norm2")
        else:
            assert torch.equal(lay.mlp.gate_up_proj.weight.float()[entry["mlp"]["ff"]:], t("mlp.up"))
            assert torch.equal(lay.norm2.weight, t("norm2"))


def test_random_weights_keep_the_padding_zero():
    from nanovllm.config import NativeConfig
    from nanovllm.models.models_map import model_dict
    model = model_dict["Pofazen"](NativeConfig(config_d()))
    model.random_init(1)
    for i in (0, 2):
        for lin, dim in ((model.layers[i].mix.proj, 1), (model.layers[i].mix.o_proj, 0)):
            used = sum(lin.output_sizes if dim else lin.input_sizes)
            assert int((lin.weight.abs().sum(dim) == 0).sum()) == lin.weight.shape[1 - dim] - used > 0
        assert model.layers[i].mix.right_norm.weight.view(model.layers[i].mix.rule.num_heads, -1).std(0).max() == 0


def test_refused_configurations():
    from nanovllm.config import NativeConfig
    from nanovllm.models.models_map import model_dict
    for change in (lambda c: c["layers"][0].update(type="recurrence"), lambda c: c["layers"][0]["mlp"].update(kind="moe")):
        cfg = config_b()
        change(cfg)
        with pytest.raises(ValueError):
            model_dict["Pofazen"](NativeConfig(cfg))


def test_wavelength_scaled_frequencies():
    """Short wavelengths keep their frequency, long ones are divided by the factor, between the two lies a blend that
    meets both ends; a transition of zero width; no scaling."""
    from nanovllm.layers.seq_mixers import WavelengthScaledRotary
    plain = WavelengthScaledRotary(32, 1e4)
    assert float(plain.freq[0]) == 1.0 and float(plain.freq[3]) == pytest.approx(1e4 ** (-6 / 32))
    sc = {"factor": 5.0, "low": 1.0, "high": 4.0, "original": 1500}
    r = WavelengthScaledRotary(32, 1e4, True, sc)
    assert torch.equal(r.freq, O.frequencies(rot(32, 1e4, (5.0, 1.0, 4.0, 1500))))
    ratio, wave = r.freq / plain.freq, 2 * math.pi / plain.freq
    assert bool((ratio[wave < 1500 / 4] == 1.0).all()) and bool(((ratio[wave > 1500] - 0.2).abs() < 1e-12).all())
    mid = ratio[(wave >= 1500 / 4) & (wave <= 1500)]
    assert mid.numel() >= 2 and bool((mid > 0.2).all()) and bool((mid < 1.0).all())
    assert bool((ratio[1:] <= ratio[:-1] + 1e-15).all())                # monotone from 1 down to 1 / factor
    step = WavelengthScaledRotary(32, 1e4, True, dict(sc, low=2.0, high=2.0))
    assert set((step.freq / plain.freq * 10).round().tolist()) == {2.0, 10.0}
    assert r.key != plain.key and WavelengthScaledRotary(32, 1e4, True, dict(sc)).key == r.key


# ------------------------------------------------------------------ the oracle's own invariants
@pytest.mark.parametrize("make", [config_a, config_d])
def test_oracle_continues_a_sequence(make):
    """A prompt in one piece equals the same prompt continued from handed-over state (keys, states, tails, shifted rows)."""
    cfg = make()
    w = O.to64(O.random_weights(cfg, seed=3))
    toks = torch.tensor(tokens_of(cfg, 26, 8))
    whole, _ = O.forward(toks, w, cfg)
    a, st = O.forward(toks[:9], w, cfg)
    b, st = O.forward(toks[9:10], w, cfg, past=st)
    c, _ = O.forward(toks[10:], w, cfg, past=st)
    assert float((torch.cat([a, b, c]) - whole).abs().max()) < 1e-9


def test_oracle_is_causal_and_looks_far_back():
    cfg = config_a()
    w = O.to64(O.random_weights(cfg, seed=4))
    toks = tokens_of(cfg, 30, 9)
    a = reference(cfg, w, toks)
    other = list(toks)
    other[12] = (other[12] + 1) % cfg["vocab"]
    b = reference(cfg, w, other)
    assert torch.equal(a[:12], b[:12]) and all(not torch.equal(a[t], b[t]) for t in range(12, 30))


def test_oracle_mask_and_recurrences():
    assert O.visible(9, {"size": 3, "keep_first": 2}) == [0, 1, 7, 8, 9]
    assert O.visible(2, {"size": 3, "keep_first": 2}) == [0, 1, 2] and O.visible(4, None) == list(range(5))
    assert O.visible(4, {"size": 1, "keep_first": 0}) == [4]
    g = torch.Generator().manual_seed(0)
    # a delta rule with beta = 1 and no decay stores the value: reading with the key returns it, a second write replaces it
    k = O.unit(torch.randn(2, 1, 6, generator=g, dtype=F64))
    k[1] = k[0]
    v = torch.randn(2, 1, 4, generator=g, dtype=F64)
    one = torch.ones(2, 1, dtype=F64)
    o, S = O.delta_rule(k, k, v, one, one, torch.zeros(1, 6, 4, dtype=F64))
    assert float((o - v).abs().max()) < 1e-5 and float((S[0].T @ k[1, 0] - v[1, 0]).abs().max()) < 1e-5
    # wkv: the first token returns its bonus alone
    r, kk, vv = (torch.randn(3, 1, 5, generator=g, dtype=F64) for _ in range(3))
    u = torch.randn(1, 5, generator=g, dtype=F64)
    o, _ = O.wkv_recurrence(r, kk, vv, torch.full((3, 1, 5), 0.5, dtype=F64), u, torch.zeros(1, 5, 5, dtype=F64))
    assert float((o[0, 0] - (r[0, 0] * u[0] * kk[0, 0]).sum() * vv[0, 0]).abs().max()) < 1e-12
    h = torch.randn(4, 6, generator=g, dtype=F64)
    assert torch.equal(O.token_shift(h, torch.zeros(6, dtype=F64)), h)
    s = O.token_shift(h, torch.ones(6, dtype=F64))
    assert not bool(s[0].any()) and torch.allclose(s[1:], h[:-1], rtol=0, atol=1e-15)
    x = torch.randn(3, 8, generator=g, dtype=F64)
    assert float((O.post_norm(x, -2.0 * x, torch.ones(8, dtype=F64), 1.0, 0.0).pow(2).mean(-1) - 1).abs().max()) < 1e-12
