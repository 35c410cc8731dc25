"""Host-side parts of Kerarax in the layer-list family: config.json reader, weight fusion, the library subset a process
serving such a model builds, the memory estimate, and self-consistency of the oracle."""
import json

import pytest
import torch

from gpustack_b200.config import LayerListConfig, ModelConfig
from gpustack_b200.weights import (layer_list_tensor_shapes, load_layer_list, load_layer_list_dir, pad_head_columns,
                                   random_layer_list_state, save_layer_list_checkpoint)
from oracle import kerarax_oracle as O

F64 = torch.float64


def _cfg():
    def layer(H, G, dk, dv, conv, mlp):
        return {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 0.3, "softcap": 12.0,
                                               "conv": conv}, "mlp": mlp}

    moe = {"kind": "moe", "expert": {"ff": 18}, "router": {"experts": 5, "top": 3}, "shared": {"ff": 22}}
    return {"architecture": "Kerarax", "vocab": 131, "width": 52, "norm": {"eps": 1e-6}, "logit_softcap": 20.0,
            "layers": [layer(3, 1, 10, 14, 3, moe), layer(4, 2, 6, 10, 1, None),
                       layer(2, 2, 12, 5, 5, dict(moe, shared=None, router={"experts": 2, "top": 1}))]}


def test_config_reader_round_trip_and_rejections(tmp_path):
    d = _cfg()
    c = LayerListConfig.from_dict(d)
    assert c.family == "layer_list" and c.residual == "output_norm" and c.norm == "layernorm_bias" and c.norm_eps == 1e-6
    assert c.sinusoidal_positions and c.embed_norm and c.logit_softcap == 20.0 and c.has_state
    a, b, z = (l.mixer for l in c.layers)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.conv_taps) == (3, 1, 10, 14, 0.3, 12.0, 3)
    assert a.plus_one and a.qk_norm and not (a.sink or a.gate or a.qkv_bias or a.window) and a.rot is None
    e = c.layers[0].mlp.moe
    assert (e.experts, e.top, e.ff, e.shared_ff, e.score, e.act) == (5, 3, 18, 22, "chosen_softmax", "relu2")
    assert e.router_bias and e.shared_gate and not e.gated and c.layers[1].mlp is None
    assert c.layers[2].mlp.moe.shared_ff == 0 and not c.layers[2].mlp.moe.shared_gate
    # cached rows: one tile width for any pair of widths in bf16, the widths themselves in 32-bit
    assert a.cache_widths() == (64, 64) and a.cache_widths(False) == (10, 14) and a.tile_sized
    wide = json.loads(json.dumps(d))
    wide["layers"][0]["mixer"].update(dim=128, vdim=96)
    m = LayerListConfig.from_dict(wide).layers[0].mixer
    assert m.cache_widths() == (128, 128) and m.tile_sized
    wide["layers"][0]["mixer"].update(dim=160, vdim=96)
    m = LayerListConfig.from_dict(wide).layers[0].mixer
    assert m.cache_widths() == (160, 96) and not m.tile_sized
    wide["layers"][0]["mixer"].update(heads=17, kv_heads=1, dim=16, vdim=16)
    assert not LayerListConfig.from_dict(wide).layers[0].mixer.tile_sized
    back = LayerListConfig.from_dict(json.loads(json.dumps(c.to_dict())))
    assert back == c
    (tmp_path / "config.json").write_text(json.dumps(d))
    assert ModelConfig.from_pretrained(str(tmp_path)) == c
    for breaker in (lambda x: x["layers"][0]["mixer"].update(heads=4, kv_heads=3),
                    lambda x: x["layers"][0]["mixer"].update(softcap=0.0),
                    lambda x: x["layers"][0]["mixer"].update(conv=0),
                    lambda x: x["layers"][0]["mixer"].update(conv=9),
                    lambda x: x["layers"][0].update(type="gla"),
                    lambda x: x["layers"][0]["mlp"].update(kind="dense"),
                    lambda x: x["layers"][0]["mlp"]["router"].update(top=6),
                    lambda x: x["layers"][0]["mlp"]["router"].update(top=0),
                    lambda x: x.update(logit_softcap=-1.0)):
        bad = json.loads(json.dumps(d))
        breaker(bad)
        with pytest.raises((ValueError, KeyError)):
            LayerListConfig.from_dict(bad)
    one = json.loads(json.dumps(d))
    for l in one["layers"]:
        l["mixer"]["conv"] = 1
    assert not LayerListConfig.from_dict(one).has_state               # one tap: nothing but pages is carried


def test_weight_fusion_layout_and_checkpoint_round_trip(tmp_path):
    d = _cfg()
    c = LayerListConfig.from_dict(d)
    W = O.random_weights(d, seed=1)
    w = load_layer_list(c, lambda k: W[k], "cpu")
    assert {k: tuple(v) for k, v in layer_list_tensor_shapes(c).items()} == O.tensor_shapes(d)
    l0, l1, l2 = w.layers
    rows = torch.cat([W["l0.mix." + n] for n in "qkv"])
    assert l0.proj.shape[0] % 8 == 0 and torch.equal(l0.proj[:rows.shape[0]], rows) and not l0.proj[rows.shape[0]:].any()
    assert l0.conv_w.dtype == torch.float32 and l0.conv_w.shape == (3, 54) and l0.conv_w.is_contiguous()
    assert torch.equal(l0.conv_w.t(), torch.cat([W[f"l0.mix.{n}.conv"] for n in "qkv"]).float())
    assert torch.equal(l0.sink, torch.zeros(3)) and l0.proj_bias is None
    assert torch.equal(l0.q_norm, W["l0.mix.q.norm"]) and torch.equal(l0.norm1_b, W["l0.norm1.b"]) and torch.equal(l0.norm2_b, W["l0.norm2.b"])
    assert torch.equal(l0.w13, torch.cat([W[f"l0.mlp.e{i}.up"] for i in range(5)]))
    assert torch.equal(l0.w2, torch.cat([W[f"l0.mlp.e{i}.down"] for i in range(5)]))
    assert torch.equal(l0.shared13, W["l0.mlp.shared.up"]) and torch.equal(l0.shared2, W["l0.mlp.shared.down"])
    # the shared expert's gate is the row behind the router's outputs
    assert l0.router.shape == (128, 52) and torch.equal(l0.router[:5], W["l0.mlp.router"])
    assert torch.equal(l0.router[5:6], W["l0.mlp.shared.sg"]) and not l0.router[6:].any()
    assert torch.equal(l0.correction, W["l0.mlp.router.b"].float())
    assert l1.norm2 is None and l1.w13 is None and l2.shared13 is None and not l2.router[2:].any()
    assert torch.equal(w.embed_norm, W["embed.norm"]) and torch.equal(w.final_norm_b, W["final.norm.b"])
    assert w.pos_freq.dtype == F64 and w.pos_freq.tolist() == pytest.approx([10000.0 ** (-2 * i / 52) for i in range(26)])
    o = pad_head_columns(W["l0.mix.o"], 3, 14, 64)
    assert o.shape == (52, 192) and torch.equal(o.view(52, 3, 64)[:, :, :14].reshape(52, 42), W["l0.mix.o"])
    assert not o.view(52, 3, 64)[:, :, 14:].any()
    bad = dict(W)
    bad["l0.mix.k.conv"] = W["l0.mix.k.conv"][:, :-1]
    with pytest.raises(ValueError):
        load_layer_list(c, lambda k: bad[k], "cpu")
    st = random_layer_list_state(c, seed=2)
    assert set(st) == set(W)
    save_layer_list_checkpoint(c, st, str(tmp_path))
    back = load_layer_list_dir(ModelConfig.from_pretrained(str(tmp_path)), str(tmp_path), "cpu")
    assert torch.equal(back.layers[2].proj[:24], st["l2.mix.q"])


def test_library_subset_of_an_output_norm_model():
    import ctypes

    from gpustack_b200 import build

    c = LayerListConfig.from_dict(_cfg())
    tag, srcs = build.layer_list_sources(c)
    assert tag == "output_norm_routed_tc" and {"postnorm.cu", "conv_attn_prep.cu", "attention_sink.cu", "attention.cu",
                                               "attention_prefill_tc.cu", "moe.cu", "moe_biased.cu"} <= set(srcs)
    assert "mlstm.cu" not in srcs and "sandwich.cu" not in srcs and "allreduce.cu" not in srcs and "norm.cu" not in srcs
    h = ctypes.CDLL(str(build.build(sources=srcs, tag=tag)))
    for n in ("b200_embed_sinusoid", "b200_output_norm_join", "b200_conv_attn_prep", "b200_attn_sink_prefill_cap",
              "b200_attn_sink_decode_cap", "b200_paged_attn_prefill_cap", "b200_paged_attn_decode_cap", "b200_moe_route_scored",
              "b200_moe_align", "b200_moe_gather_scaled", "b200_moe_grouped_gemm_ex", "b200_linear_simt_grouped_ex",
              "b200_gemm_bf16_relu2", "b200_relu2", "b200_linear_simt", "b200_sample_softcap_f32", "b200_last_error"):
        assert hasattr(h, n), n
    assert not hasattr(h, "b200_mlstm_scan") and not hasattr(h, "b200_sandwich_join")
    d = _cfg()
    for l in d["layers"]:
        l["mlp"] = None
        l["mixer"].update(dim=144)
    tag, srcs = build.layer_list_sources(LayerListConfig.from_dict(d))
    assert tag == "output_norm" and "moe.cu" not in srcs and "attention.cu" not in srcs


def test_vram_estimate_counts_padded_pages_rings_and_experts():
    from gpustack_b200.config import EngineConfig
    from gpustack_b200.resource_fit import estimate

    d = _cfg()
    c = LayerListConfig.from_dict(d)
    e16 = estimate(c, EngineConfig(max_model_len=256, max_num_seqs=4, max_num_batched_tokens=256))
    e32 = estimate(c, EngineConfig(max_model_len=256, max_num_seqs=4, max_num_batched_tokens=256, dtype="float32"))
    assert e16.weights == c.weight_bytes() and e16.kv_bytes_per_token == c.kv_bytes_per_token() == 2 * 128 * (1 + 2 + 2)
    assert e32.kv_bytes_per_token == 4 * (1 * 24 + 2 * 16 + 2 * 17)
    # rings: the last taps - 1 rows of [q | k | v] of the layers with more than one tap
    assert c.state_bytes_per_seq() == 4 * (2 * (30 + 10 + 14) + 4 * (24 + 24 + 10))
    W = O.random_weights(d, 0)
    n = sum(v.numel() for k, v in W.items() if k.split(".")[-1] not in ("norm", "norm1", "norm2", "b", "conv", "embed", "sg"))
    assert c.weight_bytes() == 2 * n


def test_oracle_mechanisms_are_consistent():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)   # noqa: E731
    x, w, b = r(7, 12), r(12), r(12)
    assert torch.allclose(O.layer_norm(x, w, b, 1e-5), torch.nn.functional.layer_norm(x, (12,), w, b, 1e-5))
    # sine and cosine of the same angle alternate; the first pair turns by one radian per position
    s = O.sinusoid(torch.arange(9), 12)
    assert torch.allclose(s[:, 0::2] ** 2 + s[:, 1::2] ** 2, torch.ones(9, 6, dtype=F64))
    assert torch.allclose(s[:, 0], torch.sin(torch.arange(9, dtype=F64))) and torch.allclose(s[3, 5], torch.cos(torch.tensor(3 * 10000 ** (-4 / 12), dtype=F64)))
    # the convolution against torch's, and its last tap on the current token
    x, w = r(20, 5), r(5, 3)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T.unsqueeze(0), (2, 0)), w.unsqueeze(1), groups=5)[0].T
    assert torch.allclose(O.causal_conv(x, w), ref) and torch.allclose(O.causal_conv(x, w)[0], w[:, 2] * x[0])
    # one more in the denominator = an ordinary softmax with an extra score of zero
    z = r(4, 6) * 3
    assert torch.allclose(O.softmax_plus_one(z), torch.softmax(torch.cat([z, torch.zeros(4, 1, dtype=F64)], -1), -1)[:, :6])
    assert float(O.softmax_plus_one(torch.full((1, 3), -60.0, dtype=F64)).sum()) < 1e-20
    # attention position by position
    q, k, v = r(11, 4, 6), r(11, 2, 6), r(11, 2, 5)
    out = O.capped_attention(q, k, v, 0.7, 2.0)
    for i, h in ((0, 0), (10, 3), (6, 1)):
        sc = 2.0 * torch.tanh(k[:i + 1, h // 2] @ q[i, h] * 0.7 / 2.0)
        p = torch.exp(sc) / (1 + torch.exp(sc).sum())
        assert torch.allclose(out[i, h], p @ v[:i + 1, h // 2])
    # routing weights are a softmax over the chosen alone
    idx, wt = O.route(torch.tensor([[1.0, -50.0, 3.0, 2.0]], dtype=F64), 2)
    assert idx.tolist() == [[2, 3]] and torch.allclose(wt, torch.softmax(torch.tensor([[3.0, 2.0]], dtype=F64), -1))
    # whole model: a prefix's logits do not depend on what follows, and no logit passes the cap
    d = _cfg()
    Wm = O.random_weights(d, seed=4)
    toks = torch.randint(0, 131, (30,), generator=g).tolist()
    full = O.forward(d, Wm, toks)
    assert torch.allclose(O.forward(d, Wm, toks[:17]), full[:17], atol=1e-9) and float(full.abs().max()) < 20.0


@pytest.mark.parametrize("name", ["odd", "tiles", "wide"])
def test_every_mechanism_shows_in_the_logits_of_the_tests_models(name, monkeypatch):
    """A mistake planted in the oracle, one mechanism at a time, moves the logits of the models that the engine tests run
    by far more than those tests' 32-bit tolerance: none of them could pass with that mechanism wrong."""
    import tests.test_kerarax_gpu as T

    cfg = T.CFGS[name]()
    W = O.random_weights(cfg, seed=3 + len(name))
    toks = T._tokens(cfg, 60, 1)
    right = O.forward(cfg, W, toks)

    def moved():
        return float((O.forward(cfg, W, toks) - right).abs().max() / right.abs().max())

    conv, cap, route, rms, ln, sin = O.causal_conv, O.soft_cap, O.route, O.head_rms_norm, O.layer_norm, O.sinusoid
    one_more_tap = lambda u, w: conv(u, torch.cat([0.2 * w[:, :1], w], 1))                                 # noqa: E731
    wrong = {
        "softmax_plus_one": lambda s: torch.softmax(s, -1),
        "causal_conv": one_more_tap,
        "soft_cap": lambda z, c: z if c != cfg["logit_softcap"] else cap(z, c),
        "route": lambda z, k: (route(z, k)[0], torch.softmax(z, -1).gather(-1, route(z, k)[0])),
        "head_rms_norm": lambda x, w, e: x / torch.sqrt((x * x).mean(-1, keepdim=True) + e) * (1 + w),
        "layer_norm": lambda x, w, b, e: ln(x, w, 0 * b, e),
        "sinusoid": lambda p, d, dt=F64: sin(p + 1, d, dt),
    }
    for fn, f in wrong.items():
        with monkeypatch.context() as m:
            m.setattr(O, fn, f)
            assert moved() > 3e-3, fn
    for leaf, w in (("mlp.shared.sg", 0.0), ("mlp.router.b", 0.0), ("mix.k.norm", 2.0), ("mix.v.conv", 0.5)):
        with monkeypatch.context() as m:
            for k in W:
                if k.endswith(leaf):
                    m.setitem(W, k, W[k] * w)
            if leaf == "mix.v.conv":                                   # (a factor alone would vanish in the output's norm)
                for k in [k for k in W if k.endswith(leaf)]:
                    m.setitem(W, k, W[k].flip(1).roll(1, 0))
            assert moved() > 3e-3, leaf
