"""Host-side parts of Bovitar in the layer-list family: config.json reader, weight fusion, shared tensors, the library subset
a process serving such a model builds, the memory estimate, scheduler bookkeeping, and self-consistency of the oracle."""
import json
import math

import pytest
import torch

from gpustack_b200.config import LayerListConfig, ModelConfig, RotarySpec
from gpustack_b200.weights import (layer_list_tensor_shapes, load_layer_list, load_layer_list_dir, random_layer_list_state,
                                   save_layer_list_checkpoint)
from oracle import bovitar_oracle as O

F64 = torch.float64


def _cfg():
    moe = {"kind": "moe", "expert": {"ff": 18}, "router": {"experts": 6, "top": 3, "scale": 1.5, "groups": {"count": 3, "keep": 2}},
           "shared": {"ff": 22}}
    par = {"type": "parallel", "mlp": moe, "mixer": {
        "left": {"heads": 3, "kv_heads": 1, "dim": 10, "vdim": 14, "conv": 3, "scale": 0.3, "softcap": 12.0,
                 "rot": {"base": 700.0, "dims": 6, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 128}}},
        "right": {"heads": 4, "vdim": 5, "state": 9, "groups": 2, "conv": 4, "norm_groups": 2}}}
    dl = {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "conv": 2},
          "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 2, "top": 1}}}
    return {"architecture": "Bovitar", "vocab": 131, "width": 52, "norm": {"eps": 1e-6}, "logit_scale": 0.4,
            "layers": [par, dict(dl, mlp=None), dict(par, weights_of=0), dl, dict(dl, weights_of=3)]}


def test_config_reader_round_trip_and_rejections(tmp_path):
    d = _cfg()
    c = LayerListConfig.from_dict(d)
    assert c.family == "layer_list" and c.residual == "pre_norm" and c.norm == "rms" and c.norm_eps == 1e-6 and c.logit_scale == 0.4
    assert c.has_state and [l.weights_of for l in c.layers] == [None, None, 0, None, 3]
    assert [c.weight_owner(l) for l in range(5)] == [0, 1, 0, 3, 3] and c.runs() == [(l, False) for l in range(5)]
    p = c.layers[0].mixer
    a, r = p.left, p.right
    assert p.kind == "side_by_side" and p.branch_norm and (p.left_scale, p.right_scale) == (0.5, 0.5)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.conv_taps) == (3, 1, 10, 14, 0.3, 12.0, 3)
    assert a.qk_norm and a.qk_norm_joint and not (a.sink or a.gate or a.qkv_bias or a.window or a.plus_one)
    assert a.rot.layout == "half" and (a.rot.dims, a.rot.wave_factor, a.rot.wave_original) == (6, 4.0, 128.0)
    assert (r.heads, r.vdim, r.state, r.groups, r.conv, r.norm_groups) == (4, 5, 9, 2, 4, 2)
    assert r.conv_width == 20 + 36 and r.proj_rows == 76 and r.row_width == 4 * 8 + 4 * 12 and r.state_width == 4 * 5 * 12
    t = c.layers[1].mixer
    assert (t.kind, t.heads, t.kv_heads, t.dim, t.vdim, t.conv) == ("delta", 4, 2, 6, 10, 2) and c.layers[1].mlp is None
    assert t.conv_width == 64 and t.proj_rows == 104 and t.row_width == 4 * 8 + 4 * 12
    e = c.layers[0].mlp.moe
    assert (e.experts, e.top, e.ff, e.shared_ff, e.scale, e.groups, e.groups_keep) == (6, 3, 18, 22, 1.5, 3, 2)
    assert e.score == "softmax" and not e.renormalize and e.act == "silu" and e.gated and not e.shared_gate
    z = c.layers[3].mlp.moe
    assert (z.groups, z.shared_ff, z.scale) == (0, 0, 1.0)
    assert a.cache_widths() == (64, 64) and a.cache_widths(False) == (10, 14) and a.tile_sized
    back = LayerListConfig.from_dict(json.loads(json.dumps(c.to_dict())))
    assert back == c
    (tmp_path / "config.json").write_text(json.dumps(d))
    assert ModelConfig.from_pretrained(str(tmp_path)) == c
    plain = json.loads(json.dumps(d))
    for l in (0, 2):
        del plain["layers"][l]["mixer"]["left"]["rot"]["scaling"]
    assert LayerListConfig.from_dict(plain).layers[0].mixer.left.rot.wave_factor == 0.0
    for breaker in (lambda x: x["layers"][0]["mixer"]["left"].update(heads=4, kv_heads=3),
                    lambda x: x["layers"][0]["mixer"]["left"].update(softcap=0.0),
                    lambda x: x["layers"][0]["mixer"]["left"].update(conv=0),
                    lambda x: x["layers"][0]["mixer"]["left"]["rot"].update(dims=12),
                    lambda x: x["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(high=0.5),
                    lambda x: x["layers"][0]["mixer"]["right"].update(groups=3),
                    lambda x: x["layers"][0]["mixer"]["right"].update(norm_groups=3),
                    lambda x: x["layers"][0]["mixer"]["right"].update(conv=9),
                    lambda x: x["layers"][1]["mixer"].update(kv_heads=3),
                    lambda x: x["layers"][1].update(type="gla"),
                    lambda x: x["layers"][0]["mlp"].update(kind="dense"),
                    lambda x: x["layers"][0]["mlp"]["router"].update(top=5),        # only 4 experts lie in two groups
                    lambda x: x["layers"][0]["mlp"]["router"]["groups"].update(count=4),
                    lambda x: x["layers"][0]["mlp"]["router"]["groups"].update(keep=4),
                    lambda x: x["layers"][2].update(weights_of=1),                 # another kind of layer
                    lambda x: x["layers"][2].update(weights_of=7),
                    lambda x: (x["layers"][0].update(weights_of=2), x["layers"][2].update(weights_of=0))):
        bad = json.loads(json.dumps(d))
        breaker(bad)
        with pytest.raises((ValueError, KeyError)):
            LayerListConfig.from_dict(bad)


def test_frequencies_on_all_three_branches():
    """Short wavelengths keep their frequency, long ones are slowed by the factor, a blend lies between -- against the rule
    written with wavelengths."""
    rot = {"base": 50.0, "dims": 16, "scaling": {"factor": 5.0, "low": 1.0, "high": 3.0, "original": 40}}
    got = RotarySpec(dims=16, base=50.0, layout="half", wave_factor=5.0, wave_original=40.0, wave_low=1.0, wave_high=3.0).frequencies()
    assert got[1] == 1.0 and got[0] == pytest.approx(O.scaled_frequencies(rot), rel=1e-14)
    kinds = set()
    for i, f in enumerate(got[0]):
        base = 50.0 ** (-i / 8)
        wave = 2 * math.pi / base
        kind = "keep" if wave < 40 / 3 else ("slow" if wave > 40 else "blend")
        kinds.add(kind)
        if kind != "blend":
            assert f == pytest.approx(base if kind == "keep" else base / 5)
        else:
            assert base / 5 < f < base
    assert kinds == {"keep", "slow", "blend"}


def test_weight_fusion_layout_shared_tensors_and_checkpoint_round_trip(tmp_path):
    d = _cfg()
    c = LayerListConfig.from_dict(d)
    W = O.random_weights(d, seed=1)
    assert {k: tuple(v) for k, v in layer_list_tensor_shapes(c).items()} == O.tensor_shapes(d)
    asked = []
    w = load_layer_list(c, lambda k: (asked.append(k), W[k])[1], "cpu")
    assert w.layers[2] is w.layers[0] and w.layers[4] is w.layers[3] and not any(k.startswith(("l2.", "l4.")) for k in asked)
    l0, l1, l3 = w.layers[0], w.layers[1], w.layers[3]
    rows = torch.cat([W["l0.mix.left." + n] for n in "qkv"] + [W["l0.mix.right.in"][:76]])
    assert l0.proj.shape[0] % 8 == 0 and torch.equal(l0.proj[:len(rows)], rows) and not l0.proj[len(rows):].any()
    assert torch.equal(l0.gates, W["l0.mix.right.in"][76:]) and l0.gates.shape == (4, 52)
    assert l0.conv_w.shape == (3, 54) and torch.equal(l0.conv_w.t(), torch.cat([W[f"l0.mix.left.{n}.conv"] for n in "qkv"]).float())
    assert l0.rec_conv_t.shape == (4, 56) and torch.equal(l0.rec_conv_t.t(), W["l0.mix.right.conv"].float())
    assert torch.equal(l0.decay_rate, torch.exp(W["l0.mix.right.A_log"].float())) and torch.equal(l0.skip, W["l0.mix.right.D"].float())
    assert torch.equal(l0.o2, W["l0.mix.right.o"]) and torch.equal(l0.left_norm, W["l0.mix.left.out"]) and l0.q_norm.shape == (30,)
    assert l0.rot_freq.dtype == F64 and l0.rot_freq.tolist() == pytest.approx(O.scaled_frequencies(d["layers"][0]["mixer"]["left"]["rot"]))
    assert l0.router.shape == (128, 52) and torch.equal(l0.router[:6], W["l0.mlp.router"]) and not l0.router[6:].any()
    assert torch.equal(l0.w13[0:2], torch.stack([W["l0.mlp.e0.gate"][0], W["l0.mlp.e0.up"][0]])) and l0.sink is None
    assert torch.equal(l1.gates, torch.cat([W["l1.mix.b"], W["l1.mix.a"]])) and l1.norm2 is None and l1.router is None
    assert torch.equal(l1.proj[:104], torch.cat([W["l1.mix." + n] for n in "qkvg"])) and l1.out_norm.shape == (10,)
    assert l3.shared13 is None and torch.equal(l3.correction, W["l3.mlp.correction"].float())
    bad = dict(W)
    bad["l1.mix.k.conv"] = W["l1.mix.k.conv"][:, :-1]
    with pytest.raises(ValueError):
        load_layer_list(c, lambda k: bad[k], "cpu")
    st = random_layer_list_state(c, seed=2)
    assert set(st) == set(W)
    save_layer_list_checkpoint(c, st, str(tmp_path))
    back = load_layer_list_dir(ModelConfig.from_pretrained(str(tmp_path)), str(tmp_path), "cpu")
    assert torch.equal(back.layers[4].proj[:12], st["l3.mix.q"])


def test_library_subset_of_a_pre_norm_model():
    import ctypes

    from gpustack_b200 import build

    c = LayerListConfig.from_dict(_cfg())
    tag, srcs = build.layer_list_sources(c)
    assert tag == "pre_norm_routed_tc" and {"prenorm.cu", "conv_attn_prep.cu", "conv_rec_prep.cu", "gated_scan.cu",
                                            "attention_sink.cu", "attention.cu", "attention_prefill_tc.cu", "moe.cu"} <= set(srcs)
    assert not {"mlstm.cu", "sandwich.cu", "allreduce.cu", "norm.cu", "postnorm.cu", "latent.cu"} & set(srcs)
    h = ctypes.CDLL(str(build.build(sources=srcs, tag=tag)))
    for n in ("b200_embed_streams", "b200_prenorm_join", "b200_conv_attn_prep_ex", "b200_rot_table", "b200_conv_rec_prep", "b200_gated_scan",
              "b200_gate_norm", "b200_attn_sink_prefill_cap", "b200_attn_sink_decode_cap", "b200_paged_attn_prefill_cap",
              "b200_paged_attn_decode_cap", "b200_moe_route_grouped", "b200_moe_align", "b200_moe_gather_scaled", "b200_moe_grouped_gemm_ex",
              "b200_linear_simt_grouped_ex", "b200_gemm_bf16_silu_mul", "b200_linear_simt", "b200_sample_softcap_f32", "b200_last_error"):
        assert hasattr(h, n), n
    assert not hasattr(h, "b200_mlstm_scan") and not hasattr(h, "b200_sandwich_join")
    d = _cfg()
    d["layers"] = [dict(d["layers"][1])]
    tag, srcs = build.layer_list_sources(LayerListConfig.from_dict(d))
    assert tag == "pre_norm" and "moe.cu" not in srcs and "attention.cu" not in srcs


def test_vram_estimate_counts_pages_states_rings_and_each_tensor_once():
    from gpustack_b200.config import EngineConfig
    from gpustack_b200.resource_fit import estimate

    d = _cfg()
    c = LayerListConfig.from_dict(d)
    e16 = estimate(c, EngineConfig(max_model_len=256, max_num_seqs=4, max_num_batched_tokens=256))
    e32 = estimate(c, EngineConfig(max_model_len=256, max_num_seqs=4, max_num_batched_tokens=256, dtype="float32"))
    assert e16.weights == c.weight_bytes() and e16.kv_bytes_per_token == c.kv_bytes_per_token() == 2 * (2 * 128)     # two runs, padded
    assert e32.kv_bytes_per_token == 2 * 4 * 24
    # per run: states, and the last taps - 1 rows of every convolution
    pair = 4 * (2 * 54 + 4 * 5 * 12 + 3 * 56)
    assert c.state_bytes_per_seq() == 2 * pair + 3 * 4 * (4 * 10 * 8 + 64)
    W = O.random_weights(d, 0)
    n = sum(v.numel() for k, v in W.items() if v.dim() == 2 and not k.endswith("conv") and k != "embed")
    assert c.weight_bytes() == 2 * n


def test_requests_take_and_return_state_slots():
    from gpustack_b200.scheduler import Request, SamplingParams, Scheduler

    s = Scheduler(num_blocks=20, block_size=16, max_num_seqs=2, max_num_batched_tokens=64, max_model_len=128, eos_token_id=None,
                  enable_prefix_caching=True, state_slots=2)
    for i in range(3):
        s.add(Request(req_id=str(i), prompt_ids=[1] * 20, params=SamplingParams(max_tokens=4, ignore_eos=True)))
    plan = s.schedule()
    assert plan is not None and s.slots.num_free == 0                   # the third request waits for a slot
    s.abort("0")
    assert s.slots.num_free == 1


def test_oracle_mechanisms_are_consistent():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)   # noqa: E731
    # the convolution against torch's, with a bias, and its last tap on the current token
    x, w, b = r(20, 5), r(5, 3), r(5)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T.unsqueeze(0), (2, 0)), w.unsqueeze(1), b, groups=5)[0].T
    assert torch.allclose(O.causal_conv(x, w, b), ref) and torch.allclose(O.causal_conv(x, w)[0], w[:, 2] * x[0])
    # a rotation keeps lengths and turns scores into functions of the distance
    rot = {"base": 100.0, "dims": 6}
    q, k = r(1, 1, 8).expand(30, 1, 8), r(1, 1, 8).expand(30, 1, 8)
    Q, K = (O.rotate_half(t.clone(), torch.arange(30), rot) for t in (q, k))
    assert torch.allclose(Q.norm(dim=-1), q.norm(dim=-1))
    S = torch.einsum("ihd,jhd->ij", Q, K)
    assert torch.allclose(S[5:, :-5].diagonal(), S[5, 0].expand(25)) and torch.equal(Q[..., 6:], q[..., 6:])
    # capped attention position by position
    q, k, v = r(11, 4, 6), r(11, 2, 6), r(11, 2, 5)
    out = O.capped_attention(q, k, v, 0.7, 2.0)
    for i, h in ((0, 0), (10, 3), (6, 1)):
        p = torch.softmax(2.0 * torch.tanh(k[:i + 1, h // 2] @ q[i, h] * 0.7 / 2.0), -1)
        assert torch.allclose(out[i, h], p @ v[:i + 1, h // 2])
    # the delta rule: with unit keys, no decay and a full step the state answers a written key with exactly its value
    T, dk, dv = 12, 5, 3
    k, v = O.unit(r(T, 1, dk), 0.0), r(T, 2, dv)
    one = torch.ones(T, 2, dtype=F64)
    assert torch.allclose(O.delta_scan(k, k, v, one, one), v)
    assert torch.allclose(O.delta_scan(k, k, v, one, 0 * one), 0 * v)
    # ... and the state-space recurrence as a sum over the past
    x, B, C, dt, A, D = r(T, 2, dv), r(T, 1, dk), r(T, 1, dk), torch.rand(T, 2, generator=g, dtype=F64), r(2), r(2)
    y = O.ssd_scan(x, B, C, dt, A, D)
    t, h = 9, 1
    want = D[h] * x[t, h]
    for s in range(t + 1):
        want = want + torch.exp(-torch.exp(A[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (B[s, 0] @ C[t, 0]) * x[s, h]
    assert torch.allclose(y[t, h], want)
    # a group is chosen by its best expert; the weights leave the correction out
    z, c = torch.log(torch.tensor([[0.4, 0.1, 0.2, 0.2, 0.05, 0.05]], dtype=F64)), torch.tensor([-9.0, -0.5, -0.1, -9.0, -0.2, -0.3], dtype=F64)
    idx, wt = O.route(z, c, {"experts": 6, "top": 3, "scale": 2.0, "groups": {"count": 3, "keep": 2}})
    assert sorted(idx[0].tolist()) == [2, 4, 5] and torch.allclose(wt.sum(), torch.tensor(0.6, dtype=F64))
    # whole model: a prefix's logits do not depend on what follows
    d = _cfg()
    Wm = O.random_weights(d, seed=4)
    toks = torch.randint(0, 131, (30,), generator=g).tolist()
    full = O.forward(d, Wm, toks)
    assert torch.allclose(O.forward(d, Wm, toks[:17]), full[:17], atol=1e-9)


@pytest.mark.parametrize("name", ["odd", "tiles", "wide"])
def test_every_mechanism_shows_in_the_logits_of_the_tests_models(name, monkeypatch):
    """A mistake planted in the oracle, one mechanism at a time, moves the logits of the models that the engine tests run
    by far more than those tests' 32-bit tolerance: none of them could pass with that mechanism wrong."""
    import tests.test_bovitar_gpu as T

    cfg = T.CFGS[name]()
    W = O.random_weights(cfg, seed=3 + len(name))
    toks = T._tokens(cfg, 60, 1)
    right = O.forward(cfg, W, toks)

    def moved(c=cfg):
        return float((O.forward(c, W, toks) - right).abs().max() / right.abs().max())

    conv, attn, unit, delta, ssd, route, rotate, softplus, grouped = (O.causal_conv, O.capped_attention, O.unit, O.delta_scan, O.ssd_scan, O.route,
                                                                      O.rotate_half, O.softplus, O.grouped_rms)

    def late_read(q, k, v, g, b):                        # the read-out misses the current token's write
        o = delta(q, k, v, g, b)
        H, G = v.shape[1], k.shape[1]
        of = torch.arange(H) // (H // G)
        own = b[..., None] * v * (q[:, of] * k[:, of]).sum(-1, keepdim=True)
        return o - own

    wrong = {
        "causal_conv": lambda u, w, b=None: conv(u, torch.cat([0.2 * w[:, :1], w], 1), b),
        "capped_attention": lambda q, k, v, s, c: attn(q, k, v, s, 1e6),
        "unit": lambda x, eps=1e-6: O.rms(x, eps),
        "delta_scan": late_read,
        "ssd_scan": lambda x, B, C, dt, A, D: ssd(x, B, C, dt, A, 0 * D),
        "softplus": lambda z: torch.clamp(z, min=0.0) + torch.log(torch.tensor(2.0, dtype=F64)) * torch.exp(-z.abs()),
        "route": lambda z, c, ro: route(z, 0 * c, ro),
        "rotate_half": lambda x, p, rot: rotate(x, 2 * p, rot),        # (a shift alone would not show)
        "grouped_rms": lambda x, n, eps: grouped(x, 1 if n > 1 else x.shape[1], eps),
    }
    for fn, f in wrong.items():
        with monkeypatch.context() as m:
            m.setattr(O, fn, f)
            assert moved() > 5e-3, fn
    # the weights renormalized; groups ignored; frequencies unscaled; one output of the pair not normed
    with monkeypatch.context() as m:
        m.setattr(O, "route", lambda z, c, ro: (lambda i, w: (i, w / w.sum(-1, keepdim=True)))(*route(z, c, ro)))
        assert moved() > 5e-3
    for change in ("groups", "scaling", "weights_of", "logit_scale"):
        bad = json.loads(json.dumps(cfg))
        for l in bad["layers"]:
            if change == "groups" and l["mlp"]:
                l["mlp"]["router"].pop("groups", None)
            if change == "scaling" and l["type"] == "parallel":
                l["mixer"]["left"]["rot"].pop("scaling", None)
        if change == "logit_scale":
            bad["logit_scale"] *= 1.5
        if change == "weights_of":
            bad["layers"] = [l for l in bad["layers"] if l.get("weights_of") is None]
            if name == "odd":                            # (their numbers would move)
                continue
        if name == "wide" and change == "groups":        # (it has none)
            continue
        assert moved(bad) > 5e-3, change
    for leaf in ("left.out", "right.out", "k.norm", "right.conv.b", "shared.down", "A_log", "dt_bias"):
        with monkeypatch.context() as m:
            for k in W:
                if k.endswith(leaf):
                    m.setitem(W, k, (W[k].float().flip(0) * 1.5 - 0.3).to(torch.bfloat16))
            assert moved() > 5e-3, leaf
