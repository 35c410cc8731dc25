"""Kerarax (layer-list decoder: a biased layer norm on every sublayer's output, sinusoidal embedding, grouped attention
over convolved q, k and v with capped scores and one more in the softmax denominator, routed relu^2 experts with a gated
shared expert, capped logits) on the GPU against the plain restatement in oracle/kerarax_oracle.py.

Every test builds its own small configuration and random weights.  Kernel tests compare one mechanism with the
oracle's function; engine tests drive LLMEngine (scheduler pools, state slots, runner step functions, CUDA graphs)
and compare logits with the oracle's whole-sequence forward.  float32 must agree to rounding, bfloat16 to bf16
rounding."""
import random

import numpy as np
import pytest
import torch

from oracle import kerarax_oracle as O

pytestmark = pytest.mark.gpu

F64 = torch.float64
BF = torch.bfloat16


def _layer(H, G, dk, dv, conv, mlp, scale=None, cap=30.0):
    return {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "conv": conv, "softcap": cap,
                                           "scale": dk ** -0.5 if scale is None else scale}, "mlp": mlp}


def _moe(E, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top},
            "shared": None if shared is None else {"ff": shared}}


def cfg_odd():
    """Nothing is a multiple of 8 and the width is odd: every product takes the CUDA-core path.  Key and value widths that
    differ, one key head for all query heads and one per query head, one to six taps, a low cap that bends most scores, a
    layer without feed-forward, one without a shared expert, every expert chosen."""
    return {"architecture": "Kerarax", "vocab": 131, "width": 51, "norm": {"eps": 1e-5}, "logit_softcap": 4.0,
            "layers": [_layer(3, 1, 10, 14, 3, _moe(5, 3, 18, 22), scale=1.3, cap=3.0), _layer(4, 2, 6, 10, 1, None, cap=50.0),
                       _layer(2, 2, 13, 7, 6, _moe(3, 3, 10, None), scale=0.9), _layer(6, 2, 70, 33, 2, _moe(2, 1, 9, 30), cap=5.0)]}


def cfg_tiles():
    """Widths that the tensor-core GEMMs take in bf16 (also the grouped ones), heads padded to 64, groups of 4 and 1."""
    return {"architecture": "Kerarax", "vocab": 256, "width": 256, "norm": {"eps": 1e-6}, "logit_softcap": 15.0,
            "layers": [_layer(4, 1, 64, 40, 4, _moe(6, 2, 256, 128), scale=0.3, cap=10.0),
                       _layer(3, 3, 32, 64, 2, _moe(4, 3, 512, 64), scale=0.4),
                       _layer(8, 2, 48, 48, 3, _moe(9, 1, 64, 192), scale=0.2, cap=20.0)]}


def cfg_plain():
    """Values a model may happen to make trivial: one tap everywhere (no state slots at all), one head, one expert, key and
    value widths alike, all experts chosen."""
    return {"architecture": "Kerarax", "vocab": 77, "width": 40, "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
            "layers": [_layer(1, 1, 8, 8, 1, _moe(1, 1, 16, 16)), _layer(2, 1, 16, 16, 1, _moe(2, 2, 8, 24), scale=1.0)]}


def cfg_wide():
    """128-wide heads, as they are and padded from either side, in groups of four (tcgen05 prefill, split-KV decode) and
    of eight; caps on both sides of the bound that lets the softmax do without a running maximum."""
    return {"architecture": "Kerarax", "vocab": 256, "width": 256, "norm": {"eps": 1e-5}, "logit_softcap": 30.0,
            "layers": [_layer(8, 2, 128, 96, 4, _moe(4, 2, 256, 256), scale=0.4, cap=25.0),
                       _layer(4, 1, 128, 128, 2, _moe(3, 1, 256, 64), scale=0.2, cap=90.0),
                       _layer(8, 1, 96, 128, 3, _moe(2, 1, 64, 64), scale=0.3)]}


CFGS = {"odd": cfg_odd, "tiles": cfg_tiles, "plain": cfg_plain, "wide": cfg_wide}


def _engine(cfg, weights, dtype, blocks=64, seqs=4, mbt=256, eager=False, max_len=512):
    from gpustack_b200.config import EngineConfig, LayerListConfig
    from gpustack_b200.engine import LLMEngine

    ecfg = EngineConfig(dtype=dtype, max_model_len=max_len, max_num_seqs=seqs, max_num_batched_tokens=mbt, num_gpu_blocks=blocks,
                        enable_prefix_caching=False, max_logit_rows=mbt, enforce_eager=eager)
    return LLMEngine.from_engine_config(ecfg, mcfg=LayerListConfig.from_dict(cfg), state_dict={k: v.cuda() for k, v in weights.items()})


def _tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def _rel(got, want):
    want = want.to(torch.float64).numpy() if isinstance(want, torch.Tensor) else want
    got = got.detach().to(torch.float64).cpu().numpy() if isinstance(got, torch.Tensor) else np.asarray(got, dtype=np.float64)
    return float(np.abs(got - want).max() / max(1e-9, np.abs(want).max()))


TOL = {"float32": 3e-5, "bfloat16": 4e-2}
KTOL = {torch.float32: 2e-5, BF: 2e-2}


def _rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def _cuts(n, sizes):
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


# ------------------------------------------------------------------------------------ mechanisms, one at a time
@pytest.mark.parametrize("D", [37, 64, 250])
@pytest.mark.parametrize("hdt", [torch.float32, BF])
def test_embedding_with_sinusoids_and_its_norm(D, hdt):
    from gpustack_b200 import ops

    table, w, b = _rnd(50, D, seed=1, dtype=BF), _rnd(D, seed=2, dtype=BF) + 1, _rnd(D, seed=3, dtype=BF)
    ids, pos = [3, 49, 0, 7, 7, 11], [0, 1, 17, 499, 200001, 65536]
    freq = torch.tensor([10000.0 ** (-2.0 * i / D) for i in range((D + 1) // 2)], dtype=F64, device="cuda")
    plain = table[ids].to(F64) + O.sinusoid(torch.tensor(pos), D)
    for norm in (False, True):
        want = O.layer_norm(plain, w.to(F64), b.to(F64), 1e-5) if norm else plain
        x, xb = torch.zeros(6, D, device="cuda"), torch.zeros(6, D, dtype=hdt, device="cuda")
        ops.embed_sinusoid(_i32(ids), _i32(pos), table.cuda(), freq, x, norm=(w.cuda(), b.cuda()) if norm else None, eps=1e-5, xb_out=xb)
        assert _rel(x, want) < 2e-6
        assert torch.equal(xb, x.to(hdt))


@pytest.mark.parametrize("D", [37, 64, 300])
@pytest.mark.parametrize("hdt", [torch.float32, BF])
def test_join_norms_the_output_and_adds_it(D, hdt):
    from gpustack_b200 import ops

    T, eps = 9, 1e-5
    x, y = _rnd(T, D, seed=1), _rnd(T, D, seed=2, scale=3.0) + 5.0        # (an output with a mean: the norm takes it off)
    pw, pb, fw, fb = (_rnd(D, seed=3 + i, dtype=BF) for i in range(4))
    d = lambda t: t.to(F64)   # noqa: E731
    z = d(x) + O.layer_norm(d(y), d(pw), d(pb), eps)
    c = lambda t: t.cuda()    # noqa: E731
    xo, ho = torch.zeros(T, D, device="cuda"), torch.zeros(T, D, dtype=hdt, device="cuda")
    ops.output_norm_join(c(x), eps, y=c(y), post=(c(pw), c(pb)), x_out=xo, h_out=ho)
    assert _rel(xo, z) < 2e-6 and torch.equal(ho, xo.to(hdt))
    inplace = c(x).clone()
    ops.output_norm_join(inplace, eps, y=c(y), post=(c(pw), c(pb)), x_out=inplace, h_out=ho)
    assert torch.equal(inplace, xo)
    # the last output, the sum and the final norm of chosen rows in one pass; the final norm alone
    rows = [7, 0, 3]
    hg = torch.zeros(3, D, dtype=hdt, device="cuda")
    ops.output_norm_join(c(x), eps, y=c(y), post=(c(pw), c(pb)), final=(c(fw), c(fb)), h_out=hg, rows=_i32(rows))
    assert _rel(hg, O.layer_norm(z, d(fw), d(fb), eps)[rows]) < (2e-6 if hdt == torch.float32 else 8e-3)
    ops.output_norm_join(c(x), eps, final=(c(fw), c(fb)), h_out=hg, rows=_i32(rows))
    assert _rel(hg, O.layer_norm(d(x), d(fw), d(fb), eps)[rows]) < (2e-6 if hdt == torch.float32 else 8e-3)
    # routed form: a token's expert rows anywhere in the row space, with and without a gated shared expert
    for K, shared in ((1, True), (3, True), (4, False)):
        yp, sh = _rnd(T * K + 5, D, seed=11), _rnd(T, D, seed=12)
        lg = _rnd(T, 8, seed=13, scale=2.0)
        pr = torch.randperm(T * K + 5, generator=torch.Generator().manual_seed(K))[:T * K]
        v = d(yp)[pr].view(T, K, D).sum(1) + (torch.sigmoid(d(lg[:, 5:6])) * d(sh) if shared else 0)
        want = d(x) + O.layer_norm(v, d(pw), d(pb), eps)
        routed = (c(yp), pr.to(torch.int32).cuda(), K, c(sh) if shared else None, c(lg)[:, 5] if shared else None)
        ops.output_norm_join(c(x), eps, routed=routed, post=(c(pw), c(pb)), x_out=xo, h_out=ho)
        assert _rel(xo, want) < 2e-6
        ops.output_norm_join(c(x), eps, routed=routed, post=(c(pw), c(pb)), final=(c(fw), c(fb)), h_out=hg, rows=_i32(rows))
        assert _rel(hg, O.layer_norm(want, d(fw), d(fb), eps)[rows]) < (2e-6 if hdt == torch.float32 else 8e-3)


PREP = [  # H, G, dk, dv, wk, wv, taps, dtype
    (3, 1, 10, 14, 10, 14, 3, torch.float32), (3, 1, 10, 14, 64, 64, 3, BF), (4, 2, 16, 8, 16, 8, 4, torch.float32),
    (4, 2, 64, 40, 64, 64, 4, BF), (2, 2, 128, 96, 128, 128, 2, BF), (8, 1, 96, 128, 128, 128, 1, BF), (5, 5, 24, 24, 24, 24, 3, BF),
    (2, 1, 13, 7, 13, 7, 7, torch.float32), (2, 1, 40, 24, 64, 64, 8, BF), (6, 3, 32, 64, 32, 64, 1, torch.float32),
    (1, 1, 200, 264, 200, 264, 2, BF), (2, 1, 160, 140, 160, 140, 3, torch.float32)]


@pytest.mark.parametrize("H,G,dk,dv,wk,wv,taps,dtype", PREP)
def test_convolution_norm_and_pages_in_portions_with_rings_that_are_used_again(H, G, dk, dv, wk, wv, taps, dtype):
    """Sequences cut into portions of 1 .. 37 rows that ride in the same launches (prompt portions and single rows), rings and
    pages in shuffled slots; a third sequence takes the first one's ring without any clearing.  Queries and pages equal the
    convolution and norm of the whole sequence; the columns behind the heads' own are zeros."""
    from gpustack_b200 import ops

    C, eps, page = (H + G) * dk + G * dv, 1e-5, 16
    cw = _rnd(taps, C, seed=1, scale=0.6)
    qn, kn = _rnd(dk, seed=2, dtype=BF) + 1, _rnd(dk, seed=3, dtype=BF) + 1
    seqs = {"a": _rnd(83, C, seed=4).to(dtype), "b": _rnd(60, C, seed=5).to(dtype), "c": _rnd(15, C, seed=6).to(dtype)}
    want = {}
    for n, u in seqs.items():
        y = O.causal_conv(u.to(F64), cw.t().to(F64))
        q, k, v = y[:, :H * dk].view(-1, H, dk), y[:, H * dk:(H + G) * dk].view(-1, G, dk), y[:, (H + G) * dk:].view(-1, G, dv)
        want[n] = (O.head_rms_norm(q, qn.to(F64), eps), O.head_rms_norm(k, kn.to(F64), eps), v)
    ring = torch.full((2, max(taps - 1, 1), C), 7.0, device="cuda") if taps > 1 else None
    kc = torch.full((20, G, page, wk), 9.0, dtype=dtype, device="cuda")
    vc = torch.full((20, G, page, wv), 9.0, dtype=dtype, device="cuda")
    tables = {"a": [7, 3, 12, 1, 9, 15], "b": [2, 14, 5, 10], "c": [6]}
    got = {n: [] for n in seqs}
    at = {n: 0 for n in seqs}
    slot = {"a": 1, "b": 0, "c": 1}
    # (prompt portions, then single rows)
    plan = [([("a", 9)], [("b", 1)]), ([("b", 2)], [("a", 1)]), ([("a", 2)], [("b", 1)]), ([("b", 5), ("a", 3)], []), ([], [("a", 1), ("b", 1)]),
            ([("a", 37), ("b", 17)], []), ([("b", 33), ("a", 30)], []), ([], [("c", 1)]), ([("c", 1)], []), ([("c", 2)], []), ([("c", 11)], [])]
    tile = 32
    for prompts, singles in plan:
        step = prompts + singles
        rows = torch.cat([seqs[n][at[n]:at[n] + m] for n, m in step]).cuda()
        wide = torch.zeros(rows.shape[0], -(-C // 8) * 8 + 8, dtype=dtype, device="cuda")
        wide[:, :C] = rows
        cu = np.cumsum([0] + [m for _, m in step]).tolist()
        slots = [tables[n][p // page] * page + p % page for n, m in step for p in range(at[n], at[n] + m)]
        qo = torch.full((rows.shape[0], H * wk), 5.0, dtype=dtype, device="cuda")
        ts = tq = None
        if prompts:
            ts, tq = (_i32(t) for t in ops.build_prefill_tiles([m for _, m in prompts], tile, [at[n] for n, _ in prompts]))
        ops.conv_attn_prep(wide, cw.cuda(), qn.cuda(), kn.cuda(), ring, _i32(cu), _i32([at[n] for n, _ in step]),
                           _i32([slot[n] for n, _ in step]), ts, tq, tile, len(prompts), len(singles), _i32(slots), qo, kc, vc, H, G, dk,
                           dv, eps)
        for (n, m), o in zip(step, cu):
            got[n].append(qo[o:o + m].cpu())
            at[n] += m
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    for n in seqs:
        assert at[n] == len(seqs[n])
        q = torch.cat(got[n]).view(-1, H, wk)
        assert _rel(q[..., :dk], want[n][0]) < tol and not q[..., dk:].any(), n
        for cache, w, ref, width in ((kc, wk, want[n][1], dk), (vc, wv, want[n][2], dv)):
            r = torch.stack([cache[tables[n][p // page], :, p % page] for p in range(at[n])]).cpu()
            assert _rel(r[..., :width], ref) < tol and not r[..., width:].any(), n
    for b in set(range(20)) - {t for tb in tables.values() for t in tb}:
        assert float(kc[b].float().min()) == 9.0                       # nobody else's page was touched
    if ring is not None:
        for n, s in (("b", 0), ("c", 1)):
            for p in range(at[n] - taps + 1, at[n]):
                assert torch.equal(ring[s, p % (taps - 1)].cpu(), seqs[n][p].float())


@pytest.mark.parametrize("taps,dtype", [(4, BF), (3, torch.float32), (6, torch.float32)])
def test_the_first_and_the_last_tap_reach_exactly_as_far_as_they_should(taps, dtype):
    """One row of the sequence stands out.  The row taps - 1 later still sees it, the next does not -- in a portion, across
    the border of two portions and in single rows; rows that are not written (slot -1) leave pages and nothing else."""
    from gpustack_b200 import ops

    H, G, dk, dv = 1, 1, 16, 16
    C, n = 48, 24
    cw = torch.ones(taps, C)
    for cuts in ([n], [1] * n, [8 + taps - 2, 1, 1, n - 8 - taps], [8, 1, n - 9]):
        u = torch.zeros(n, C, dtype=dtype)
        u[7] = 100.0
        ring = torch.full((1, taps - 1, C), 3.0, device="cuda")
        vc = torch.zeros(3, 1, 16, dv, dtype=dtype, device="cuda")
        kc = torch.zeros(3, 1, 16, dk, dtype=dtype, device="cuda")
        at = 0
        for m in cuts:
            single = m == 1 and at > 0
            ts, tq = (None, None) if single else (_i32(t) for t in ops.build_prefill_tiles([m], 16, [at]))
            q = torch.zeros(m, dk, dtype=dtype, device="cuda")
            ops.conv_attn_prep(u[at:at + m].cuda(), cw.cuda(), None, None, ring, _i32([0, m]), _i32([at]), _i32([0]), ts, tq, 16,
                               0 if single else 1, 1 if single else 0, _i32([16 + p if p != 9 else -1 for p in range(at, at + m)]),
                               q, kc, vc, H, G, dk, dv, 1e-5)
            at += m
        seen = [p for p in range(n) if float(vc.view(-1, dv)[16 + p, 0]) == 100.0]
        assert seen == [p for p in range(7, 7 + taps) if p != 9], (cuts, seen)


def _paged(k, v, G, wk, wv, dtype, seed, extra=5):
    """k [T, G, dk], v [T, G, dv] in shuffled pages (junk elsewhere), heads padded with zeros -> caches and block table."""
    T = k.shape[0]
    nb = -(-T // 16)
    g = torch.Generator().manual_seed(seed)
    perm = (torch.randperm(nb + extra, generator=g) + 1)[:nb]
    kc = torch.full((nb + extra + 1, G, 16, wk), 50.0, dtype=dtype)
    vc = torch.full((nb + extra + 1, G, 16, wv), 50.0, dtype=dtype)
    for p in range(T):
        b = int(perm[p // 16])
        for c, t in ((kc, k), (vc, v)):
            c[b, :, p % 16] = 0.0
            c[b, :, p % 16, :t.shape[2]] = t[p].to(dtype)
    return kc.cuda(), vc.cuda(), perm.to(torch.int32).view(1, -1).cuda()


ATT = [  # H, G, dk, dv, wk, wv, cap, route
    (3, 1, 10, 14, 10, 14, 3.0, "generic32"), (4, 2, 70, 33, 70, 33, 30.0, "generic32"), (4, 2, 24, 40, 24, 40, 8.0, "generic16"),
    (6, 3, 64, 48, 64, 64, 20.0, "generic16"), (4, 1, 64, 40, 64, 64, 30.0, "decode"), (16, 1, 40, 64, 64, 64, 5.0, "decode"),
    (2, 2, 96, 128, 128, 128, 50.0, "decode"), (8, 2, 128, 96, 128, 128, 30.0, "tc"), (8, 1, 100, 128, 128, 128, 4.0, "tc"),
    (4, 1, 128, 128, 128, 128, 90.0, "tc"), (8, 1, 128, 128, 128, 128, 54.0, "tc")]


@pytest.mark.parametrize("H,G,dk,dv,wk,wv,cap,route", ATT)
@pytest.mark.parametrize("start", [0, 1, 37])
def test_capped_attention_with_one_more_in_the_denominator(H, G, dk, dv, wk, wv, cap, route, start):
    """Prompt portions that begin at 0, 1 and 37 and single rows at many lengths, over shuffled pages with junk in foreign
    ones; scores of several times the cap among small ones.  All scores low: the extra one takes most of the softmax."""
    from gpustack_b200 import ops

    dtype = torch.float32 if route == "generic32" else BF
    n = 150
    for shift, scale in ((0.0, 4.0 * cap / 30 / dk ** 0.5), (0.0, 0.5 / dk ** 0.5), (-3.0, 1.0 / dk ** 0.5)):
        q, k, v = _rnd(n, H, dk, seed=1), _rnd(n, G, dk, seed=2), _rnd(n, G, dv, seed=3)
        k[:, :, 0], q[:, :, 0] = 1.0, shift / scale * min(1.0, dk ** 0.5 / 8)         # a common offset of every score
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        want = O.capped_attention(q.to(F64), k.to(F64), v.to(F64), scale, cap)
        kc, vc, bt = _paged(k, v, G, wk, wv, dtype, seed=4)
        qp = torch.zeros(n, H, wk, dtype=dtype)
        qp[..., :dk] = q
        rows = qp[start:].reshape(n - start, H * wk).contiguous().cuda()
        zero = torch.zeros(H, device="cuda")
        tile = ops.attn_prefill_tile(H, G) if route == "tc" else 16
        ts, tq = (_i32(t) for t in ops.build_prefill_tiles([n - start], tile, [start]))
        out = torch.full((n - start, H * wv), 3.0, dtype=dtype, device="cuda")
        cu, ctx = _i32([0, n - start]), _i32([start])
        if route == "tc":
            ops.paged_attn_prefill_ex(rows, rows.stride(0), kc, vc, bt, cu, ctx, ts, tq, out, H, G, wk, scale, sink=zero, softcap=cap)
        else:
            ops.attn_sink_prefill(rows, -1, kc, vc, bt, cu, ctx, ts, tq, zero, out, H, G, wk, wv, scale, tile_rows=tile, softcap=cap)
        got = out.view(-1, H, wv)
        tol = KTOL[dtype]
        assert _rel(got[..., :dv], want[start:]) < tol and not got[..., dv:].any()
        lens = sorted({1, 2, 15, 16, 17, 33, 64, 100, 149, 150})
        lens = [m for m in lens if m > start]
        one = torch.stack([qp[m - 1] for m in lens]).reshape(len(lens), H * wk).cuda()
        btb = bt.repeat(len(lens), 1)
        for splits in ((1,) if route.startswith("generic") else (1, 3)):
            od = torch.full((len(lens), H * wv), 3.0, dtype=dtype, device="cuda")
            if route.startswith("generic"):
                ops.attn_sink_decode(one, -1, kc, vc, btb, _i32(lens), zero, od, H, G, wk, wv, scale, softcap=cap)
            else:
                ws = ops.attn_decode_workspace(len(lens), H, wk, splits, "cuda")
                ops.paged_attn_decode(one, one.stride(0), kc, vc, btb, _i32(lens), od, H, G, wk, scale, num_splits=splits,
                                      workspace=ws, sink=zero, softcap=cap)
            assert _rel(od.view(-1, H, wv)[..., :dv], want[[m - 1 for m in lens]]) < tol, splits


@pytest.mark.parametrize("route,H,G,W", [("generic32", 2, 1, 24), ("generic16", 2, 1, 24), ("decode", 4, 1, 64), ("tc", 8, 2, 128), ("tc", 8, 1, 128)])
@pytest.mark.parametrize("far", [0, 15, 16, 63, 64, 127, 128, 255, 383])
def test_one_far_key_stands_out_and_a_later_one_stays_invisible(route, H, G, W, far):
    """Among 400 keys one reaches the cap (its value is 5, the others' about 0): the rows behind it answer about 5, the rows
    before it do not; the next key after a single row would win if it were seen."""
    from gpustack_b200 import ops

    dtype = torch.float32 if route == "generic32" else BF
    n, cap = 400, 20.0
    q, k, v = torch.ones(n, H, W), _rnd(n, G, W, seed=1, scale=0.05), _rnd(n, G, W, seed=2, scale=0.01)
    k[far], v[far] = 1.0, 5.0
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    scale = 30.0 / W                                                  # score 30 -> capped to 20 tanh(1.5) = 18.1
    want = O.capped_attention(q.to(F64), k.to(F64), v.to(F64), scale, cap)
    assert float(want[far:].min()) > 4.9 and (far == 0 or float(want[:far].max()) < 0.1)
    kc, vc, bt = _paged(k, v, G, W, W, dtype, seed=3)
    rows, zero = q.reshape(n, H * W).cuda(), torch.zeros(H, device="cuda")
    for start in sorted({0, max(0, far - 1), far, min(n - 2, far + 1), 390}):
        tile = ops.attn_prefill_tile(H, G) if route == "tc" else 16
        ts, tq = (_i32(t) for t in ops.build_prefill_tiles([n - start], tile, [start]))
        out = torch.zeros(n - start, H * W, dtype=dtype, device="cuda")
        args = (kc, vc, bt, _i32([0, n - start]), _i32([start]), ts, tq)
        if route == "tc":
            ops.paged_attn_prefill_ex(rows[start:], H * W, *args, out, H, G, W, scale, sink=zero, softcap=cap)
        else:
            ops.attn_sink_prefill(rows[start:], -1, *args, zero, out, H, G, W, W, scale, tile_rows=tile, softcap=cap)
        assert float((out.view(-1, H, W).cpu().to(F64) - want[start:]).abs().max()) < (1e-4 if dtype == torch.float32 else 5e-2)
    lens = [m for m in (far, far + 1, far + 2, n) if 1 <= m <= n]
    one, btb, od = rows[:len(lens)].contiguous(), bt.repeat(len(lens), 1), torch.zeros(len(lens), H * W, dtype=dtype, device="cuda")
    if route.startswith("generic"):
        ops.attn_sink_decode(one, -1, kc, vc, btb, _i32(lens), zero, od, H, G, W, W, scale, softcap=cap)
    else:
        ws = ops.attn_decode_workspace(len(lens), H, W, 4, "cuda")
        ops.paged_attn_decode(one, H * W, kc, vc, btb, _i32(lens), od, H, G, W, scale, num_splits=4, workspace=ws, sink=zero, softcap=cap)
    assert float((od.view(-1, H, W).cpu().to(F64) - want[[m - 1 for m in lens]]).abs().max()) < (1e-4 if dtype == torch.float32 else 5e-2)


@pytest.mark.parametrize("E,top", [(1, 1), (5, 3), (8, 8), (33, 4), (70, 2), (256, 16)])
def test_routing_by_chosen_logits(E, top):
    """The bias takes part in the choice and in the weights; logits hundreds apart, where a softmax over all outputs would
    leave nothing of the smaller ones, are still ranked and weighted."""
    from gpustack_b200 import ops
    from gpustack_b200.lib import check, load

    T = 50
    z, b = _rnd(T, E, seed=E, scale=3.0), _rnd(E, seed=E + 1, scale=3.0)
    z[10:20] *= 60.0
    idx, wt = O.route((z + b).to(F64), top)
    lg = torch.full((T, E + 3), 1e4, device="cuda")                    # columns behind the outputs are no candidates
    lg[:, :E] = z.cuda()
    ids, w = _i32([0] * (T * top)), torch.zeros(T * top, device="cuda")
    check(load().b200_moe_route_scored(lg.data_ptr(), lg.stride(0), b.cuda().data_ptr(), ids.data_ptr(), w.data_ptr(), T, E, top, 1.0, 2, 1,
                                       torch.cuda.current_stream().cuda_stream))
    torch.cuda.synchronize()
    assert torch.equal(ids.view(T, top).cpu().long(), idx)
    assert float((w.view(T, top).cpu().to(F64) - wt).abs().max()) < 1e-6


@pytest.mark.parametrize("D,ff,fs,E,top,dtype", [(51, 18, 22, 5, 3, torch.float32), (52, 18, 22, 5, 3, BF), (256, 256, 128, 6, 2, BF),
                                                  (256, 512, 64, 3, 1, BF), (256, 64, 64, 12, 3, BF), (256, 256, 128, 6, 2, torch.float32),
                                                  (128, 48, None, 4, 2, torch.float32)])
@pytest.mark.parametrize("T", [1, 7, 150])
def test_relu2_experts_with_a_gated_shared_one_and_the_norm_behind_them(D, ff, fs, E, top, dtype, T):
    """Router, choice, expert products (CUDA-core and tensor-core routes), shared expert and its gate, combine + norm + sum."""
    from gpustack_b200 import ops

    mlp = _moe(E, top, ff, fs)
    cfg = {"architecture": "Kerarax", "vocab": 3, "width": D, "norm": {"eps": 1e-5}, "logit_softcap": 1.0, "layers": [_layer(1, 1, 8, 8, 1, mlp)]}
    W = {k[len("l0.mlp."):]: v for k, v in O.random_weights(cfg, seed=D + E).items() if k.startswith("l0.mlp.")}
    W["router"] = (W["router"].float() * 4).to(BF)                     # decided choices
    x = _rnd(T, D, seed=5).to(dtype)
    want = O.moe_ff(x.to(F64), {k: v.to(F64) for k, v in W.items()}, mlp)
    n_out = E + (fs is not None)
    router = torch.zeros(-(-n_out // 128) * 128, D, dtype=BF)
    router[:E] = W["router"]
    if fs is not None:
        router[E] = W["shared.sg"][0]
    ws = ops.RoutedWorkspace(T, top, n_out, D, ff, dtype, "cuda")
    xc = x.cuda()
    shared = None
    if fs is not None:
        act = torch.zeros(T, fs, dtype=dtype, device="cuda")
        ops.linear(xc, W["shared.up"].cuda(), act, relu2=True)
        shared = ws.shared[:T]
        ops.linear(act, W["shared.down"].cuda(), shared)
    w1 = torch.cat([W[f"e{e}.up"] for e in range(E)]).cuda()
    w2 = torch.cat([W[f"e{e}.down"] for e in range(E)]).cuda()
    ops.routed_experts(xc, router.cuda(), W["router.b"].float().cuda(), w1, w2, ws, None, E, 0, top, 1.0, ff, 0.0, act="relu2",
                       score="chosen_softmax", combine=False)
    pw, pb, x0 = _rnd(D, seed=6, dtype=BF), _rnd(D, seed=7, dtype=BF), _rnd(T, D, seed=8)
    xo = torch.zeros(T, D, device="cuda")
    ops.output_norm_join(x0.cuda(), 1e-5, routed=(ws.yp, ws.pair_row, top, shared, None if fs is None else ws.logits[:T, E]),
                         post=(pw.cuda(), pb.cuda()), x_out=xo)
    ref = x0.to(F64) + O.layer_norm(want, pw.to(F64), pb.to(F64), 1e-5)
    assert _rel(xo, ref) < (1e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("V", [77, 640, 5000])
def test_sampler_caps_the_logits_in_its_pass(V):
    from gpustack_b200 import ops

    z = _rnd(6, V, seed=V, scale=20.0)
    z[2, 5] = 4000.0
    want = O.soft_cap(z.to(F64), 15.0)
    lg = z.cuda().clone()
    got = ops.sample(lg, torch.zeros(6, device="cuda"), _i32([0] * 6), softcap=15.0)
    assert float((lg.cpu().to(F64) - want).abs().max()) < 1e-5
    for i in range(6):
        assert int(got[i]) == int(lg[i].cpu().argmax())
    # a hot row draws from the capped distribution: flat logits of the cap's size leave every token a chance
    lg = torch.full((512, V), 0.0, device="cuda")
    lg[:, 3] = 1e6
    temps = torch.ones(512, device="cuda")
    drawn = ops.sample(lg, temps, _i32(list(range(1, 513))), softcap=1.0)
    share = float((drawn == 3).float().mean())
    assert share < 0.12 and len(set(drawn.tolist())) > 40             # e / (e + V - 1)
    plain = torch.zeros(2, V, device="cuda")
    plain[:, 1] = 100.0
    ops.sample(plain, torch.zeros(2, device="cuda"), _i32([0, 0]))
    assert float(plain[0, 1]) == 100.0                                 # no cap: the logits stay as they are


# ------------------------------------------------------------------------------------ whole models through the engine
def _close(got, want, dtype):
    """float32: every logit to rounding.  bfloat16: rounding may overturn a router's close call, which moves that position by
    more than rounding does, while a fault of the cache, the rings or the batch moves most positions: at most one position in
    twenty may be off, and the typical one is well inside."""
    if dtype == "float32":
        return _rel(got, want) < TOL[dtype]
    want = want.to(torch.float64).numpy() if isinstance(want, torch.Tensor) else np.asarray(want, dtype=np.float64)
    err = np.abs(np.asarray(got, dtype=np.float64) - want).max(axis=1) / np.abs(want).max()
    return float(np.mean(err > TOL[dtype])) <= 0.05 and float(np.median(err)) < TOL[dtype] / 2


@pytest.fixture(scope="module", params=list(CFGS))
def model(request):
    cfg = CFGS[request.param]()
    return cfg, O.random_weights(cfg, seed=3 + len(request.param))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_logits_and_every_layer(model, dtype):
    cfg, W = model
    toks = _tokens(cfg, 70, 1)
    trail = []
    want = O.forward(cfg, W, toks, trace=trail)
    eng = _engine(cfg, W, dtype)
    seen = eng.runner.layer_trace = []
    got = eng.replay_step([("a", toks, list(range(len(toks))))], ["a"])
    eng.runner.layer_trace = None
    assert len(seen) == len(cfg["layers"]) == len(trail)
    for l in range(len(seen)):
        assert _close(seen[l].cpu().numpy(), trail[l], dtype), f"residual stream after layer {l}"
    assert _close(got, want, dtype)
    # the serving path (the last output folded into the final norm) gives the same logits as the traced one
    again = eng.replay_step([("b", toks, list(range(len(toks))))], ["b"])
    assert _rel(again, got) < (1e-6 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_and_single_tokens_match_the_whole_prompt(model, dtype):
    """One prompt, token by token, and portions of changing size down to two tokens (pages of 16, one to six taps: cuts inside
    and at their borders): the logits at a position do not depend on the cut."""
    cfg, W = model
    toks = _tokens(cfg, 90, 2)
    want = O.forward(cfg, W, toks)
    eng = _engine(cfg, W, dtype)
    whole = eng.replay_step([("w", toks, list(range(len(toks))))], ["w"])
    one = np.concatenate([eng.replay_step([("t", toks[i:i + 1], [0])], ["t"] if i == len(toks) - 1 else []) for i in range(len(toks))])
    parts, pos = [], 0
    for c in _cuts(len(toks), [2, 3, 11, 16, 2, 17, 1, 5, 31, 2]):
        parts.append(eng.replay_step([("p", toks[pos:pos + c], list(range(c)))], ["p"] if pos + c == len(toks) else []))
        pos += c
    parts = np.concatenate(parts)
    for got in (whole, one, parts):
        assert _close(got, want, dtype)
    if dtype == "float32":
        assert _rel(one, whole) < 1e-5 and _rel(parts, whole) < 1e-5
    assert eng.sched.pool.num_free == eng.sched.pool.num_total


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_of_unequal_requests_with_reused_pages_and_slots(model, dtype):
    """Five requests of unequal length through four sequence / state slots and too few pages for all of them at once:
    portions of some ride beside single tokens of others, a finished request's pages and rings go to the next one.  Every
    request's logits equal those of the request alone."""
    cfg, W = model
    lens = [61, 9, 120, 33, 47]
    reqs = {f"r{i}": _tokens(cfg, n, 20 + i) for i, n in enumerate(lens)}
    want = {k: O.forward(cfg, W, t).numpy() for k, t in reqs.items()}
    eng = _engine(cfg, W, dtype, blocks=17, seqs=4)     # 16 pages: the five requests need 19, so pages are reused
    at = {k: 0 for k in reqs}
    got = {k: [] for k in reqs}
    plan = [[("r0", 30), ("r1", 2)], [("r0", 1), ("r1", 7), ("r2", 50)], [("r0", 1), ("r2", 17), ("r3", 33)],
            [("r0", 29), ("r2", 1)], [("r2", 1), ("r4", 2)], [("r2", 51), ("r4", 1)], [("r4", 1)], [("r4", 43)]]
    for step in plan:
        entries, end = [], []
        for rid, n in step:
            lo = at[rid]
            entries.append((rid, reqs[rid][lo:lo + n], list(range(n))))
            at[rid] = lo + n
            if at[rid] == len(reqs[rid]):
                end.append(rid)
        out = eng.replay_step(entries, end)
        off = 0
        for rid, n in step:
            got[rid].append(out[off:off + n])
            off += n
    assert all(at[k] == len(reqs[k]) for k in reqs)
    for k in reqs:
        assert _close(np.concatenate(got[k]), want[k], dtype), k
    assert eng.sched.pool.num_free == eng.sched.pool.num_total
    if eng.runner.mcfg.has_state:
        assert eng.sched.slots.num_free == 4
    assert eng.runner.stats.get("mixed_steps", 0) >= 4 and eng.runner.stats["decode_steps"] >= 1


def _random_cfg(rng):
    """A random model: order, head counts, widths (odd and tile-sized), taps, caps, experts and constants all drawn anew."""
    D = rng.choice([47, 48, 64, 96, 128, 192, 256, 320])
    layers = []
    for _ in range(rng.randint(2, 5)):
        G = rng.choice([1, 2, 3, 4])
        H = G * rng.choice([1, 2, 3, 4, 8])
        dk, dv = rng.choice([8, 16, 20, 24, 32, 64, 80, 128, 144]), rng.choice([8, 12, 16, 32, 40, 64, 128])
        E = rng.choice([1, 2, 3, 6, 17])
        mlp = _moe(E, rng.randint(1, min(E, 5)), rng.choice([16, 24, 64, 96, 128, 256]), rng.choice([None, 8, 40, 64, 200]))
        layers.append(_layer(H, G, dk, dv, rng.choice([1, 2, 3, 4, 5, 8]), mlp if rng.random() < 0.85 else None,
                             scale=rng.choice([dk ** -0.5, 0.2, 0.7]), cap=rng.choice([2.0, 15.0, 30.0, 50.0])))
    return {"architecture": "Kerarax", "vocab": rng.choice([100, 257, 1000]), "width": D, "norm": {"eps": rng.choice([1e-5, 1e-6])},
            "logit_softcap": rng.choice([2.0, 10.0, 30.0, 100.0]), "layers": layers}


@pytest.mark.parametrize("seed,dtype", [(s, "float32") for s in range(201, 209)] + [(s, "bfloat16") for s in range(211, 215)])
def test_random_configurations(seed, dtype):
    """Whole prompt, and two requests in portions beside single tokens, against the oracle."""
    rng = random.Random(seed)
    cfg = _random_cfg(rng)
    W = O.random_weights(cfg, seed=seed)
    t1, t2 = _tokens(cfg, 150, seed), _tokens(cfg, 70, seed + 1)
    w1, w2 = O.forward(cfg, W, t1), O.forward(cfg, W, t2)
    eng = _engine(cfg, W, dtype, blocks=20)

    def ok(got, want):
        if dtype == "float32":
            return _rel(got, want) < TOL[dtype]
        err = np.abs(got - want.numpy()).max(axis=1) / np.abs(want.numpy()).max()     # (many experts: close calls)
        return float(np.median(err)) < TOL[dtype]

    assert ok(eng.replay_step([("a", t1, list(range(150)))], ["a"]), w1)
    toks, at, got = {"x": t1, "y": t2}, {"x": 0, "y": 0}, {"x": [], "y": []}
    for step in ([("x", 37), ("y", 2)], [("x", 2), ("y", 30)], [("x", 1), ("y", 1)], [("x", 64), ("y", 1)], [("x", 1), ("y", 36)], [("x", 45)]):
        entries, end = [], []
        for rid, n in step:
            entries.append((rid, toks[rid][at[rid]:at[rid] + n], list(range(n))))
            at[rid] += n
            if at[rid] == len(toks[rid]):
                end.append(rid)
        out, off = eng.replay_step(entries, end), 0
        for rid, n in step:
            got[rid].append(out[off:off + n])
            off += n
    assert ok(np.concatenate(got["x"]), w1) and ok(np.concatenate(got["y"]), w2)
    assert eng.sched.pool.num_free == eng.sched.pool.num_total


@pytest.mark.parametrize("name,dtype", [("odd", "float32"), ("wide", "bfloat16")])
def test_long_decoding_through_the_graphs(name, dtype):
    """300 single-token steps after a short prompt through the captured decode graphs: the rings pass through 300 updates, the
    decode kernels walk 20 pages."""
    cfg = CFGS[name]()
    W = O.random_weights(cfg, seed=5)
    toks = _tokens(cfg, 320, 9)
    want = O.forward(cfg, W, toks)
    eng = _engine(cfg, W, dtype)
    out = [eng.replay_step([("a", toks[:20], list(range(20)))], [])]
    for i in range(20, len(toks)):
        out.append(eng.replay_step([("a", toks[i:i + 1], [0])], ["a"] if i == len(toks) - 1 else []))
    assert _close(np.concatenate(out), want, dtype)
    assert eng.runner.stats["graph_replays"] >= 290


def test_a_model_whose_far_token_decides_the_logits():
    """Weights that make one early token the only thing attention answers to: its embedding is large and every query points at
    its key, so the logits 300 positions later change with it -- in the oracle and in the engine alike, whole, in portions
    and decoded."""
    cfg = {"architecture": "Kerarax", "vocab": 40, "width": 64, "norm": {"eps": 1e-6}, "logit_softcap": 10.0,
           "layers": [_layer(2, 1, 32, 24, 2, None, scale=0.8, cap=25.0)]}
    W = O.random_weights(cfg, seed=1)
    u = torch.ones(64)
    W["embed"] = (_rnd(40, 64, seed=2, scale=0.3)).to(BF)
    W["embed"][7] += u * torch.tensor([1.0, -1.0]).repeat(32) * 4          # token 7 points one way, with no mean
    key = torch.tensor([1.0, -1.0]).repeat(32) / 8
    W["l0.mix.k"] = (torch.outer(torch.ones(32), key) + 0.05 * _rnd(32, 64, seed=3)).to(BF)
    W["l0.mix.q"] = (torch.outer(torch.ones(64), torch.ones(64) * 0) + 0.2 * _rnd(64, 64, seed=4).abs()).to(BF)
    base = [t if t != 7 else 8 for t in _tokens(cfg, 310, 5)]
    spiked = list(base)
    spiked[3] = 7
    wa, wb = O.forward(cfg, W, base), O.forward(cfg, W, spiked)
    moved = float((wa[250:] - wb[250:]).abs().max())
    assert moved > 0.05                                                # the early token shows 300 positions later
    eng = _engine(cfg, W, "float32", mbt=320)
    for toks, want in ((base, wa), (spiked, wb)):
        got = eng.replay_step([("w", toks, list(range(310)))], ["w"])
        assert _rel(got, want) < TOL["float32"]
        parts, pos = [], 0
        for c in _cuts(280, [50, 2, 77]) + [1] * 30:
            parts.append(eng.replay_step([("p", toks[pos:pos + c], list(range(c)))], ["p"] if pos + c == 310 else []))
            pos += c
        assert _rel(np.concatenate(parts), want) < TOL["float32"]


@pytest.mark.parametrize("name,dtype,eager", [("odd", "float32", True), ("tiles", "bfloat16", False), ("plain", "bfloat16", False),
                                              ("wide", "bfloat16", False)])
def test_greedy_generation_through_the_scheduler(name, dtype, eager):
    """LLMEngine.generate: continuous batching of six prompts over four sequence and state slots, chunked prefill
    (token budget 48), decode steps.  The oracle is teacher-forced on the engine's tokens; wherever its top-2 margin
    is decisive the engine's token is its argmax."""
    from gpustack_b200.scheduler import SamplingParams

    cfg = CFGS[name]()
    W = O.random_weights(cfg, seed=8)
    prompts = [_tokens(cfg, n, 40 + n) for n in (5, 70, 23, 1, 64, 17)]
    eng = _engine(cfg, W, dtype, blocks=40, seqs=4, mbt=48, eager=eager)
    outs = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    tol = 1e-4 if dtype == "float32" else 4e-2
    checked, wrong = 0, []
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        lg = O.forward(cfg, W, p + o)
        for t in range(12):
            row = lg[len(p) - 1 + t]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) > tol * float(row.abs().max()):
                checked += 1
                if int(row.argmax()) != o[t]:
                    wrong.append((len(p), t))
    # (bf16: a router's close call may flip and move one position by more than the margin)
    assert checked >= 40 and len(wrong) <= (0 if dtype == "float32" else 2), wrong
    assert eng.sched.pool.num_free == eng.sched.pool.num_total
