"""Bovitar (layer-list decoder: pre-norm layers that may share tensors, a gated delta rule, capped rotary attention over
convolved q / k / v beside a state-space recurrence, experts chosen inside the best groups with a shared one) on the GPU
against the plain restatement in oracle/bovitar_oracle.py.

Every test builds its own small configuration and random weights.  Kernel tests compare one mechanism with the
oracle's function; engine tests drive LLMEngine (scheduler pools, state slots, runner step functions, CUDA graphs)
and compare logits with the oracle's whole-sequence forward.  float32 must agree to rounding, bfloat16 to bf16
rounding."""
import random

import numpy as np
import pytest
import torch

from oracle import bovitar_oracle as O

pytestmark = pytest.mark.gpu

F64 = torch.float64
BF = torch.bfloat16


def _delta(H, G, dk, dv, conv, mlp):
    return {"type": "delta", "mixer": {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "conv": conv}, "mlp": mlp}


def _parallel(left, right, mlp):
    """left (H, G, dk, dv, conv, rotated, scale, cap, scaling), right (H, vdim, state, groups, conv, norm_groups)."""
    H, G, dk, dv, conv, dims, scale, cap, scaling = left
    rot = {"dims": dims, "base": 5000.0}
    if scaling:
        rot["scaling"] = scaling
    r = dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right))
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "conv": conv, "rot": rot, "scale": scale,
                               "softcap": cap}, "right": r}}


def _moe(E, top, ff, shared, groups=None, scale=1.0):
    ro = {"experts": E, "top": top, "scale": scale}
    if groups:
        ro["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": ro, "shared": None if shared is None else {"ff": shared}}


def _same(l, j):
    return dict(l, weights_of=j)


def cfg_odd():
    """Nothing is a multiple of 8 and the width is odd: every product takes the CUDA-core path.  Widths that all differ, one
    key head for all and one per head, one to six taps, rotated parts of a head, frequencies on all three branches, a layer
    without feed-forward, one without shared expert, layers that use another's tensors (before and after a third)."""
    sc = {"factor": 3.0, "low": 1.5, "high": 6.0, "original": 90}
    L = [_parallel((3, 1, 10, 14, 3, 6, 1.1, 3.0, sc), (2, 7, 9, 1, 5, 1), _moe(6, 2, 18, 22, (3, 1), 1.7)), _delta(4, 2, 13, 6, 2, None),
         _parallel((4, 2, 6, 70, 1, 6, 0.4, 40.0, None), (6, 5, 33, 3, 2, 5), _moe(5, 3, 10, None)),
         _delta(3, 3, 70, 33, 6, _moe(4, 1, 9, 30, (4, 1), 0.6))]
    return {"architecture": "Bovitar", "vocab": 131, "width": 51, "norm": {"eps": 1e-5}, "logit_scale": 0.7,
            "layers": [L[0], L[1], _same(L[0], 0), L[2], _same(L[1], 1), L[3]]}


def cfg_tiles():
    """Widths that the tensor-core GEMMs take in bf16 (also the grouped ones), heads padded to 64, states of 64 and 128."""
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}
    L = [_delta(4, 2, 64, 32, 3, _moe(8, 3, 128, 64, (2, 1), 2.0)),
         _parallel((4, 1, 64, 40, 4, 32, 0.3, 10.0, sc), (8, 16, 128, 2, 4, 4), _moe(4, 2, 256, 128, (4, 3)))]
    return {"architecture": "Bovitar", "vocab": 256, "width": 256, "norm": {"eps": 1e-6}, "logit_scale": 0.5,
            "layers": [L[0], L[1], _same(L[0], 0), _same(L[1], 1)]}


def cfg_plain():
    """Values a model may happen to make trivial: one tap, one head, one group, one expert, key and value widths alike, the
    whole head rotated, no scaling, one norm group, a logit scale of one; no shared tensors."""
    return {"architecture": "Bovitar", "vocab": 77, "width": 40, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "layers": [_parallel((1, 1, 8, 8, 1, 8, 0.35, 30.0, None), (1, 8, 8, 1, 1, 1), _moe(1, 1, 16, 16, (1, 1))),
                       _delta(1, 1, 16, 16, 1, _moe(2, 2, 8, 24))]}


def cfg_delta_only():
    """No attention at all: no pages are read, every layer is a recurrence."""
    return {"architecture": "Bovitar", "vocab": 90, "width": 64, "norm": {"eps": 1e-6}, "logit_scale": 2.0,
            "layers": [_delta(6, 2, 24, 40, 4, _moe(6, 2, 64, 64, (3, 2))), _delta(2, 1, 136, 20, 3, None)]}


def cfg_wide():
    """128-wide heads, as they are and padded from either side, in groups of four (tcgen05 prefill, split-KV decode) and
    of eight; caps on both sides of the bound that lets the softmax do without a running maximum."""
    sc = {"factor": 2.0, "low": 1.0, "high": 3.0, "original": 40}
    L = [_parallel((8, 2, 128, 96, 4, 64, 0.2, 25.0, sc), (4, 64, 128, 1, 4, 2), _moe(4, 2, 256, 256)),
         _parallel((8, 1, 96, 128, 3, 96, 0.1, 90.0, None), (2, 128, 64, 2, 3, 1), None), _delta(2, 2, 128, 128, 4, _moe(3, 1, 256, 64))]
    return {"architecture": "Bovitar", "vocab": 256, "width": 256, "norm": {"eps": 1e-5}, "logit_scale": 0.3,
            "layers": [L[0], L[1], L[2], _same(L[0], 0)]}


CFGS = {"odd": cfg_odd, "tiles": cfg_tiles, "plain": cfg_plain, "delta_only": cfg_delta_only, "wide": cfg_wide}


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


TOL = 5e-5                                 # 32-bit logits against the oracle's


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


# Steps of (prompt portions, then single rows) that carry sequences a (83), b (60) and c (15) from start to end; c takes a's
# slot and ring afterwards, without any clearing
LENS = {"a": 83, "b": 60, "c": 15}
SLOT = {"a": 1, "b": 0, "c": 1}
PLAN = [([("a", 9)], [("b", 1)]), ([("b", 2)], [("a", 1)]), ([("a", 2)], [("b", 1)]), ([("b", 5), ("a", 3)], []), ([], [("a", 1), ("b", 1)]),
        ([("a", 37), ("b", 17)], []), ([("b", 33), ("a", 30)], []), ([], [("c", 1)]), ([("c", 1)], []), ([("c", 2)], []), ([("c", 11)], [])]


def _steps(tile=32):
    """Every step of PLAN as (entries with their first position, cu, ctx, slots, tiles, portions, singles)."""
    from gpustack_b200 import ops

    at = {n: 0 for n in LENS}
    for prompts, singles in PLAN:
        step = [(n, m, at[n]) for n, m in prompts + singles]
        ts = tq = None
        if prompts:
            ts, tq = (_i32(t) for t in ops.build_prefill_tiles([m for _, m in prompts], tile, [at[n] for n, _ in prompts]))
        cu = np.cumsum([0] + [m for _, m, _ in step]).tolist()
        yield step, cu, _i32(cu), _i32([p for _, _, p in step]), _i32([SLOT[n] for n, _, _ in step]), ts, tq, len(prompts), len(singles)
        for n, m, _ in step:
            at[n] += m
    assert at == LENS


# ------------------------------------------------------------------------------------ mechanisms, one at a time
REC = [  # segments (heads, width, factor of the unit norm or None), taps, bias, dtype
    (((2, 10, 0.3), (2, 10, 1.0), (3, 14, None)), 3, False, torch.float32), (((2, 64, 0.125), (2, 64, 1.0), (4, 32, None)), 4, False, BF),
    (((4, 16, None), (1, 24, None), (1, 24, None)), 4, True, BF), (((3, 7, None), (1, 9, None), (1, 9, None)), 5, True, torch.float32),
    (((1, 136, 0.1), (1, 136, 1.0), (2, 20, None)), 2, False, torch.float32), (((5, 40, 1.0), (5, 40, 2.0), (5, 8, None)), 1, False, BF),
    (((2, 200, 1.0), (2, 200, 1.0), (2, 264, None)), 8, False, BF), (((2, 128, 1.0), (2, 128, 1.0), (2, 128, None)), 2, False, torch.float32)]


@pytest.mark.parametrize("segs,taps,biased,dtype", REC)
def test_recurrence_inputs_in_portions_with_rings_that_are_used_again(segs, taps, biased, dtype):
    """Convolution, silu and unit norms over portions of 1 .. 37 rows that ride in the same launches, rings in shuffled slots;
    the rows equal those of the whole sequence, and the columns behind a head's own are zeros."""
    from gpustack_b200 import ops

    C = sum(h * w for h, w, _ in segs)
    cw, cb = _rnd(taps, C, seed=1, scale=0.6), _rnd(C, seed=2) if biased else None
    seqs = {n: _rnd(m, C, seed=4 + i).to(dtype) for i, (n, m) in enumerate(LENS.items())}
    wides = [-(-w // 4) * 4 for _, w, _ in segs]
    W = sum(h * p for (h, _, _), p in zip(segs, wides))
    ring = torch.full((2, taps - 1, C), 7.0, device="cuda") if taps > 1 else None
    got = {n: [] for n in seqs}
    for step, cu, cu_d, ctx, slots, ts, tq, n_p, n_s in _steps():
        rows = torch.cat([seqs[n][p:p + m] for n, m, p in step])
        wide = torch.full((rows.shape[0], 8 + -(-C // 8) * 8), 9.0, dtype=dtype, device="cuda")
        wide[:, 8:8 + C] = rows.cuda()                                 # the convolved channels start at a column of their own
        out = torch.full((rows.shape[0], W + 4), 5.0, device="cuda")
        ops.conv_rec_prep(wide[:, 8:], cw.cuda(), None if cb is None else cb.cuda(), ring, cu_d, ctx, slots, ts, tq, 32, n_p, n_s, segs, out)
        assert float(out[:, W:].min()) == 5.0                          # nothing behind the row
        for (n, m, _), o in zip(step, cu):
            got[n].append(out[o:o + m, :W].cpu())
    for n, u in seqs.items():
        y = O.silu(O.causal_conv(u.to(F64), cw.t().to(F64), None if cb is None else cb.to(F64)))
        g, c, o = torch.cat(got[n]), 0, 0
        for (h, w, unit), p in zip(segs, wides):
            ref = y[:, c:c + h * w].view(-1, h, w)
            ref = ref if unit is None else O.unit(ref) * unit
            mine = g[:, o:o + h * p].view(-1, h, p)
            assert _rel(mine[..., :w], ref) < 3e-6 and not mine[..., w:].any(), (n, w)
            c, o = c + h * w, o + h * p
    if ring is not None:
        for n, s in (("b", 0), ("c", 1)):
            for p in range(LENS[n] - taps + 1, LENS[n]):
                assert torch.equal(ring[s, p % (taps - 1)].cpu(), seqs[n][p].float())


PREP = [  # H, G, dk, dv, wk, wv, taps, rotated, half layout, joint, dtype
    (3, 1, 10, 14, 10, 14, 3, 6, True, True, torch.float32), (3, 1, 10, 14, 64, 64, 3, 6, True, True, BF),
    (4, 2, 16, 8, 16, 8, 4, 16, True, True, torch.float32), (4, 2, 64, 40, 64, 64, 4, 32, True, True, BF),
    (2, 2, 128, 96, 128, 128, 2, 128, True, True, BF), (8, 1, 96, 128, 128, 128, 1, 96, True, True, BF),
    (20, 4, 128, 128, 128, 128, 4, 64, True, True, BF), (5, 5, 24, 24, 24, 24, 3, 24, False, True, BF),
    (2, 1, 13, 7, 13, 7, 7, 4, True, True, torch.float32), (2, 1, 40, 24, 64, 64, 8, 40, False, True, BF),
    (6, 3, 32, 64, 32, 64, 1, 16, True, False, torch.float32), (4, 2, 24, 24, 64, 64, 2, 8, False, False, BF),
    (2, 1, 160, 140, 160, 140, 3, 100, True, True, torch.float32), (3, 3, 16, 16, 16, 16, 2, 0, True, True, BF)]


@pytest.mark.parametrize("H,G,dk,dv,wk,wv,taps,dims,half,joint,dtype", PREP)
def test_attention_inputs_normed_over_the_whole_projection_and_rotated(H, G, dk, dv, wk, wv, taps, dims, half, joint, dtype):
    """Convolution, norm (over all heads at once, or per head), rotation, pages: portions of 1 .. 37 rows and single rows with
    rings and pages in shuffled slots equal the whole sequence; columns behind the heads' own are zeros."""
    from gpustack_b200 import ops

    C, eps, page = (H + G) * dk + G * dv, 1e-5, 16
    cw = _rnd(taps, C, seed=1, scale=0.6)
    qn, kn = (_rnd(n * dk if joint else dk, seed=2 + n, dtype=BF) + 1 for n in (H, G))
    rot = {"dims": dims, "base": 300.0}
    freq = torch.tensor(O.scaled_frequencies(rot), dtype=F64, device="cuda")
    seqs = {n: _rnd(m, C, seed=14 + i).to(dtype) for i, (n, m) in enumerate(LENS.items())}

    def turn(x):
        if not dims:
            return x
        if half:
            return O.rotate_half(x, torch.arange(x.shape[0]), rot)
        perm = list(range(0, dims, 2)) + list(range(1, dims, 2)) + list(range(dims, dk))     # pairs (2i, 2i + 1) side by side
        out = torch.empty_like(x)
        out[..., perm] = O.rotate_half(x[..., perm], torch.arange(x.shape[0]), rot)
        return out

    want = {}
    for n, u in seqs.items():
        y = O.causal_conv(u.to(F64), cw.t().to(F64))
        q, k, v = torch.split(y, [H * dk, G * dk, G * dv], dim=-1)
        if joint:
            q, k = O.rms(q, eps) * qn.to(F64), O.rms(k, eps) * kn.to(F64)
        q, k = q.reshape(-1, H, dk), k.reshape(-1, G, dk)
        if not joint:
            q, k = O.rms(q, eps) * qn.to(F64), O.rms(k, eps) * kn.to(F64)
        want[n] = (turn(q), turn(k), v.reshape(-1, G, dv))
    ring = torch.full((2, taps - 1, C), 7.0, device="cuda") if taps > 1 else None
    kc = torch.full((20, G, page, wk), 9.0, dtype=dtype, device="cuda")
    vc = torch.full((20, G, page, wv), 9.0, dtype=dtype, device="cuda")
    tables = {"a": [7, 3, 12, 1, 9, 15], "b": [2, 14, 5, 10], "c": [6]}
    got = {n: [] for n in seqs}
    for step, cu, cu_d, ctx, slots, ts, tq, n_p, n_s in _steps():
        rows = torch.cat([seqs[n][p:p + m] for n, m, p in step])
        wide = torch.zeros(rows.shape[0], -(-C // 8) * 8 + 8, dtype=dtype, device="cuda")
        wide[:, :C] = rows.cuda()
        where = [tables[n][p // page] * page + p % page for n, m, p0 in step for p in range(p0, p0 + m)]
        qo = torch.full((rows.shape[0], H * wk), 5.0, dtype=dtype, device="cuda")
        pos = _i32([p for _, m, p0 in step for p in range(p0, p0 + m)])
        cs = ops.rot_table(pos, freq, torch.zeros(len(pos), dims // 2, 2, device="cuda")) if dims else None
        ops.conv_attn_prep(wide, cw.cuda(), qn.cuda(), kn.cuda(), ring, cu_d, ctx, slots, ts, tq, 32, n_p, n_s, _i32(where), qo, kc, vc, H, G,
                           dk, dv, eps, joint_norm=joint, rot_dims=dims, half_layout=half, cos_sin=cs)
        for (n, m, _), o in zip(step, cu):
            got[n].append(qo[o:o + m].cpu())
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    for n in seqs:
        q = torch.cat(got[n]).view(-1, H, wk)
        assert _rel(q[..., :dk], want[n][0]) < tol and not q[..., dk:].any(), n
        if n == "a":
            continue
        for cache, w, ref, width in ((kc, wk, want[n][1], dk), (vc, wv, want[n][2], dv)):
            r = torch.stack([cache[tables[n][p // page], :, p % page] for p in range(LENS[n])]).cpu()
            assert _rel(r[..., :width], ref) < tol and not r[..., width:].any(), n
    for b in set(range(20)) - {t for tb in tables.values() for t in tb}:
        assert float(kc[b].float().min()) == 9.0                       # nobody else's page was touched
    if ring is not None:
        for n, s in (("b", 0), ("c", 1)):
            for p in range(LENS[n] - taps + 1, LENS[n]):
                assert torch.equal(ring[s, p % (taps - 1)].cpu(), seqs[n][p].float())


@pytest.mark.parametrize("position", [0, 1, 4095, 131071, 1000003])
def test_rotation_far_from_the_start(position):
    """A single row at a large position: the angle is formed and reduced before it is rounded to 32 bits."""
    from gpustack_b200 import ops

    H, G, dk = 2, 1, 32
    rot = {"dims": 32, "base": 20.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}}
    u = _rnd(1, (H + 2 * G) * dk, seed=1)
    one = torch.ones(H * dk, dtype=BF, device="cuda")
    q, kc, vc = torch.zeros(1, H * dk, device="cuda"), *(torch.zeros(1, G, 16, dk, device="cuda") for _ in range(2))
    freq = torch.tensor(O.scaled_frequencies(rot), dtype=F64, device="cuda")
    ops.conv_attn_prep(u.cuda(), torch.ones(1, u.shape[1], device="cuda"), one, one[:G * dk], None, _i32([0, 1]), _i32([position]), _i32([0]), None,
                       None, 16, 0, 1, _i32([3]), q, kc, vc, H, G, dk, dk, 0.0, joint_norm=True, rot_dims=32, half_layout=True,
                       cos_sin=ops.rot_table(_i32([position]), freq, torch.zeros(1, 16, 2, device="cuda")))
    x = O.rms(u[:, :H * dk].to(F64), 0.0).view(1, H, dk)
    assert _rel(q.view(1, H, dk), O.rotate_half(x, torch.tensor([position]), rot)) < 2e-6


SCAN = [(4, 2, 10, 14), (3, 3, 33, 6), (2, 1, 64, 40), (6, 2, 96, 32), (2, 2, 128, 70), (1, 1, 7, 1), (2, 1, 136, 20), (1, 1, 300, 9)]


def _scan_case(H, G, dk, dv, T, seed):
    r = lambda *s, i=0, k=1.0: _rnd(*s, seed=seed * 10 + i, scale=k)   # noqa: E731
    q, k, v = O.unit(r(T, G, dk, i=1)), O.unit(r(T, G, dk, i=2)), r(T, H, dv, i=3)
    return q, k, v, r(T, H, i=4), r(T, H, i=5, k=2.0)


@pytest.mark.parametrize("H,G,dk,dv", SCAN)
@pytest.mark.parametrize("delta", [True, False])
def test_scans_in_portions_with_slots_that_are_used_again(H, G, dk, dv, delta):
    """Both recurrences over portions of 1 .. 37 rows and single rows that ride in the same launches, states in shuffled
    slots; a third sequence starts from zero in the first one's slot."""
    from gpustack_b200 import ops

    rate, bias, skip = torch.exp(_rnd(H, seed=1) - 1.0), _rnd(H, seed=2) - 1.0, _rnd(H, seed=3)
    kp, vp = -(-dk // 4) * 4, -(-dv // 4) * 4
    W = 2 * G * kp + H * vp
    S = torch.full((2, H, dv, kp), 3.0, device="cuda")
    S[..., dk:] = 0.0
    cases = {n: _scan_case(H, G, dk, dv, m, i + 1) for i, (n, m) in enumerate(LENS.items())}
    got = {n: [] for n in cases}
    for step, cu, cu_d, ctx, slots, ts, tq, n_p, n_s in _steps():
        T = cu[-1]
        x, gates = torch.zeros(T, W + 4, device="cuda"), torch.full((T, 2 * H + 3), 50.0, device="cuda")
        for (n, m, p), o in zip(step, cu):
            q, k, v, a, b = (t[p:p + m].cuda() for t in cases[n])
            x[o:o + m, :G * kp].view(m, G, kp)[..., :dk] = k
            x[o:o + m, G * kp:2 * G * kp].view(m, G, kp)[..., :dk] = q
            x[o:o + m, 2 * G * kp:W].view(m, H, vp)[..., :dv] = v
            if delta:
                gates[o:o + m, :H], gates[o:o + m, H:2 * H] = b, a
            else:
                gates[o:o + m, :H] = a
        out = torch.full((T, H * dv), 9.0, device="cuda")
        ops.gated_scan(x, G * kp, 0, 2 * G * kp, gates, rate.cuda(), bias.cuda(), None if delta else skip.cuda(), cu_d, ctx, slots, S, out, H, G,
                       dk, dv, delta, max_len=max(m for _, m, _ in step))
        for (n, m, _), o in zip(step, cu):
            got[n].append(out[o:o + m].view(m, H, dv).cpu())
    for n, c in cases.items():
        q, k, v, a, b = (t.to(F64) for t in c)
        sp = O.softplus(a + bias.to(F64))
        if delta:
            want = O.delta_scan(q, k, v, torch.exp(-rate.to(F64) * sp), torch.sigmoid(b))
        else:
            want = O.ssd_scan(v, k, q, sp, torch.log(rate.to(F64)), skip.to(F64))
        assert _rel(torch.cat(got[n]), want) < 5e-6, n
    assert not S[..., dk:].any()                                       # columns behind dk stay zero


@pytest.mark.parametrize("delta", [True, False])
def test_one_early_write_is_still_read_a_thousand_tokens_later(delta):
    """A state that hardly decays: one token's value is 100, all others are small; a query along that token's key reads it
    back at the end -- whole, in portions, token by token -- and an erased one (the delta rule writes zero there) not."""
    from gpustack_b200 import ops

    H = G = 1
    dk, dv, T, mark = 16, 8, 1000, 137
    k = torch.zeros(T, 1, dk)
    k[:, 0, 1:] = O.unit(_rnd(T, dk - 1, seed=1))
    k[mark, 0] = 0.0
    k[mark, 0, 0] = 1.0
    v = _rnd(T, 1, dv, seed=2, scale=0.01)
    v[mark] = 100.0
    erase = {False: v, True: v.clone()}
    ke = k.clone()
    ke[700, 0] = ke[mark, 0]
    erase[True][700] = 0.0
    q = torch.zeros(T, 1, dk)
    q[:, 0, 0] = 1.0
    a = torch.full((T, 1), -8.0)                       # softplus about 3e-4
    for gone in ((False, True) if delta else (False,)):
        kk, vv = (ke if gone else k), erase[gone]
        sp = O.softplus(a.to(F64))
        if delta:
            b = torch.full((T, 1), 9.0)
            want = O.delta_scan(q.to(F64), kk.to(F64), vv.to(F64), torch.exp(-0.1 * sp), torch.sigmoid(b.to(F64)))
        else:
            b = None
            want = O.ssd_scan(vv.to(F64), kk.to(F64), q.to(F64), sp, torch.log(torch.tensor([0.1], dtype=F64)), torch.zeros(1, dtype=F64))
        last = float(want[-1].abs().max())
        assert (last < 0.1) if gone else (last > (50.0 if delta else 0.02))
        x = torch.cat([q.view(T, dk), kk.view(T, dk), vv.view(T, dv)], 1).cuda()
        gates = (torch.cat([b, a], 1) if delta else a).cuda()
        for cuts in ([T], _cuts(T, [100, 2, 17, 16, 1]), [T - 40] + [1] * 40):
            S, outs, at = torch.full((1, 1, dv, dk), 7.0, device="cuda"), [], 0
            for m in cuts:
                o = torch.zeros(m, dv, device="cuda")
                ops.gated_scan(x[at:at + m], 0, dk, 2 * dk, gates[at:at + m], torch.full((1,), 0.1, device="cuda"), torch.zeros(1, device="cuda"),
                               None, _i32([0, m]), _i32([at]), _i32([0]), S, o, H, G, dk, dv, delta, max_len=m)
                outs.append(o.cpu())
                at += m
            # (the decay is a 32-bit number just below one: its rounding, up to 2^-25, compounds once per token)
            assert _rel(torch.cat(outs), want.view(T, dv)) < 1e-5 + T * 2.0 ** -25, (gone, len(cuts))


@pytest.mark.parametrize("C,parts", [(48, 1), (48, 3), (35, 5), (512, 2), (640, 10), (1024, 64), (4096, 1), (8192, 64), (5000, 1250)])
@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_gate_before_and_after_the_grouped_norm(C, parts, dtype):
    from gpustack_b200 import ops

    T, z_col = 5, 12
    y, z, w = _rnd(T, C, seed=1), _rnd(T, C + z_col + 4, seed=2).to(dtype), _rnd(C, seed=3, dtype=BF) + 1
    y[:, :C // parts] *= 40.0                                          # parts of very different size
    out = torch.zeros(T, C, dtype=dtype, device="cuda")
    ops.gate_norm(y.cuda(), z.cuda(), z_col, w.cuda(), out, parts, 1e-5)
    want = O.grouped_rms(y.to(F64) * O.silu(z[:, z_col:z_col + C].to(F64)), parts, 1e-5) * w.to(F64)
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    assert _rel(out, want) < tol
    # ... and the norm of every piece, one weight vector for all of them, before the gate
    shared = w[:C // parts].contiguous()
    ops.gate_norm(y.cuda(), z.cuda(), z_col, shared.cuda(), out, parts, 1e-5, gate_after=True)
    want = O.grouped_rms(y.to(F64), parts, 1e-5) * shared.to(F64).repeat(parts) * O.silu(z[:, z_col:z_col + C].to(F64))
    assert _rel(out, want) < tol


@pytest.mark.parametrize("D", [37, 64, 300, 5000])
@pytest.mark.parametrize("hdt", [torch.float32, BF])
def test_join_takes_in_every_kind_of_output(D, hdt):
    """One row, a pair of mixers' outputs each normed first, a routed feed-forward's rows with and without a shared expert;
    in place, for chosen rows only, with the logit scale, and the sum alone."""
    from gpustack_b200 import ops

    T, eps = 9, 1e-5
    x, y, y2 = _rnd(T, D, seed=1), _rnd(T, D, seed=2, scale=3.0), _rnd(T, D, seed=3, scale=0.1)
    w, w1, w2 = (_rnd(D, seed=4 + i, dtype=BF) for i in range(3))
    d, c = (lambda t: t.to(F64)), (lambda t: t.cuda())   # noqa: E731
    forms = [({}, d(x)), ({"y": c(y)}, d(x) + d(y)),
             ({"pair": (c(y), c(y2), c(w1), c(w2), 0.5, 0.25)}, d(x) + 0.5 * O.rms(d(y), eps) * d(w1) + 0.25 * O.rms(d(y2), eps) * d(w2))]
    for K, shared in ((1, True), (3, False), (4, True)):
        yp = _rnd(T * K + 5, D, seed=11)
        pr = torch.randperm(T * K + 5, generator=torch.Generator().manual_seed(K))[:T * K]
        want = d(x) + d(yp)[pr].view(T, K, D).sum(1) + (d(y2) if shared else 0)
        forms.append(({"routed": (c(yp), pr.to(torch.int32).cuda(), K, c(y2) if shared else None)}, want))
    rows = [7, 0, 3]
    tol = 2e-6 if hdt == torch.float32 else 8e-3
    for kw, want in forms:
        xo, ho = torch.zeros(T, D, device="cuda"), torch.zeros(T, D, dtype=hdt, device="cuda")
        ops.prenorm_join(c(x), c(w), eps, x_out=xo, h_out=ho, **kw)
        assert _rel(xo, want) < 2e-6 and _rel(ho, O.rms(want, eps) * d(w)) < tol, list(kw)
        inplace = c(x).clone()
        ops.prenorm_join(inplace, c(w), eps, x_out=inplace, h_out=ho, **kw)
        assert torch.equal(inplace, xo)
        alone = torch.zeros(T, D, device="cuda")
        ops.prenorm_join(c(x), None, eps, x_out=alone, **kw)
        assert torch.equal(alone, xo)
        hg = torch.zeros(3, D, dtype=hdt, device="cuda")
        ops.prenorm_join(c(x), c(w), eps, h_out=hg, rows=_i32(rows), out_scale=0.3, **kw)
        assert _rel(hg, 0.3 * (O.rms(want, eps) * d(w))[rows]) < tol


@pytest.mark.parametrize("E,top,groups", [(8, 3, (4, 2)), (6, 2, (3, 2)), (6, 1, (6, 1)), (12, 6, (2, 1)), (9, 9, None), (1, 1, (1, 1)),
                                          (64, 8, (8, 3)), (250, 16, (25, 4)), (256, 4, (256, 9))])
def test_experts_are_chosen_inside_the_best_groups(E, top, groups):
    """The correction steers groups and choice but not the weights; all corrected scores negative, so that a banned expert
    counted as zero would win."""
    from gpustack_b200 import ops
    from gpustack_b200.lib import check, load

    T = 60
    for shift in (0.0, -3.0):
        z, b = _rnd(T, E, seed=E, scale=2.0), _rnd(E, seed=E + 1, scale=0.2) + shift
        ro = {"experts": E, "top": top, "scale": 1.7}
        if groups:
            ro["groups"] = {"count": groups[0], "keep": groups[1]}
        idx, wt = O.route(z.to(F64), b.to(F64), ro)
        lg = torch.full((T, E + 3), 1e4, device="cuda")                # columns behind the outputs are no candidates
        lg[:, :E] = z.cuda()
        ids, w = _i32([0] * (T * top)), torch.zeros(T * top, device="cuda")
        gn, gk = groups or (0, 0)
        check(load().b200_moe_route_grouped(lg.data_ptr(), lg.stride(0), b.cuda().data_ptr(), ids.data_ptr(), w.data_ptr(), T, E, top, 1.7, 0, 0,
                                            gn, gk, torch.cuda.current_stream().cuda_stream))
        torch.cuda.synchronize()
        assert torch.equal(ids.view(T, top).cpu().long(), idx)
        assert float((w.view(T, top).cpu().to(F64) - wt).abs().max()) < 1e-6
    with pytest.raises(Exception):
        ops.check(load().b200_moe_route_grouped(lg.data_ptr(), lg.stride(0), None, ids.data_ptr(), w.data_ptr(), T, E, top, 1.0, 0, 0, E + 1, 1,
                                                torch.cuda.current_stream().cuda_stream))


@pytest.mark.parametrize("D,ff,fs,E,top,groups,dtype", [(51, 18, 22, 6, 3, (3, 2), torch.float32), (52, 18, 22, 5, 3, None, BF),
                                                         (256, 128, 128, 6, 2, (2, 1), BF), (256, 256, 64, 3, 1, None, BF),
                                                         (256, 64, None, 12, 3, (4, 2), BF), (256, 256, 128, 6, 2, (3, 3), torch.float32)])
@pytest.mark.parametrize("T", [1, 7, 150])
def test_routed_experts_with_a_shared_one(D, ff, fs, E, top, groups, dtype, T):
    """Router, choice, gated products (CUDA-core and tensor-core routes), shared expert, and the sum in the join."""
    from gpustack_b200 import ops
    from gpustack_b200.config import LayerListConfig
    from gpustack_b200.weights import load_layer_list

    mlp = _moe(E, top, ff, fs, groups, 1.3)
    cfg = {"architecture": "Bovitar", "vocab": 3, "width": D, "norm": {"eps": 1e-5}, "logit_scale": 1.0, "layers": [_delta(1, 1, 8, 8, 1, mlp)]}
    W = O.random_weights(cfg, seed=D + E)
    lw = load_layer_list(LayerListConfig.from_dict(cfg), lambda n: W[n], "cuda").layers[0]
    x = _rnd(T, D, seed=5).to(dtype)
    want = O.moe_ff(x.to(F64), {k[len("l0.mlp."):]: v.to(F64) for k, v in W.items() if k.startswith("l0.mlp.")}, mlp)
    ws = ops.RoutedWorkspace(T, top, E, D, ff, dtype, "cuda")
    shared = None
    if fs is not None:
        act, shared = torch.zeros(T, fs, dtype=dtype, device="cuda"), ws.shared[:T]
        ops.gated_linear(x.cuda(), lw.shared13, act, "silu")
        ops.linear(act, lw.shared2, shared)
    gn, gk = groups or (0, 0)
    ops.routed_experts(x.cuda(), lw.router, lw.correction, lw.w13, lw.w2, ws, None, E, 0, top, 1.3, ff, 0.0, act="silu", renormalize=False,
                       combine=False, groups=gn, groups_keep=gk)
    x0 = _rnd(T, D, seed=8)
    xo = torch.zeros(T, D, device="cuda")
    ops.prenorm_join(x0.cuda(), None, 1e-5, routed=(ws.yp, ws.pair_row, top, shared), x_out=xo)
    assert _rel(xo.cpu() - x0, want) < (1e-5 if dtype == torch.float32 else 3e-2)


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
    (3, 1, 10, 14, 10, 14, 3.0, "generic32"), (4, 2, 70, 33, 70, 33, 30.0, "generic32"), (4, 2, 40, 40, 64, 64, 20.0, "decode"),
    (6, 2, 64, 48, 64, 64, 50.0, "decode"), (8, 2, 128, 96, 128, 128, 30.0, "tc"), (8, 1, 96, 128, 128, 128, 90.0, "tc")]


@pytest.mark.parametrize("H,G,dk,dv,wk,wv,cap,route", ATT)
@pytest.mark.parametrize("far", [0, 16, 63, 127, 255])
def test_capped_softmax_without_a_sink_and_one_far_key(H, G, dk, dv, wk, wv, cap, route, far):
    """Capped scores and an ordinary softmax: scores so low that anything else in the denominator would take most of it.  Then
    one key among 300 stands out: rows behind it answer with its value, rows before it and its own future do not."""
    from gpustack_b200 import ops

    dtype = torch.float32 if route == "generic32" else BF
    n, tol = 300, (2e-5 if route == "generic32" else 2e-2)
    for spike in (False, True):
        scale = 3.0 * cap / dk if spike else 1.5 / dk ** 0.5
        if spike:
            q, k, v = torch.ones(n, H, dk), _rnd(n, G, dk, seed=1, scale=0.05), _rnd(n, G, dv, seed=2, scale=0.01)
            k[far], v[far] = 1.0, 5.0
        else:
            q, k, v = _rnd(n, H, dk, seed=1), _rnd(n, G, dk, seed=2), _rnd(n, G, dv, seed=3)
            k[:, :, 0], q[:, :, 0] = -1.0, 0.8 * cap / scale                                # every score far below zero
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        want = O.capped_attention(q.to(F64), k.to(F64), v.to(F64), scale, cap)
        kc, vc, bt = _paged(k, v, G, wk, wv, dtype, seed=4)
        qp = torch.zeros(n, H, wk, dtype=dtype)
        qp[..., :dk] = q
        start = max(0, far - 3)
        rows = qp[start:].reshape(n - start, H * wk).contiguous().cuda()
        tile = ops.attn_prefill_tile(H, G) if route == "tc" else 16
        ts, tq = (_i32(t) for t in ops.build_prefill_tiles([n - start], tile, [start]))
        out = torch.full((n - start, H * wv), 3.0, dtype=dtype, device="cuda")
        args = (kc, vc, bt, _i32([0, n - start]), _i32([start]), ts, tq)
        if route == "tc":
            ops.paged_attn_prefill_ex(rows, rows.stride(0), *args, out, H, G, wk, scale, softcap=cap)
        else:
            ops.attn_sink_prefill(rows, -1, *args, None, out, H, G, wk, wv, scale, tile_rows=tile, softcap=cap)
        got = out.view(-1, H, wv)
        assert _rel(got[..., :dv], want[start:]) < tol and not got[..., dv:].any()
        lens = sorted({m for m in (1, far, far + 1, far + 2, 100, n) if m >= 1})
        one = torch.stack([qp[m - 1] for m in lens]).reshape(len(lens), H * wk).cuda()
        btb, od = bt.repeat(len(lens), 1), torch.full((len(lens), H * wv), 3.0, dtype=dtype, device="cuda")
        if route == "generic32":
            ops.attn_sink_decode(one, -1, kc, vc, btb, _i32(lens), None, od, H, G, wk, wv, scale, softcap=cap)
        else:
            ws = ops.attn_decode_workspace(len(lens), H, wk, 3, "cuda")
            ops.paged_attn_decode(one, one.stride(0), kc, vc, btb, _i32(lens), od, H, G, wk, scale, num_splits=3, workspace=ws, softcap=cap)
        err = od.view(-1, H, wv)[..., :dv].cpu().to(F64) - want[[m - 1 for m in lens]]
        assert float(err.abs().max()) < tol * max(1.0, float(want.abs().max()))


# ------------------------------------------------------------------------------------ whole models through the engine
def _close(got, want, dtype):
    """float32: every logit to rounding.  bfloat16: every position within a tenth, the typical one within a fiftieth."""
    if dtype == "float32":
        return _rel(got, want) < TOL
    want = want.to(torch.float64).numpy() if isinstance(want, torch.Tensor) else np.asarray(want, dtype=np.float64)
    err = np.abs(np.asarray(got, dtype=np.float64) - want).max(axis=1) / np.abs(want).max()
    return float(err.max()) < 0.1 and float(np.median(err)) < 0.02


def _decided(W, dtype):
    """In bfloat16 rounding may overturn a router's close call, and the recurrences carry that position's jump on to all that
    follow.  So the bfloat16 runs get corrections so far apart that every token's choice is decided (the weights, which do not
    use them, still depend on the token); the choice itself is tested in 32-bit and on its own."""
    if dtype == "float32":
        return W
    out = dict(W)
    for n, t in W.items():
        if n.endswith("mlp.correction"):
            out[n] = 1.5 * torch.randperm(t.numel(), generator=torch.Generator().manual_seed(len(n) + t.numel())).to(BF)
    return out


@pytest.fixture(scope="module", params=list(CFGS))
def model(request):
    cfg = CFGS[request.param]()
    return cfg, O.random_weights(cfg, seed=3 + len(request.param))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompt_logits_and_every_layer(model, dtype):
    cfg, W = model[0], _decided(model[1], dtype)
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
    """One prompt, token by token, and portions of changing size down to two tokens (pages and scan chunks of 16, one to six
    taps: cuts inside and at their borders): the logits at a position do not depend on the cut."""
    cfg, W = model[0], _decided(model[1], dtype)
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
        assert _rel(one, whole) < 2e-5 and _rel(parts, whole) < 2e-5
    assert eng.sched.pool.num_free == eng.sched.pool.num_total


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_of_unequal_requests_with_reused_pages_and_slots(model, dtype):
    """Five requests of unequal length through four sequence / state slots and too few pages for all of them at once:
    portions of some ride beside single tokens of others, a finished request's pages, states and rings go to the next one.
    Every request's logits equal those of the request alone."""
    cfg, W = model[0], _decided(model[1], dtype)
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
    assert eng.sched.pool.num_free == eng.sched.pool.num_total and eng.sched.slots.num_free == 4
    assert eng.runner.stats.get("mixed_steps", 0) >= 4 and eng.runner.stats["decode_steps"] >= 1


def _random_cfg(rng):
    """A random model: order, kinds, head counts, widths (odd and tile-sized), taps, caps, groups and constants drawn anew."""
    D = rng.choice([47, 48, 64, 96, 128, 192, 256, 320])
    layers = []
    for _ in range(rng.randint(2, 5)):
        if layers and rng.random() < 0.25:
            j = rng.randrange(len(layers))
            while layers[j].get("weights_of") is not None:
                j = layers[j]["weights_of"]
            layers.append(_same(layers[j], j))
            continue
        gs, n = rng.choice([1, 2, 3, 5]), rng.choice([1, 2, 4])
        keep = rng.randint(1, gs)
        mlp = _moe(gs * n, rng.randint(1, min(keep * n, 6)), rng.choice([16, 24, 64, 96, 128]), rng.choice([None, 8, 40, 64, 200]),
                   rng.choice([None, (gs, keep)]) if keep == gs else (gs, keep), rng.choice([1.0, 2.5]))
        mlp = mlp if rng.random() < 0.85 else None
        G = rng.choice([1, 2, 3])
        H = G * rng.choice([1, 2, 4, 8])
        dk, dv = rng.choice([8, 16, 20, 24, 32, 64, 80, 128, 144]), rng.choice([8, 12, 16, 32, 40, 64, 128])
        if rng.random() < 0.4:
            layers.append(_delta(H, G, dk, dv, rng.choice([1, 2, 3, 4, 5, 8]), mlp))
            continue
        sc = rng.choice([None, {"factor": rng.choice([2.0, 8.0]), "low": 1.0, "high": rng.choice([2.0, 4.0]), "original": rng.choice([32, 100, 2048])}])
        rg = rng.choice([1, 2])
        rh = rg * rng.choice([1, 2, 3])
        p = rng.choice([6, 8, 16, 32, 50, 64])
        ng = rng.choice([g for g in range(1, rh * p + 1) if rh * p % g == 0 and rh * p // g >= 4 and g <= 8])
        layers.append(_parallel((H, G, dk, dv, rng.choice([1, 2, 3, 4, 6]), rng.choice([d for d in (4, 8, 16, 64, dk) if d <= dk]),
                                 rng.choice([dk ** -0.5, 0.2]), rng.choice([2.0, 15.0, 50.0]), sc),
                                (rh, p, rng.choice([5, 8, 16, 40, 64, 128]), rg, rng.choice([1, 2, 3, 4, 7]), ng), mlp))
    return {"architecture": "Bovitar", "vocab": rng.choice([100, 257, 1000]), "width": D, "norm": {"eps": rng.choice([1e-5, 1e-6])},
            "logit_scale": rng.choice([0.1, 1.0, 3.0]), "layers": layers}


@pytest.mark.parametrize("seed,dtype", [(s, "float32") for s in range(301, 313)] + [(s, "bfloat16") for s in range(321, 327)])
def test_random_configurations(seed, dtype):
    """Whole prompt, and two requests in portions beside single tokens, against the oracle."""
    rng = random.Random(seed)
    cfg = _random_cfg(rng)
    W = _decided(O.random_weights(cfg, seed=seed), dtype)
    t1, t2 = _tokens(cfg, 110, seed), _tokens(cfg, 70, seed + 1)
    w1, w2 = O.forward(cfg, W, t1), O.forward(cfg, W, t2)
    eng = _engine(cfg, W, dtype, blocks=20)

    assert _close(eng.replay_step([("a", t1, list(range(110)))], ["a"]), w1, dtype)
    toks, at, got = {"x": t1, "y": t2}, {"x": 0, "y": 0}, {"x": [], "y": []}
    for step in ([("x", 37), ("y", 2)], [("x", 2), ("y", 30)], [("x", 1), ("y", 1)], [("x", 24), ("y", 1)], [("x", 1), ("y", 36)], [("x", 45)]):
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
    assert _close(np.concatenate(got["x"]), w1, dtype) and _close(np.concatenate(got["y"]), w2, dtype)
    assert eng.sched.pool.num_free == eng.sched.pool.num_total


@pytest.mark.parametrize("name,dtype", [("odd", "float32"), ("tiles", "float32"), ("wide", "bfloat16")])
def test_long_decoding_through_the_graphs(name, dtype):
    """300 single-token steps after a short prompt through the captured decode graphs: states and rings pass through 300
    updates, the decode kernels walk 20 pages."""
    cfg = CFGS[name]()
    W = _decided(O.random_weights(cfg, seed=5), dtype)
    toks = _tokens(cfg, 320, 9)
    want = O.forward(cfg, W, toks)
    eng = _engine(cfg, W, dtype)
    out = [eng.replay_step([("a", toks[:20], list(range(20)))], [])]
    for i in range(20, len(toks)):
        out.append(eng.replay_step([("a", toks[i:i + 1], [0])], ["a"] if i == len(toks) - 1 else []))
    assert _close(np.concatenate(out), want, dtype)
    assert eng.runner.stats["graph_replays"] >= 290


def test_a_repeated_layer_keeps_a_state_of_its_own():
    """Two layers on one set of tensors: zeroing ONE of the two layers' states (or pages) between portions changes what
    follows, each differently, and zeroing both differs again -- no layer reads the other's."""
    cfg = cfg_tiles()
    W = O.random_weights(cfg, seed=6)
    toks = _tokens(cfg, 60, 3)
    eng = _engine(cfg, W, "float32")
    assert eng.runner.w.layers[2] is eng.runner.w.layers[0]

    def run(clear):
        eng.replay_step([("a", toks[:40], [])], [])
        for l in clear:
            for t in [s for s in (eng.runner.state[l] or ()) if s is not None] + [c for c in (eng.runner.k_cache[l],) if c is not None]:
                t.zero_()
        return eng.replay_step([("a", toks[40:], list(range(20)))], ["a"])

    base = run([])
    assert _rel(base, O.forward(cfg, W, toks)[40:]) < TOL
    outs = [run(c) for c in ([0], [2], [0, 2], [1], [3], [1, 3])]
    for i, a in enumerate(outs):
        assert _rel(a, base) > 1e-3
        for b in outs[:i]:
            assert _rel(a, b) > 1e-3
    assert np.array_equal(run([]), base)


def test_a_model_whose_far_token_decides_the_logits():
    """One early token is the only thing attention answers to, and the recurrences hardly forget: the logits 300 positions
    later change with it -- in the oracle and in the engine alike, whole, in portions and decoded."""
    cfg = {"architecture": "Bovitar", "vocab": 40, "width": 64, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
           "layers": [_parallel((2, 1, 32, 24, 2, 8, 0.8, 25.0, None), (2, 16, 24, 1, 3, 1), None), _delta(2, 1, 24, 16, 3, None)]}
    W = O.random_weights(cfg, seed=1)
    key = torch.tensor([1.0, -1.0]).repeat(32)
    W["embed"] = _rnd(40, 64, seed=2, scale=0.3).to(BF)
    W["embed"][7] += key * 4                                           # token 7 points one way
    W["l0.mix.left.k"] = (torch.outer(torch.ones(32), key / 8) + 0.05 * _rnd(32, 64, seed=3)).to(BF)
    W["l0.mix.left.q"] = (0.2 * _rnd(64, 64, seed=4).abs()).to(BF)
    for n in ("l0.mix.right.", "l1.mix."):
        W[n + "A_log"] = torch.full_like(W[n + "A_log"], -5.0)         # slow decays
    base = [t if t != 7 else 8 for t in _tokens(cfg, 310, 5)]
    spiked = list(base)
    spiked[3] = 7
    wa, wb = O.forward(cfg, W, base), O.forward(cfg, W, spiked)
    assert float((wa[250:] - wb[250:]).abs().max()) > 0.02             # the early token shows 300 positions later
    eng = _engine(cfg, W, "float32", mbt=320)
    for toks, want in ((base, wa), (spiked, wb)):
        got = eng.replay_step([("w", toks, list(range(310)))], ["w"])
        assert _rel(got, want) < TOL
        parts, pos = [], 0
        for c in _cuts(280, [50, 2, 77]) + [1] * 30:
            parts.append(eng.replay_step([("p", toks[pos:pos + c], list(range(c)))], ["p"] if pos + c == 310 else []))
            pos += c
        assert _rel(np.concatenate(parts), want) < TOL


@pytest.mark.parametrize("name,dtype,eager", [("odd", "float32", True), ("tiles", "bfloat16", False), ("plain", "bfloat16", False),
                                              ("delta_only", "float32", False), ("wide", "bfloat16", False)])
def test_greedy_generation_through_the_scheduler(name, dtype, eager):
    """LLMEngine.generate: continuous batching of six prompts over four sequence and state slots, chunked prefill
    (token budget 48), decode steps.  The oracle is teacher-forced on the engine's tokens; wherever its top-2 margin
    is decisive the engine's token is its argmax."""
    from gpustack_b200.scheduler import SamplingParams

    cfg = CFGS[name]()
    W = _decided(O.random_weights(cfg, seed=8), dtype)
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
    assert checked >= 40 and not wrong, wrong
    assert eng.sched.pool.num_free == eng.sched.pool.num_total
