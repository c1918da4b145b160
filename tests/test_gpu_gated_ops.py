"""Kernels of the gated layer-list decoders, each mechanism alone, against plain PyTorch (B200)."""
from types import SimpleNamespace

import pytest
import torch

from conftest import pkg, rel_err
from oracle import sefalorn_ref as ref

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
TOL = {BF: 1e-2, F32: 2e-5}


def randn(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def status():
    return torch.zeros(64, dtype=torch.int32, device=DEV)


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------- glue


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width,ld", [(192, 192), (204, 256), (2048, 2048), (33, 64), (8100, 8128)])
def test_residual_norm(ops, width, ld, dtype):
    P = pkg("gated").Pending
    M, top = 7, 3

    def padded(*shape, seed, dt=dtype, shift=0.0):
        t = torch.zeros(*shape, ld)
        t[..., :width] = shift + randn(*shape, width, seed=seed)
        return t.to(dt)

    x = padded(M, seed=1, dt=F32) * 3 + torch.arange(M)[:, None] * (torch.arange(ld) < width)  # rows with a mean of their own
    d, w = padded(M, seed=2), padded(seed=4, dt=F32, shift=1.0)
    b, g = padded(seed=5, dt=F32), torch.rand(M, ld, generator=torch.Generator().manual_seed(6)).to(dtype)
    rows, pairs = padded(11, seed=7), torch.randint(-1, 11, (M, top), generator=torch.Generator().manual_seed(8), dtype=torch.int32)
    pw = torch.rand(M, top, generator=torch.Generator().manual_seed(9))
    summed = torch.stack([sum((pw[m, k].double() * rows[pairs[m, k]].double() if pairs[m, k] >= 0 else torch.zeros(ld).double())
                              for k in range(top)) for m in range(M)])
    dv = [t.to(DEV) for t in (d, b, g, rows, pairs, pw, w)]
    D, Bi, G, Ro, Pa, Pw, Wt = dv
    for pend, add in ((None, 0.0), (P(G, dense=D, bias=Bi), (d.double() + b.double()) * g.double()), (P(G, dense=D), d.double() * g.double()),
                      (P(G, expert_rows=Ro, row_of_pair=Pa, pair_weight=Pw), summed * g.double())):
        xg = x.to(DEV)
        for center in (True, False):
            if not center:
                xg = x.to(DEV)
            out = ops.residual_norm(xg, pend, Wt, 1e-3, width, center, dtype=dtype).cpu()
            total = x.double() + add
            assert float((xg.cpu().double() - total).abs().max()) < 1e-4  # the residual stays fp32
            f = ref.layer_norm if center else (lambda a, c, e: ref.rms_unit(a, e) * c)
            assert rel_err(out[:, :width], f(total[:, :width], w.double()[:width], 1e-3)) < TOL[dtype] and not out[:, width:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,D", [(8, 2, 64), (6, 6, 4), (5, 1, 128), (32, 4, 128), (7, 7, 192)])
def test_mix_heads(ops, H, G, D, dtype):
    q, mix = randn(9, H, D, seed=1, dtype=dtype), randn(H, H, seed=2)
    got = ops.mix_heads(q.to(DEV), mix.to(DEV), G).cpu().view(9, H, G, D)
    per = H // G
    want = torch.stack([torch.einsum("hg,mgd->mhd", mix[:, c * per:(c + 1) * per].double(), q[:, c * per:(c + 1) * per].double())
                        for c in range(G)], 2)
    assert rel_err(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("taps", [1, 2, 4, 18, 35])
def test_conv_silu_in_portions_and_decoded(ops, taps, dtype):
    """Any cut of a sequence - portions of every size down to two tokens, decode rows in between, each run twice - gives the
    whole sequence's convolution, whatever the slot's last user left."""
    C, T = 144, 75
    x, w = randn(T, C, seed=5, dtype=dtype), randn(taps, C, seed=6, dtype=dtype)
    want = ref.silu(ref.causal_conv(x.double(), w.double().T.contiguous()))
    xg, wg = x.to(DEV), w.to(DEV)
    for cuts in ([T], [2, 3, 1, 16, 14, 2, 37], [15, 1, 1, 1, 14, 43], [1] * 40 + [35], [31, 2, 42]):
        ring = torch.full((3, taps, C), 9.0, dtype=dtype, device=DEV) if taps > 1 else None
        st, got, at = status(), [], 0
        for n in cuts:
            for _ in range(2 if n == 1 else 1):
                y = ops.conv_silu(xg[at:at + n], wg, ring, torch.full((n,), 1, dtype=torch.int32, device=DEV),
                                  torch.arange(at, at + n, dtype=torch.int32, device=DEV), n > 1, st)
            got.append(y.cpu())
            at += n
        ops.read_status(st, "conv")
        assert rel_err(torch.cat(got), want) < TOL[dtype], (taps, cuts)
        if ring is not None:
            assert bool((ring[[0, 2]] == 9.0).all())
    st = status()
    ops.conv_silu(xg[:1], wg, torch.zeros(3, taps, C, dtype=dtype, device=DEV), i32(3), i32(5), False, st)
    with pytest.raises(RuntimeError):
        ops.read_status(st, "a slot outside the ring")


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("groups,size,ld,shared", [(4, 64, 64, True), (3, 20, 32, True), (1, 1024, 1024, False), (5, 100, 112, False),
                                                   (1, 1500, 1536, False), (2, 1040, 1040, True)])
def test_group_norm_gate(ops, groups, size, ld, shared, dtype):
    o, w = torch.zeros(6, groups, ld), torch.zeros(groups, ld)
    o[..., :size] = randn(6, groups, size, seed=1) * torch.logspace(-2, 2, groups)[None, :, None]  # groups of very different sizes
    w[:, :size] = 1 + 0.3 * randn(groups, size, seed=2)
    g = randn(6, groups, ld, seed=3, dtype=dtype)
    if shared:
        w = w[:1].expand(groups, ld)
    out = torch.full((6, groups * ld + 64), 7.0, dtype=dtype, device=DEV)
    ops.group_norm_gate(o.to(DEV), (w[0] if shared else w).contiguous().view(-1).to(DEV), g.to(DEV).view(6, -1), 1e-4, size, shared, 1.7,
                        out[:, 64:])
    want = ref.rms_unit(o[..., :size].double(), 1e-4) * w[:, :size].double() * g[..., :size].double() * 1.7
    got = out[:, 64:].cpu().view(6, groups, ld)
    assert rel_err(got[..., :size], want) < TOL[dtype] and not got[..., size:].any() and bool((out[:, :64] == 7.0).all())


# -------------------------------------------------------------- attention


def columns(pool):
    """[blocks, heads, 16, D] -> [blocks, heads * D / 64, 16, 64]."""
    nb, G, page, D = pool.shape
    return pool.view(nb, G, page, D // 64, 64).transpose(2, 3).reshape(nb, G * D // 64, page, 64).contiguous()


def attention_case(T, H, G, dk, dv, window, dtype, seed, spare=4):
    """Raw queries, the mixing matrix, mixed queries, keys, values, penalties, and the keys and values in shuffled pages."""
    q = randn(T, H, dk, seed=seed, dtype=dtype)
    talk = (torch.eye(H) + randn(H, H, seed=seed + 5) * 0.3).bfloat16()
    per, scale = H // G, dk ** -0.5
    qm = torch.cat([torch.einsum("hg,tgd->thd", scale * talk[:, c * per:(c + 1) * per].double(), q[:, c * per:(c + 1) * per].double())
                    for c in range(G)], -1)
    k, v = randn(T, G, dk, seed=seed + 1, dtype=dtype), randn(T, G, dv, seed=seed + 2, dtype=dtype)
    bias = 0.5 * torch.rand(H, min(window, T + 40), generator=torch.Generator().manual_seed(seed + 3)) * torch.arange(min(window, T + 40)).sqrt()
    pages = -(-T // 16)
    order = torch.randperm(pages + spare, generator=torch.Generator().manual_seed(seed + 4))[:pages]
    for i in (40, 96, 150):  # the score of the row's last seen and of the first unseen key would be far above all others
        for j in (i - window + 1, i - window):
            if 0 <= j and i < T:
                m = qm[i, (i + j) % H].float()
                k[j] = (m.view(G, dk) * 8 / m.pow(2).sum()).to(dtype)
    kp, vp = torch.full((pages + spare, G, 16, dk), 3.0, dtype=dtype), torch.full((pages + spare, G, 16, dv), 3.0, dtype=dtype)
    for t in range(T):
        kp[order[t // 16], :, t % 16], vp[order[t // 16], :, t % 16] = k[t], v[t]
    return q, talk, scale, qm, k, v, bias, columns(kp), columns(vp), order.to(torch.int32)


def attention_want(qm, k, v, bias, window, rows, positions):
    """Rows of the windowed softmax, straight."""
    H, per = qm.shape[1], qm.shape[1] // k.shape[1]
    out = torch.zeros(len(rows), H, v.shape[2], dtype=torch.float64)
    for r, (row, i) in enumerate(zip(rows, positions)):
        lo = max(0, i - window + 1)
        kk = k[lo:i + 1].double().flatten(1)
        s = qm[row].double() @ kk.T - bias[:, torch.arange(i - lo, -1, -1)].double()
        p = torch.softmax(s, -1)
        for h in range(H):
            out[r, h] = p[h] @ v[lo:i + 1, h // per].double()
    return out


SHAPES = [(8, 2, 64, 64), (16, 2, 192, 128), (12, 4, 192, 64), (40, 8, 128, 128), (3, 1, 64, 64), (10, 5, 64, 256), (14, 7, 64, 192), (6, 2, 128, 192), (5, 5, 64, 128), (32, 4, 128, 128), (24, 1, 64, 64), (2, 1, 192, 320), (64, 4, 128, 128),
          (12, 3, 64, 256), (50, 2, 192, 256)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("window", [1, 16, 33, 100, 1000])
@pytest.mark.parametrize("H,G,dk,dv", SHAPES)
def test_mixed_attention(ops, H, G, dk, dv, window, dtype):
    """Decode rows at page borders, at the sequence's start and around the window's edge, and prompt chunks of several sizes.
    For some rows one key just inside the window and one just outside is made to stand out."""
    T = 170
    q, talk, scale, qm, k, v, bias, kp, vp, order = attention_case(T, H, G, dk, dv, window, dtype, seed=H + dk + window)
    Q, QM, KP, VP, B, O, mix = (t.to(DEV) for t in (q, qm.to(dtype), kp, vp, ops.pad_distances(bias), order, (talk.float() * scale)))
    rows = [0, 1, 15, 16, 17, 31, 32, 40, 47, 48, 96, 99, 100, 150, 169]
    pos = torch.tensor(rows, dtype=torch.int32, device=DEV)
    st = status()
    table = O[None].expand(len(rows), -1).contiguous()
    want = 1.3 * attention_want(qm, k, v, bias, window, rows, rows)
    for raw in (False, True) if ops.mixed_attn_mixes(H, G, dk, dv, dtype) else (False,):
        for split in (None, 32, 0) if not raw else (None, 64):
            out = torch.full((len(rows), H * dv + 32), 7.0, dtype=dtype, device=DEV)
            ops.mixed_attn((Q if raw else QM)[rows].contiguous(), KP, VP, G, table, pos, B, window, out, 1.3, st, split, mix=mix if raw else None)
            ops.read_status(st, "decode rows")
            assert rel_err(out[:, : H * dv].cpu().view(-1, H, dv), want) < 1.5 * TOL[dtype], (raw, split)
            assert bool((out[:, H * dv:] == 7.0).all())
    form = ops.mixed_attn_prefill_form(H, G, dk, dv, dtype)
    if not form:
        return
    full = 1.3 * attention_want(qm, k, v, bias, window, range(T), range(T))
    for first, n in ((0, 170), (0, 2), (16, 2), (33, 100), (90, 80), (168, 2), (95, 16)):
        out = torch.full((n, H * dv + 32), 7.0, dtype=dtype, device=DEV)
        more = dict(talk=talk.to(DEV), scale=scale) if form == 2 else {}
        ops.mixed_attn_prefill((Q if form == 2 else QM)[first:first + n].contiguous(), KP, VP, G, O, first, B, window, out, 1.3, st, **more)
        ops.read_status(st, "prompt chunk")
        assert rel_err(out[:, : H * dv].cpu().view(n, H, dv), full[first:first + n]) < 1.5 * TOL[dtype], (first, n)
        assert bool((out[:, H * dv:] == 7.0).all())


def test_mixed_attention_reports_bad_pages_and_positions(ops):
    q, talk, scale, qm, k, v, bias, kp, vp, order = attention_case(40, 8, 2, 64, 64, 32, BF, 1)
    QM, KP, VP, B, O = (t.to(DEV) for t in (qm.to(BF), kp, vp, ops.pad_distances(bias), order))
    out = torch.empty(1, 512, dtype=BF, device=DEV)
    for table, pos in ((torch.full((1, 3), 99, dtype=torch.int32, device=DEV), i32(20)), (O[None].contiguous(), i32(48))):
        st = status()
        ops.mixed_attn(QM[:1].contiguous(), KP, VP, 2, table, pos, B, 32, out, 1.0, st)
        with pytest.raises(RuntimeError):
            ops.read_status(st, "bad page or position")


# ------------------------------------------------------------ recurrences


def recurrence_case(T, H, G, d, dv, delta, dtype, seed):
    act = randn(T, 2 * G * d + H * dv, seed=seed, dtype=dtype)
    w = SimpleNamespace(qk_heads=G)
    if delta:
        w.a_log, w.dt_bias = -3.0 + 2 * randn(H, seed=seed + 1), randn(H, seed=seed + 2)
        ba = randn(T, 2 * H, seed=seed + 3) * 2
    else:
        w.decay, ba = 1.0 - torch.logspace(-0.3, -4, H), None
    q, k = act[:, : G * d].double().view(T, G, d), act[:, G * d:2 * G * d].double().view(T, G, d)
    v = act[:, 2 * G * d:].double().view(T, H, dv)
    per = H // G
    if delta:
        beta = torch.sigmoid(ba[:, :H].double())
        g = torch.exp(-torch.exp(w.a_log.double()) * torch.nn.functional.softplus(ba[:, H:].double() + w.dt_bias.double()))
        want = torch.stack([ref.delta_rule(ref.unit(q[:, h // per]) * d ** -0.5, ref.unit(k[:, h // per]), v[:, h], beta[:, h], g[:, h])
                            for h in range(H)], 1)
    else:
        want = torch.stack([ref.decay_attention(q[:, h], k[:, h], v[:, h], float(w.decay[h])) for h in range(H)], 1)
    w = SimpleNamespace(**{n: (t.to(DEV) if torch.is_tensor(t) else t) for n, t in vars(w).items()})
    return act, ba, w, want


def run_recurrence(ops, A, BA, w, state, at, n, d, dv, H, delta, how, st):
    """n tokens of the sequence in slot 1 from position `at` on, by the kernel `how`."""
    o = torch.empty(n, H, dv, device=DEV)
    slots, pos = torch.full((n,), 1, dtype=torch.int32, device=DEV), torch.arange(at, at + n, dtype=torch.int32, device=DEV)
    ba, q_scale = None if BA is None else BA[at:at + n], d ** -0.5 if delta else 1.0
    if how == "chunk":
        ops.state_chunk(A[at:at + n], w, state, slots, pos, o, st, ba=ba, q_scale=q_scale)
    elif how == "step":
        ops.state_step(A[at:at + n], w, state, slots, pos, o, st)
    else:
        ops.state_scan(A[at:at + n], w, state, slots, pos, o, n > 1, st, ba=ba, q_scale=q_scale)
    return o.cpu().double()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("delta", [True, False])
@pytest.mark.parametrize("H,G,d,dv", [(4, 4, 64, 64), (4, 2, 128, 128), (3, 3, 16, 48), (6, 2, 48, 32), (2, 1, 32, 144), (2, 2, 208, 64),
                                      (1, 1, 304, 16), (2, 2, 64, 256), (2, 2, 112, 16), (20, 20, 48, 128), (19, 19, 80, 128)])
def test_recurrence_in_portions_and_decoded(ops, H, G, d, dv, delta, dtype):
    """Any cut of a sequence gives the whole sequence's recurrence, by every kernel that takes the portion: portions from two
    tokens on, over and at the borders of the kernels' inner blocks, decode rows in between (each run twice); other slots keep
    their states."""
    if not delta and H != G:
        pytest.skip("one query/key head per head")
    T = 200
    act, ba, w, want = recurrence_case(T, H, G, d, dv, delta, dtype, seed=H + d)
    A, BA = act.to(DEV), None if ba is None else ba.to(DEV)
    scale = want.abs().amax(0, keepdim=True).clamp_min(1e-6)
    blocked = ops.state_chunk_supported(d, dv, dtype)
    for cuts in ([T], [2, 3, 1, 15, 17, 2, 64, 1, 1, 94], [64, 64, 72], [1] * 20 + [130, 50], [33, 65, 2, 100], [63, 1, 128, 8]):
        for how in ("scan", "chunk") if blocked else ("scan",):
            state = torch.full((3, 2, H, d, dv), 9.0, device=DEV)
            st, got, at = status(), [], 0
            for n in cuts:
                kernel = how if n > 1 else "step" if not delta and how == "chunk" and ops.state_step_supported(d, dv) else "scan"
                for _ in range(2 if n == 1 else 1):
                    o = run_recurrence(ops, A, BA, w, state, at, n, d, dv, H, delta, kernel, st)
                got.append(o)
                at += n
            ops.read_status(st, "recurrence")
            err = float(((torch.cat(got) - want) / scale).abs().max())
            assert err < (2e-4 if dtype == BF else 2e-5), (how, cuts, err)
            assert bool((state[[0, 2]] == 9.0).all())


def test_recurrence_with_extreme_decays(ops):
    """Decays of 0 and 1 and step sizes near 0 and 1 in the blocked kernel; keys that repeat (the inverse is far from 1)."""
    H, d, dv, T = 4, 64, 32, 150
    for delta in (True, False):
        act, ba, w, want = recurrence_case(T, H, H, d, dv, delta, BF, seed=9)
        if delta:
            act[20:140, H * d:2 * H * d] = act[20:21, H * d:2 * H * d]
            ba[:, :H] = torch.tensor([8.0, 8.0, -8.0, 0.0])
            ba[:, H:] = torch.tensor([-20.0, 40.0, -20.0, 1.0])
            ba[100] = -ba[100]
            a_log, dt = w.a_log.cpu().double(), w.dt_bias.cpu().double()
            q, k, v = (
                act[:, :H * d].double().view(T, H, d), act[:, H * d:2 * H * d].double().view(T, H, d), act[:, 2 * H * d:].double().view(T, H, dv))
            g = torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(ba[:, H:].double() + dt))
            want = torch.stack([ref.delta_rule(ref.unit(q[:, h]) * d ** -0.5, ref.unit(k[:, h]), v[:, h], torch.sigmoid(ba[:, h].double()), g[:, h])
                                for h in range(H)], 1)
        else:
            w.decay = torch.tensor([0.0, 1.0, 1e-6, 0.5], device=DEV)
            q, k, v = act[:, :H * d].double().view(T, H, d), act[:, H * d:2 * H * d].double().view(T, H, d), act[:, 2 * H * d:].double().view(T, H, dv)
            want = torch.stack([ref.decay_attention(q[:, h], k[:, h], v[:, h], float(w.decay[h])) for h in range(H)], 1)
        state, st = torch.full((3, 2, H, d, dv), 9.0, device=DEV), status()
        got = run_recurrence(ops, act.to(DEV), None if ba is None else ba.to(DEV), w, state, 0, T, d, dv, H, delta, "chunk", st)
        assert float(((got - want) / want.abs().amax(0, keepdim=True)).abs().max()) < 3e-4, delta
        ops.read_status(st, "recurrence")


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,d,dv,taps,size", [(4, 4, 64, 64, 4, 64), (6, 2, 48, 32, 1, 20), (4, 1, 128, 128, 3, 128), (2, 2, 16, 272, 7, 260)])
def test_decode_step_of_the_gated_delta_rule(ops, H, G, d, dv, taps, size, dtype):
    """The one-kernel decode step (convolution, recurrence, head norm, gate) against the same in separate kernels, on top of a
    prompt chunk and of other decode steps; every step run twice."""
    T, C = 40, 2 * G * d + H * dv
    pre, conv = randn(T, C, seed=1, dtype=dtype), randn(taps, C, seed=2, dtype=dtype)
    pre.view(T, C)[:, 2 * G * d:].view(T, H, dv)[..., size:] = 0
    _, ba, w, _ = recurrence_case(T, H, G, d, dv, True, dtype, seed=3)
    w.conv, w.head_norm = conv.to(DEV), (1 + 0.3 * randn(dv, seed=4)).to(DEV)
    g = randn(T, H * dv, seed=5, dtype=dtype).to(DEV)
    P, BA, q_scale = pre.to(DEV), ba.to(DEV), d ** -0.5
    rings = [torch.full((3, taps, C), 7.0, dtype=dtype, device=DEV) if taps > 1 else None for _ in range(2)]
    states, st = [torch.full((3, 2, H, d, dv), 9.0, device=DEV) for _ in range(2)], status()
    for at, n in [(0, 11)] + [(i, 1) for i in range(11, T)]:
        slots, pos = torch.full((n,), 2, dtype=torch.int32, device=DEV), torch.arange(at, at + n, dtype=torch.int32, device=DEV)
        outs = []
        for which in range(2 if n == 1 else 1):
            out = torch.full((n, H * dv + 16), 5.0, dtype=dtype, device=DEV)
            for _ in range(2):
                if which == 1:
                    ops.state_step(P[at:at + n], w, states[1], slots, pos, None, st, ba=BA[at:at + n], q_scale=q_scale, ring=rings[1],
                                   gate=g[at:at + n], eps=1e-5, size=size, scale=1.4, out=out)
                    continue
                a = ops.conv_silu(P[at:at + n], w.conv, rings[0], slots, pos, n > 1, st)
                o = torch.empty(n, H, dv, device=DEV)
                ops.state_scan(a, w, states[0], slots, pos, o, n > 1, st, ba=BA[at:at + n], q_scale=q_scale)
                ops.group_norm_gate(o, w.head_norm, g[at:at + n], 1e-5, size, True, 1.4, out)
                if n > 1:
                    break
            outs.append(out)
        if n > 1:  # the prompt chunk goes to both
            states[1].copy_(states[0])
            if taps > 1:
                rings[1].copy_(rings[0])
        else:
            assert rel_err(outs[1][:, : H * dv], outs[0][:, : H * dv]) < (1e-2 if dtype == BF else 2e-5) and bool((outs[1][:, H * dv:] == 5.0).all())
            assert rel_err(states[1], states[0]) < 1e-5
            if taps > 1:
                assert torch.equal(rings[1], rings[0])
    ops.read_status(st, "delta step")


def test_recurrence_rows_are_independent_sequences(ops):
    """A decode step's rows with slots and positions in any order; a row at position 0 starts from zeros."""
    H, d, dv, T = 2, 32, 32, 12
    act, ba, w, want = recurrence_case(T, H, H, d, dv, True, F32, seed=3)
    A, BA = act.to(DEV), ba.to(DEV)
    state, st = torch.full((4, 2, H, d, dv), 5.0, device=DEV), status()
    lag = {3: 0, 0: 4, 2: 7}  # slot -> steps it starts later
    for step in range(T):
        live = [s for s in lag if step >= lag[s]]
        at = torch.tensor([step - lag[s] for s in live], device=DEV)
        o = torch.empty(len(live), H, dv, device=DEV)
        ops.state_scan(A[at].contiguous(), w, state, i32(*live), at.int(), o, False, st, ba=BA[at].contiguous(), q_scale=d ** -0.5)
        assert rel_err(o, want[at.cpu()]) < 2e-5
    assert bool((state[1] == 5.0).all())
    ops.read_status(st, "rows")
    ops.state_scan(A[:1], w, state, i32(4), i32(0), torch.empty(1, H, dv, device=DEV), False, st, ba=BA[:1], q_scale=1.0)
    with pytest.raises(RuntimeError):
        ops.read_status(st, "a slot outside the states")


# ---------------------------------------------------------------- experts


@pytest.mark.parametrize("E,K,scale", [(8, 2, 1.5), (12, 12, 1.0), (300, 8, 0.3), (1, 1, 2.0), (40, 20, 1.0)])
def test_sigmoid_routing(ops, E, K, scale):
    lg = randn(50, E, seed=E) * 3
    ids, w = ops.moe_route_sigmoid(lg.to(DEV), K, scale)
    want_ids, want_w = ref.route(lg.double(), K, scale)
    assert torch.equal(ids.cpu().long(), want_ids) and rel_err(w, want_w) < 1e-5


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,E,K,W,F,tile", [(1, 4, 2, 64, 128, None), (37, 8, 2, 192, 128, None), (300, 5, 3, 256, 384, None),
                                             (130, 16, 4, 128, 256, 32), (200, 3, 1, 320, 128, 64), (256, 64, 8, 512, 128, None)])
def test_experts(ops, T, E, K, W, F, tile, dtype):
    """Sorted rows and both products; experts without a token and experts with several tiles."""
    x = randn(T, W, seed=1, dtype=dtype)
    gate, up, down = (randn(E, a, b, seed=s, dtype=dtype, scale=b ** -0.5) for s, a, b in ((2, F, W), (3, F, W), (4, W, F)))
    lg = randn(T, E, seed=5)
    lg[:, 0] += 3.0  # crowded
    if E > 4:
        lg[:, E - 1] -= 100.0  # nobody
    ids = torch.topk(lg, K, -1).indices.int()
    lay = pkg("layered")
    w13 = torch.stack([lay.interleave_glu(gate[e], up[e]) for e in range(E)]).to(DEV)
    ws = torch.zeros(ops.moe_permute_workspace_bytes(T, E, K), dtype=torch.uint8, device=DEV)
    st = status()
    p = ops.moe_permute_copy(ids.to(DEV), x.to(DEV), E, ws, None if dtype == F32 else tile)
    rows = p.row_of_pair.cpu().long()
    assert sorted(rows.flatten().tolist()) == list(range(T * K))
    assert torch.equal(p.rows.cpu()[rows], x[:, None].expand(T, K, W))
    h = ops.moe_gate_up(p, w13, st)
    y = ops.moe_down(p, h, down.to(DEV), st)
    ops.read_status(st, "experts"), ops.read_status(ws, "permutation")
    hr = h.cpu()[rows]
    for t in range(0, T, 7):
        for k in range(K):
            e = int(ids[t, k])
            a = ref.silu(gate[e].double() @ x[t].double()) * (up[e].double() @ x[t].double())
            assert rel_err(hr[t, k], a) < TOL[dtype]
            assert rel_err(y.cpu()[rows[t, k]], down[e].double() @ hr[t, k].double()) < TOL[dtype]


@pytest.mark.parametrize("dtype", [BF, F32])
def test_projection_with_biases_and_activations(ops, dtype):
    M, K, st = 70, 128, status()
    x, w, b = randn(M, K, seed=1, dtype=dtype), randn(64 + 2 * 32 + 48 + 96 + 5, K, seed=2, dtype=dtype, scale=K ** -0.5), randn(64 + 64 + 48 + 96 + 5, seed=3)
    q, a, g, f = (torch.empty(M, n, dtype=t, device=DEV) for n, t in ((64, F32), (48, dtype), (96, dtype), (5, F32)))
    pool = torch.zeros(8, 2, 16, 32, dtype=dtype, device=DEV)
    table = torch.randperm(8, generator=torch.Generator().manual_seed(1))[None].expand(M, -1).int().contiguous().to(DEV)
    ops.proj_split(x.to(DEV), w.to(DEV), [(ops.SEG_F32, q), (ops.SEG_PAGES, pool), (ops.SEG_ROWS, a, ops.ACT_SILU),
                                          (ops.SEG_ROWS, g, ops.ACT_SIGMOID), (ops.SEG_F32, f)],
                   positions=torch.arange(M, dtype=torch.int32, device=DEV), block_table=table, status=st, col_bias=b.to(DEV))
    ops.read_status(st, "projection")
    y = x.double() @ w.double().T + b.double()
    pages = torch.stack([pool.cpu()[int(table[0, t // 16]), :, t % 16].reshape(-1) for t in range(M)])
    for got, want in ((q, y[:, :64]), (pages, y[:, 64:128]), (a, ref.silu(y[:, 128:176])), (g, torch.sigmoid(y[:, 176:272])), (f, y[:, 272:])):
        assert rel_err(got, want) < TOL[dtype]
