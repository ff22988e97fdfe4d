"""Each mechanism of the Kipedra decoder alone, against the plain implementation in ``kipedra_oracle``.

As in ``test_mixers``: the CPU ops and, where there is a GPU, the kernels in fp32 and bf16; sequences in portions cut at
awkward places, in batches beside other sequences, on pages and slots in shuffled order that held other requests.
"""
import pytest
import torch
from torch.nn.functional import pad

import kipedra_oracle as O
from test_mixers import LENGTHS, Pages, Step, be, close, cuts, rnd  # noqa: F401


def plans():
    """Both sequences whole in one step, and the portions of ``SCHEDULE``."""
    yield [([(0, n, 3 - i) for i, n in enumerate(LENGTHS)], [(i, 0, n) for i, n in enumerate(LENGTHS)])]
    yield list(cuts())


# ---- attention -----------------------------------------------------------------------------------
ATTN = [  # heads, kv heads, dim, vdim, window, rotated dims, taps
    (4, 2, 32, 16, 13, 32, 4),
    (6, 2, 64, 64, 100, 24, 3),
    (3, 1, 96, 40, 17, 12, 2),
    (8, 8, 128, 128, 16, 64, 4),
    (4, 1, 128, 96, 1, 128, 6),
    (18, 1, 64, 128, 29, 64, 1),
    (2, 1, 160, 200, 33, 20, 5),
    (2, 2, 264, 20, 64, 8, 4),       # wider than the vectorised kernel takes
    (3, 3, 22, 30, 9, 10, 9),        # nothing is a multiple of four
    (2, 1, 36, 32, 500, 6, 4),
]


@pytest.mark.parametrize("shape", ATTN, ids=lambda s: "-".join(map(str, s)))
def test_attention(be, shape):
    """Projections to output heads: convolutions, interleaved rotation, window."""
    from tgi_b200 import ops
    from tgi_b200.models.arch import MixerSpec
    from tgi_b200.models.mixers import RotaryTables

    dev, dt = be
    H, G, d, dv, window, rot, taps = shape
    scale = 1.3 * d ** -0.5
    tab = RotaryTables(128, dev).get(MixerSpec("attention", H, G, d, dv, rot_dims=rot, rot_base=500.0))
    dk, dvp = ops.attention_pitch(d, dv, dt, dev)
    widths = (H * d, G * d, G * dv)
    offs = [0, (widths[0] + 7) // 8 * 8]
    offs.append(offs[1] + (widths[1] + 7) // 8 * 8)
    proj = [rnd(i + 1, n, offs[2] + (widths[2] + 7) // 8 * 8).to(dt) for i, n in enumerate(LENGTHS)]
    conv = [rnd(5 + i, w, taps, std=0.7) for i, w in enumerate(widths)]
    want = []
    for p in proj:
        q, k, v = (O.causal_conv(p.double()[:, o:o + w], c.double()) for o, w, c in zip(offs, widths, conv))
        want.append(O.attend(O.rotate_pairs(q.view(-1, H, d), rot, 500.0), O.rotate_pairs(k.view(-1, G, d), rot, 500.0),
                             v.view(-1, G, dv), scale, window))
    weights = ops.conv_weights(conv, dev)
    for steps in plans():
        pg = Pages(dev, dt, G, dk, dvp)
        past = torch.full((4, taps - 1, sum(widths)), 3.0, dtype=dt, device=dev)
        got = [torch.zeros(n, H, dv) for n in LENGTHS]
        for parts, rows in steps:
            st = Step(parts, dev)
            x = torch.cat([proj[i][a:b] for i, a, b in rows]).to(dev)
            q = ops.rotate_norm_store(x, offs, st.positions, tab.cos_sin, pg.slots(rows), pg.k, pg.v, H, G, d, dv, rot, False,
                                      1e-3, interleaved=True,
                                      conv=ops.ShortConv(weights, past, st.cu, st.kv, st.slots, st.max_q == 1))
            o = ops.paged_attention(q, pg.k, pg.v, pg.table([r[0] for r in rows]), st.cu, st.kv, scale, window=window,
                                    max_q=st.max_q, max_kv=st.max_kv)
            t = 0
            for i, a, b in rows:
                got[i][a:b] = o[t:t + b - a, :, :dv].float().cpu()
                t += b - a
        for i in range(2):
            close(got[i], want[i], dt)
        assert (pg.k[..., d:] == 0).all() and (pg.v[..., dv:] == 0).all()
        assert (past[1] == 3.0).all()                             # a slot nobody held


@pytest.mark.parametrize("inter,conv,norm,mix", [(True, False, False, False), (False, True, True, True), (True, True, True, False),
                                                 (True, False, True, True), (False, True, False, False)])
def test_other_combinations(be, inter, conv, norm, mix):
    """Rotation layout, convolution, unit norm and value mixing are independent of each other."""
    from tgi_b200 import ops
    from tgi_b200.utils.rotary import RotaryTable, scaled_frequencies

    import fuzuvik_oracle as F

    dev, dt = be
    H, G, d, dv, rot, taps, n = 4, 2, 64, 48, 32, 4, 23
    tab = RotaryTable.from_frequencies(scaled_frequencies(300.0, rot), 64).to(dev)
    widths = (H * d, G * d, G * dv)
    offs = [0, widths[0], widths[0] + widths[1]]
    x, first = rnd(1, n, sum(widths)).to(dt), rnd(2, n, widths[2]).to(dt)
    w = [rnd(3 + i, c, taps) for i, c in enumerate(widths)]
    parts = [x.double()[:, o:o + c] for o, c in zip(offs, widths)]
    if conv:
        parts = [O.causal_conv(p, c.double()) for p, c in zip(parts, w)]
    turn = (lambda y: O.rotate_pairs(y, rot, 300.0)) if inter else (lambda y: F.rotate(y, {"dims": rot, "base": 300.0}))
    q, k = (turn(p.view(n, -1, d)) for p in parts[:2])
    if norm:
        q, k = O.rms(q, 1e-3), O.rms(k, 1e-3)
    v = 0.7 * parts[2] + 0.3 * first.double() if mix else parts[2]
    st = Step([(0, n, 0)], dev)
    past = ops.ShortConv(ops.conv_weights(w, dev), torch.zeros(1, taps - 1, sum(widths), dtype=dt, device=dev), st.cu, st.kv,
                         st.slots, False) if conv else None
    kc, vc = torch.zeros(2, 16, G, d, dtype=dt, device=dev), torch.zeros(2, 16, G, dv, dtype=dt, device=dev)
    slots = torch.arange(n, dtype=torch.int32, device=dev)
    got = ops.rotate_norm_store(x.to(dev), offs, st.positions, tab.cos_sin, slots, kc, vc, H, G, d, dv, rot, norm, 1e-3,
                                first.to(dev) if mix else None, 0.3, inter, past)
    close(got, q, dt)
    close(kc.view(-1, G, d)[:n], k, dt)
    close(vc.view(-1, G, dv)[:n].reshape(n, -1), v, dt)


@pytest.mark.parametrize("dims", [(128, 128), (64, 64), (256, 256), (40, 24)], ids=str)
@pytest.mark.parametrize("window", [1, 16, 25, 130])
def test_window_edge(be, dims, window):
    """One key draws nearly all the weight of its query: seen as the oldest key of the window, not seen one further back, in
    prompts of several tiles, short portions and decoded tokens."""
    from tgi_b200 import ops

    dev, dt = be
    d, dv = dims
    L = 330
    dk, dvp = ops.attention_pitch(d, dv, dt, dev)
    for qpos in (window, 160, 255, L - 1):
        for key in (qpos - window + 1, qpos - window):
            if key < 0:
                continue
            q, k, v = rnd(1, L, 2, d, std=0.1), rnd(2, L, 1, d, std=0.1), rnd(3, L, 1, dv)
            q[qpos], k[key, 0] = 0, 0
            q[qpos, :, 3], k[key, 0, 3] = 7.0, 7.0
            q, k, v = q.to(dt), k.to(dt), v.to(dt)
            js = [j for j in range(L) if O.sees(qpos, j, window)]
            s = q[qpos].double() @ k[js, 0].double().t() * 0.25
            want = torch.softmax(s, -1) @ v[js, 0].double()
            alone = v[key, 0].double()
            assert bool((want - alone).norm() < 0.1 * alone.norm()) == (key == qpos - window + 1)
            pg = Pages(dev, dt, 1, dk, dvp, blocks=45)
            sl = pg.slots([(0, 0, L)]).long()
            pg.k.view(-1, 1, dk)[sl, :, :d] = k.to(dev)
            pg.v.view(-1, 1, dvp)[sl, :, :dv] = v.to(dev)
            qq = pad(q, (0, dk - d)).to(dev)
            for start, n in ((0, qpos + 1), (max(0, qpos - 1), min(2, qpos + 1)), (qpos, 1)):
                st = Step([(start, n, 0)], dev)
                o = ops.paged_attention(qq[start:start + n], pg.k, pg.v, pg.table([0]), st.cu, st.kv, 0.25, window=window,
                                        max_q=n, max_kv=qpos + 1)
                close(o[-1, :, :dv].float(), want, dt)


# ---- delta rule ----------------------------------------------------------------------------------
def delta_case(dt, G, H, d, dv, taps):
    case, off = {"offs": []}, 0
    widths = [G * d, G * d, H * dv, H, H]
    for w in widths:
        case["offs"].append(off)
        off += (w + 7) // 8 * 8
    case["proj"] = [rnd(i + 1, n, off).to(dt) for i, n in enumerate(LENGTHS)]
    case["conv"] = [rnd(7 + i, c, taps, std=0.7) for i, c in enumerate(widths[:3])]
    case["a_log"], case["dt_bias"] = rnd(11, H), rnd(12, H) - 2.0
    want = []
    for x in case["proj"]:
        x = x.double()
        cv = [O.silu(O.causal_conv(x[:, o:o + w], c.double())) for o, w, c in zip(case["offs"], widths, case["conv"])]
        of = [h // (H // G) for h in range(H)]
        b, a = (x[:, o:o + H] for o in case["offs"][3:])
        g = torch.exp(-torch.exp(case["a_log"].double()) * O.softplus(a + case["dt_bias"].double()))
        o = O.delta_scan((O.unit(cv[0].view(-1, G, d)) * d ** -0.5)[:, of], O.unit(cv[1].view(-1, G, d))[:, of],
                         cv[2].view(-1, H, dv), g, torch.sigmoid(b))
        want.append((o, g))
    return case, want


@pytest.mark.parametrize("shape", [(2, 4, 24, 40, 4), (3, 3, 64, 64, 2), (1, 2, 100, 33, 3), (2, 2, 128, 128, 4), (1, 1, 150, 8, 5),
                                   (1, 3, 256, 20, 4), (2, 2, 16, 132, 1), (2, 4, 64, 260, 9), (2, 4, 128, 64, 7), (1, 1, 1, 4, 2),
                                   (1, 2, 30, 50, 3), (3, 6, 32, 32, 4)], ids=str)
def test_delta_rule(be, shape):
    """Convolutions, unit norms, decays per head and the scan, on slots that held other states."""
    from tgi_b200 import ops

    dev, dt = be
    G, H, d, dv, taps = shape
    case, want = delta_case(dt, *shape)
    pitch = ops.recurrent_pitch(d, dev)
    conv, a_log, bias = ops.conv_weights(case["conv"], dev), case["a_log"].to(dev), case["dt_bias"].to(dev)
    at = case["offs"][4]
    for steps in plans():
        past = torch.full((4, taps - 1, 2 * G * d + H * dv), 3.0, dtype=dt, device=dev)
        state = torch.full((4, H, dv, pitch), 5.0, device=dev)
        got = [torch.zeros(n, H, dv) for n in LENGTHS]
        for parts, rows in steps:
            st = Step(parts, dev)
            x = torch.cat([case["proj"][i][a:b] for i, a, b in rows]).to(dev)
            r = ops.delta_inputs(x, case["offs"], x[:, at:at + H], conv, a_log, bias, st.cu, st.kv, st.slots, past, G, H, d,
                                 pitch, dv, st.max_q == 1, True)
            assert r[3].shape == (x.shape[0], H)
            close(r[3], torch.cat([want[i][1][a:b] for i, a, b in rows]), torch.float32)
            o = ops.delta_scan(*r, st.cu, st.kv, st.slots, state, d, st.max_q)
            t = 0
            for i, a, b in rows:
                got[i][a:b] = o[t:t + b - a].cpu()
                t += b - a
        for i in range(2):
            close(got[i], want[i][0], dt)
        assert (state[1] == 5.0).all() and (past[1] == 3.0).all()


@pytest.mark.parametrize("portion", [1, 2, 7])
def test_delta_far_write(be, portion):
    """A value written once comes back 200 tokens later where the head keeps its state, and shrunk by the product of the
    decays where it forgets; a head that forgets everything at one token has lost it."""
    from tgi_b200 import ops

    dev, dt = be
    if dt != torch.float32:
        pytest.skip("the scan is fp32 whatever the activations")
    H, d, dv, n = 3, 32, 24, 203
    q, k, v = torch.zeros(n, H, d), torch.zeros(n, H, d), rnd(1, n, H, dv)
    k[0, :, 5] = 1.0
    for t in range(1, n):
        k[t, :, 6 + t % 8] = 1.0
    q[-1, :, 5] = 1.0
    g = torch.ones(n, H)
    g[:, 1] = 0.97
    g[101, 2] = 0.0
    beta = torch.full((n, H), 0.5)
    state = torch.zeros(1, H, dv, d, device=dev)
    for t in range(0, n, portion):
        m = min(portion, n - t)
        st = Step([(t, m, 0)], dev)
        o = ops.delta_scan(*(x[t:t + m].to(dev).contiguous() for x in (q, k, v, g, beta, (q * k).sum(-1))), st.cu, st.kv, st.slots,
                           state, d, m)
    close(o[-1, 0], 0.5 * v[0, 0], torch.float32)
    close(o[-1, 1], 0.5 * v[0, 1] * 0.97 ** (n - 1), torch.float32, tol32=1e-3)
    assert (o[-1, 2] == 0).all()


@pytest.mark.parametrize("batch", [1, 40, 130])
@pytest.mark.parametrize("dims", [(64, 64), (128, 96)], ids=str)
def test_scan_layouts(be, batch, dims):
    """Few and many sequences take different layouts of the state over lanes."""
    from tgi_b200 import ops

    dev, dt = be
    if dt != torch.float32 or (dev.type == "cpu" and batch > 1):
        pytest.skip("one layout on the CPU; the scan is fp32")
    d, dv, H, n = dims[0], dims[1], 2, 19
    k, q, v = (rnd(i, batch, n, H, w) for i, w in enumerate((d, d, dv)))
    k, q = O.unit(k), O.unit(q)
    g, beta = torch.sigmoid(rnd(4, batch, n, H) + 1), torch.sigmoid(rnd(5, batch, n, H))
    state, outs, a = torch.zeros(batch, H, dv, d, device=dev), [], 0
    for m in (13, 1, 5):
        st = Step([(a, m, batch - 1 - i) for i in range(batch)], dev)
        row = lambda x: x[:, a:a + m].reshape(batch * m, *x.shape[2:]).to(dev).contiguous()
        outs.append(ops.delta_scan(row(q), row(k), row(v), row(g), row(beta), row((q * k).sum(-1)), st.cu, st.kv, st.slots, state,
                                   d, m).cpu().view(batch, m, H, dv))
        a += m
    for i in {0, batch // 2, batch - 1}:
        close(torch.cat(outs, 1)[i], O.delta_scan(*(x[i].double() for x in (q, k, v, g, beta))), torch.float32)


def test_padding_rows(be):
    """Rows of a captured batch without a sequence (length 0, slot -1) leave every pool as it is."""
    from tgi_b200 import ops
    from tgi_b200.utils.rotary import RotaryTable, scaled_frequencies

    dev, dt = be
    if dev.type == "cpu":
        pytest.skip("captured batches exist on the GPU only")
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    cu, kv, slots, pages = i32([0, 1, 2, 3]), i32([0, 1, 0]), i32([-1, 1, -1]), i32([-1, 5, -1])
    for d in (32, 30):                                            # vectorised and plain kernel
        C = 4 * d + 2 * d + 2 * 16
        tab = RotaryTable.from_frequencies(scaled_frequencies(300.0, d - d % 4), 64).to(dev)
        past = torch.full((2, 3, C), 3.0, dtype=dt, device=dev)
        kc, vc = torch.full((1, 16, 2, d), 7.0, dtype=dt, device=dev), torch.full((1, 16, 2, 16), 7.0, dtype=dt, device=dev)
        ops.rotate_norm_store(rnd(1, 3, C).to(dt).to(dev), [0, 4 * d, 6 * d], i32([0, 0, 0]), tab.cos_sin, pages, kc, vc, 4, 2, d,
                              16, d - d % 4, False, 1e-5, interleaved=True,
                              conv=ops.ShortConv(ops.conv_weights([rnd(2, C, 4)], dev), past, cu, kv, slots, True))
        assert (past[0] == 3.0).all() and not (past[1] == 3.0).any()
        kept = [r for r in range(16) if r != 5]
        assert (kc[0, kept] == 7.0).all() and (vc[0, kept] == 7.0).all() and not (kc[0, 5] == 7.0).any()
    case, _ = delta_case(dt, 2, 4, 24, 40, 4)
    past = torch.full((2, 3, 2 * 48 + 160), 3.0, dtype=dt, device=dev)
    state = torch.full((2, 4, 40, 32), 5.0, device=dev)
    x = case["proj"][0][:3].to(dev)
    r = ops.delta_inputs(x, case["offs"], x[:, case["offs"][4]:][:, :4], ops.conv_weights(case["conv"], dev),
                         case["a_log"].to(dev), case["dt_bias"].to(dev), cu, kv, slots, past, 2, 4, 24, 32, 40, True, True)
    ops.delta_scan(*r, cu, kv, slots, state, 24, 1)
    assert (state[0] == 5.0).all() and (past[0] == 3.0).all() and not (state[1] == 5.0).any()


@pytest.mark.parametrize("groups,width", [(3, 24), (4, 128), (1, 1500), (1, 30), (2, 1028)])
def test_gated_norm(be, groups, width):
    from tgi_b200 import ops

    dev, dt = be
    T, n = 5, groups * width
    for extra in (0, -n % 8):
        o, gate, w = rnd(1, T, groups, width), rnd(2, T, n + 16).to(dt), rnd(3, width)
        y = ops.gated_norm(o.to(dev), gate.to(dev)[:, 8:8 + n], w.to(dev), 1e-2, groups, n + extra, "silu")
        close(y[:, :n], (O.rms(o.double(), 1e-2) * w.double()).reshape(T, n) * O.silu(gate[:, 8:8 + n].double()), dt)
        assert (y[:, n:] == 0).all()


# ---- residual stream -----------------------------------------------------------------------------
@pytest.mark.parametrize("width", [80, 203, 4096, 6144, 20000])
def test_two_additions_two_norms(be, width):
    """The stream takes both outputs, scaled, in 32 bits; both norms see the same stream; weights are deviations from one."""
    from tgi_b200 import ops

    dev, dt = be
    T = 6
    x, w1, w2 = rnd(1, T, width), rnd(2, width).to(dt), rnd(3, width).to(dt)
    a, b = rnd(4, T, width).to(dt), rnd(5, T, width).to(dt)
    to = lambda t: t.to(dev)
    y1, y2, r = ops.residual_norm((to(a), to(b)), to(x), to(w1), 1e-2, scale=0.3, unit_offset=True, weight2=to(w2))
    want = x.double() + 0.3 * (a.double() + b.double())
    close(r, want, torch.float32)
    close(y1, O.norm(want, w1.double(), 1e-2), dt)
    close(y2, O.norm(want, w2.double(), 1e-2), dt)
    y1, y2, r = ops.residual_norm(None, to(x), to(w1), 1e-2, scale=0.3, unit_offset=True, weight2=to(w2))
    close(y2, O.norm(x.double(), w2.double(), 1e-2), dt)
    assert (r.cpu() == x).all()
    y1, r = ops.residual_norm(to(a), to(x), to(w1), 1e-2, scale=-1.5, unit_offset=True)      # a layer without feed-forward
    close(y1, O.norm(x.double() - 1.5 * a.double(), w1.double(), 1e-2), dt)
    rows = torch.tensor([5, 0], dtype=torch.int32, device=dev)
    y1, none = ops.residual_norm((to(a), to(b)), to(x), to(w1), 1e-2, rows, keep=False, scale=0.3, unit_offset=True)
    assert none is None
    close(y1, O.norm(want, w1.double(), 1e-2)[[5, 0]], dt)
    big = torch.full((1, width), 4096.0, device=dev)              # small additions to large values are kept
    tiny = torch.full((1, width), 0.0625, device=dev, dtype=dt)
    assert (ops.residual_norm((tiny, tiny), big, to(w1), 1e-2, scale=0.5)[1] == 4096.0625).all()


# ---- feed-forward --------------------------------------------------------------------------------
@pytest.mark.parametrize("ff", [96, 40, 50, 33])
def test_gated_gelu(be, ff):
    from tgi_b200 import ops

    dev, dt = be
    x = (rnd(1, 9, 2 * ff) * 3).to(dt)
    close(ops.act_and_mul(x.to(dev), "gelu_tanh"), O.gelu_tanh(x[:, :ff].double()) * x[:, ff:].double(), dt)
    close(ops.activation(x.to(dev), "relu2"), O.relu_squared(x.double()), dt)


@pytest.mark.parametrize("tokens,experts,width,top", [(1, 10, 80, 3), (5, 64, 256, 8), (37, 16, 1000, 1), (600, 40, 320, 6),
                                                      (513, 33, 264, 2), (3, 256, 4096, 12), (20, 4, 44, 4), (7, 130, 2048, 5)])
def test_router(be, tokens, experts, width, top):
    """Logits in 32 bits; the correction decides who is chosen and leaves the weights alone."""
    from tgi_b200 import ops
    from tgi_b200.models.layers import FastLinear

    dev, dt = be
    x, w, corr = rnd(1, tokens, width).to(dt), rnd(2, experts, width, std=1.5 * width ** -0.5).to(dt), rnd(3, experts, std=0.3)
    z = x.double() @ w.double().t()
    ids, wts = O.route(z, corr.double(), top, 2.5)
    if top < experts:
        c = (torch.sigmoid(z) + corr.double()).sort(-1, descending=True).values
        clear = c[:, top - 1] - c[:, top] > 1e-4
    else:
        clear = torch.ones(tokens, dtype=torch.bool)
    gw, gi = ops.moe_route_sigmoid(x.to(dev), FastLinear(w.to(dev)).weight, corr.to(dev), top, 2.5)
    dense = lambda i, v: torch.zeros(tokens, experts, dtype=torch.float64).scatter_(1, i.long().cpu(), v.double().cpu())
    close(dense(gi, gw)[clear], dense(ids, wts)[clear], torch.float32)
    assert clear.double().mean() > 0.9
    close(gw.sum(-1), torch.full((tokens,), 2.5), torch.float32)
    if experts > 2 * top:
        plain = O.route(z, torch.zeros(experts, dtype=torch.float64), top, 2.5)[0]
        assert tokens < 5 or not torch.equal(plain.sort(-1).values, ids.sort(-1).values)


@pytest.mark.parametrize("tokens,experts,width,ff,top", [(1, 10, 80, 40, 3), (7, 4, 256, 96, 2), (70, 6, 100, 44, 3), (300, 8, 512, 264, 2),
                                                         (9, 5, 36, 21, 5), (33, 12, 64, 520, 9), (129, 3, 128, 64, 1)])
def test_experts(be, tokens, experts, width, ff, top):
    """Ungated squared-relu experts on their routed rows: experts without a token, one that gets all of them, odd sizes."""
    from tgi_b200 import ops

    dev, dt = be
    x = rnd(1, tokens, width).to(dt)
    up, down = rnd(2, experts, ff, width, std=width ** -0.5).to(dt), rnd(3, experts, width, ff, std=ff ** -0.5).to(dt)
    order = torch.stack([torch.randperm(experts - 1, generator=torch.Generator().manual_seed(t)) for t in range(tokens)])
    ids = order[:, :top].clone() if top < experts else torch.arange(experts).expand(tokens, -1)      # the last expert: nobody
    if top < experts:
        for t in range(tokens):                                   # expert 0: everybody
            if 0 not in ids[t]:
                ids[t, t % top] = 0
    wts = torch.rand(tokens, top, generator=torch.Generator().manual_seed(9)) + 0.1
    want = torch.zeros(tokens, width, dtype=torch.float64)
    for t in range(tokens):
        for e, w in zip(ids[t].tolist(), wts[t]):
            want[t] += w.double() * (down[e].double() @ O.relu_squared(up[e].double() @ x[t].double()))
    wu, wd = ops.plain_expert_weights(up.to(dev), down.to(dev))
    got = ops.moe_plain_experts(x.to(dev), wu, wd, wts.to(dev), ids.to(torch.int32).to(dev), "relu2")
    assert got.dtype == dt
    close(got, want, dt)
    if dev.type == "cuda":
        from tgi_b200.ops import cuda as K

        assert K.check_status(dev) == 0
