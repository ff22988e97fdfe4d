"""Each mechanism of the hybrid decoders alone, against the plain implementation in ``fuzuvik_oracle``.

Every test runs on the CPU ops and, where there is a GPU, on the kernels in fp32 and bf16.  Sequences arrive in
portions cut at awkward places, in batches beside other sequences, on pages and slots in shuffled order.
"""
import math

import pytest
import torch

import fuzuvik_oracle as O

BACKENDS = ["cpu-f32", pytest.param("cuda-f32", marks=pytest.mark.gpu), pytest.param("cuda-bf16", marks=pytest.mark.gpu)]


@pytest.fixture(params=BACKENDS)
def be(request):
    dev, dt = request.param.split("-")
    return torch.device(dev), torch.float32 if dt == "f32" else torch.bfloat16


def rnd(seed, *shape, std=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std


def close(got, want, dtype, tol32=2e-5, tol16=1.2e-2):
    """Root mean square of the difference against that of the expected values."""
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    err = ((got - want).pow(2).mean() / want.pow(2).mean().clamp_min(1e-30)).sqrt().item()
    assert err < (tol32 if dtype == torch.float32 else tol16), err


class Step:
    """Metadata of one ragged step: ``parts`` is a list of ``(start, n, slot)``."""

    def __init__(self, parts, dev):
        cu = [0]
        for _, n, _ in parts:
            cu.append(cu[-1] + n)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
        self.cu, self.kv = i32(cu), i32([s + n for s, n, _ in parts])
        self.slots = i32([x for _, _, x in parts])
        self.positions = i32([s + i for s, n, _ in parts for i in range(n)])
        self.max_q, self.max_kv = max(n for _, n, _ in parts), max(s + n for s, n, _ in parts)


# portions of two sequences of 70 and 41 tokens: single tokens, two tokens, a long stretch, one sequence left out
SCHEDULE = [((0, 1), (0, 5)), ((1, 2), (5, 1)), ((3, 30), None), (None, (6, 2)), ((33, 1), (8, 1)), ((34, 1), (9, 1)),
            ((35, 17), (10, 30)), ((52, 2), (40, 1)), ((54, 16), None)]
LENGTHS = (70, 41)


def cuts(slots=(2, 0)):
    """``(parts, rows of the sequences in this step)`` of every step of ``SCHEDULE``."""
    for entry in SCHEDULE:
        parts = [(p[0], p[1], slots[i]) for i, p in enumerate(entry) if p]
        rows = [(i, p[0], p[0] + p[1]) for i, p in enumerate(entry) if p]
        yield parts, rows


# ---- attention -----------------------------------------------------------------------------------
class Pages:
    def __init__(self, dev, dtype, hkv, dk, dv, blocks=24, bs=16):
        g = torch.Generator().manual_seed(9)
        order = (torch.randperm(blocks - 1, generator=g) + 1).tolist()
        half = len(order) // 2
        self.tables = [order[:half], order[half:2 * half]]
        self.bs, self.dev = bs, dev
        self.k = torch.zeros(blocks, bs, hkv, dk, dtype=dtype, device=dev)
        self.v = torch.zeros(blocks, bs, hkv, dv, dtype=dtype, device=dev)

    def table(self, which):
        return torch.tensor([self.tables[i] for i in which], dtype=torch.int32, device=self.dev)

    def slots(self, rows):
        return torch.tensor([self.tables[i][t // self.bs] * self.bs + t % self.bs for i, a, b in rows for t in range(a, b)],
                            dtype=torch.int32, device=self.dev)


ATTN = [  # heads, kv heads, dim, vdim, chunk, rotated dims, scaling
    (4, 2, 32, 16, 48, 32, (8.0, 1.0, 4.0, 256.0)),
    (6, 2, 64, 64, 100, 32, None),
    (3, 1, 96, 40, 17, 96, (4.0, 1.0, 2.0, 64.0)),
    (8, 8, 128, 128, 16, 64, None),
    (4, 1, 128, 128, 0, 128, (2.0, 0.5, 8.0, 96.0)),
    (2, 1, 160, 200, 33, 20, None),
    (2, 2, 264, 20, 64, 8, None),
    (18, 1, 128, 96, 29, 128, None),
]


@pytest.mark.parametrize("shape", ATTN, ids=lambda s: "-".join(str(x) for x in s[:5]))
def test_attention(be, shape):
    """Projections to output heads, in portions and in one piece: rotation, unit RMS, value mixing, chunks, sink."""
    from tgi_b200 import ops
    from tgi_b200.models.arch import MixerSpec
    from tgi_b200.models.mixers import RotaryTables

    dev, dt = be
    H, G, d, dv, chunk, rot, scaling = shape
    eps, lam, scale = 1e-3, 0.35, 1.7 * d ** -0.5
    spec = MixerSpec("attention", H, G, d, dv, rot_dims=rot, rot_base=500.0, rot_scaling=scaling)
    tab = RotaryTables(128, dev).get(spec)
    dk, dvp = ops.attention_pitch(d, dv, dt, dev)
    offs = [0, H * d + 8, H * d + 8 + G * d]
    proj = [rnd(i + 1, n, offs[2] + G * dv + 3).to(dt) for i, n in enumerate(LENGTHS)]
    first = [rnd(i + 5, n, G * dv).to(dt) for i, n in enumerate(LENGTHS)]
    want = []
    for p, f in zip(proj, first):
        p, f = p.double(), f.double()
        rotd = {"dims": rot, "base": 500.0}
        if scaling:
            rotd["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
        q = O.rms(O.rotate(p[:, :H * d].view(-1, H, d), rotd), eps)
        k = O.rms(O.rotate(p[:, offs[1]:offs[1] + G * d].view(-1, G, d), rotd), eps)
        v = (1 - lam) * p[:, offs[2]:offs[2] + G * dv] + lam * f
        want.append(O.attend(q, k, v.view(-1, G, dv), scale, chunk))
    for whole in (True, False):
        pg = Pages(dev, dt, G, dk, dvp)
        got = [torch.zeros(n, H, dv) for n in LENGTHS]
        steps = [([(0, n, i) for i, n in enumerate(LENGTHS)], [(i, 0, n) for i, n in enumerate(LENGTHS)])] if whole else cuts()
        for parts, rows in steps:
            st = Step(parts, dev)
            x = torch.cat([proj[i][a:b] for i, a, b in rows]).to(dev)
            f = torch.cat([first[i][a:b] for i, a, b in rows]).to(dev)
            q = ops.rotate_norm_store(x, offs, st.positions, tab.cos_sin, pg.slots(rows), pg.k, pg.v, H, G, d, dv, rot, True,
                                      eps, f, lam)
            o = ops.paged_attention(q, pg.k, pg.v, pg.table([r[0] for r in rows]), st.cu, st.kv, scale, max_q=st.max_q,
                                    max_kv=st.max_kv, chunk=chunk, sink=True)
            t = 0
            for i, a, b in rows:
                got[i][a:b] = o[t:t + b - a, :, :dv].float().cpu()
                t += b - a
        for i in range(2):
            close(got[i], want[i], dt)
        assert (pg.k[..., d:] == 0).all() and (pg.v[..., dv:] == 0).all()


@pytest.mark.parametrize("dims", [(128, 128), (64, 64), (256, 256), (40, 24)], ids=str)
@pytest.mark.parametrize("chunk", [16, 24, 64])
def test_chunk_edge(be, dims, chunk):
    """One key draws nearly all the weight of its query: the query sees it if it is the first of the chunk and does not
    if it is the last of the chunk before; prompts of several tiles and decoded tokens."""
    from tgi_b200 import ops

    dev, dt = be
    d, dv = dims
    L = 330
    dk, dvp = ops.attention_pitch(d, dv, dt, dev)
    for qpos in (chunk * 4, chunk * 4 + chunk - 1, L - 1):
        first = qpos // chunk * chunk
        for key in (first, first - 1):
            q, k, v = rnd(1, L, 2, d, std=0.1), rnd(2, L, 1, d, std=0.1), rnd(3, L, 1, dv)
            q[qpos], k[key, 0] = 0, 0
            q[qpos, :, 3], k[key, 0, 3] = 6.0, 6.0
            if key != qpos:
                k[qpos, 0, 3] = 0
            q, k, v = q.to(dt), k.to(dt), v.to(dt)
            js = [j for j in range(L) if O.sees(qpos, j, chunk)]
            want = O.sink_softmax(q[qpos].double() @ k[js, 0].double().t() * 0.25) @ v[js, 0].double()
            alone = v[key, 0].double()
            hit = (want - alone).norm() < 0.1 * alone.norm()
            assert bool(hit) == (key == first)
            pg = Pages(dev, dt, 1, dk, dvp, blocks=45)
            sl = pg.slots([(0, 0, L)]).long()
            pg.k.view(-1, 1, dk)[sl, :, :d] = k.to(dev)
            pg.v.view(-1, 1, dvp)[sl, :, :dv] = v.to(dev)
            qq = torch.nn.functional.pad(q, (0, dk - d)).to(dev)
            for start, n in ((0, qpos + 1), (max(0, qpos - 1), 2), (qpos, 1)):
                st = Step([(start, n, 0)], dev)
                o = ops.paged_attention(qq[start:start + n], pg.k, pg.v, pg.table([0]), st.cu, st.kv, 0.25, max_q=n,
                                        max_kv=qpos + 1, chunk=chunk, sink=True)
                close(o[-1, :, :dv].float(), want, dt)


def test_sink(be):
    """Scores far below 0 leave the output near zero (the sink takes the weight), scores far above leave it alone; the
    keys of a decode step are split over several blocks."""
    from tgi_b200 import ops

    dev, dt = be
    L, d = 500, 128
    for shift in (-8.0, -1.0, 0.0, 9.0):
        q, k, v = torch.zeros(1, 4, d), torch.zeros(L, 1, d), rnd(3, L, 1, d) + 1.0
        q[:, :, 0], k[:, 0, 0] = 4.0, shift
        k[:, 0, 1:] = rnd(4, L, d - 1, std=0.1)
        q, k, v = q.to(dt), k.to(dt), v.to(dt)
        s = (k[:, 0].double() @ q[0].double().t()).t() * 0.25
        want = O.sink_softmax(s) @ v[:, 0].double()
        pg = Pages(dev, dt, 1, d, d, blocks=69)
        sl = pg.slots([(0, 0, L)]).long()
        pg.k.view(-1, 1, d)[sl] = k.to(dev)
        pg.v.view(-1, 1, d)[sl] = v.to(dev)
        for n in (1, 2):
            st = Step([(L - n, n, 0)], dev)
            o = ops.paged_attention(q.expand(n, -1, -1).contiguous().to(dev), pg.k, pg.v, pg.table([0]), st.cu, st.kv, 0.25,
                                    max_q=n, max_kv=L, sink=True)
            close(o[-1].float(), want, dt)


# ---- recurrences ---------------------------------------------------------------------------------
def delta_case(dt, G, H, d, dv, taps, rank=16):
    """Random projections of two sequences and their parameters, the expected read-outs from the oracle."""
    case = {"offs": [], "w": {}}
    widths = [G * d, G * d, H * dv, H]
    off = 0
    for w in widths:
        case["offs"].append(off)
        off += (w + 7) // 8 * 8
    case["proj"] = [rnd(i + 1, n, off).to(dt) for i, n in enumerate(LENGTHS)]
    case["a"] = [rnd(i + 3, n, H * d).to(dt) for i, n in enumerate(LENGTHS)]
    case["conv"] = [rnd(7 + i, c, taps, std=0.7) for i, c in enumerate((G * d, G * d, H * dv))]
    case["a_log"], case["dt_bias"] = rnd(11, H), rnd(12, H * d) - 2.0
    want = []
    for x, a in zip(case["proj"], case["a"]):
        x, a = x.double(), a.double()
        cv = [O.silu(O.causal_conv(x[:, o:o + w], c.double())) for o, w, c in zip(case["offs"], widths, case["conv"])]
        of = [h // (H // G) for h in range(H)]
        q = (O.unit(cv[0].view(-1, G, d)) * d ** -0.5)[:, of]
        k = O.unit(cv[1].view(-1, G, d))[:, of]
        beta = torch.sigmoid(x[:, case["offs"][3]:case["offs"][3] + H])
        g = torch.exp(-torch.exp(case["a_log"].double())[None, :, None]
                      * torch.nn.functional.softplus(a + case["dt_bias"].double()).view(-1, H, d))
        want.append((O.delta_scan(q, k, cv[2].view(-1, H, dv), g, beta), g))
    return case, want


DELTA = [(2, 4, 24, 40, 4), (3, 3, 64, 64, 2), (1, 2, 100, 33, 3), (2, 2, 128, 128, 4), (1, 1, 150, 8, 5), (1, 3, 256, 20, 4),
         (2, 2, 16, 132, 1), (2, 4, 64, 260, 9), (2, 4, 128, 64, 7), (1, 2, 30, 50, 3)]


@pytest.mark.parametrize("shape", DELTA, ids=str)
def test_delta_rule(be, shape):
    """Convolutions, unit norms, decays and the scan: in one piece and in portions over slots that held other states."""
    from tgi_b200 import ops

    dev, dt = be
    G, H, d, dv, taps = shape
    case, want = delta_case(dt, *shape)
    pitch = ops.recurrent_pitch(d, dev)
    conv, a_log, bias = ops.conv_weights(case["conv"], dev), case["a_log"].to(dev), case["dt_bias"].to(dev)
    for whole in (True, False):
        conv_state = torch.full((4, taps - 1, 2 * G * d + H * dv), 3.0, dtype=dt, device=dev)
        state = torch.full((4, H, dv, pitch), 5.0, device=dev)
        got = [torch.zeros(n, H, dv) for n in LENGTHS]
        for parts, rows in ([([(0, n, 3 - i) for i, n in enumerate(LENGTHS)], [(i, 0, n) for i, n in enumerate(LENGTHS)])]
                            if whole else cuts()):
            st = Step(parts, dev)
            x = torch.cat([case["proj"][i][a:b] for i, a, b in rows]).to(dev)
            a_pre = torch.cat([case["a"][i][a:b] for i, a, b in rows]).to(dev)
            q, k, v, g, beta, qk = ops.delta_inputs(x, case["offs"], a_pre, conv, a_log, bias, st.cu, st.kv, st.slots,
                                                    conv_state, G, H, d, pitch, dv, st.max_q == 1)
            for j, (i, a, b) in enumerate(rows):
                lo, hi = int(st.cu[j]), int(st.cu[j + 1])
                close(g[lo:hi, :, :d], want[i][1][a:b], torch.float32)
            o = ops.delta_scan(q, k, v, g, beta, qk, st.cu, st.kv, st.slots, state, d, st.max_q)
            t = 0
            for i, a, b in rows:
                got[i][a:b] = o[t:t + b - a].cpu()
                t += b - a
        for i in range(2):
            close(got[i], want[i][0], dt)
        assert (state[1] == 5.0).all() and (conv_state[1] == 3.0).all()      # a slot nobody held


def test_delta_far_write(be):
    """A value written under a key that is never touched again comes back after a long decode when the decay is 1, and is
    gone where its channel forgets; single-token steps only."""
    from tgi_b200 import ops

    dev, dt = be
    if dt != torch.float32:
        pytest.skip("the scan is fp32 whatever the activations")
    H, d, dv, n = 2, 32, 24, 200
    q, k, v = torch.zeros(n, H, 32), torch.zeros(n, H, 32), rnd(1, n, H, dv)
    k[0, :, 5] = 1.0
    for t in range(1, n):
        k[t, :, 6 + t % 8] = 1.0
    q[-1, :, 5] = 1.0
    g = torch.ones(n, H, 32)
    g[:, 1, 5] = 0.9
    beta = torch.full((n, H), 0.5)
    state = torch.zeros(1, H, dv, 32, device=dev)
    for t in range(n):
        st = Step([(t, 1, 0)], dev)
        one = [x[t:t + 1].to(dev).contiguous() for x in (q, k, v, g, beta, (q * k).sum(-1))]
        o = ops.delta_scan(one[0], one[1], one[2], one[3], one[4], one[5], st.cu, st.kv, st.slots, state, d, 1)
    close(o[0, 0], 0.5 * v[0, 0], torch.float32)
    close(o[0, 1], 0.5 * v[0, 1] * 0.9 ** (n - 1), torch.float32, tol32=1e-3)


@pytest.mark.parametrize("shape", [(3, 16, 24), (2, 64, 40), (4, 32, 64), (1, 128, 128), (2, 200, 7)], ids=str)
def test_decay_attention(be, shape):
    from tgi_b200 import ops

    dev, dt = be
    H, d, dv = shape
    decay = [0.2, 0.9, 0.999, 1.0][4 - H:]
    offs = [0, (H * d + 7) // 8 * 8, 2 * ((H * d + 7) // 8 * 8)]
    proj = [rnd(i + 1, n, offs[2] + H * dv + 5).to(dt) for i, n in enumerate(LENGTHS)]
    want = [O.lightning_scan(*(O.silu(p.double()[:, o:o + w]).view(-1, H, w // H)
                               for o, w in zip(offs, (H * d, H * d, H * dv))), decay) for p in proj]
    for whole in (True, False):
        state = torch.full((4, H, dv, ops.recurrent_pitch(d, dev)), -2.0, device=dev)
        got = [torch.zeros(n, H, dv) for n in LENGTHS]
        for parts, rows in ([([(0, n, 3 - i) for i, n in enumerate(LENGTHS)], [(i, 0, n) for i, n in enumerate(LENGTHS)])]
                            if whole else cuts()):
            st = Step(parts, dev)
            x = torch.cat([proj[i][a:b] for i, a, b in rows]).to(dev)
            o = ops.decay_scan(x, offs, torch.tensor(decay, device=dev), st.cu, st.kv, st.slots, state, H, d, dv, st.max_q)
            t = 0
            for i, a, b in rows:
                got[i][a:b] = o[t:t + b - a].cpu()
                t += b - a
        for i in range(2):
            close(got[i], want[i], dt)
        assert (state[1] == -2.0).all()


@pytest.mark.parametrize("batch", [1, 40, 130])
@pytest.mark.parametrize("dims", [(64, 64), (128, 96)], ids=str)
def test_scan_layouts(be, batch, dims):
    """Few and many sequences in a step take different layouts of the state over lanes: prompts, then more tokens."""
    from tgi_b200 import ops

    dev, dt = be
    if dev.type == "cpu" and batch > 1:
        pytest.skip("one layout on the CPU")
    d, dv, H, lens = dims[0], dims[1], 2, (13, 6)
    pitch = ops.recurrent_pitch(d, dev)
    n = sum(lens)
    k, q, v = (rnd(i, batch, n, H, w) for i, w in enumerate((d, d, dv)))
    k, q = O.unit(k), O.unit(q)
    g, beta = torch.sigmoid(rnd(4, batch, n, H, d) + 2), torch.sigmoid(rnd(5, batch, n, H))
    decay = torch.tensor([0.7, 0.98])
    y = torch.cat([x.reshape(batch, n, -1) for x in (q, k, v)], -1).to(dt)
    s1, s2 = (torch.zeros(batch, H, dv, pitch, device=dev) for _ in range(2))
    pad = lambda x, value=0.0: torch.nn.functional.pad(x, (0, pitch - d), value=value)
    a = 0
    outs = [[], []]
    for m in lens:
        st = Step([(a, m, batch - 1 - i) for i in range(batch)], dev)
        row = lambda x: x[:, a:a + m].reshape(batch * m, *x.shape[2:]).to(dev).contiguous()
        outs[0].append(ops.delta_scan(row(pad(q)), row(pad(k)), row(v), row(pad(g)), row(beta), row((q * k).sum(-1)), st.cu,
                                      st.kv, st.slots, s1, d, m).cpu().view(batch, m, H, dv))
        outs[1].append(ops.decay_scan(row(y), [0, H * d, 2 * H * d], decay.to(dev), st.cu, st.kv, st.slots, s2, H, d, dv,
                                      m).cpu().view(batch, m, H, dv))
        a += m
    for i in {0, batch // 2, batch - 1}:
        close(torch.cat(outs[0], 1)[i], O.delta_scan(*(x[i].double() for x in (q, k, v, g, beta))), torch.float32)
        c = [O.silu(t.double()).view(n, H, -1) for t in y[i].split([H * d, H * d, H * dv], -1)]
        close(torch.cat(outs[1], 1)[i], O.lightning_scan(*c, decay.tolist()), torch.float32)


def test_padding_rows(be):
    """Rows of a captured batch without a sequence (length 0, slot -1) leave every pool as it is."""
    from tgi_b200 import ops

    dev, dt = be
    if dev.type == "cpu":
        pytest.skip("captured batches exist on the GPU only")
    case, _ = delta_case(dt, 2, 4, 24, 40, 4)
    cu = torch.arange(4, dtype=torch.int32, device=dev)
    kv = torch.tensor([0, 1, 0], dtype=torch.int32, device=dev)
    slots = torch.tensor([-1, 1, -1], dtype=torch.int32, device=dev)
    conv_state = torch.full((2, 3, 2 * 48 + 160), 3.0, dtype=dt, device=dev)
    state = torch.full((2, 4, 40, 32), 5.0, device=dev)
    r = ops.delta_inputs(case["proj"][0][:3].to(dev), case["offs"], case["a"][0][:3].to(dev),
                         ops.conv_weights(case["conv"], dev), case["a_log"].to(dev), case["dt_bias"].to(dev), cu, kv, slots,
                         conv_state, 2, 4, 24, 32, 40, True)
    ops.delta_scan(*r, cu, kv, slots, state, 24, 1)
    assert (state[0] == 5.0).all() and (conv_state[0] == 3.0).all() and not (state[1] == 5.0).any()


# ---- norms, residual, activation -----------------------------------------------------------------
@pytest.mark.parametrize("groups,width", [(3, 24), (4, 128), (1, 1500), (1, 30), (2, 1028)])
def test_gated_norm(be, groups, width):
    from tgi_b200 import ops

    dev, dt = be
    T, n = 5, groups * width
    for pad in (0, -n % 8):
        o, gate, w = rnd(1, T, groups, width), rnd(2, T, n + 16).to(dt), rnd(3, width)
        y = ops.gated_norm(o.to(dev), gate.to(dev)[:, 8:8 + n], w.to(dev), 1e-2, groups, n + pad)
        want = (O.rms(o.double(), 1e-2) * w.double()).reshape(T, n) * torch.sigmoid(gate[:, 8:8 + n].double())
        close(y[:, :n], want, dt)
        assert (y[:, n:] == 0).all()


@pytest.mark.parametrize("width", [80, 203, 4096, 6144, 20000])
def test_residual_norm(be, width):
    from tgi_b200 import ops

    dev, dt = be
    T = 7
    ids = torch.tensor([3, 0, 9, 9, 1, 5, 2], dtype=torch.int32, device=dev)
    table, w, delta = rnd(1, 10, width).to(dt), rnd(2, width).to(dt), rnd(3, T, width).to(dt)
    r = ops.embed_residual(ids, table.to(dev), 2.5)
    x = table.double()[ids.long().cpu()] * 2.5
    close(r, x, torch.float32)
    y, r1 = ops.residual_norm(None, r, w.to(dev), 1e-2)
    close(y, O.rms(x, 1e-2) * w.double(), dt)
    y, r2 = ops.residual_norm(delta.to(dev), r1, w.to(dev), 1e-2)
    x = x + delta.double()
    close(r2, x, torch.float32)
    close(y, O.rms(x, 1e-2) * w.double(), dt)
    rows = torch.tensor([6, 2], dtype=torch.int32, device=dev)
    y, none = ops.residual_norm(delta.to(dev), r1, w.to(dev), 1e-2, rows, keep=False)
    assert none is None
    close(y, (O.rms(x, 1e-2) * w.double())[[6, 2]], dt)
    # a stream of large values and small additions keeps them
    big = torch.full((1, width), 4096.0, device=dev)
    _, r3 = ops.residual_norm(torch.full((1, width), 0.0625, device=dev, dtype=dt), big, w.to(dev), 1e-2)
    assert (r3 == 4096.0625).all()


def test_erf_gelu(be):
    from tgi_b200 import ops

    dev, dt = be
    x = torch.cat([torch.linspace(-6, 6, 1001), rnd(1, 30)]).to(dt)
    close(ops.activation(x.to(dev), "gelu"), O.gelu_erf(x.double()), dt)


def test_sliced_product(be):
    """A column slice of a wider matrix is multiplied in place; odd inner sizes are padded."""
    from tgi_b200 import ops
    from tgi_b200.models.mixers import pad_columns, stack_rows

    dev, dt = be
    x = rnd(1, 37, 200).to(dt)
    w = rnd(2, 50, 24).to(dt)
    close(ops.linear(x.to(dev)[:, 104:128], w.to(dev)), x[:, 104:128].double() @ w.double().t(), dt)
    long = rnd(7, 700, 64).to(dt)        # many rows over a short inner dimension
    close(ops.linear_shallow(long.to(dev)[:, 32:56], w.to(dev)), long[:, 32:56].double() @ w.double().t(), dt)
    w = rnd(3, 50, 21).to(dt)
    close(ops.linear(x[:, :21].contiguous().to(dev), pad_columns(w.to(dev))), x[:, :21].double() @ w.double().t(), dt)
    m, offs = stack_rows([rnd(4, 5, 200).to(dt).to(dev), rnd(5, 16, 200).to(dt).to(dev), rnd(6, 3, 200).to(dt).to(dev)])
    assert offs == [0, 8, 24] and m.shape[0] == 32
    y = ops.linear(x.to(dev), m)
    close(y[:, 24:27], x.double() @ rnd(6, 3, 200).to(dt).double().t(), dt)
    assert (y[:, 5:8] == 0).all()


def test_split_decode_workspace_of_several_head_sizes():
    """Layers of different head sizes share the workspace of split decode steps: both its parts grow to what each needs, and
    what captured steps may still use is not freed."""
    from types import SimpleNamespace

    from tgi_b200.ops.cuda import _attention_parts

    st = SimpleNamespace(attn_part_o=None, attn_part_ml=None, kept={}, device=torch.device("cpu"))
    first = _attention_parts(st, 24, 256)
    o, ml = _attention_parts(st, 90, 64)                   # fewer outputs, more rows
    assert o is first[0] and o.numel() >= 90 * 64 and ml.numel() >= 90 * 2 and ml is not first[1]
    assert any(t is first[1] for t in st.kept["outgrown"])
    assert _attention_parts(st, 90, 64)[1] is ml
