"""Each mechanism of the Sobivik decoder alone, against the plain implementation in ``sobivik_oracle``.

As in ``test_mixers``: the CPU ops and, where there is a GPU, the kernels in fp32 and bf16; sequences in portions cut at
awkward places, in batches beside other sequences, on pages and slots in shuffled order that held other requests.
"""
import math
import random

import numpy as np
import pytest
import torch

import sobivik_oracle as O
from test_mixers import LENGTHS, Pages, Step, be, close, cuts, rnd  # noqa: F401
from tgi_b200.utils import synthetic as syn

SLOTS = (2, 0)          # of the two sequences in pools of three


def plans():
    """Both sequences whole in one step, and the portions of ``SCHEDULE``."""
    yield [([(0, n, s) for n, s in zip(LENGTHS, SLOTS)], [(i, 0, n) for i, n in enumerate(LENGTHS)])]
    yield list(cuts(SLOTS))


def mixer_for(be, layer, width, seed=1):
    """The product's mixer of one layer, and its tensors."""
    from tgi_b200.models.arch import ModelConfig
    from tgi_b200.models.mixers import RotaryTables, load_mixer

    dev, dt = be
    cfg = syn.sobivik_config([layer], width=width, eps=1e-3)
    sd = {k: v.to(torch.bfloat16) for k, v in syn.sobivik_state_dict(cfg, seed=seed).items()}
    w = syn.DictWeights({k: v.to(dev) for k, v in sd.items()}, dev, dt, bare_names=True)
    mixer = load_mixer(ModelConfig(cfg).mixers[0], "l0.mix", w, 0, 1e-3, None, RotaryTables(512, dev), "l0.canon1")
    return mixer, (lambda n: sd[n].double())


def run(mixer, x, steps, expand=None, blocks=24):
    """Outputs of both sequences ``x`` brought as ``steps`` say; sequences with at least ``expand`` tokens have keys and values
    written out."""
    from tgi_b200.models import mixers
    from tgi_b200.models.decoder import ForwardMeta

    dev, dt, s = mixer.device, mixer.dtype, mixer.spec
    pg = Pages(dev, dt, 1, 8, 8, blocks=blocks)
    cache = mixer.page_tensors(blocks, 16, dev) + mixer.state_tensors(3, dev)
    for t in cache:                             # what another request left: any finite value, zeros where nobody writes
        used = (torch.rand(t.shape, generator=torch.Generator().manual_seed(3)) * 4 - 2).to(t)
        if s.kind == "latent":
            t[..., :s.kv_rank] = used[..., :s.kv_rank]
            t[..., mixer.off_rot:mixer.off_rot + s.rot_dims] = used[..., mixer.off_rot:mixer.off_rot + s.rot_dims]
        else:
            n = s.dim if s.kind == "decay" else 2 * s.dim if t is cache[0] else s.vdim
            t[..., :n] = used[..., :n]
    got = [torch.zeros(*y.shape) for y in x]
    for parts, rows in steps:
        st = Step(parts, dev)
        tables = pg.table([r[0] for r in rows])
        meta = ForwardMeta(None, st.positions, pg.slots(rows), tables, st.cu, st.kv, st.max_q, st.max_kv, state_slots=st.slots)
        if expand is not None:
            slots = [(t[:, None].numpy() * 16 + np.arange(16)).reshape(-1).astype(np.int32) for t in tables.cpu()]
            plan = mixers.plan_expansion(s.window, [a for _, a, _ in rows], [b - a for _, a, b in rows], slots)
            if plan is not None:
                meta.expansions = {s.window: mixers.Expansion(*(torch.from_numpy(v).to(dev) for v in plan[0]), *plan[1])}
        y = mixer(torch.cat([x[i][a:b] for i, a, b in rows]).to(dev), None, meta, None, cache).float().cpu()
        t = 0
        for i, a, b in rows:
            got[i][a:b] = y[t:t + b - a]
            t += b - a
    return got


# ---- mixers: hidden rows to hidden rows ------------------------------------------------------------
RETENTION = [(3, 24, 20, None), (4, 64, 40, [0.25, 0.9, 0.999, 1.0]), (1, 128, 256, None), (2, 200, 7, [0.5, 0.98]), (5, 10, 30, None),
             (2, 32, 128, [0.0, 0.984375])]


@pytest.mark.parametrize("shape", RETENTION, ids=lambda s: "-".join(map(str, s[:3])))
def test_retention(be, shape):
    layer = syn.sobivik_retention(*shape)
    mixer, W = mixer_for(be, layer, 72)
    x = [rnd(i + 1, n, 72).to(be[1]) for i, n in enumerate(LENGTHS)]
    want = [O.retention(y.double(), W, "l0.mix.", layer["mixer"], 1e-3) for y in x]
    for steps in plans():
        for g, w in zip(run(mixer, x, steps), want):
            close(g, w, be[1], tol16=2e-2)


LATENT = [  # heads, dim, vdim, query rank, rank, rotated dims, window, YaRN
    (4, 24, 20, 32, 40, 8, 13, (4.0, 8.0, 1.0, 128)),
    (8, 128, 128, 192, 512, 64, 30, (40.0, 32.0, 1.0, 4096)),
    (3, 10, 14, 21, 30, 6, 17, None),
    (1, 16, 8, 1, 64, 2, 5, (2.0, 4.0, 4.0, 64)),
    (20, 32, 96, 130, 128, 16, 1, (3.0, 16.0, 2.0, 100)),
    (2, 200, 136, 72, 600, 40, 50, None),           # wider than the tensor-core kernels take
    (5, 64, 72, 88, 192, 32, 64, None),
]


@pytest.mark.parametrize("shape", LATENT, ids=lambda s: "-".join(str(x) for x in s[:7]))
def test_latent_attention(be, shape, monkeypatch):
    """Latents of queries and of keys, halves rotated, sinks, window, gate per element; up-projections absorbed or written out."""
    from tgi_b200.models import mixers

    H, d, dv, qr, rank, rot, window, scaling = shape
    layer = syn.sobivik_latent(H, d, dv, qr, rank, rot, window, 500.0, scaling, scale=1.4 * (d + rot) ** -0.5)
    mixer, W = mixer_for(be, layer, 72)
    x = [rnd(i + 1, n, 72).to(be[1]) for i, n in enumerate(LENGTHS)]
    want = [O.latent_attention(y.double(), W, "l0.mix.", layer["mixer"], 1e-3) for y in x]
    for expand in (None, 1, 16):                # none, every portion, only longer ones beside the others
        if expand is not None and mixer.full is None:
            continue
        monkeypatch.setattr(mixers, "EXPAND_TOKENS", expand or 10 ** 9)
        for steps in plans():
            for g, w in zip(run(mixer, x, steps, expand), want):
                close(g, w, be[1], tol16=2e-2)


ATTN = [  # heads, kv heads, dim, vdim, window, kept
    (4, 2, 12, 28, 20, 3),
    (8, 2, 64, 128, 16, 4),              # sizes of the tensor-core kernels
    (18, 1, 40, 88, 9, 5),               # more query maps of a key head than one tile of decoding holds
    (6, 6, 32, 64, 33, 17),
    (3, 1, 22, 30, 1, 1),
    (2, 2, 100, 256, 25, 20),
    (2, 1, 130, 20, 31, 2),              # wider than the tensor-core kernels take
    (4, 4, 64, 100, 24, 0),
    (4, 1, 16, 40, 0, 0),                # everything visible
]


@pytest.mark.parametrize("shape", ATTN, ids=lambda s: "-".join(map(str, s)))
def test_differential_attention(be, shape):
    H, G, d, dv, window, keep = shape
    layer = syn.sobivik_attention(H, G, d, dv, window, keep, 0.35, scale=2.0 * d ** -0.5)
    mixer, W = mixer_for(be, layer, 72)
    assert abs(mixer.map_lambda - float(O.strength(W, "l0.mix.", 0.35))) < 1e-9 and abs(mixer.map_lambda - 0.35) > 1e-3
    x = [rnd(i + 1, n, 72).to(be[1]) for i, n in enumerate(LENGTHS)]
    want = [O.differential_attention(y.double(), W, "l0.mix.", layer["mixer"], 1e-3) for y in x]
    for steps in plans():
        for g, w in zip(run(mixer, x, steps), want):
            close(g, w, be[1], tol16=3e-2)


# ---- kept first tokens -------------------------------------------------------------------------------
def one_loud_key(L, G, H, d, dv, qpos, key, dt):
    """Queries and keys of small scores but for one key that the query at ``qpos`` gives nearly all its weight."""
    q, k, v = rnd(1, L, H, d, std=0.1), rnd(2, L, G, d, std=0.1), rnd(3, L, G, dv)
    q[qpos, :, 3 % d], k[key, :, 3 % d] = 7.0, 7.0
    return q.to(dt), k.to(dt), v.to(dt)


@pytest.mark.parametrize("keep,window", [(1, 1), (4, 16), (20, 25), (70, 64), (130, 40), (200, 130), (5, 300)], ids=str)
@pytest.mark.parametrize("dims", [(4, 2, 128, 128), (20, 2, 128, 128), (4, 2, 64, 64), (2, 2, 256, 256), (4, 2, 40, 24)], ids=str)
def test_kept_tokens_and_window_edge(be, dims, keep, window):
    """The last kept token is seen from anywhere, the next one only inside the window; the window's own edge stays where it is.
    Prompts of several tiles, short portions and decoded tokens."""
    from tgi_b200 import ops

    dev, dt = be
    H, G, d, dv = dims
    L, pitch = 330, ops.attention_pitch(dims[2], dims[3], be[1], be[0])
    for qpos in (keep, min(keep + window, L - 2), 128 + 15, L - 1):
        for key in sorted({keep - 1, keep, 0, qpos - window + 1, qpos - window}):
            if key < 0 or key > qpos:
                continue
            q, k, v = one_loud_key(L, G, H, d, dv, qpos, key, dt)
            seen = [j for j in range(L) if O.sees(qpos, j, window, keep)]
            want = torch.stack([torch.softmax(k[seen, h // (H // G)].double() @ q[qpos, h].double() * 0.4, 0) @ v[seen, h // (H // G)].double()
                                for h in range(H)])
            alone = v[key].double().repeat_interleave(H // G, 0)
            assert bool((want - alone).norm() < 0.1 * alone.norm()) == (key in seen)
            pg = Pages(dev, dt, G, *pitch, blocks=45)
            at = pg.slots([(0, 0, L)]).long()
            pg.k.view(-1, G, pitch[0])[at, :, :d], pg.v.view(-1, G, pitch[1])[at, :, :dv] = k.to(dev), v.to(dev)
            i32 = lambda z: torch.tensor(z, dtype=torch.int32, device=dev)
            for n in (1, 2, 20, qpos + 1):
                if n > qpos + 1:
                    continue
                part = torch.nn.functional.pad(q[qpos + 1 - n:qpos + 1], (0, pitch[0] - d)).to(dev)
                o = ops.paged_attention(part, pg.k, pg.v, pg.table([0]), i32([0, n]), i32([qpos + 1]), 0.4, window=window, max_q=n,
                                        max_kv=qpos + 1, keep=keep)
                close(o[-1, :, :dv], want, dt)


@pytest.mark.parametrize("heads,kv_heads,d", [(8, 2, 128), (40, 2, 128), (4, 4, 64), (3, 1, 40)], ids=str)
def test_kept_tokens_of_many_sequences(be, heads, kv_heads, d):
    """Single tokens of sequences of all lengths in one step, in a batch that is split over keys and in one that is not."""
    from tgi_b200 import ops

    dev, dt = be
    window, keep = 50, 21
    pitch, _ = ops.attention_pitch(d, d, dt, dev)
    for lens in ([700, 3], [1, 20, 21, 22, 70, 71, 72, 0, 16, 17, 300, 333] + [30 + 7 * i for i in range(40)]):
        rng = random.Random(1)
        per = [-(-n // 16) for n in lens]
        order = rng.sample(range(1, sum(per) + 1), sum(per))
        table = torch.zeros(len(lens), max(per), dtype=torch.int32)
        k, v = (torch.zeros(sum(per) + 1, 16, kv_heads, pitch) for _ in range(2))
        k[..., :d], v[..., :d] = rnd(1, *k.shape[:3], d), rnd(2, *v.shape[:3], d)
        q = torch.nn.functional.pad(rnd(3, len(lens), heads, d), (0, pitch - d))
        k, v, q = k.to(dt), v.to(dt), q.to(dt)
        want = torch.zeros(len(lens), heads, d)
        for b, n in enumerate(lens):
            table[b, :per[b]] = torch.tensor(order[sum(per[:b]):sum(per[:b + 1])])
            seen = [j for j in range(n) if O.sees(n - 1, j, window, keep)]
            if n:
                kb, vb = (t[table[b, :per[b]].long()].reshape(-1, kv_heads, pitch)[seen].double().repeat_interleave(heads // kv_heads, 1) for t in (k, v))
                p = torch.softmax(torch.einsum("hd,lhd->hl", q[b].double(), kb) * 1.5 * d ** -0.5, -1)
                want[b] = torch.einsum("hl,lhd->hd", p, vb)[:, :d]
        i32 = lambda z: torch.tensor(z, dtype=torch.int32, device=dev)
        got = ops.paged_attention(q.to(dev), k.to(dev), v.to(dev), table.to(dev), i32(list(range(len(lens) + 1))), i32(lens),
                                  1.5 * d ** -0.5, window=window, max_q=1, max_kv=max(lens), keep=keep) if dev.type == "cuda" or 0 not in lens else None
        if got is None:                         # the plain ops want a key for every query
            continue
        live = torch.tensor(lens) > 0
        close(got[live.to(dev)][..., :d], want[live], dt)


# ---- sinks of latent attention -------------------------------------------------------------------------
@pytest.mark.parametrize("heads,rank,rot,window", [(8, 40, 8, -1), (32, 512, 64, 100), (5, 64, 16, 33), (64, 128, 32, -1)], ids=str)
def test_latent_sinks(be, heads, rank, rot, window):
    """Sinks from nothing to everything: decoded tokens of many sequences (most shared between workers), portions of one."""
    from tgi_b200 import ops

    dev, dt = be
    lens = [1, 2, 700, 15, 16, 17, 64, 65, 300, 129, 511] + [40 + 3 * i for i in range(20)]
    off, width = ops.latent_layout(rank, rot, dt, dev)
    per = [-(-n // 16) for n in lens]
    order = random.Random(1).sample(range(1, sum(per) + 1), sum(per))
    table = torch.zeros(len(lens), max(per), dtype=torch.int32)
    pages, q = torch.zeros(sum(per) + 1, 16, 1, width), torch.zeros(len(lens), heads, width)
    for lo, n in ((0, rank), (off, rot)):
        pages[..., lo:lo + n], q[..., lo:lo + n] = rnd(1 + lo, sum(per) + 1, 16, 1, n), rnd(2 + lo, len(lens), heads, n)
    pages, q, scale = pages.to(dt), q.to(dt), 2.0 * (rank + rot) ** -0.5
    sink = rnd(6, heads, std=3.0)
    sink[0], sink[1], sink[2] = -60.0, 0.0, 80.0
    rows = lambda b, n: pages[table[b, :per[b]].long()].reshape(-1, 1, width)[:n].double()
    for b in range(len(lens)):
        table[b, :per[b]] = torch.tensor(order[sum(per[:b]):sum(per[:b + 1])])

    def last(b, n, qq):
        k = rows(b, n)
        full = torch.cat([torch.zeros(n - len(qq), heads, width, dtype=torch.float64), qq.double()])
        seen = k if window < 0 else k[max(0, n - window):]
        s = torch.cat([full[-1] @ seen[:, 0].T * scale, sink.double()[:, None]], 1)
        return torch.softmax(s, -1)[:, :-1] @ seen[:, 0, :rank]

    want = torch.stack([last(b, n, q[b:b + 1]) for b, n in enumerate(lens)])
    assert want[:, 2].abs().max() < 1e-6
    i32 = lambda z: torch.tensor(z, dtype=torch.int32, device=dev)
    got = ops.latent_attention(q.to(dev), pages.to(dev), rank, table.to(dev), i32(list(range(len(lens) + 1))), i32(lens), scale, window,
                               1, max(lens), sink=sink.to(dev))[..., :rank]
    close(got, want, dt)
    assert got[:, 2].abs().max() < 1e-6
    for b, n in ((2, 5), (8, 70), (3, 15)):     # the last n tokens of a sequence in one step
        qq = torch.zeros(n, heads, width)
        for lo, c in ((0, rank), (off, rot)):
            qq[..., lo:lo + c] = rnd(9 + lo, n, heads, c)
        qq = qq.to(dt)
        got = ops.latent_attention(qq.to(dev), pages.to(dev), rank, table[b:b + 1].to(dev), i32([0, n]), i32([lens[b]]), scale, window, n,
                                   lens[b], sink=sink.to(dev))[-1, :, :rank]
        close(got, last(b, lens[b], qq), dt)


def test_sinks_with_keys_written_out(be):
    from tgi_b200 import ops
    from tgi_b200.models.mixers import Expansion

    dev, dt = be
    if dev.type != "cuda" or dt != torch.bfloat16:
        pytest.skip("written-out keys are a bf16 kernel")
    H, L = 4, 300
    sink = torch.tensor([-60.0, 0.0, 4.0, 80.0])
    i32 = lambda z: torch.tensor(z, dtype=torch.int32, device=dev)
    for dk, n, window in ((128, 300, 37), (192, 41, 200), (128, 2, 16)):
        q, k, v = rnd(1, n, H, dk).to(dt), rnd(2, 304, H, dk).to(dt), rnd(3, 304, H, 128).to(dt)
        full = torch.cat([torch.zeros(L - n, H, dk, dtype=dt), q])
        want = O.attend(full.double(), k[:L].double(), v[:L].double(), dk ** -0.5, window=window, sink=sink.double())[L - n:]
        plan = Expansion(None, torch.arange(19, dtype=torch.int32, device=dev)[None], i32([L]), None, True, 0)
        o = torch.zeros(n, H, 128, dtype=dt, device=dev)
        ops.expanded_attention(q.to(dev), torch.cat([k.reshape(304, -1), v.reshape(304, -1)], 1).contiguous().to(dev), plan, i32([0, n]),
                               dk ** -0.5, window, n, None, o, sink.to(dev))
        for h in range(3):
            close(o[:, h], want[:, h], dt)
        assert o[:, 3].abs().max() < 1e-6


# ---- maps --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims", [(5, 5, 24, 8, 64, 16), (8, 2, 64, 128, 128, 128), (3, 1, 11, 30, 22, 30), (4, 2, 64, 300, 512, 512)], ids=str)
def test_maps(be, dims):
    """Places of the maps in key rows and queries, rows without a slot; difference, norm, factor and gate of the outputs."""
    from tgi_b200 import ops

    dev, dt = be
    H, G, d, dv, Dk, Dv = dims
    n, up = 37, lambda z: (z + 7) // 8 * 8
    offs = [0, up(2 * H * d), up(2 * H * d) + up(2 * G * d)]
    x = rnd(1, n, offs[2] + up(G * dv) + 8).to(dt)
    slots = torch.randperm(64, generator=torch.Generator().manual_seed(1))[:n].int()
    slots[4] = -1
    kc, vc = torch.zeros(4, 16, G, Dk, dtype=dt, device=dev), torch.zeros(4, 16, G, Dv, dtype=dt, device=dev)
    q = ops.map_store(x.to(dev), offs, slots.to(dev), kc, vc, H, G, d, dv).cpu()
    maps = x[:, :2 * H * d].view(n, H, 2, d)
    assert torch.equal(q[:, 0::2, :d], maps[:, :, 0]) and torch.equal(q[:, 1::2, d:2 * d], maps[:, :, 1])
    assert (q[:, 0::2, d:] == 0).all() and (q[:, 1::2, :d] == 0).all() and (q[..., 2 * d:] == 0).all()
    ok = slots >= 0
    assert torch.equal(kc.cpu().view(-1, G, Dk)[slots[ok].long(), :, :2 * d], x[ok, offs[1]:offs[1] + 2 * G * d].view(-1, G, 2 * d))
    assert torch.equal(vc.cpu().view(-1, G, Dv)[slots[ok].long(), :, :dv], x[ok, offs[2]:offs[2] + G * dv].view(-1, G, dv))
    assert (kc != 0).any(-1).sum() == (n - 1) * G and (kc[..., 2 * d:] == 0).all() and (vc[..., dv:] == 0).all()

    a, g = rnd(5, n, 2 * H, Dv).to(dt), rnd(6, n, H + 3).to(dt)
    a[3] = 1e-3 * a[3]                          # the constant inside the root counts
    y = a[..., :dv].double()
    for gate in (None, g[:, 3:]):
        want = O.difference(y[:, 0::2], y[:, 1::2], -0.7, 0.25, 1e-3)
        if gate is not None:
            want = want * O.sigmoid(gate.double())[:, :, None]
        got = ops.map_difference(a.to(dev), None if gate is None else g.to(dev)[:, 3:], -0.7, 0.75, 1e-3, dv)
        close(got, want.reshape(n, -1), dt)
        close(got[3], want[3].reshape(-1), dt)


# ---- stream ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [72, 80, 1001, 4096, 20000])
def test_stream_step(be, width):
    """Norm of the output, addition, weighted sum with the new result among the kept ones, norm, factor; chosen rows."""
    from tgi_b200 import ops

    dev, dt = be
    T, eps = 9, 1e-2
    r, d, w, post = rnd(1, T, width), rnd(2, T, width, std=0.05).to(dt), rnd(3, width).to(dt), rnd(4, width).to(dt)
    streams, avg = rnd(5, 7, T, width), rnd(6, 5)
    rows = torch.tensor([8, 0, 3], dtype=torch.int32)
    to = lambda t: None if t is None else t.to(dev)
    for delta, p, average in ((None, None, None), (d, None, None), (d, post, None), (d, post, avg), (None, None, avg), (d, post, avg[:1])):
        new = r.double() + (0 if delta is None else delta.double() if p is None else O.over_rms(delta.double(), eps) * p.double())
        total = new if average is None else O.average([*streams[:len(average) - 1].double(), new], average.double())
        want = O.over_rms(total, eps) * w.double()
        kept = streams.clone().to(dev)
        y, res = ops.stream_step(to(delta), to(p), to(r), to(w), eps, average=to(average), streams=kept, gain=0.4)
        close(y, 0.4 * want, dt)
        close(res, total, torch.float32)
        if average is not None:
            close(kept[len(average) - 1], new, torch.float32)
            same = [i for i in range(7) if i != len(average) - 1]
            assert torch.equal(kept.cpu()[same], streams[same])
        before = kept.clone()
        y, res = ops.stream_step(to(delta), to(p), to(r), to(w), eps, rows.to(dev), keep=False, average=to(average), streams=kept)
        close(y, want[rows.long()], dt)
        assert res is None and torch.equal(kept, before)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 9])
@pytest.mark.parametrize("width", [24, 72, 1000, 1001])
def test_input_convolution(be, taps, width):
    """Behind the norm, in portions of all lengths and single tokens, on slots that held other requests."""
    from tgi_b200 import ops
    from tgi_b200.models.mixers import InputConv

    dev, dt = be
    conv = InputConv(rnd(7, width, taps).to(torch.bfloat16), dt, dev)
    x, w, k = [rnd(i + 1, n, width) for i, n in enumerate(LENGTHS)], rnd(3, width).to(dt), rnd(7, width, taps).to(torch.bfloat16).double()
    want = []
    for y in x:
        h = (O.over_rms(y.double(), 1e-3) * w.double()).to(dt).double()         # kept as it is stored
        want.append(h + O.causal_conv(h, k))
    for steps in plans():
        state = conv.state(3, dev)
        assert tuple(state.shape) == (3, taps - 1, width)
        state += 2.0
        for parts, rows in steps:
            st = Step(parts, dev)
            got, _ = ops.stream_step(None, None, torch.cat([x[i][a:b] for i, a, b in rows]).to(dev), w.to(dev), 1e-3,
                                     conv=ops.ShortConv(conv.weight, state, st.cu, st.kv, st.slots, st.max_q == 1))
            close(got, torch.cat([want[i][a:b] for i, a, b in rows]), dt)
        assert (state[1] == 2.0).all()


def test_padding_rows(be):
    """Rows of a captured batch without a sequence (length 0, slot -1) leave every state as it is."""
    from tgi_b200 import ops

    dev, dt = be
    if dev.type != "cuda":
        pytest.skip("captured batches exist on the GPU only")
    W, i32 = 64, lambda z: torch.tensor(z, dtype=torch.int32, device=dev)
    state, w = torch.full((3, 3, W), 5.0, dtype=dt, device=dev), torch.ones(4, W, device=dev)
    conv = ops.ShortConv(w, state, i32([0, 1, 2, 3]), i32([7, 0, 0]), i32([1, -1, -1]), True)
    out, _ = ops.stream_step(None, None, rnd(1, 3, W).to(dev), torch.ones(W, dtype=dt, device=dev), 1e-5, conv=conv)
    assert torch.isfinite(out).all() and (state[0] == 5).all() and (state[2] == 5).all() and (state[1, :2] == 5).all()
    assert (state[1, 2] != 5).all()
    kc = torch.zeros(2, 16, 2, 64, dtype=dt, device=dev)
    vc = kc.clone()
    ops.map_store(torch.ones(3, 512, dtype=dt, device=dev), [0, 256, 384], i32([-1, -1, -1]), kc, vc, 4, 2, 32, 64)
    assert not kc.any() and not vc.any()


# ---- scan --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("batch", [1, 40, 130])
@pytest.mark.parametrize("dims", [(64, 64), (128, 96), (40, 33)], ids=str)
def test_scan_without_activation(be, batch, dims):
    """Few and many sequences take different layouts; prompts, more tokens, single tokens; k's factor; states far from zero."""
    from tgi_b200 import ops

    dev, dt = be
    if dev.type == "cpu" and batch > 1:
        pytest.skip("one layout on the CPU")
    d, dv, H, lens = dims[0], dims[1], 2, (13, 6, 1, 1)
    n, up = sum(lens), lambda z: (z + 7) // 8 * 8
    decay = torch.tensor([0.7, 0.998])
    q, k, v = (rnd(i, batch, n, H, w) for i, w in enumerate((d, d, dv)))
    offs = [0, up(H * d), 2 * up(H * d)]
    y = torch.zeros(batch, n, offs[2] + up(H * dv))
    for o, t in zip(offs, (q, k, v)):
        y[..., o:o + t.shape[2] * t.shape[3]] = t.flatten(2)
    y = y.to(dt)
    state = torch.full((batch, H, dv, ops.recurrent_pitch(d, dev)), 3.0, device=dev)
    a, outs = 0, []
    for m in lens:
        st = Step([(a, m, batch - 1 - i) for i in range(batch)], dev)
        outs.append(ops.decay_scan(y[:, a:a + m].reshape(batch * m, -1).to(dev).contiguous(), offs, decay.to(dev), st.cu, st.kv, st.slots,
                                   state, H, d, dv, m, "", d ** -0.5).cpu().view(batch, m, H, dv))
        a += m
    for i in {0, batch // 2, batch - 1}:
        c = [y[i, :, o:o + H * w].double().view(n, H, w) for o, w in zip(offs, (d, d, dv))]
        close(torch.cat(outs, 1)[i], O.retain(*c, decay.tolist()), torch.float32)


def test_far_token_in_the_state(be):
    """What one token wrote hundreds of tokens ago is what is left of it, through prompts, portions and single tokens."""
    from tgi_b200 import ops

    dev, dt = be
    H, d, dv, n = 3, 32, 16, 400
    decay, pitch = [0.5, 0.99, 1.0], ops.recurrent_pitch(32, be[0])
    offs = [0, H * d, 2 * H * d]
    y = torch.zeros(n, offs[2] + H * dv)
    y[0, H * d:2 * H * d].view(H, d)[:, 5] = 2.0
    y[0, offs[2]:] = rnd(1, H * dv)
    y[n - 1, :H * d].view(H, d)[:, 5] = 1.5
    y = y.to(dt)
    for portions in ([n], [1] * n, [350, 1, 2, 46, 1], [2] * (n // 2)):
        state, at = torch.ones(1, H, dv, pitch, device=dev), 0
        for m in portions:
            st = Step([(at, m, 0)], dev)
            o = ops.decay_scan(y[at:at + m].to(dev), offs, torch.tensor(decay, device=dev), st.cu, st.kv, st.slots, state, H, d, dv, m, "", 0.25)
            at += m
        v = y[0, offs[2]:].double().view(H, dv)
        for h in range(1, H):
            close(o[-1, h], 0.75 * v[h] * decay[h] ** (n - 1), torch.float32, tol32=1e-3)
        assert o[-1, 0].abs().max() < 1e-30


def test_rotation_in_halves_by_reordered_rows(be):
    """Rotating neighbours of reordered projections gives the scores that rotating halves gives; far positions."""
    from tgi_b200.models.arch import MixerSpec
    from tgi_b200.models.mixers import RotaryTables

    rot = {"dims": 12, "base": 5000.0, "scaling": dict(zip(("factor", "fast", "slow", "original"), (8.0, 16.0, 1.0, 256)))}
    spec = MixerSpec("latent", 1, 1, 8, 8, rot_dims=12, rot_base=5000.0, rot_yarn=(8.0, 16.0, 1.0, 256))
    tab = RotaryTables(400, be[0]).get(spec).cos_sin.cpu().double()
    x = rnd(1, 400, 1, 12).double()
    want = O.rotate_halves(x, rot)[:, 0]
    order = torch.arange(12).view(2, 6).t().reshape(-1)
    u, v = x[:, 0, order][:, 0::2], x[:, 0, order][:, 1::2]
    got = torch.stack([u * tab[:, :6] - v * tab[:, 6:], v * tab[:, :6] + u * tab[:, 6:]], -1).flatten(1)
    assert (got - want[:, order]).abs().max() < 1e-5 and abs(O.yarn(12, 5000.0, rot["scaling"])[1] - (0.1 * math.log(8) + 1)) < 1e-12
