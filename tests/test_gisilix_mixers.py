"""Each mechanism of the Gisilix decoder alone, against the plain implementation in ``gisilix_oracle``.

As in ``test_mixers``: the CPU ops and, where there is a GPU, the kernels in fp32 and bf16; sequences in portions cut at
awkward places, in batches beside other sequences, on pages in shuffled order that held other requests.
"""
import random

import numpy as np
import pytest
import torch

import gisilix_oracle as O
from test_mixers import LENGTHS, Pages, Step, be, close, cuts, rnd  # noqa: F401
from tgi_b200.utils import synthetic as syn


def plans():
    """Both sequences whole in one step, and the portions of ``SCHEDULE``."""
    yield [([(0, n, 0) for n in LENGTHS], [(i, 0, n) for i, n in enumerate(LENGTHS)])]
    yield list(cuts())


def mixer_for(be, layer, width, seed=1):
    """The product's mixer of one layer, and its tensors."""
    from tgi_b200.models.arch import ModelConfig
    from tgi_b200.models.mixers import RotaryTables, load_mixer

    dev, dt = be
    cfg = syn.gisilix_config([layer], width=width, eps=1e-3)
    sd = {k: v.to(torch.bfloat16) for k, v in syn.gisilix_state_dict(cfg, seed=seed).items()}
    w = syn.DictWeights({k: v.to(dev) for k, v in sd.items()}, dev, dt, bare_names=True)
    return load_mixer(ModelConfig(cfg).mixers[0], "l0.mix", w, 0, 1e-3, None, RotaryTables(512, dev)), (lambda n: sd[n].double())


def meta_for(st, rows, pg, expand):
    """Step metadata as the engine builds it; sequences with at least ``expand`` tokens have their keys written out."""
    from tgi_b200.models import mixers
    from tgi_b200.models.decoder import ForwardMeta

    tables = pg.table([r[0] for r in rows])
    meta = ForwardMeta(None, st.positions, pg.slots(rows), tables, st.cu, st.kv, st.max_q, st.max_kv)
    if expand is not None:
        slots = [(t[:, None].numpy() * 16 + np.arange(16)).reshape(-1).astype(np.int32) for t in tables.cpu()]
        meta.expansions = {}
        for window in expand[1]:
            plan = mixers.plan_expansion(window, [a for _, a, _ in rows], [b - a for _, a, b in rows], slots)
            if plan is not None:
                meta.expansions[window] = mixers.Expansion(*(torch.from_numpy(x).to(pg.dev) for x in plan[0]), *plan[1])
    return meta


def run(mixer, x, steps, expand=None, blocks=24):
    """Outputs of both sequences ``x`` brought as ``steps`` say."""
    dev, dt = mixer.device, mixer.dtype
    pg = Pages(dev, dt, 1, 8, 8, blocks=blocks)
    cache = mixer.cache_tensors(blocks, 16, 1, dev)
    for t in cache:                             # what another request left: any finite value, zeros where nobody writes
        used = (torch.rand(t.shape, generator=torch.Generator().manual_seed(3)) * 4 - 2).to(t)
        if mixer.spec.kind == "latent":
            r, o = mixer.spec.kv_rank, mixer.off_rot
            t[..., :r] = used[..., :r]
            t[..., o:o + mixer.spec.rot_dims] = used[..., o:o + mixer.spec.rot_dims]
        else:
            n = mixer.spec.dim if t is cache[0] else mixer.spec.vdim
            t[..., :n] = used[..., :n]
    got = [torch.zeros(*y.shape) for y in x]
    for parts, rows in steps:
        meta = meta_for(Step(parts, dev), rows, pg, expand)
        y = mixer(torch.cat([x[i][a:b] for i, a, b in rows]).to(dev), None, meta, None, cache).float().cpu()
        t = 0
        for i, a, b in rows:
            got[i][a:b] = y[t:t + b - a]
            t += b - a
    return got


# ---- latent attention ----------------------------------------------------------------------------
LATENT = [  # heads, dim, rotated dims, vdim, rank, window, YaRN
    (4, 24, 8, 20, 40, 13, (4.0, 8.0, 1.0, 128)),
    (8, 128, 64, 128, 512, 30, (40.0, 32.0, 1.0, 4096)),
    (6, 64, None, 64, 256, None, None),
    (3, 10, 6, 14, 30, 17, None),
    (1, 16, 2, 8, 64, 5, (2.0, 4.0, 4.0, 64)),
    (20, 32, 16, 32, 128, 1, (3.0, 16.0, 2.0, 100)),
    (2, 200, 40, 136, 600, 50, None),           # wider than the tensor-core kernels take
    (40, 64, 128, 96, 192, 40, None),
    (16, 100, None, 128, 500, None, None),
]


@pytest.mark.parametrize("shape", LATENT, ids=lambda s: "-".join(str(x) for x in s[:6]))
def test_latent_attention(be, shape, monkeypatch):
    """Hidden rows to hidden rows: latent norm, rotations, absorbed up-projections or written-out keys, window, head gates."""
    from tgi_b200.models import mixers

    H, d, rot, dv, rank, window, scaling = shape
    layer = (syn.gisilix_latent(H, d, dv, rank, scale=1.4 * d ** -0.5) if rot is None else
             syn.gisilix_rotated_latent(H, d, dv, rank, rot, window, 500.0, scaling, scale=1.4 * (d + rot) ** -0.5))
    mixer, W = mixer_for(be, layer, 72)
    x = [rnd(i + 1, n, 72).to(be[1]) for i, n in enumerate(LENGTHS)]
    want = [O.latent_attention(y.double(), W, "l0.mix.", layer["mixer"], 1e-3) for y in x]
    for expand in (None, 1, 16):                # none, every portion, only longer ones beside the others
        if expand is not None and mixer.full is None:
            continue
        monkeypatch.setattr(mixers, "EXPAND_TOKENS", expand or 10 ** 9)
        for steps in plans():
            got = run(mixer, x, steps, None if expand is None else (expand, [window or 0]))
            for g, w in zip(got, want):
                close(g, w, be[1])


@pytest.mark.parametrize("expand", [False, True])
@pytest.mark.parametrize("window", [1, 16, 25, 64, 130])
def test_latent_window_edge(be, window, expand):
    """One key draws nearly all the weight of its query: seen as the oldest key of the window, not seen one further back, in
    prompts of several tiles, short portions and decoded tokens."""
    from tgi_b200 import ops
    from tgi_b200.models.mixers import Expansion

    dev, dt = be
    H, rank, rot, L = 2, 40, 8, 330
    if expand and (dev.type != "cuda" or dt != torch.bfloat16):
        pytest.skip("written-out keys are a bf16 kernel")
    off, width = ops.latent_layout(rank, rot, dt, dev)
    for qpos in (window, 63, 64, 160, L - 1):
        for key in (qpos - window + 1, qpos - window):
            if key < 0:
                continue
            q, k = torch.zeros(L, H, width), torch.zeros(L, width)
            for lo, n in ((0, rank), (off, rot)):
                q[..., lo:lo + n], k[:, lo:lo + n] = rnd(lo + 1, L, H, n, std=0.1), rnd(lo + 2, L, n, std=0.1)
            q[qpos, :, off + 3], k[key, off + 3], k[key, :rank] = 7.0, 7.0, rnd(8, rank)     # the rotated part decides
            q, k = q.to(dt), k.to(dt)
            seen = [j for j in range(L) if O.sees(qpos, j, window)]
            p = torch.softmax(q[qpos].double() @ k[seen].double().t() * 0.4, -1)
            want = p @ k[seen, :rank].double()
            alone = k[key, :rank].double()
            assert bool((want - alone).norm() < 0.1 * alone.norm()) == (key == qpos - window + 1)
            pg = Pages(dev, dt, 1, 8, 8, blocks=45)
            table = pg.table([0])
            i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
            pages = torch.zeros(45, 16, 1, width, dtype=dt, device=dev)
            pages.view(-1, width)[pg.slots([(0, 0, L)]).long()] = k.to(dev)
            for n in (1, 2, 20, qpos + 1):
                if n > qpos + 1:
                    continue
                cu, kv = i32([0, n]), i32([qpos + 1])
                if expand:
                    dk, v = 128, torch.zeros(336, H, 256, dtype=dt, device=dev)      # keys: rotated part in front
                    v[:L, :, :rot], v[:L, :, rot:rot + rank] = k[:, None, off:off + rot].to(dev), k[:, None, :rank].to(dev)
                    both = torch.cat([v[..., :dk].reshape(336, -1), torch.nn.functional.pad(v[..., rot:rot + rank], (0, 128 - rank)).reshape(336, -1)], 1)
                    qq = torch.zeros(n, H, dk, dtype=dt, device=dev)
                    part = q[qpos + 1 - n:qpos + 1].to(dev)
                    qq[..., :rot], qq[..., rot:rot + rank] = part[..., off:off + rot], part[..., :rank]
                    plan = Expansion(None, torch.arange(21, dtype=torch.int32, device=dev)[None], kv, None, True, 0)
                    o = torch.zeros(n, H, 128, dtype=dt, device=dev)
                    ops.expanded_attention(qq, both.contiguous(), plan, cu, 0.4, window, n, None, o)
                else:
                    o = ops.latent_attention(q[qpos + 1 - n:qpos + 1].to(dev).contiguous(), pages, rank, table, cu, kv, 0.4, window, n, qpos + 1)
                close(o[-1, :, :rank], want, dt)


@pytest.mark.parametrize("heads,rank,rot,window", [(8, 40, 8, -1), (32, 512, 64, -1), (32, 512, 64, 100), (5, 64, 0, 33), (64, 128, 32, -1)],
                         ids=str)
def test_latent_decode_of_many_sequences(be, heads, rank, rot, window):
    """Single tokens of sequences from one key to hundreds: most are shared between CTAs, padding rows bring nothing."""
    from tgi_b200 import ops

    dev, dt = be
    lens = [1, 2, 700, 15, 16, 17, 63, 64, 65, 300, 0, 128, 129, 511, 33, 90, 0] + [40 + 3 * i for i in range(20)]
    off, width = ops.latent_layout(rank, rot, dt, dev)
    rng = random.Random(1)
    per = [-(-n // 16) for n in lens]
    order = rng.sample(range(1, sum(per) + 1), sum(per))
    table = torch.zeros(len(lens), max(per), dtype=torch.int32)
    pages, q = torch.zeros(sum(per) + 1, 16, 1, width), torch.zeros(len(lens), heads, width)
    for lo, n in ((0, rank), (off, rot)):
        pages[..., lo:lo + n], q[..., lo:lo + n] = rnd(1 + lo, sum(per) + 1, 16, 1, n), rnd(2 + lo, len(lens), heads, n)
    pages, q, gate = pages.to(dt), q.to(dt), rnd(5, len(lens), heads + 3).to(dt)
    want, scale = torch.zeros(len(lens), heads, rank), 2.0 * (rank + rot) ** -0.5
    for b, n in enumerate(lens):
        table[b, :per[b]] = torch.tensor(order[sum(per[:b]):sum(per[:b + 1])])
        if n:
            k = pages[table[b, :per[b]].long()].reshape(-1, width)[:n].double()
            k = k[max(0, n - window):] if window > 0 else k
            p = torch.softmax(q[b].double() @ k.t() * scale, -1)
            want[b] = p @ k[:, :rank] * O.sigmoid(gate[b, 3:].double())[:, None]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    got = ops.latent_attention(q.to(dev), pages.to(dev), rank, table.to(dev), i32(list(range(len(lens) + 1))), i32(lens), scale, window,
                               1, max(lens), gate.to(dev)[:, 3:])[..., :rank]
    if dev.type == "cuda":
        live = torch.tensor(lens) > 0
        assert (got[~live.to(dev)] == 0).all()
        close(got[live.to(dev)], want[live], dt)
    else:
        for b, n in enumerate(lens):
            if n:
                close(got[b], want[b], dt)


# ---- attention with row norms, temperature, caps, sinks and a gate ---------------------------------
ATTN = [  # heads, kv heads, dim, vdim, every, cap
    (4, 2, 24, 16, 20, 9.0),
    (8, 2, 128, 128, 7, 30.0),
    (6, 6, 48, 64, 1, 4.0),
    (3, 1, 22, 30, 33, 2.0),
    (16, 1, 64, 40, 64, 50.0),
    (2, 2, 256, 256, 16, 15.0),
    (2, 1, 264, 20, 25, 5.0),
]


@pytest.mark.parametrize("shape", ATTN, ids=lambda s: "-".join(map(str, s)))
def test_attention(be, shape):
    H, G, d, dv, every, cap = shape
    layer = syn.gisilix_attention(H, G, d, dv, 0.4, every, cap, scale=3.0 * d ** -0.5)
    mixer, W = mixer_for(be, layer, 72)
    x = [rnd(i + 1, n, 72).to(be[1]) for i, n in enumerate(LENGTHS)]
    mx = layer["mixer"]
    want = [O.attention(y.double(), O.attention_keys(y.double(), W, "l0.mix.", mx, 1e-3), W, "l0.mix.", mx, 1e-3) for y in x]
    for steps in plans():
        for g, w in zip(run(mixer, x, steps), want):
            close(g, w, be[1], tol16=2e-2)


@pytest.mark.parametrize("dims", [(128, 128), (64, 64), (256, 256), (40, 24)], ids=str)
def test_capped_scores_and_sinks(be, dims):
    """Scores far past the cap, a far key whose capped score still stands out, sinks from nothing to everything."""
    from tgi_b200 import ops

    dev, dt = be
    d, dv = dims
    H, G, L, cap = 4, 2, 300, 6.0
    dk, dvp = ops.attention_pitch(d, dv, dt, dev)
    sink = torch.tensor([-30.0, 0.0, 5.5, 60.0])
    for n in (1, 3, L):
        q, k, v = rnd(1, n, H, d, std=0.3), rnd(2, L, G, d, std=0.3), rnd(3, L, G, dv)
        q[-1, :, 2], k[7, :, 2] = 20.0, 30.0                     # raw score 60: capped to 6, e^6 against about 300 others
        q, k, v = q.to(dt), k.to(dt), v.to(dt)
        full = torch.cat([torch.zeros(L - n, H, d, dtype=dt), q])
        want = O.attend(full.double(), k.double(), v.double(), 0.1, cap=cap, sink=sink.double())[L - n:]
        assert want[-1, 3].abs().max() < 1e-6 and (want[-1, 0] - v[7, 0].double()).norm() < 0.7 * v[7, 0].double().norm()
        pg = Pages(dev, dt, G, dk, dvp, blocks=45)
        at = pg.slots([(0, 0, L)]).long()
        pg.k.view(-1, G, dk)[at, :, :d], pg.v.view(-1, G, dvp)[at, :, :dv] = k.to(dev), v.to(dev)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
        got = ops.paged_attention(torch.nn.functional.pad(q, (0, dk - d)).to(dev), pg.k, pg.v, pg.table([0]), i32([0, n]), i32([L]), 0.1,
                                  softcap=cap, max_q=n, max_kv=L, sink=sink.to(dev))
        for h in range(3):
            close(got[:, h, :dv], want[:, h], dt)
        assert got[:, 3].abs().max() < 1e-6


def test_row_norm_temperature_and_store(be):
    """Means over all heads (one loud head quiets the others), the step of the temperature, rows without a slot, queries only."""
    from tgi_b200 import ops

    dev, dt = be
    H, G, d, dv, n = 5, 2, 24, 8, 50
    offs = [0, H * d, H * d + G * d]
    x = rnd(1, n, offs[2] + G * dv + 8)
    x[:, :d] *= 20
    x = x.to(dt)
    wq, wk = rnd(2, H * d, std=0.3) + 1, rnd(3, G * d, std=0.3) + 1
    pos = torch.tensor([3 * i for i in range(n)], dtype=torch.int32)
    y = x.double()
    t = O.temperature(pos, 0.7, 16)
    assert t[4] == t[0] != t[5]                 # positions 12 and 15
    q = O.rms_norm(y[:, :H * d], wq.double(), 1e-3).view(n, H, d) * t[:, None, None]
    k = O.rms_norm(y[:, offs[1]:offs[2]], wk.double(), 1e-3).view(n, G, d)
    slots = torch.randperm(64, generator=torch.Generator().manual_seed(1))[:n].int()
    slots[4] = -1
    kc, vc = torch.zeros(4, 16, G, 32, dtype=dt, device=dev), torch.zeros(4, 16, G, 16, dtype=dt, device=dev)
    args = (pos.to(dev), slots.to(dev), kc, vc, wq.to(dev))
    got = ops.row_norm_store(x.to(dev), offs, *args, wk.to(dev), 1e-3, H, G, d, dv, 32, (0.7, 16))
    close(got[..., :d], q, dt)
    ok = slots >= 0
    close(kc.view(-1, G, 32)[slots[ok].long()][..., :d], k[ok], dt)
    close(vc.view(-1, G, 16)[slots[ok].long()][..., :dv], y[ok, offs[2]:offs[2] + G * dv].view(-1, G, dv), dt)
    assert (got[..., d:] == 0).all() and (kc[..., d:] == 0).all() and (kc != 0).any(-1).sum() == 49 * G
    before = kc.clone()
    alone = ops.row_norm_store(x[:, :H * d + 8].to(dev), [0], *args, None, 1e-3, H, G, d, dv, 32, (0.7, 16))
    assert torch.equal(alone, got) and torch.equal(kc, before)


# ---- stream, rotation, feed-forward ----------------------------------------------------------------
@pytest.mark.parametrize("width", [72, 80, 1001, 4096, 20000])
def test_layer_norm_on_the_stream(be, width):
    from tgi_b200 import ops

    dev, dt = be
    r, w, b = rnd(1, 9, width) + 30.0, rnd(2, width).to(dt), rnd(3, width).to(dt)
    d1, d2 = rnd(4, 9, width).to(dt), rnd(5, 9, width).to(dt)
    rows = torch.tensor([8, 0, 3], dtype=torch.int32)
    for delta in (None, d1, (d1, d2)):
        parts = () if delta is None else delta if isinstance(delta, tuple) else (delta,)
        total = r.double() + sum((p.double() for p in parts), torch.zeros(9, width, dtype=torch.float64))
        want = O.layer_norm(total, w.double(), b.double(), 1e-2)
        moved = None if delta is None else tuple(p.to(dev) for p in parts) if len(parts) > 1 else parts[0].to(dev)
        y, res = ops.residual_norm(moved, r.to(dev), w.to(dev), 1e-2, layer=True, bias=b.to(dev))
        close(y, want, dt)
        close(res, total, torch.float32)
        y, res = ops.residual_norm(moved, r.to(dev), w.to(dev), 1e-2, rows.to(dev), keep=False, layer=True, bias=b.to(dev))
        close(y, want[rows.long()], dt)
        assert res is None


@pytest.mark.parametrize("dims,base,sc", [(64, 10000.0, (40.0, 32.0, 1.0, 4096)), (32, 20000.0, (2.0, 32.0, 1.0, 512)),
                                          (8, 300.0, (4.0, 2.0, 2.0, 64)), (2, 50.0, (8.0, 1.0, 0.5, 32)),
                                          (16, 1000.0, (1.0, 32.0, 1.0, 100)), (24, 500.0, None)])
def test_rotary_table(dims, base, sc):
    from tgi_b200.models.arch import MixerSpec
    from tgi_b200.models.mixers import RotaryTables

    tab = RotaryTables(3000, torch.device("cpu")).get(MixerSpec("latent", 1, 1, 8, 8, rot_dims=dims, rot_base=base, rot_yarn=sc)).cos_sin
    freq, amp = O.yarn(dims, base, None if sc is None else dict(zip(("factor", "fast", "slow", "original"), sc)))
    ang = torch.arange(3000).double()[:, None] * torch.tensor(freq, dtype=torch.float64)
    assert (tab.double() - amp * torch.cat([ang.cos(), ang.sin()], 1)).abs().max() < 1e-6
    if sc and sc[0] > 1 and dims > 8:
        assert freq[0] == 1.0 and freq[-1] < base ** (-(dims - 2) / dims) * 0.9 and amp > 1


@pytest.mark.parametrize("T,width,E,top", [(1, 80, 10, 3), (37, 100, 5, 1), (600, 128, 40, 8), (5, 64, 3, 3), (9, 72, 200, 12)])
def test_router(be, T, width, E, top):
    from tgi_b200 import ops
    from tgi_b200.models.layers import FastLinear

    dev, dt = be
    x, w = rnd(1, T, width).to(dt), rnd(2, E, width, std=width ** -0.5).to(dt)
    bias = rnd(3, E, std=1.5)
    z = x.double() @ w.double().T + bias.double()
    want_id, want_w = O.route(z, top)
    if E > top:
        assert T < 5 or (want_id != O.route(z - bias.double(), top)[0]).any()      # the bias takes part in the choice
    gw, gi = ops.moe_route_softmax(x.to(dev), FastLinear(w.to(dev)).weight, bias.to(dev), top)
    sure = (lambda s: (s[:, :-1] - s[:, 1:]).min(-1).values > 1e-4)(torch.sort(z, -1, descending=True).values[:, :top + 1])
    assert sure.float().mean() > 0.8 or T == 1
    assert torch.equal(gi.cpu().long()[sure], want_id[sure])
    close(gw.cpu()[sure], want_w[sure], torch.float32)
    assert (gw.sum(-1).cpu() - 1).abs().max() < 1e-5
    big = ops.moe_route_softmax(x.to(dev), FastLinear(w.to(dev)).weight, bias.to(dev) + 300.0, top)[0]      # no overflow
    close(big.cpu()[sure], want_w[sure], torch.float32, tol32=1e-4)


@pytest.mark.parametrize("T,width,ff,E,top", [(1, 80, 24, 10, 3), (45, 100, 21, 5, 1), (300, 128, 64, 16, 4), (7, 64, 40, 3, 3), (33, 72, 8, 30, 11)])
def test_gated_experts(be, T, width, ff, E, top):
    from tgi_b200 import ops

    dev, dt = be
    x = rnd(1, T, width).to(dt)
    sd = {f"e{e}.{n}": rnd(10 + 3 * e + i, *s, std=s[1] ** -0.5).to(dt) for e in range(E)
          for i, (n, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))}
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(t))[:top] for t in range(T)]).int()
    wts = torch.softmax(rnd(4, T, top), -1)
    want = torch.zeros(T, width, dtype=torch.float64)
    for t in range(T):
        for e, p in zip(ids[t].tolist(), wts[t].double()):
            want[t] += p * O.dense(x[t:t + 1].double(), lambda n: sd[n].double(), f"e{e}.")[0]
    up, down, gate = (torch.stack([sd[f"e{e}.{n}"] for e in range(E)]).to(dev) for n in ("up", "down", "gate"))
    wu, wd = ops.plain_expert_weights(up, down, gate)
    close(ops.moe_plain_experts(x.to(dev), wu, wd, wts.to(dev), ids.to(dev), "silu", True), want, dt)
    swapped = ops.plain_expert_weights(gate, down, up)       # gate and up are not interchangeable
    with pytest.raises(AssertionError):
        close(ops.moe_plain_experts(x.to(dev), *swapped, wts.to(dev), ids.to(dev), "silu", True), want, dt, tol16=5e-2)


def test_plan_of_written_out_keys(monkeypatch):
    """Sequences with many tokens, the first key their window shows rounded down to a group, gaps, the limit on rows."""
    from tgi_b200.models import mixers

    monkeypatch.setattr(mixers, "EXPAND_TOKENS", 10)
    slots = [np.arange(1000 * i, 1000 * i + 400, dtype=np.int32) for i in range(4)]
    starts, counts = [0, 100, 50, 5], [20, 40, 1, 9]
    (rows, tables, kv, queries), (every, rest) = mixers.plan_expansion(24, starts, counts, slots)
    first = (100 - 23) // 16 * 16
    assert kv.tolist() == [20, 140 - first, 0, 0] and (every, rest) == (False, 9) and queries.tolist() == list(range(60))
    assert rows[:20].tolist() == list(range(20)) and set(rows[20:32]) == {0} and rows[32:32 + kv[1]].tolist() == list(range(1000 + first, 1140))
    assert len(rows) % 16 == 0 and tables[0, :2].tolist() == [0, 1] and tables[1, :5].tolist() == [2, 3, 4, 5, 6][:5]
    (rows, tables, kv, _), (every, rest) = mixers.plan_expansion(0, [0, 100], [20, 40], slots[:2])
    assert kv.tolist() == [20, 140] and (every, rest) == (True, 0)
    assert mixers.plan_expansion(0, [5, 0], [1, 9], slots[:2]) is None
    monkeypatch.setattr(mixers, "EXPAND_ROWS", 64)
    (rows, _, kv, queries), (every, rest) = mixers.plan_expansion(0, [100, 0], [40, 20], slots[:2])
    assert kv.tolist() == [0, 20] and (every, rest) == (False, 40) and queries.tolist() == list(range(40, 60)) and len(rows) == 32
