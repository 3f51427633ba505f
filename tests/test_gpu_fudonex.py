"""Fudonex family on the GPU against the float64 oracle (oracle/fudonex_oracle.py): every mechanism alone through its
operator, then whole models through the serving path (ScheduleBatch → worker → kernels, decode through the captured CUDA
graphs) under every way of cutting and batching the same tokens, then greedy generation through the semi-PD engine."""
import pytest
import torch

from oracle import fudonex_oracle as F
from tests import fudonex_helpers as C
from tests import rimidra_helpers as H

pytestmark = pytest.mark.gpu

DEV = "cuda"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _close(got, want, dtype, what="", tol32=2e-5, tol16=3e-2):
    tol = tol32 if dtype == torch.float32 else tol16
    err = (got.double().cpu() - want.double().cpu()).abs().max().item()
    ref = want.double().abs().max().item() + 1e-9
    assert err <= tol * ref, f"{what}: max abs err {err:.3e} vs ref max {ref:.3e}"


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def i64(x):
    return torch.tensor(x, dtype=torch.int64, device=DEV)


# =================================================================================================
# mechanisms alone
# =================================================================================================
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [7, 36, 256, 1000, 4096, 8200])
def test_residual_update_with_the_norm_on_the_output(dtype, width):
    from semi_pd_b200 import ops
    dt = DT[dtype]
    g = torch.Generator().manual_seed(width)
    T, eps = 5, 1e-3
    x = torch.randn(T, width, generator=g) * 3
    y = (torch.randn(T, width, generator=g) * 0.3).to(dt)
    coef = torch.randn(width, generator=g)
    w = (torch.randn(width, generator=g) * 0.3).to(dt)
    xd = x.to(DEV)
    _close(ops.residual_postnorm(xd, None, None, eps, dt), x, dt, "operand alone", tol32=1e-7, tol16=5e-3)
    _close(xd, x, torch.float32, "nothing was added", tol32=1e-9)
    h = ops.residual_postnorm(xd, y.to(DEV), coef.to(DEV), eps, dt)
    x1 = x.double() + F.unit_rms(y.double(), eps) * coef.double()
    _close(xd, x1, torch.float32, "update", tol32=1e-6)
    _close(h, x1, dt, "next operand", tol32=1e-6, tol16=5e-3)
    h = ops.residual_postnorm(xd, y.to(DEV), coef.to(DEV), eps, dt, weight=w.to(DEV), weight_offset=1.0)
    x2 = x1 + F.unit_rms(y.double(), eps) * coef.double()
    _close(xd, x2, torch.float32, "second update", tol32=1e-6)
    _close(h, F.rms_norm_around_one(x2, w, eps), dt, "norm of the sum", tol32=2e-6, tol16=1e-2)
    h = ops.residual_postnorm(xd, None, None, eps, dt, weight=w.to(DEV), weight_offset=1.0)
    _close(h, F.rms_norm_around_one(x2, w, eps), dt, "norm alone", tol32=2e-6, tol16=1e-2)


def test_logit_cap():
    from semi_pd_b200 import ops
    z = torch.linspace(-200, 200, 3 * 77).view(3, 77)
    _close(ops.softcap_f32_(z.to(DEV), 13.0), F.soft_cap(z.double(), 13.0), torch.float32, "cap", tol32=1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kvh,dk,dv,rot,paired", [
    (4, 2, 16, 24, 8, False), (1, 1, 10, 6, 10, False), (8, 4, 64, 64, 64, False), (2, 1, 6, 4, 0, False),
    (4, 2, 32, 128, 32, False), (5, 1, 128, 64, 128, False), (3, 1, 128, 256, 64, False), (20, 4, 128, 128, 128, False),
    (2, 1, 300, 36, 100, False), (4, 2, 64, 32, 64, True)])
def test_norms_before_the_rotation(dtype, heads, kvh, dk, dv, rot, paired):
    """q, k, v as slices of one wider row: biases, a norm per head with a weight on q and k and without one on v, rotation
    with a table whose cos and sin carry a magnitude, k and v scattered into cache pools."""
    from semi_pd_b200 import ops
    dt = DT[dtype]
    T, eps = 5, 1e-2
    g = torch.Generator().manual_seed(dk * 31 + dv + heads)
    sizes = [heads * dk, kvh * dk, kvh * dv]
    row = torch.randn(T, sum(sizes) + (8 if dk % 8 == 0 else 3), generator=g).to(dt)
    qb, kb, vb = (torch.randn(n, generator=g) for n in sizes)
    qw, kw = 1 + 0.3 * torch.randn(dk, generator=g), 1 + 0.3 * torch.randn(dk, generator=g)
    pos, loc = [0, 1, 77, 300, 599], [9, 2, 5, 11, 3]
    spec = {"dims": rot, "base": 300.0, "scaling": {"factor": 3.0, "original": 80, "fast": 3.0, "slow": 0.5}}
    table = None
    if rot:
        f, mag = F.rotary_frequencies(spec)
        ang = torch.arange(600, dtype=torch.float64)[:, None] * f[None]
        table = (torch.cat([ang.cos(), ang.sin()], -1) * mag).float().to(DEV)
    rd = row.to(DEV)
    q, k, v = rd[:, : sum(sizes)].split(sizes, -1)
    k_pool, v_pool = torch.zeros(12, kvh * dk, device=DEV, dtype=dt), torch.zeros(12, kvh * dv, device=DEV, dtype=dt)
    q_out = torch.empty(T, heads * dk, device=DEV, dtype=dt)
    ops.rotary_segments([
        ops.rotary_segment(q, q_out, heads, dk, rot, bias=qb.to(DEV), norm_eps=eps, norm_weight=qw.to(DEV)),
        ops.rotary_segment(k, k_pool, kvh, dk, rot, bias=kb.to(DEV), to_pool=True, norm_eps=eps, norm_weight=kw.to(DEV)),
        ops.rotary_segment(v, v_pool, kvh, dv, 0, bias=vb.to(DEV), to_pool=True, norm_eps=eps),
    ], i64(pos), table, dt, loc=i64(loc), paired=paired)
    rq, rk, rv = (t.double() for t in row[:, : sum(sizes)].split(sizes, -1))
    q64 = F.rms_norm((rq + qb.double()).view(T, heads, dk), qw, eps)
    k64 = F.rms_norm((rk + kb.double()).view(T, kvh, dk), kw, eps)
    if paired:  # the same rotation on channels reordered from pairs to halves and back
        perm = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2), torch.arange(rot, dk)])
        q64, k64 = (F.rotate(t[..., perm], pos, spec)[..., torch.argsort(perm)] for t in (q64, k64))
    else:
        q64, k64 = F.rotate(q64, pos, spec), F.rotate(k64, pos, spec)
    _close(q_out, q64.reshape(T, -1), dt, "q", tol16=1e-2)
    _close(k_pool[loc], k64.reshape(T, -1), dt, "k", tol16=1e-2)
    _close(v_pool[loc], F.unit_rms((rv + vb.double()).view(T, kvh, dv), eps).reshape(T, -1), dt, "v", tol16=1e-2)
    assert float(k_pool[0].abs().max()) == 0 and float(v_pool[1].abs().max()) == 0, "other slots stay untouched"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,groups,part", [(5, 1, 96), (3, 4, 24), (7, 5, 3), (2, 1, 4096), (1, 2, 1000), (2, 1, 14000)])
def test_gate_before_a_norm_of_equal_parts(dtype, rows, groups, part):
    from semi_pd_b200 import ops
    dt = DT[dtype]
    g = torch.Generator().manual_seed(part)
    n = groups * part
    y = torch.randn(rows, n, generator=g) * torch.rand(n, generator=g) * 4
    wide = torch.randn(rows, n + 16, generator=g).to(dt)
    w = (1 + 0.2 * torch.randn(n, generator=g)).to(dt)
    got = ops.gated_group_norm(y.to(DEV), wide.to(DEV)[:, 8: 8 + n], w.to(DEV), groups, 1e-3)
    want = F.gated_group_norm(y.double(), wide.double()[:, 8: 8 + n], w, groups, 1e-3)
    _close(got, want, dt, "gated group norm", tol32=5e-6, tol16=1e-2)


class _Portions:
    """Two sequences fed in unequal portions (one idle in one of them), then decoded beside a padded row; then the first
    one's slot is used again by a new sequence.  `run(rows_a, rows_b, kw)` gets the row ranges of both sequences."""

    SLOTS = [4, 2]
    CUTS = ((3, 1), (1, 2), (17, 0), (2, 40), (35, 5))  # single tokens, pairs, odd and even counts, several kernel blocks

    def __init__(self):
        self.lens = [sum(c[i] for c in self.CUTS) + 3 for i in (0, 1)]

    def extends(self):
        at = [0, 0]
        for n in self.CUTS:
            yield ([(at[0], at[0] + n[0]), (at[1], at[1] + n[1])],
                   dict(req_pool_indices=i64(self.SLOTS), prefix_lens=i32(at), extend_lens=i32(list(n)),
                        extend_start_loc=i32([0, n[0]])))
            at = [at[0] + n[0], at[1] + n[1]]

    def decodes(self):
        at = [sum(c[0] for c in self.CUTS), sum(c[1] for c in self.CUTS)]
        for _ in range(3):
            yield at, dict(req_pool_indices=i64(self.SLOTS + [4]), seq_lens=i64([at[0] + 1, at[1] + 1, 1]),
                           out_cache_loc=i64([9, 3, 0]))
            at = [at[0] + 1, at[1] + 1]

    def again(self, n):
        return dict(req_pool_indices=i64([4]), prefix_lens=i32([0]), extend_lens=i32([n]), extend_start_loc=i32([0]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("channels,taps,bias", [(48, 4, True), (24, 1, True), (37, 3, False), (1100, 2, True), (264, 8, False),
                                                (5, 5, True), (40, 6, False), (16, 7, True)])
def test_short_convolution_keeps_its_last_inputs(dtype, channels, taps, bias):
    from semi_pd_b200 import ops
    dt = DT[dtype]
    P = _Portions()
    g = torch.Generator().manual_seed(channels + taps)
    seqs = [torch.randn(n, channels, generator=g).to(dt) for n in P.lens]
    w = (torch.randn(channels, taps, generator=g) * 0.6).to(dt)
    b = torch.randn(channels, generator=g).to(dt) if bias else None
    want = [F.short_conv(s.double(), w, b) for s in seqs]
    state = torch.full((6, max(taps - 1, 1) * channels), 50.0, device=DEV) if taps > 1 else None  # stale values
    wd, bd = w.T.contiguous().to(DEV), b.to(DEV) if bias else None

    def run(x, **kw):  # the input is a slice of a wider row
        wide = torch.cat([torch.full((x.shape[0], 8), 9.0, dtype=dt), x, torch.full((x.shape[0], 8), 9.0, dtype=dt)], 1)
        return ops.short_conv(wide.to(DEV)[:, 8: 8 + channels], wd, bd, state, **kw)

    for (ra, rb), kw in P.extends():
        got = run(torch.cat([seqs[0][ra[0]:ra[1]], seqs[1][rb[0]:rb[1]]]), max_extend_len=40, **kw)
        _close(got, torch.cat([want[0][ra[0]:ra[1]], want[1][rb[0]:rb[1]]]), dt, f"portion {ra} {rb}", tol16=1e-2)
    for at, kw in P.decodes():
        got = run(torch.stack([seqs[0][at[0]], seqs[1][at[1]], seqs[1][0]]), **kw)
        _close(got[:2], torch.stack([want[0][at[0]], want[1][at[1]]]), dt, f"decoding {at}", tol16=1e-2)
    got = run(seqs[1][:3], max_extend_len=3, **P.again(3))
    _close(got, want[1][:3], dt, "slot used again", tol16=1e-2)


RECURRENCES = [
    # heads, key heads, head_dim, v_dim
    (4, 2, 16, 24), (2, 1, 32, 64), (3, 3, 64, 40), (2, 1, 128, 128), (4, 4, 96, 32), (1, 1, 1, 5), (3, 1, 7, 3), (2, 2, 160, 40),
    (1, 1, 256, 33), (6, 2, 20, 36), (2, 1, 66, 34),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("form", ["ssd", "delta"])
@pytest.mark.parametrize("heads,kh,dk,dv", RECURRENCES)
def test_head_decay_recurrence(form, dtype, heads, kh, dk, dv):
    """Both recurrences in portions of odd and even length, decoding beside a padded row, a slot used again; q, k, v and
    the gate projections are slices of one wider row; decays from nearly none to nearly all."""
    from semi_pd_b200 import ops
    dt = DT[dtype]
    P = _Portions()
    g = torch.Generator().manual_seed(dk * 7 + dv + heads)
    sizes = [kh * dk, kh * dk, heads * dv, heads, heads]
    seqs = [torch.randn(n, sum(sizes), generator=g).to(dt) for n in P.lens]
    dt_bias, a_log = torch.rand(heads, generator=g) * 4 - 4, torch.rand(heads, generator=g) * 5 - 4
    skip = torch.randn(heads, generator=g) if form == "ssd" else None
    scale = dk ** -0.5 if form == "delta" else 1.0
    want = []
    for s in seqs:
        q, k, v, z, b = (t.double() for t in s.split(sizes, -1))
        q, k, v = q.view(-1, kh, dk), k.view(-1, kh, dk), v.view(-1, heads, dv)
        step, decay = F.head_decay(z, a_log, dt_bias)
        if form == "ssd":
            o = F.ssd_recurrence(v, k, q, step, decay, skip)
        else:
            o = F.delta_recurrence(F.unit_vector(q) * scale, F.unit_vector(k), v, torch.sigmoid(b), decay)
        want.append(o.reshape(len(s), -1))
    state = torch.full((6, heads, dv, dk), 7.0, device=DEV)  # stale values that position 0 must ignore
    par = dict(num_heads=heads, num_k_heads=kh, head_dim=dk, v_dim=dv, form=form, dt_bias=dt_bias.to(DEV),
               a_log=a_log.to(DEV), skip=skip.to(DEV) if skip is not None else None, q_scale=scale, unit_eps=F.UNIT_EPS)

    def run(rows, **kw):
        q, k, v, z, b = rows.to(DEV).split(sizes, -1)
        return ops.head_decay_recurrence(q, k, v, z, state, b=b if form == "delta" else None, **par, **kw)

    tol = dict(tol32=2e-5, tol16=2e-5)  # everything inside is fp32 whatever the inputs' dtype
    for (ra, rb), kw in P.extends():
        got = run(torch.cat([seqs[0][ra[0]:ra[1]], seqs[1][rb[0]:rb[1]]]), **kw)
        _close(got, torch.cat([want[0][ra[0]:ra[1]], want[1][rb[0]:rb[1]]]), dt, f"portion {ra} {rb}", **tol)
    for at, kw in P.decodes():
        got = run(torch.stack([seqs[0][at[0]], seqs[1][at[1]], seqs[1][0]]), **kw)
        _close(got[:2], torch.stack([want[0][at[0]], want[1][at[1]]]), dt, f"decoding {at}", **tol)
    got = run(seqs[1][:5], **P.again(5))
    _close(got, want[1][:5], dt, "slot used again", **tol)
    assert float((state[[0, 1, 3, 5]] - 7.0).abs().max()) == 0, "other slots stay untouched"


def test_recurrence_does_not_depend_on_the_cut():
    """Bit for bit where the pairs of tokens fall the same way, to rounding where they do not."""
    from semi_pd_b200 import ops
    g = torch.Generator().manual_seed(3)
    T, Hh, d = 50, 2, 64
    x = torch.randn(T, 3 * Hh * d + 2 * Hh, generator=g).to(DEV)
    q, k, v, z, b = x.split([Hh * d] * 3 + [Hh, Hh], -1)
    par = dict(num_heads=Hh, num_k_heads=Hh, head_dim=d, v_dim=d, form="delta", dt_bias=torch.zeros(Hh, device=DEV) - 2,
               a_log=torch.zeros(Hh, device=DEV) - 2, q_scale=d ** -0.5)

    def run(cuts):
        state, at, out = torch.zeros(2, Hh, d, d, device=DEV), 0, []
        for n in cuts:
            r = slice(at, at + n)
            out.append(ops.head_decay_recurrence(q[r], k[r], v[r], z[r], state, i64([1]), b=b[r], prefix_lens=i32([at]),
                                                 extend_lens=i32([n]), extend_start_loc=i32([0]), **par))
            at += n
        return torch.cat(out)

    whole = run([50])
    assert torch.equal(whole, run([2, 16, 30, 2]))
    assert (whole - run([1, 7, 3, 39])).abs().max() < 2e-6 * whole.abs().max()


# ---- attention over a window and pooled blocks -----------------------------------------------------------------
class _Runs:
    """Requests over shuffled runs of `run_len` consecutive slots, with block rows behind them."""

    def __init__(self, lens, run_len, size, seed=0):
        g = torch.Generator().manual_seed(seed)
        need = [-(-n // run_len) for n in lens]
        self.runs = sum(need) + 3
        order = torch.randperm(self.runs, generator=g).tolist()
        self.slots, self.r2t = [], torch.zeros(len(lens) + 2, max(lens) + 4, dtype=torch.int32)
        self.req = list(range(1, len(lens) + 1))
        for r, n, m in zip(self.req, lens, need):
            runs, order = order[:m], order[m:]
            pos = torch.arange(n)
            s = torch.tensor(runs)[pos // run_len] * run_len + 1 + pos % run_len
            self.slots.append(s)
            self.r2t[r, :n] = s.to(torch.int32)
        self.base = self.runs * run_len + 1
        self.per = -(-run_len // size)
        self.rows = self.base + self.runs * self.per
        self.blocks = (size, run_len, self.base)

    def block_rows(self, i):
        size, run_len, base = self.blocks
        last = self.slots[i][size - 1:: size] - 1
        return base + last // run_len * self.per + last % run_len // size


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,run_len,row", [(1, 16, 24), (2, 16, 6), (5, 16, 40), (16, 16, 128), (24, 16, 8), (32, 128, 512),
                                              (7, 128, 1100), (600, 64, 16)])
def test_block_means(dtype, size, run_len, row):
    """Rows of the blocks that a batch completes, and no others, in portions and in decoding."""
    from semi_pd_b200 import ops
    dt = DT[dtype]
    lens = [max(3 * size + 2, 20), 2 * size + 1]
    lay = _Runs(lens, run_len, size, seed=size)
    g = torch.Generator().manual_seed(row)
    k, v = torch.randn(lay.base, row, generator=g).to(dt), torch.randn(lay.base, row + 8, generator=g).to(dt)
    kp, vp = torch.full((lay.rows, row), 77.0, dtype=dt), torch.full((lay.rows, row + 8), 77.0, dtype=dt)
    kp[: lay.base], vp[: lay.base] = k, v
    kp, vp, r2t = kp.to(DEV), vp.to(DEV), lay.r2t.to(DEV)
    done = [0, 0]
    cut = [(size - 1 or 1, 1), (1, size), (size + 3, 0)]
    for n in cut + [(10 ** 6, 10 ** 6)]:  # the last portion: all but two tokens
        n = [max(min(m, l - 2 - d), 0) for m, l, d in zip(n, lens, done)]
        ops.pool_key_blocks(kp, vp, r2t, i64(lay.req), lay.blocks, prefix_lens=i32(done), extend_lens=i32(n),
                            max_extend_len=max(n) if max(n) else 1)
        done = [a + b for a, b in zip(done, n)]
    for _ in range(2):  # decoding beside a padded row (its page starts with slot 0)
        done = [d + 1 for d in done]
        ops.pool_key_blocks(kp, vp, r2t, i64(lay.req + [0]), lay.blocks, seq_lens=i64(done + [size]))
    assert done == lens
    written = set()
    for i, n in enumerate(lens):
        rows = lay.block_rows(i)
        assert len(rows) == n // size
        for b, r in enumerate(rows.tolist()):
            tok = lay.slots[i][b * size: (b + 1) * size]
            _close(kp[r], k[tok].double().mean(0), dt, f"key block {b}", tol32=1e-6, tol16=5e-3)
            _close(vp[r], v[tok].double().mean(0), dt, f"value block {b}", tol32=1e-6, tol16=5e-3)
            written.add(r)
    rest = [r for r in range(lay.base, lay.rows) if r not in written]
    assert not rest or float((kp[rest].float() - 77).abs().max()) == 0, "rows of incomplete blocks stay untouched"
    assert torch.equal(kp[: lay.base].cpu(), k) and torch.equal(vp[: lay.base].cpu(), v)


ATTN_CASES = [
    # name, H, G, dk, dv, window, block, run_len
    ("small", 4, 2, 16, 24, 12, 8, 16),
    ("one", 1, 1, 6, 5, 1, 1, 16),
    ("pairs-of-tokens", 3, 3, 10, 4, 1, 2, 16),
    ("tiles", 8, 2, 64, 64, 40, 16, 128),
    ("tiles-wide-keys", 4, 1, 128, 64, 70, 5, 128),
    ("tiles-32", 4, 2, 32, 32, 33, 3, 32),
    ("group-decode", 6, 2, 40, 64, 20, 24, 16),
    ("long-blocks", 2, 1, 16, 16, 9, 50, 32),
    ("many-heads", 20, 1, 64, 64, 30, 7, 128),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ATTN_CASES, ids=[c[0] for c in ATTN_CASES])
def test_attention_over_window_and_blocks(dtype, case):
    """Ragged portions and decoding.  Chosen queries look sharply at the key just inside their window while the key just
    outside attracts twice as much, or at the last block they see while the block that is not yet seen (its tokens lie
    between the blocks and the window: they are not seen at all) attracts twice as much, or at the first block of all."""
    from semi_pd_b200 import ops
    _, Hh, G, dk, dv, window, size, run_len = case
    dt = DT[dtype]
    lens, pre = [263, 41, 1, 150], [200, 0, 0, 149]
    lay = _Runs(lens, run_len, size, seed=dk)
    g = torch.Generator().manual_seed(dk + dv)
    sinks = torch.randn(Hh, generator=g) + 1
    kp, vp = torch.zeros(lay.rows, G * dk, dtype=dt), torch.zeros(lay.rows, G * dv, dtype=dt)
    qs, wants = [], []
    gain = 6.0
    for i, (n, p0) in enumerate(zip(lens, pre)):
        q, k = torch.randn(n, Hh, dk, generator=g), torch.randn(n, G, dk, generator=g)
        v = torch.randn(n, G, dv, generator=g)
        picks = {n - 1: "edge", p0 + (n - p0) // 2: "block", p0 + (n - p0) // 3: "first"}
        for t, what in picks.items():
            h = Hh - 1
            kk, d = k[:, h // (Hh // G)], q[t, h] / q[t, h].norm()
            q[t, h] = d * gain
            nb = max(t - window + 1, 0) // size
            if what == "edge" and t >= window:
                kk[t - window + 1], kk[t - window] = d * gain, d * gain * 2
            elif what == "block" and nb:
                kk[(nb - 1) * size: nb * size] = d * gain
                kk[nb * size: max(t - window + 1, nb * size)] = d * gain * 2
            elif what == "first" and nb:
                kk[:size] = d * gain
        q, k, v = q.to(dt), k.to(dt), v.to(dt)
        wants.append(F.windowed_pooled_attention(q.double(), k.double(), v.double(), 0.4, window=window, pool=size, sinks=sinks))
        qs.append(q)
        kp[lay.slots[i]], vp[lay.slots[i]] = k.reshape(n, -1), v.reshape(n, -1)
    kp, vp, r2t, req = kp.to(DEV), vp.to(DEV), lay.r2t.to(DEV), i64(lay.req)
    kw = dict(num_q_heads=Hh, num_kv_heads=G, head_dim=dk, v_dim=dv, sm_scale=0.4, window=window, sinks=sinks.to(DEV),
              blocks=lay.blocks)
    for a, b in ((([0] * 4), pre), (pre, lens)):  # the prefixes' blocks, then the portions'
        ext = [y - x for x, y in zip(a, b)]
        ops.pool_key_blocks(kp, vp, r2t, req, lay.blocks, prefix_lens=i32(a), extend_lens=i32(ext), max_extend_len=max(ext))
    ext = [n - p for n, p in zip(lens, pre)]
    q_ext = torch.cat([q[p:].reshape(n - p, -1) for q, n, p in zip(qs, lens, pre)]).to(DEV)
    want_ext = torch.cat([w[p:].reshape(n - p, -1) for w, n, p in zip(wants, lens, pre)])
    starts = [sum(ext[:i]) for i in range(4)]
    for bound in (max(ext), 0):  # the tensor-core prefill kernel where it applies, and the CUDA-core one
        got = ops.attn_general(q_ext, kp, vp, r2t, req, prefix_lens=i32(pre), extend_lens=i32(ext),
                               extend_start_loc=i32(starts), max_extend_len=bound, **kw)
        _close(got, want_ext, dt, f"portions (bound {bound})", tol16=2e-2)
    q_dec = torch.stack([q[-1].reshape(-1) for q in qs]).to(DEV)
    got = ops.attn_general(q_dec, kp, vp, r2t, req, seq_lens=i64(lens), **kw)
    _close(got, torch.stack([w[-1].reshape(-1) for w in wants]), dt, "decoding", tol16=2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_decoded_position_around_the_block_edges(dtype):
    """Token-by-token decoding with blocks written as they complete: positions before, at and after the first window, every
    block's first appearance, runs' borders."""
    from semi_pd_b200 import ops
    dt = DT[dtype]
    n, window, size, run_len, Hh, G, dk = 75, 7, 6, 16, 4, 2, 32
    lay = _Runs([n], run_len, size, seed=1)
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(n, x, dk, generator=g).to(dt) for x in (Hh, G, G))
    q = (q.float() * 2).to(dt)
    want = F.windowed_pooled_attention(q.double(), k.double(), v.double(), 0.3, window=window, pool=size)
    kp, vp = (torch.full((lay.rows, G * dk), 30.0, dtype=dt, device=DEV) for _ in range(2))  # stale rows show
    r2t, req = lay.r2t.to(DEV), i64(lay.req)
    got = []
    for t in range(n):
        s = lay.slots[0][t]
        kp[s], vp[s] = k[t].reshape(-1).to(DEV), v[t].reshape(-1).to(DEV)
        ops.pool_key_blocks(kp, vp, r2t, req, lay.blocks, seq_lens=i64([t + 1]))
        got.append(ops.attn_general(q[t].reshape(1, -1).to(DEV), kp, vp, r2t, req, seq_lens=i64([t + 1]), num_q_heads=Hh,
                                    num_kv_heads=G, head_dim=dk, v_dim=dk, sm_scale=0.3, window=window, blocks=lay.blocks))
    err = (torch.cat(got).double().cpu() - want.reshape(n, -1)).abs().max(-1).values
    assert err.max() <= (1e-5 if dtype == "float32" else 3e-2) * want.abs().max(), f"worst at position {int(err.argmax())}"


def test_attention_refuses_blocks_it_cannot_place():
    from semi_pd_b200 import ops
    z = torch.zeros(1, 16, device=DEV)
    pool = torch.zeros(40, 16, device=DEV)
    kw = dict(num_q_heads=1, num_kv_heads=1, head_dim=16, v_dim=16, sm_scale=1.0, seq_lens=i64([1]))
    r2t = torch.zeros(2, 8, dtype=torch.int32, device=DEV)
    for bad in (dict(window=-1, blocks=(4, 16, 33)), dict(window=4, blocks=(4, 0, 33)), dict(window=4, blocks=(4, 16, 0)),
                dict(window=4, blocks=(4, 16, 33), slopes=torch.zeros(1, device=DEV))):
        with pytest.raises(RuntimeError):
            ops.attn_general(z, pool, pool, r2t, i64([1]), **kw, **bad)


# =================================================================================================
# whole models through the serving path
# =================================================================================================
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, make in C.CONFIGS.items():
        cfg = make()
        weights = C.make_weights(name, cfg)
        out[name] = (cfg, weights, H.write_model(tmp_path_factory.mktemp(name), cfg, weights))
    return out


_oracle_cache = {}


def _oracle(models, name, tokens):
    key = (name, tuple(tokens))
    if key not in _oracle_cache:
        cfg, weights, _ = models[name]
        _oracle_cache[key] = F.forward(cfg, weights, list(tokens))
    return _oracle_cache[key]


def _check(got, want, dtype, what):
    err = H.rel_err(got, want)
    # unit vectors and norms over a handful of channels amplify 16-bit rounding: the small-size configuration's sharp test
    # is the 32-bit one
    tol = H.TOL[dtype] * (2.5 if dtype == "bfloat16" and what.startswith("ones") else 1)
    if dtype == "float32":
        assert err.max().item() < tol, f"{what}: worst relative error {err.max().item():.3e} at row {int(err.argmax())}"
        return
    # 16-bit: a sharp softmax between two close keys amplifies the rounding of a few rows
    assert err.median().item() < tol / 2, f"{what}: median {err.median().item():.3e}"
    assert err.max().item() < 3 * tol and (err > tol).sum().item() <= max(2, 0.02 * len(err)), \
        f"{what}: worst {err.max().item():.3e}, {(err > tol).sum()} rows off"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(C.CONFIGS))
def test_residual_after_every_layer(models, name, dtype):
    cfg, weights, folder = models[name]
    s = H.open_session(folder, dtype, max_tokens=256, max_requests=2, cuda_graph=False)
    model = s.worker.model_runner.model
    got = {}
    model._layer_hook = lambda i, x: got.__setitem__(i, x.double().cpu())
    toks = H.prompt(45, cfg["vocab"], 19)
    s.step([{"id": "a", "tokens": toks, "want": []}])
    model._layer_hook = None
    want = []
    F.forward(cfg, weights, toks, layers_out=want)
    assert len(got) == len(want) == len(cfg["layers"])
    for r, ref in enumerate(want):
        rel = ((got[r] - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt()).item()
        assert rel < (1e-5 if dtype == "float32" else 5e-2), f"layer {r}: relative RMS error {rel:.3e}"


LENGTHS = (1, 2, 13, 150)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(C.CONFIGS))
def test_model_every_schedule(models, name, dtype):
    """Whole prompts, prompt + token-by-token decoding, portions of changing size down to two tokens, and mixed batches of
    unequal requests — each position against the whole-sequence oracle; all of it in one small pool, so request slots
    (convolution and matrix states) and cache runs (token and block rows) are used again throughout."""
    if name == "far" and dtype == "bfloat16":
        pytest.skip("the sharp configuration is a 32-bit test: 16-bit rounding flips its near-ties")
    cfg, _, folder = models[name]
    s = H.open_session(folder, dtype, max_tokens=640, max_requests=4)
    V = cfg["vocab"]
    prompts = {n: H.prompt(n, V, seed=n) for n in LENGTHS}
    full = lambda n: list(range(n))
    for n, toks in prompts.items():
        got = s.step([{"id": f"w{n}", "tokens": toks, "want": full(n)}])
        s.end([f"w{n}"])
        _check(got, _oracle(models, name, toks), dtype, f"{name} whole {n}")
    for n, cut in ((13, 4), (150, 118)):
        toks = prompts[n]
        rows = [s.step([{"id": "d", "tokens": toks[:cut], "want": full(cut)}])]
        for p in range(cut, n):
            rows.append(s.step([{"id": "d", "tokens": [toks[p]], "want": [0]}]))
        s.end(["d"])
        _check(torch.cat(rows), _oracle(models, name, toks), dtype, f"{name} decode {n}")
    toks, rows, at = prompts[150], [], 0
    for size in (2, 3, 64, 2, 5, 1, 1, 40, 2, 30):
        rows.append(s.step([{"id": "c", "tokens": toks[at:at + size], "want": full(size)}]))
        at += size
    assert at == 150
    s.end(["c"])
    _check(torch.cat(rows), _oracle(models, name, toks), dtype, f"{name} portions")
    plan = {"a": prompts[150], "b": prompts[13], "c": prompts[2], "d": H.prompt(70, V, 70), "e": H.prompt(31, V, 31)}
    cuts = {"a": [64, 2, 1, 1, 50, 1, 31], "b": [1, 1, 1, 5, 5], "c": [2], "d": [3, 60, 1, 1, 1, 1, 1, 1, 1],
            "e": [30, 1]}
    order = [["a", "b", "c", "d"], ["a", "b", "d"], ["a", "b", "d", "e"], ["a", "b", "d", "e"], ["a", "b", "d"],
             ["a", "d"], ["a", "d"], ["d"], ["d"]]
    at, idx, got = {k: 0 for k in plan}, {k: 0 for k in plan}, {k: [] for k in plan}
    for live in order:
        entries, ends = [], []
        for r in live:
            n = cuts[r][idx[r]]
            entries.append({"id": r, "tokens": plan[r][at[r]:at[r] + n], "want": full(n)})
            at[r] += n
            idx[r] += 1
            if at[r] == len(plan[r]):
                ends.append(r)
        out, o = s.step(entries), 0
        for e in entries:
            got[e["id"]].append(out[o:o + len(e["tokens"])])
            o += len(e["tokens"])
        s.end(ends)
    for r, toks in plan.items():
        assert at[r] == len(toks)
        _check(torch.cat(got[r]), _oracle(models, name, toks), dtype, f"{name} mixed {r}")


@pytest.mark.parametrize("name", ["far", "uneven"])
def test_long_decoding_and_far_tokens(models, name):
    """330 tokens, 320 of them decoded one by one across runs of the cache, blocks longer than a run included; and a change
    of the FIRST token (which only blocks and recurrent states still carry) moves the last logits by what the oracle
    says."""
    cfg, _, folder = models[name]
    s = H.open_session(folder, "float32", max_tokens=768, max_requests=2)
    V = cfg["vocab"]
    toks = H.prompt(330, V, 9)
    other = [(toks[0] + 1) % V] + toks[1:]
    last = {}
    for rid, seq in (("x", toks), ("y", other)):
        rows = [s.step([{"id": rid, "tokens": seq[:10], "want": list(range(10))}])]
        for p in range(10, 330):
            rows.append(s.step([{"id": rid, "tokens": [seq[p]], "want": [0]}]))
        s.end([rid])
        got = torch.cat(rows).cpu()
        _check(got, _oracle(models, name, seq), "float32", f"{name} {rid}")
        last[rid] = got[-1].double()
    want_moved = _oracle(models, name, toks)[329] - _oracle(models, name, other)[329]
    if name == "far":
        assert want_moved.abs().max() > 1e-2, "the test's weights do not carry the first token this far"
    assert ((last["x"] - last["y"]) - want_moved).abs().max() < 0.05 * want_moved.abs().max() + 1e-4


def test_sharp_attention_sees_every_key_and_block(models):
    """With the sharp weights a query's output is mostly one key's or block's value, wherever it is: every row of a
    300-token prompt must match, as a whole and in portions and single tokens across the run borders of the pool."""
    cfg, _, folder = models["far"]
    s = H.open_session(folder, "float32", max_tokens=512, max_requests=2)
    toks = H.prompt(300, cfg["vocab"], 3)
    want = _oracle(models, "far", toks)
    got = s.step([{"id": "w", "tokens": toks, "want": list(range(300))}])
    s.end(["w"])
    _check(got, want, "float32", "sharp whole")
    rows, at = [], 0
    for size in [120, 7, 1, 1, 2, 125] + [1] * 10 + [34]:
        rows.append(s.step([{"id": "p", "tokens": toks[at:at + size], "want": list(range(size))}]))
        at += size
    assert at == 300
    _check(torch.cat(rows), want, "float32", "sharp portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_engine_greedy_generation(models, name, dtype):
    from semi_pd_b200.configs import ServerArgs
    from semi_pd_b200.semi_pd_scheduler import SemiPDEngine
    cfg, weights, folder = models[name]
    V, n_new = cfg["vocab"], 24
    sa = ServerArgs(model_path=folder, dtype=dtype, load_format="auto", max_total_tokens=4096,
                    max_running_requests=8, context_length=512, enable_semi_pd=True, cuda_graph_bs=[1, 2, 4, 8],
                    chunked_prefill_size=48, max_prefill_tokens=256)
    eng = SemiPDEngine(sa, gpu_id=0, prefill_sm_percent=50, decode_sm_percent=50)
    try:
        prompts = [H.prompt(n, V, seed=100 + n) for n in (5, 33, 120, 61, 2, 77)]
        rids = [eng.submit(p, n_new) for p in prompts]
        done = {r.rid: r for r in eng.wait(len(rids), timeout=120)}
    finally:
        eng.shutdown()
    margin_floor = 1e-3 if dtype == "float32" else 0.4
    compared = 0
    for rid, p in zip(rids, prompts):
        out = done[rid].output_ids
        assert len(out) == n_new
        logits = F.forward(cfg, weights, list(p) + list(out))  # one pass over what was generated
        for t, tok in enumerate(out):
            row = logits[len(p) - 1 + t]
            top2 = row.topk(2).values
            if float(top2[0] - top2[1]) < margin_floor:
                continue  # a near tie: either token is a correct greedy choice after the same history
            compared += 1
            assert tok == int(row.argmax()), f"{rid}: token {t} differs from the oracle's greedy choice"
    assert compared >= 30
