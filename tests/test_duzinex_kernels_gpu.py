"""Each kernel of the Duzinex design alone against the plain implementation of ``plain_duzinex``: sizes that a thread's or a
block's share divides and does not, states carried through portions over reused slots, keys on both sides of every edge."""
import numpy as np
import pytest
import torch

import plain_duzinex as pd

pytestmark = pytest.mark.gpu

DEV = "cuda"
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
KERNEL_TOL = {"float32": 6e-6, "bfloat16": 1.2e-2}


def ops():
    from fieldrun_b200.csrc import ops as o
    return o


def dev(a, dtype=None):
    t = torch.as_tensor(np.ascontiguousarray(a))
    if dtype is not None:
        t = t.to(dtype)
    return t.to(DEV).contiguous()


def f32(a):
    return dev(np.asarray(a, dtype=np.float32))


def f64(t):
    return t.detach().float().cpu().numpy().astype(np.float64)


def as32(a):
    return np.asarray(a, dtype=np.float32).astype(np.float64)


def rounded(a, dtype):
    """The values as the device holds them in ``dtype``."""
    return f64(torch.as_tensor(np.asarray(a, dtype=np.float32)).to(TORCH[dtype]))


def close(got, ref, tol, what=""):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, (got.shape, ref.shape)
    assert np.isfinite(got).all(), what
    err = np.abs(got - ref).max() / max(np.abs(ref).max(), 1e-30)
    assert err <= tol, f"{what}: relative error {err:.3e} > {tol:.1e}"


class Tables:
    """A step's tables on the device: sequences in ``slots`` that continue at ``starts`` with ``q_lens`` new tokens each."""

    def __init__(self, slots, starts, q_lens):
        cu = np.concatenate([[0], np.cumsum(q_lens)]).astype(np.int32)
        self.num_seqs, self.max_q_len = len(slots), int(max(q_lens))
        self.seq_slot = dev(np.asarray(slots, dtype=np.int32))
        self.seq_start = dev(np.asarray(starts, dtype=np.int32))
        self.cu_q_len = dev(cu)
        self.tok_seq = dev(np.repeat(np.arange(len(slots)), q_lens).astype(np.int32))


def in_steps(lengths, portions):
    """Step s holds the s-th portion of every sequence that still has one: (sequences, starts, sizes)."""
    at = [0] * len(lengths)
    for s in range(max(len(p) for p in portions)):
        live = [b for b in range(len(lengths)) if s < len(portions[b])]
        yield live, [at[b] for b in live], [portions[b][s] for b in live]
        for b in live:
            at[b] += portions[b][s]
    assert at == list(lengths)


def cut(length, sizes):
    """``length`` in portions that go through ``sizes`` again and again."""
    out = []
    while sum(out) < length:
        out.append(min(sizes[len(out) % len(sizes)], length - sum(out)))
    return out


# ------------------------------------------------------------------------------------------- norm and token shift

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [40, 31, 700, 1028])
@pytest.mark.parametrize("fused", [True, False])
def test_norm_and_token_shift_through_portions_over_reused_slots(dtype, width, fused):
    """Portions of even and odd sizes (a portion of an even size reads and writes the same copy of the state), down to one
    token; updates of every form on the way; a second turn takes the slots of the first."""
    rng = np.random.default_rng(width)
    w, b, alpha, share = as32(rng.normal(size=width)), as32(rng.normal(size=width)), as32([0.6]), as32(rng.normal(size=width))
    t = {"n": w, "n.b": b, "n.alpha": alpha[0]}
    offset, slots_of = 12, [3, 0, 2]
    state = torch.full((4, 2, offset + width), 5.0, device=DEV)
    for turn, (lengths, sizes) in enumerate((((45, 1, 20), ((2, 4, 1, 3), (1,), (17, 3))), ((9, 1100, 64), ((1,), (1000, 100), (64,))))):
        state[:, :, offset:] = 0.0                                    # what the cache does when it hands a slot out
        xs = [as32(rng.normal(size=(n, width)) * 2) for n in lengths]
        updates = [[as32(rng.normal(size=(n, width))) for _ in range(2)] for n in lengths]
        vector = as32(rng.normal(size=width))
        got, streams = [[] for _ in lengths], [[] for _ in lengths]
        for step, (live, starts, counts) in enumerate(in_steps(lengths, [cut(n, s) for n, s in zip(lengths, sizes)])):
            rows = lambda source: f32(np.concatenate([source[q][s:s + c] for q, s, c in zip(live, starts, counts)]))
            x = rows(xs)
            deltas = tuple(rows([u[i] for u in updates]) for i in range(2))
            ctx = Tables([slots_of[q] for q in live], starts, counts)
            out = torch.empty(x.shape, dtype=TORCH[dtype], device=DEV)
            stream = torch.empty_like(x)
            args = dict(deltas=deltas, vector=f32(vector))
            if fused:
                ops().dyt_rows(x, (f32(w), f32(b), f32(alpha)), out, stream=stream, shift=(f32(share), ctx, state, offset), **args)
            else:
                h = torch.empty_like(x)
                ops().dyt_rows(x, (f32(w), f32(b), f32(alpha)), h, stream=x, **args)
                stream = x
                ops().token_shift(h, out, shift=(f32(share), ctx, state, offset))
            at = 0
            for q, c in zip(live, counts):
                got[q].append(f64(out[at:at + c]))
                streams[q].append(f64(stream[at:at + c]))
                at += c
        for q, n in enumerate(lengths):
            v = xs[q] + updates[q][0] + updates[q][1] + vector
            close(np.concatenate(streams[q]), v, 1e-6, "stream")
            close(np.concatenate(got[q]), pd.token_shift(pd.dynamic_tanh(v, t, "n"), share), KERNEL_TOL[dtype], f"turn {turn}, sequence {q}")
    assert (state[:, :, :offset] == 5.0).all() and (state[1, :, offset:] == 0.0).all()     # nobody else's state was touched


@pytest.mark.parametrize("width", [36, 45])
def test_norm_of_chosen_rows_and_without_updates(width):
    rng = np.random.default_rng(width)
    x, d = as32(rng.normal(size=(30, width))), as32(rng.normal(size=(30, width)))
    w, b, alpha = as32(rng.normal(size=width)), as32(rng.normal(size=width)), as32([-0.8])
    t = {"n": w, "n.b": b, "n.alpha": alpha[0]}
    norm = (f32(w), f32(b), f32(alpha))
    rows = np.array([29, 0, 7, 7], dtype=np.int32)
    out = torch.empty((4, width), device=DEV)
    ops().dyt_rows(f32(x), norm, out, deltas=(f32(d),), rows=dev(rows))
    close(f64(out), pd.dynamic_tanh(x + d, t, "n")[rows], 1e-6)
    out = torch.empty((30, width), device=DEV)
    ops().dyt_rows(f32(x), norm, out)
    close(f64(out), pd.dynamic_tanh(x, t, "n"), 1e-6)


def test_a_shift_that_would_overwrite_its_neighbours_input_is_refused():
    o = ops()
    x = torch.zeros((2, 8), device=DEV)
    norm = tuple(torch.ones(n, device=DEV) for n in (8, 8, 1))
    with pytest.raises(o.KernelError):
        o.dyt_rows(x, norm, torch.empty_like(x), deltas=(x.clone(),), stream=x,
                   shift=(torch.ones(8, device=DEV), Tables([0], [0], [2]), torch.zeros((1, 2, 8), device=DEV), 0))


# ------------------------------------------------------------------------------------------- activation, difference of maps

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [20, 33, 1024, 3000, 9216, 40000])
@pytest.mark.parametrize("rows", [3, 70])
def test_normed_powers(dtype, width, rows):
    rng = np.random.default_rng(width)
    z = as32(rng.normal(size=(rows, width)) * rng.uniform(0.05, 20.0, size=(rows, 1)))
    z[1] *= 1e-3                                                     # small enough that eps decides the cube's norm
    act = as32([0.7, -0.4, 0.9, 0.15])
    out = torch.empty((rows, width), dtype=TORCH[dtype], device=DEV)
    ops().poly_norm(f32(z), f32(act), 1e-5, out)
    want = pd.poly_norm(z, act, 1e-5)
    for r in range(rows):
        close(f64(out[r:r + 1]), want[r:r + 1], KERNEL_TOL[dtype], f"row {r}")


@pytest.mark.parametrize("heads,kv_heads,vd", [(4, 2, 40), (3, 3, 7), (8, 1, 64), (6, 2, 130)])
def test_difference_of_two_maps(heads, kv_heads, vd):
    rng = np.random.default_rng(vd)
    rows, group = 9, heads // kv_heads
    a = as32(rng.normal(size=(rows, heads, 2, vd)))                  # head by head, [map 1, map 2]
    a[2, :, 1] = a[2, :, 0] * 1.6                                    # nearly cancels: the norm brings what is left to full size
    lam = as32([0.62])
    maps = a.reshape(rows, kv_heads, group, 2, vd).transpose(0, 1, 3, 2, 4)
    out = torch.empty((rows, heads * vd), device=DEV)
    ops().map_difference(f32(maps.reshape(rows, -1)), out, heads=heads, kv_heads=kv_heads, v_dim=vd, lam=f32(lam), eps=1e-4, factor=0.7)
    want = pd.difference_of_maps(a[:, :, 0], a[:, :, 1], lam[0], 0.3, 1e-4).reshape(rows, -1)
    for r in range(rows):
        close(f64(out[r]), want[r], 3e-5 if r == 2 else 3e-6, f"row {r}")


# ------------------------------------------------------------------------------------------- the two recurrences

def gru_plain(proj, c, bz, bx):
    z, u, g = pd.sigmoid(proj[:, :c] + bz), proj[:, c:2 * c] + bx, proj[:, 2 * c:3 * c]
    return pd.min_gru(z, u) * pd.silu(g)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("channels", [33, 17, 128, 200])
def test_gated_recurrence_carries_its_state_through_portions_and_reused_slots(dtype, channels):
    rng = np.random.default_rng(channels)
    stride, offset, slots_of = 3 * channels + 5, 4, [2, 0, 3]
    bz, bx = as32(rng.normal(size=channels)), as32(rng.normal(size=channels))
    state = torch.full((4, 2, offset + channels), 3.0, device=DEV)
    for lengths, sizes in (((300, 1, 21), ((129, 2, 1, 128), (1,), (2, 5))), ((40, 260, 9), ((1,), (257, 3), (8, 1)))):
        state[:, :, offset:] = 0.0
        rows = [as32(rng.normal(size=(n, stride)) * 3) for n in lengths]
        got = [[] for _ in lengths]
        for live, starts, counts in in_steps(lengths, [cut(n, s) for n, s in zip(lengths, sizes)]):
            proj = f32(np.concatenate([rows[q][s:s + n] for q, s, n in zip(live, starts, counts)]))
            out = torch.empty((proj.shape[0], channels), dtype=TORCH[dtype], device=DEV)
            ops().min_gru(proj, 0, channels, 2 * channels, f32(bz), f32(bx), Tables([slots_of[q] for q in live], starts, counts), state,
                          offset, out)
            at = 0
            for q, n in zip(live, counts):
                got[q].append(f64(out[at:at + n]))
                at += n
        for q in range(3):
            close(np.concatenate(got[q]), gru_plain(rows[q], channels, bz, bx), KERNEL_TOL[dtype], f"sequence {q}")
    assert (state[:, :, :offset] == 3.0).all() and (state[1, :, offset:] == 0.0).all()


def test_gated_recurrence_holds_a_token_for_a_thousand_steps_and_forgets_at_once():
    """Gates of 1e-4: a large first candidate still counts after 1,500 tokens, and a decay rounded to float32 would have drifted
    by then; then a gate of nearly one (1 - z = 1e-9) drops the state but for its billionth part."""
    rng = np.random.default_rng(5)
    n, c = 1502, 40
    proj = as32(rng.normal(size=(n, 3 * c)) * 0.1)
    proj[:, :c] = as32(np.log(1e-4 / (1 - 1e-4)) + 0.01 * rng.normal(size=(n, c)))
    proj[0, :c], proj[0, c:2 * c] = 30.0, 1e5
    proj[1500, :c] = 20.7
    proj[:, 2 * c:] = 2.0
    zero = np.zeros(c)
    want = gru_plain(proj, c, zero, zero)
    for sizes in ((n,), (64,), (1,)):
        state = torch.zeros((1, 2, c), device=DEV)
        got, at = [], 0
        for count in cut(n, sizes):
            out = torch.empty((count, c), device=DEV)
            ops().min_gru(f32(proj[at:at + count]), 0, c, 2 * c, f32(zero), f32(zero), Tables([0], [at], [count]), state, 0, out)
            got.append(f64(out))
            at += count
        got = np.concatenate(got)
        for t in (1, 700, 1499, 1500, 1501):
            close(got[t], want[t], 1e-2 if t >= 1500 else 6e-6, f"portions of {sizes}, token {t}")


def retention_case(rng, rows, heads, dim, vdim):
    return as32(rng.normal(size=(rows, 2 * heads * dim + 2 * heads * vdim + 3)))


def retention_plain(proj, heads, dim, vdim, decay, eps, dtype):
    n, qk, v = proj.shape[0], heads * dim, heads * vdim
    q, k = proj[:, :qk].reshape(n, heads, dim), proj[:, qk:2 * qk].reshape(n, heads, dim)
    values, gate = proj[:, 2 * qk:2 * qk + v].reshape(n, heads, vdim), proj[:, 2 * qk + v:2 * qk + 2 * v]
    o = pd.retention(q, k * dim ** -0.5, values, decay)
    return pd.rms_divide(o, eps).reshape(n, v) * pd.silu(gate)


def run_retention(proj, heads, dim, vdim, decay, eps, ctx, state, offset, dtype):
    qk, v = heads * dim, heads * vdim
    out = torch.empty((proj.shape[0], v), dtype=TORCH[dtype], device=DEV)
    raw = torch.full((proj.shape[0], v), float("nan"), device=DEV)
    chunks = dtype == "bfloat16" and ctx.max_q_len >= 2 and ops().retention_chunks_take(dim, vdim)
    if chunks:                                               # rows on 16 bytes, as the part lays them out
        proj = np.concatenate([proj, np.zeros((proj.shape[0], -proj.shape[1] % 16))], axis=1)
    ops().retention(dev(proj, torch.bfloat16) if chunks else f32(proj), (0, qk, 2 * qk, 2 * qk + v), ops().retention_decays(decay, DEV), ctx, state, offset, out, raw, heads=heads,
                    dim=dim, vdim=vdim, k_scale=dim ** -0.5, eps=eps)
    return f64(out)


# in bfloat16 a prompt's q, k and v are rounded to bfloat16 on their way into the tensor cores
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 32, 32), (3, 20, 36), (1, 5, 7), (2, 64, 64), (1, 128, 128), (2, 48, 80), (1, 200, 33),
                                            (1, 256, 256), (2, 64, 200), (4, 128, 64), (1, 16, 144)])
def test_retention_carries_its_state_through_portions_and_reused_slots(dtype, heads, dim, vdim):
    rng = np.random.default_rng(dim + vdim)
    decay = [0.97, 0.5, 0.999, 0.0][:heads]
    offset, slots_of = 8, [2, 0, 3]
    state = torch.full((4, 2, offset + heads * dim * vdim), 3.0, device=DEV)
    for lengths, sizes in (((150, 1, 21), ((70, 2, 1, 64), (1,), (17, 3))), ((40, 200, 9), ((1,), (129, 63, 8), (8, 1)))):
        state[:, :, offset:] = 0.0
        rows = [retention_case(rng, n, heads, dim, vdim) for n in lengths]
        if dtype == "bfloat16":
            rows = [rounded(r, dtype) for r in rows]
        got = [[] for _ in lengths]
        for live, starts, counts in in_steps(lengths, [cut(n, s) for n, s in zip(lengths, sizes)]):
            out = run_retention(np.concatenate([rows[q][s:s + n] for q, s, n in zip(live, starts, counts)]), heads, dim, vdim, decay, 1e-5,
                                Tables([slots_of[q] for q in live], starts, counts), state, offset, dtype)
            at = 0
            for q, n in zip(live, counts):
                got[q].append(out[at:at + n])
                at += n
        for q in range(3):
            close(np.concatenate(got[q]), retention_plain(rows[q], heads, dim, vdim, decay, 1e-5, dtype), KERNEL_TOL[dtype], f"sequence {q}")
    assert (state[:, :, :offset] == 3.0).all() and (state[1, :, offset:] == 0.0).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_retention_reads_a_token_hundreds_of_steps_back_and_none_behind_a_decay_of_zero(dtype):
    """One write at token 3 that only the last query reads (every other key is orthogonal to it), with decays that keep it, fade it
    to a known share, and drop it: what the last token gives is that write's value times decay^distance."""
    rng = np.random.default_rng(31)
    heads, dim, vdim, n = 3, 64, 64, 700
    decay = [1.0, 0.9990234375, 0.0]
    proj = rounded(retention_case(rng, n, heads, dim, vdim), "bfloat16")
    qk, v = heads * dim, heads * vdim
    for h in range(heads):
        k = proj[:, qk + h * dim:qk + (h + 1) * dim]
        k[:, 0] = 0.0                                        # a view: channel 0 of every key ...
        k[3, :], k[3, 0] = 0.0, 8.0                          # ... belongs to token 3 alone
        proj[-1, h * dim:(h + 1) * dim] = 0.0
        proj[-1, h * dim] = 4.0
    values = proj[3, 2 * qk:2 * qk + v].reshape(heads, vdim)
    want = retention_plain(proj, heads, dim, vdim, decay, 1e-5, dtype)
    direct = [pd.rms_divide(decay[h] ** (n - 4) * 32.0 * dim ** -0.5 * values[h], 1e-5) for h in range(heads)]
    assert np.allclose(want[-1], np.concatenate(direct) * pd.silu(proj[-1, 2 * qk + v:2 * qk + 2 * v]))
    assert np.abs(want[-1][:2 * vdim]).max() > 0.5 and np.abs(want[-1][2 * vdim:]).max() == 0.0
    for sizes in ((n,), (64,), (699, 1), (1,)):
        state = torch.zeros((1, 2, heads * dim * vdim), device=DEV)
        at, last = 0, None
        for count in cut(n, sizes):
            last = run_retention(proj[at:at + count], heads, dim, vdim, decay, 1e-5, Tables([0], [at], [count]), state, 0, dtype)[-1]
            at += count
        close(last[:2 * vdim], want[-1][:2 * vdim], 2e-5 if dtype == "float32" else 6e-3, f"portions of {sizes}")
        assert np.abs(last[2 * vdim:]).max() < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_retention_over_thousands_of_tokens_keeps_a_decay_close_to_one_exact(dtype):
    rng = np.random.default_rng(32)
    heads, dim, vdim, n = 1, 16, 16, 3000
    decay = [1.0 - 3e-4]                                     # no float32 number: rounded, it would be off at every token
    proj = rounded(np.abs(retention_case(rng, n, heads, dim, vdim)) * 0.5, "bfloat16")       # everything adds up
    want = retention_plain(proj, heads, dim, vdim, decay, 1e-5, dtype)
    state = torch.zeros((1, 2, dim * vdim), device=DEV)
    got = run_retention(proj, heads, dim, vdim, decay, 1e-5, Tables([0], [0], [n]), state, 0, dtype)
    close(got, want, 6e-6 if dtype == "float32" else 6e-3, "whole")
    s = np.zeros((dim, vdim))
    for t in range(n):
        s = decay[0] * s + np.outer(proj[t, dim:2 * dim], proj[t, 2 * dim:2 * dim + vdim]) * dim ** -0.5
    close(f64(state[0, n & 1]).reshape(dim, vdim), s, 3e-6, "state")


# ------------------------------------------------------------------------------------------- attention

SCALE = 0.2


def scrambled_pages(rng, lengths, k_heads, v_heads, dim, vdim, dtype, spare=3):
    """Keys [slot][T, K, dim], values [slot][T, V, vdim] and room for them in pages of 64 in a scrambled order."""
    per = [(n + 63) // 64 for n in lengths]
    pages = sum(per) + spare
    order = rng.permutation(pages)
    table = np.full((len(lengths), max(per) + 1), -1, dtype=np.int32)
    keys, values, at = [], [], 0
    for s, n in enumerate(lengths):
        keys.append(rounded(rng.normal(size=(n, k_heads, dim)), dtype))
        values.append(rounded(rng.normal(size=(n, v_heads, vdim)), dtype))
        for i in range(per[s]):
            table[s, i] = order[at]
            at += 1
    return keys, values, np.zeros((pages, k_heads, 64, dim)), np.zeros((pages, v_heads, vdim, 64)), table


def lay_into_pages(keys, values, kc, vc, table):
    for s in range(len(keys)):
        for j in range(keys[s].shape[0]):
            page = table[s, j // 64]
            kc[page, :, j % 64] = keys[s][j]
            vc[page, :, :, j % 64] = values[s][j]


def plain_maps(q, keys, values, rows, window, keep, softcap):
    """q [R, Q, dim] in the kernels' order of heads [value head, map, query head of the group]; one map's attention per run of
    query heads.  Returns [R, Q, vdim]."""
    k_heads, v_heads = keys[0].shape[1], values[0].shape[1]
    share = k_heads // v_heads
    out = []
    for r, (s, p) in enumerate(rows):
        v = np.repeat(values[s], share, axis=1)
        out.append(pd.map_attention(q[r:r + 1], keys[s], v, scale=SCALE, window=window, keep_first=keep, softcap=softcap, positions=[p])[0])
    return np.stack(out)


def differential_case(rng, heads, kv_heads, dim, vdim, seqs, window, keep, softcap, dtype):
    """Sequences (start, new tokens): keys, values and queries, and what the plain implementation makes of them.  For the last
    query of the last sequence these keys are made to stand out: the first one inside its window, the one just outside, the last
    of the kept first tokens and the next one."""
    maps = 2
    lengths = [start + n for start, n in seqs]
    keys, values, kc, vc, table = scrambled_pages(rng, lengths, maps * kv_heads, kv_heads, dim, vdim, dtype)
    rows = [(s, start + i) for s, (start, n) in enumerate(seqs) for i in range(n)]
    q = rounded(rng.normal(size=(len(rows), maps * heads, dim)), dtype)
    last, position = len(seqs) - 1, lengths[-1] - 1
    group = heads // kv_heads
    w = window or 10 ** 6
    for place, value in ((position - w + 1, 5.0), (position - w, -9.0), (keep - 1, 3.0), (keep, 11.0)):
        if 0 <= place < position:
            keys[last][place] = rounded(q[-1, ::group] * 2.0, dtype)
            values[last][place] = value
    lay_into_pages(keys, values, kc, vc, table)
    lam, factor, eps = as32([0.55]), 0.7, 1e-5
    a = plain_maps(q, keys, values, rows, window, keep, softcap)
    split = a.reshape(len(rows), kv_heads, 2, group, vdim)
    want = pd.difference_of_maps(split[:, :, 0], split[:, :, 1], lam[0], 1 - factor, eps).reshape(len(rows), heads * vdim)
    t = TORCH[dtype]
    return dict(q=dev(q.reshape(len(rows), -1), t), kc=dev(kc, t), vc=dev(vc, t), table=dev(table), rows=rows, maps=a.reshape(len(rows), -1),
                want=want, difference=dict(lam=f32(lam), eps=eps, factor=factor),
                args=dict(num_heads=2 * heads, num_kv_heads=2 * kv_heads, head_dim=dim, v_dim=vdim, scale=SCALE, window=window,
                          keep_first=keep, softcap=softcap, maps=2))


MASKS = [(64, 5, 4.0), (100, 70, None), (130, 64, 20.0), (7, 0, None), (64, 200, 3.0), (None, 0, 5.0), (300, 1, None)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 24, 40), (3, 3, 16, 16), (6, 1, 10, 7), (2, 1, 100, 200)])
@pytest.mark.parametrize("window,keep,softcap", MASKS)
def test_maps_with_window_and_first_tokens_in_the_general_kernel(dtype, heads, kv_heads, dim, vdim, window, keep, softcap):
    rng = np.random.default_rng(dim + (window or 0))
    c = differential_case(rng, heads, kv_heads, dim, vdim, [(0, 80), (140, 3), (63, 2), (0, 1), (250, 3), (420, 1)], window, keep, softcap, dtype)
    n = len(c["rows"])
    maps = torch.full((n, c["maps"].shape[1]), 7.0, device=DEV)
    ops().attention_generic(c["q"], c["kc"], c["vc"], c["table"], dev(np.array([p for _, p in c["rows"]], dtype=np.int32)),
                            dev(np.array([s for s, _ in c["rows"]], dtype=np.int32)), maps, **c["args"])
    close(f64(maps), c["maps"], 3e-6, "the maps")                    # the output is float32 in both modes
    out = torch.empty((n, heads * vdim), dtype=TORCH[dtype], device=DEV)
    ops().map_difference(maps, out, heads=heads, kv_heads=kv_heads, v_dim=vdim, **c["difference"])
    close(f64(out), c["want"], 2e-5 if dtype == "float32" else 1.2e-2, "the difference")


def test_the_kept_tokens_and_the_windows_edges_show():
    """The case above for one query: with every other score small, moving an edge by one token changes the output at once."""
    seen = {}
    for window, keep in ((50, 4), (51, 4), (50, 5), (50, 0)):
        c = differential_case(np.random.default_rng(78), 1, 1, 32, 32, [(420, 1)], 50, 4, None, "float32")
        c["args"].update(window=window, keep_first=keep)
        maps = torch.empty((1, 64), device=DEV)
        ops().attention_generic(c["q"], c["kc"], c["vc"], c["table"], dev(np.array([420], dtype=np.int32)),
                                dev(np.array([0], dtype=np.int32)), maps, **c["args"])
        seen[(window, keep)] = f64(maps)[0, :32].mean()
    base = seen[(50, 4)]
    assert all(abs(v - base) > 0.5 for key, v in seen.items() if key != (50, 4)), seen


TC_SIZES = [(4, 2, 32, 64), (6, 1, 64, 128), (2, 2, 64, 64), (3, 1, 128, 128), (4, 4, 32, 32), (4, 1, 96, 96)]


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", TC_SIZES)
@pytest.mark.parametrize("window,keep,softcap", MASKS)
@pytest.mark.parametrize("kernel", ["attention_decode_mma", "attention_decode_tma"])
def test_one_token_kernels_join_two_maps(heads, kv_heads, dim, vdim, window, keep, softcap, kernel):
    if kernel == "attention_decode_tma" and dim not in (64, 128):
        pytest.skip("the TMA kernel takes key heads of 64 and 128")
    rng = np.random.default_rng(dim + heads + (window or 0))
    w = window or 500
    c = differential_case(rng, heads, kv_heads, dim, vdim, [(999, 1), (256, 1), (63, 1), (0, 1), (512, 1), (w, 1), (w - 1, 1),
                                                            (keep + w, 1), (2 * w + 331, 1)], window, keep, softcap, "bfloat16")
    positions = np.array([p for _, p in c["rows"]], dtype=np.int32)
    chunks = (int(positions.max()) + 256) // 256
    n = len(positions)
    for per_block in ((None,) if kernel == "attention_decode_mma" else (None, 1, 3)):
        part_o = torch.full((n, 2 * heads, chunks, vdim), float("nan"), device=DEV)
        part_ml = torch.full((n, 2 * heads, chunks, 2), float("nan"), device=DEV)
        out = torch.full((n, heads * vdim), 7.0, dtype=torch.bfloat16, device=DEV)
        extra = {} if kernel == "attention_decode_mma" else {"chunks_per_block": per_block}
        getattr(ops(), kernel)(c["q"], c["kc"], c["vc"], c["table"], dev(positions), dev(np.arange(n, dtype=np.int32)), part_o, part_ml, out,
                               max_chunks=chunks, difference=c["difference"], **extra, **c["args"])
        ops().tc_status_check(DEV)
        close(f64(out), c["want"], 2.5e-2, f"{kernel}, {per_block} chunks a block")


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", TC_SIZES)
@pytest.mark.parametrize("window,keep,softcap", MASKS)
@pytest.mark.parametrize("kernel", ["attention_prefill_mma", "attention_prefill_tc"])
def test_many_token_kernels_leave_two_maps_in_float32(heads, kv_heads, dim, vdim, window, keep, softcap, kernel):
    if kernel == "attention_prefill_tc" and dim not in (64, 128):
        pytest.skip("the tcgen05 kernel takes key heads of 64 and 128")
    rng = np.random.default_rng(3 * dim + heads + (window or 0))
    seqs = [(0, 140), (130, 17), (0, 1), (63, 80), (300, 129), (420, 140)]
    c = differential_case(rng, heads, kv_heads, dim, vdim, seqs, window, keep, softcap, "bfloat16")
    tile = 128 if kernel == "attention_prefill_tc" else 16
    tile_seq = np.concatenate([np.full((n + tile - 1) // tile, b) for b, (_, n) in enumerate(seqs)]).astype(np.int32)
    tile_q0 = np.concatenate([np.arange(0, n, tile) for _, n in seqs]).astype(np.int32)
    q_lens = np.array([n for _, n in seqs], dtype=np.int32)
    cu = np.concatenate([[0], np.cumsum(q_lens)]).astype(np.int32)
    maps = torch.full((len(c["rows"]), 2 * heads * vdim), 7.0, device=DEV)
    getattr(ops(), kernel)(c["q"], c["kc"], c["vc"], c["table"], dev(tile_seq), dev(tile_q0), dev(np.arange(len(seqs), dtype=np.int32)),
                           dev(np.array([s for s, _ in seqs], dtype=np.int32)), dev(q_lens), dev(cu), maps, **c["args"])
    ops().tc_status_check(DEV)
    close(f64(maps), c["maps"], 1.2e-2, kernel)
    if kernel == "attention_prefill_tc" and ops().attention_pair_takes(dim, vdim):
        # both maps, their difference and its norm in one kernel
        out = torch.full((len(c["rows"]), heads * vdim), 7.0, dtype=torch.bfloat16, device=DEV)
        ops().attention_pair_tc(c["q"], c["kc"], c["vc"], c["table"], dev(tile_seq), dev(tile_q0), dev(np.arange(len(seqs), dtype=np.int32)),
                                dev(np.array([s for s, _ in seqs], dtype=np.int32)), dev(q_lens), dev(cu), out, heads=heads, v_heads=kv_heads,
                                head_dim=dim, v_dim=vdim, scale=SCALE, window=window, keep_first=keep, softcap=softcap, **c["difference"])
        ops().tc_status_check(DEV)
        close(f64(out), c["want"], 2.5e-2, "one kernel")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens", [5, 100])
@pytest.mark.parametrize("dim,vdim,rot", [(24, 40, 16), (10, 7, 10), (64, 128, 32), (12, 12, 0)])
def test_queries_and_keys_of_two_maps_turned_and_laid_into_pages(dtype, tokens, dim, vdim, rot):
    rng = np.random.default_rng(dim + tokens)
    heads, kv = 4, 2
    q_heads, k_heads, base = 2 * heads, 2 * kv, 300.0
    row = as32(rng.normal(size=(tokens, (q_heads + k_heads) * dim + kv * vdim)))
    bias = as32(rng.normal(size=row.shape[1]))
    start, slot = 60, 1
    positions = np.arange(start, start + tokens)
    table = np.array([[-1] * 4, [4, 2, 5, 1]], dtype=np.int32)
    t = TORCH[dtype]
    kc, vc = torch.zeros((6, k_heads, 64, dim), dtype=t, device=DEV), torch.zeros((6, kv, vdim, 64), dtype=t, device=DEV)
    q = torch.empty((tokens, q_heads * dim), dtype=t, device=DEV)
    cos = sin = None
    if rot:
        from fieldrun_b200.parts import build_position
        cos, sin = build_position({"kind": "rotary", "rotary_dim": rot, "theta": base, "pairing": "interleaved"}).tables(256, DEV)
    ops().qkv_prepare(f32(row), None, None, 1e-6, cos, sin, dev(positions.astype(np.int32)), dev(np.full(tokens, slot, dtype=np.int32)),
                      dev(table), q, kc, vc, num_heads=q_heads, num_kv_heads=k_heads, num_v_heads=kv, head_dim=dim, rotary_dim=rot,
                      interleaved=True, write_cache=True, bias=f32(bias), v_dim=vdim)
    full = row + bias
    wq, wk = full[:, :q_heads * dim].reshape(tokens, q_heads, dim), full[:, q_heads * dim:(q_heads + k_heads) * dim].reshape(tokens, k_heads, dim)
    if rot:
        wq, wk = pd.rotate_neighbours(wq, positions, rot, base), pd.rotate_neighbours(wk, positions, rot, base)
    wv = full[:, (q_heads + k_heads) * dim:].reshape(tokens, kv, vdim)
    close(f64(q).reshape(wq.shape), wq, KERNEL_TOL[dtype], "queries")
    kc, vc = f64(kc), f64(vc)
    close(np.stack([kc[table[slot, p // 64], :, p % 64] for p in positions]), wk, KERNEL_TOL[dtype], "keys")
    close(np.stack([vc[table[slot, p // 64], :, :, p % 64] for p in positions]), wv, KERNEL_TOL[dtype], "values")
