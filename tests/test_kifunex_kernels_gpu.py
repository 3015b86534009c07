"""Each mechanism of the Kifunex design alone against the plain implementation of ``plain_kifunex``: the copies of the stream in
every form of update, values that are keys before their rotation, the rotation's blended frequencies, attention with keys on
both sides of a window's edge, the experts' choice and weights with the shared expert, the head."""
import numpy as np
import pytest
import torch

import plain_kifunex as pk

pytestmark = pytest.mark.gpu

DEV = "cuda"
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
KERNEL_TOL = {"float32": 6e-6, "bfloat16": 1.2e-2}
BOTH = pytest.mark.parametrize("dtype", ["float32", "bfloat16"])


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


# ------------------------------------------------------------------------------------------- copies of the stream

class Copies:
    """Copies, updates and constants of a case, as arrays, and what the plain implementation makes of them."""

    def __init__(self, rows, streams, width, top=3, equal=False, seed=0):
        rng = np.random.default_rng(1000 * streams + width + seed)
        self.rows, self.streams, self.width, self.equal = rows, streams, width, equal
        self.x = as32(rng.normal(size=(rows, width) if equal else (rows, streams, width)) * 2)
        self.ya, self.d0, self.d1 = (as32(rng.normal(size=(rows, width))) for _ in range(3))
        self.y, self.ew = as32(rng.normal(size=(rows * top + 5, width))), as32(rng.uniform(size=(rows, top)))
        self.rowmap = rng.permutation(rows * top + 5)[:rows * top].astype(np.int32)
        self.mix, self.oa, self.ob, self.gather = (as32(rng.normal(size=s)) for s in ((streams, streams), streams, streams, streams))
        self.w, self.b, self.alpha = as32(1 + 0.2 * rng.normal(size=width)), as32(rng.normal(size=width)), as32([0.37])
        self.experts_sum = np.einsum("tk,tkd->td", self.ew, self.y[self.rowmap].reshape(rows, top, width))

    def full(self):
        return np.repeat(self.x[:, None, :], self.streams, axis=1) if self.equal else self.x

    def after(self, first, second):
        new = pk.spread_update(self.full(), self.ya if first else 0.0 * self.ya, self.mix, self.oa)
        yb = {"none": 0.0, "tensor": self.d0, "two": self.d0 + self.d1, "experts": self.experts_sum,
              "all": self.d0 + self.d1 + self.experts_sum}[second]
        return new + np.einsum("td,s->tsd", np.broadcast_to(yb, (self.rows, self.width)), self.ob)

    def normed(self, u):
        t = {"n": self.w, "n.b": self.b, "n.alpha": self.alpha[0]}
        return pk.dynamic_tanh(u, t, "n")

    def args(self, first, second):
        out = dict(mix=f32(self.mix), gather=f32(self.gather), norm=(f32(self.w), f32(self.b), f32(self.alpha)))
        if first:
            out["first"] = (f32(self.ya), f32(self.oa))
        if second != "none":
            out["second"] = {"tensor": (f32(self.d0),), "two": (f32(self.d0), f32(self.d1)), "experts": (),
                             "all": (f32(self.d0), f32(self.d1))}[second]
            out["second_out"] = f32(self.ob)
            if second in ("experts", "all"):
                out["experts"] = (f32(self.y), f32(self.ew), dev(self.rowmap))
        return out


@BOTH
@pytest.mark.parametrize("streams,width", [(1, 40), (2, 96), (3, 1100), (4, 512), (5, 64), (8, 132), (4, 257), (9, 40), (64, 36)])
def test_copies_updated_summed_and_normed_in_one_pass(dtype, streams, width):
    for equal in (False, True):
        c = Copies(19, streams, width, equal=equal)
        for first, second in ((True, "none"), (False, "tensor"), (True, "two"), (False, "experts"), (True, "all")):
            what = f"equal copies {equal}, first {first}, second {second}"
            v = c.after(first, second)
            u = pk.gather_streams(v, c.gather)
            args = c.args(first, second)
            for store in (False, True):
                x = f32(c.x)
                kept = (torch.full((19, streams, width), 7.0, device=DEV) if equal else x) if store else None
                out = torch.full((19, width), 7.0, dtype=TORCH[dtype], device=DEV)
                out32 = torch.full((19, width), 7.0, device=DEV)
                ops().stream_copies(x, streams, store=kept, out=out, out32=out32, **args)
                close(f64(out32), c.normed(u), 2e-5, f"{what}, stored {store}: the norm in float32")
                close(f64(out), c.normed(u), max(2e-5, KERNEL_TOL[dtype]), f"{what}, stored {store}: the norm")
                if store:
                    close(f64(kept), v, 5e-6, what + ": the copies")
                else:
                    assert np.array_equal(f64(x), c.x), "the copies were written although they should not be"
            picked = np.array([18, 0, 7, 7], dtype=np.int32)
            few = torch.full((4, width), 7.0, dtype=TORCH[dtype], device=DEV)
            ops().stream_copies(f32(c.x), streams, rows=dev(picked), out=few, **args)
            close(f64(few), c.normed(u)[picked], max(2e-5, KERNEL_TOL[dtype]), what + ": chosen rows")
        # without constants: the copies as they are, added up; without a norm: the sum itself
        plain = torch.full((19, width), 7.0, device=DEV)
        ops().stream_copies(f32(c.x), streams, out32=plain)
        close(f64(plain), c.full().sum(axis=1), 5e-6, "the plain sum")


@pytest.mark.parametrize("rows", [300, 700, 2100])
@pytest.mark.parametrize("streams,width", [(4, 96), (3, 50)])
def test_many_rows_a_block_takes_several(rows, streams, width):
    c = Copies(rows, streams, width, top=5)
    v = c.after(True, "all")
    x, out = f32(c.x), torch.empty((rows, width), device=DEV)
    ops().stream_copies(x, streams, store=x, out=out, **c.args(True, "all"))
    close(f64(x), v, 5e-6, "the copies")
    close(f64(out), c.normed(pk.gather_streams(v, c.gather)), 2e-5, "the norm")


def test_wrong_shapes_are_refused_before_the_launch():
    from fieldrun_b200.csrc.ops import KernelError
    x, out = torch.zeros((3, 2, 8), device=DEV), torch.zeros((3, 8), device=DEV)
    with pytest.raises(KernelError):
        ops().stream_copies(x, 3, out32=out)
    with pytest.raises(KernelError):
        ops().stream_copies(x, 2, out32=out, mix=torch.zeros((3, 3), device=DEV))
    with pytest.raises(KernelError):
        ops().stream_copies(x, 2, out32=out, first=(out, None))
    with pytest.raises(KernelError):
        ops().stream_copies(x[:, 0].contiguous(), 2, out32=out, store=torch.zeros((3, 3, 8), device=DEV))


@BOTH
def test_a_norm_with_statistics_reads_copies_too(dtype):
    """The design's norm goes through the kernel that holds it; any other norm gets the summed row."""
    from test_parts_gpu import Stepper, lib, source
    _, config, _, parts, _ = lib()
    rng = np.random.default_rng(5)
    c = Copies(11, 3, 60)
    w = as32(1 + 0.1 * rng.normal(size=60))
    part = parts.build_part("norm", config.PartSpec("rmsnorm", {"width": 60, "eps": 1e-4}, {"weight": "n.w"}), TORCH[dtype])
    part.load(source({"n.w": w}, dtype))
    stepper = Stepper([], dtype)
    ctx = stepper.engine.StepContext(stepper.workspace, TORCH[dtype], [0], [0], [11])
    update = parts.CopiesUpdate(f32(c.mix), first=f32(c.ya), first_out=f32(c.oa), second=f32(c.d0), second_out=f32(c.ob))
    x = f32(c.x)
    kept, act, act32 = part.forward_copies(ctx, x, update, 3, gather=f32(c.gather), want32=True, store=True)
    v = c.after(True, "tensor")
    u = pk.gather_streams(v, c.gather)
    want = u / np.sqrt((u * u).mean(axis=-1, keepdims=True) + 1e-4) * w
    assert kept.data_ptr() == x.data_ptr()
    close(f64(kept), v, 5e-6, "copies")
    close(f64(act), want, max(2e-5, KERNEL_TOL[dtype]), "norm")
    close(f64(act32), want, 2e-5, "norm in float32")


# ------------------------------------------------------------------------------------------- attention

@BOTH
@pytest.mark.parametrize("tokens", [5, 100])
@pytest.mark.parametrize("heads,kv,dim,rot,biased", [(4, 2, 24, 16, False), (3, 3, 10, 10, True), (5, 1, 64, 48, False), (2, 1, 12, 0, True),
                                                     (6, 2, 128, 128, False)])
def test_values_are_the_keys_as_projected(dtype, tokens, heads, kv, dim, rot, biased):
    rng = np.random.default_rng(dim + tokens)
    row = as32(rng.normal(size=(tokens, (heads + kv) * dim)))
    bias = as32(rng.normal(size=row.shape[1])) if biased else 0.0 * row[0]
    start, slot = 60, 1
    positions = np.arange(start, start + tokens)
    table = np.array([[-1] * 4, [4, 2, 5, 1]], dtype=np.int32)
    t = TORCH[dtype]
    kc, vc = torch.zeros((6, kv, 64, dim), dtype=t, device=DEV), torch.zeros((6, kv, dim, 64), dtype=t, device=DEV)
    q = torch.empty((tokens, heads * dim), dtype=t, device=DEV)
    blend = {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 150.0}
    cos = sin = None
    if rot:
        from fieldrun_b200.parts import build_position
        cos, sin = build_position({"kind": "rotary", "rotary_dim": rot, "theta": 400.0, "pairing": "half",
                                   "frequency_blend": blend}).tables(256, DEV)
    ops().qkv_prepare(f32(row), None, None, 1e-6, cos, sin, dev(positions.astype(np.int32)), dev(np.full(tokens, slot, dtype=np.int32)),
                      dev(table), q, kc, vc, num_heads=heads, num_kv_heads=kv, head_dim=dim, rotary_dim=rot, interleaved=False,
                      write_cache=True, bias=f32(bias) if biased else None, values_from_keys=True)
    full = row + bias
    wq, wv = full[:, :heads * dim].reshape(tokens, heads, dim), full[:, heads * dim:].reshape(tokens, kv, dim)
    freq = pk.rotation_frequencies(rot, 400.0, blend)
    wq, wk = pk.rotate_halves(wq, positions, freq), pk.rotate_halves(wv, positions, freq)
    close(f64(q).reshape(wq.shape), wq, KERNEL_TOL[dtype], "queries")
    kc, vc = f64(kc), f64(vc)
    close(np.stack([kc[table[slot, p // 64], :, p % 64] for p in positions]), wk, KERNEL_TOL[dtype], "keys")
    close(np.stack([vc[table[slot, p // 64], :, :, p % 64] for p in positions]), wv, KERNEL_TOL[dtype], "values")


SCALE = 0.2


def windowed_case(rng, heads, kv_heads, dim, seqs, window, dtype):
    """Sequences (start, new tokens) over scrambled pages.  For the last query of the last sequence these keys stand out: the
    first one inside its window, the one just outside it, and an early one."""
    lengths = [start + n for start, n in seqs]
    per = [(n + 63) // 64 for n in lengths]
    order, at = rng.permutation(sum(per) + 3), 0
    table = np.full((len(lengths), max(per) + 1), -1, dtype=np.int32)
    for s, count in enumerate(per):
        table[s, :count] = order[at:at + count]
        at += count
    keys = [rounded(rng.normal(size=(n, kv_heads, dim)), dtype) for n in lengths]
    values = [rounded(rng.normal(size=(n, kv_heads, dim)), dtype) for n in lengths]
    rows = [(s, start + i) for s, (start, n) in enumerate(seqs) for i in range(n)]
    q = rounded(rng.normal(size=(len(rows), heads, dim)), dtype)
    last, position = len(seqs) - 1, lengths[-1] - 1
    for place, value in ((position - (window or 300) + 1, 5.0), (position - (window or 300), -9.0), (3, 11.0)):
        if 0 <= place < position:
            keys[last][place] = rounded(q[-1, ::heads // kv_heads] * 3.0, dtype)
            values[last][place] = value
    kc, vc = np.zeros((len(order), kv_heads, 64, dim)), np.zeros((len(order), kv_heads, dim, 64))
    for s in range(len(lengths)):
        for j in range(lengths[s]):
            kc[table[s, j // 64], :, j % 64] = keys[s][j]
            vc[table[s, j // 64], :, :, j % 64] = values[s][j]
    want = np.stack([pk.windowed_attention(q[r:r + 1], keys[s], values[s], scale=SCALE, window=window, positions=[p])[0]
                     for r, (s, p) in enumerate(rows)])
    t = TORCH[dtype]
    return dict(q=dev(q.reshape(len(rows), -1), t), kc=dev(kc, t), vc=dev(vc, t), table=dev(table), rows=rows,
                want=want.reshape(len(rows), -1), args=dict(num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, v_dim=dim, scale=SCALE,
                                                            window=window))


WINDOWS = [1, 7, 64, 100, 130, 256, None]


@BOTH
@pytest.mark.parametrize("heads,kv_heads,dim", [(4, 2, 24), (3, 3, 9), (12, 1, 64), (24, 1, 80)])
@pytest.mark.parametrize("window", WINDOWS)
def test_window_in_the_general_kernel(dtype, heads, kv_heads, dim, window):
    c = windowed_case(np.random.default_rng(dim + (window or 0)), heads, kv_heads, dim, [(0, 80), (140, 3), (63, 2), (0, 1), (250, 3), (420, 1)],
                      window, dtype)
    out = torch.full((len(c["rows"]), heads * dim), 7.0, dtype=TORCH[dtype], device=DEV)
    ops().attention_generic(c["q"], c["kc"], c["vc"], c["table"], dev(np.array([p for _, p in c["rows"]], dtype=np.int32)),
                            dev(np.array([s for s, _ in c["rows"]], dtype=np.int32)), out, **c["args"])
    close(f64(out), c["want"], KERNEL_TOL[dtype])


TC_SIZES = [(10, 1, 64), (16, 1, 32), (6, 2, 128), (4, 4, 64), (12, 2, 96)]


@pytest.mark.parametrize("heads,kv_heads,dim", TC_SIZES)
@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("kernel", ["attention_decode_mma", "attention_decode_tma"])
def test_window_in_the_one_token_kernels(heads, kv_heads, dim, window, kernel):
    if kernel == "attention_decode_tma" and dim not in (64, 128):
        pytest.skip("the TMA kernel takes key heads of 64 and 128")
    w = window or 500
    c = windowed_case(np.random.default_rng(dim + heads + w), heads, kv_heads, dim,
                      [(999, 1), (256, 1), (63, 1), (0, 1), (512, 1), (w, 1), (w - 1, 1), (2 * w + 331, 1)], window, "bfloat16")
    positions = np.array([p for _, p in c["rows"]], dtype=np.int32)
    chunks, n = (int(positions.max()) + 256) // 256, len(positions)
    part_o = torch.full((n, heads, chunks, dim), float("nan"), device=DEV)
    part_ml = torch.full((n, heads, chunks, 2), float("nan"), device=DEV)
    out = torch.full((n, heads * dim), 7.0, dtype=torch.bfloat16, device=DEV)
    getattr(ops(), kernel)(c["q"], c["kc"], c["vc"], c["table"], dev(positions), dev(np.arange(n, dtype=np.int32)), part_o, part_ml, out,
                           max_chunks=chunks, **c["args"])
    ops().tc_status_check(DEV)
    close(f64(out), c["want"], 1.2e-2, kernel)


@pytest.mark.parametrize("heads,kv_heads,dim", TC_SIZES)
@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("kernel", ["attention_prefill_mma", "attention_prefill_tc"])
def test_window_in_the_many_token_kernels(heads, kv_heads, dim, window, kernel):
    if kernel == "attention_prefill_tc" and dim not in (64, 128):
        pytest.skip("the tcgen05 kernel takes key heads of 64 and 128")
    seqs = [(0, 140), (130, 17), (0, 1), (63, 80), (300, 129), (420, 140)]
    c = windowed_case(np.random.default_rng(3 * dim + heads + (window or 0)), heads, kv_heads, dim, seqs, window, "bfloat16")
    tile = 128 if kernel == "attention_prefill_tc" else 16
    tile_seq = np.concatenate([np.full((n + tile - 1) // tile, b) for b, (_, n) in enumerate(seqs)]).astype(np.int32)
    tile_q0 = np.concatenate([np.arange(0, n, tile) for _, n in seqs]).astype(np.int32)
    q_lens = np.array([n for _, n in seqs], dtype=np.int32)
    cu = np.concatenate([[0], np.cumsum(q_lens)]).astype(np.int32)
    out = torch.full((len(c["rows"]), heads * dim), 7.0, dtype=torch.bfloat16, device=DEV)
    getattr(ops(), kernel)(c["q"], c["kc"], c["vc"], c["table"], dev(tile_seq), dev(tile_q0), dev(np.arange(len(seqs), dtype=np.int32)),
                           dev(np.array([s for s, _ in seqs], dtype=np.int32)), dev(q_lens), dev(cu), out, **c["args"])
    ops().tc_status_check(DEV)
    close(f64(out), c["want"], 1.2e-2, kernel)


def attention_part(dtype, hidden, m, tensors):
    from test_parts_gpu import lib, source
    _, config, _, parts, _ = lib()
    rot = m.get("rot") or {}
    position = {"kind": "rotary", "rotary_dim": rot["dims"], "theta": rot["base"], "pairing": "half"} if rot else None
    if rot.get("scaling"):
        position["frequency_blend"] = rot["scaling"]
    part = parts.build_part("mixer", config.PartSpec(
        "gqa_attention", {"hidden_size": hidden, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                          "values_from_keys": True, "qk_norm": "none", "position": position, "softmax_scale": m["scale"],
                          "window": (m.get("mask") or {}).get("size")}, {"q_proj": "q", "k_proj": "k", "o_proj": "o"}), TORCH[dtype])
    part.load(source(tensors, dtype))
    return part


@BOTH
@pytest.mark.parametrize("heads,kv,dim,window,rot", [(2, 1, 64, 90, 32), (2, 2, 20, 65, 20), (4, 2, 32, 128, 16)])
def test_one_key_that_stands_out_at_a_windows_edge(dtype, heads, kv, dim, window, rot):
    """Through the part and its cache: a row far back whose key every later query wants.  The last query sees it if it is
    window - 1 rows back and not if it is window rows back, whether the rows come whole, in portions or one by one, over a page
    border too; and it gets the key's value unturned."""
    from test_parts_gpu import Stepper
    hidden = 48
    rng = np.random.default_rng(dim)
    tensors = {"q": rng.normal(size=(heads * dim, hidden)) * 0.05, "k": rng.normal(size=(kv * dim, hidden)) * 0.05,
               "o": rng.normal(size=(hidden, heads * dim)) * 0.3}
    # input entry 0 makes queries and keys of one direction that no rotation touches much (the slowest pair), the others noise
    slow = rot // 2 - 1
    for h in range(heads):
        tensors["q"][h * dim:(h + 1) * dim, 0] = 0.0
        tensors["q"][h * dim + slow, 0] = 3.0
    for h in range(kv):
        tensors["k"][h * dim:(h + 1) * dim, 1] = 0.0
        tensors["k"][h * dim + slow, 1] = 3.0
    tensors = {k: rounded(v, "bfloat16") for k, v in tensors.items()}
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": 0.4, "mask": {"size": window},
         "rot": {"dims": rot, "base": 1e6, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}}}
    part = attention_part(dtype, hidden, m, tensors)
    seen = {}
    for back in (window - 1, window):
        length = 3 * window + 5
        act = rng.normal(size=(length, hidden)) * 0.3
        act[:, 0], act[:, 1] = 1.0, 0.0                       # every row asks ...
        act[length - 1 - back, 1] = 6.0                       # ... for this one
        act = rounded(act, "bfloat16")
        want = pk.attention_mixer(act, tensors, "", m)
        rows = dev(act, TORCH[dtype])
        for sizes in ([length], [window, 2, length - window - 2], [length - 3, 1, 1, 1], [40] * (length // 40) + [length % 40]):
            stepper = Stepper([part.cache_need()], dtype)
            part.prepare(stepper.cache.max_tokens, DEV)
            other = stepper.cache.alloc()                     # another sequence holds pages in between
            stepper.context([other], [70])
            stepper.cache.end_step([other], [70])
            slot, at, got = stepper.cache.alloc(), 0, []
            for count in [s for s in sizes if s]:
                ctx = stepper.context([slot], [count])
                got.append(f64(part.forward(ctx, rows[at:at + count].contiguous(), stepper.cache.line(0), True)))
                stepper.cache.end_step([slot], [count])
                at += count
            close(np.concatenate(got), want, 2e-5 if dtype == "float32" else 1.5e-2, f"{back} rows back, portions {sizes[:4]}")
        seen[back] = np.abs(want[-1]).max()
    assert seen[window - 1] > 5 * seen[window], seen


# ------------------------------------------------------------------------------------------- experts and head

@BOTH
@pytest.mark.parametrize("hidden,experts,top,ff,shared,scale", [(96, 7, 3, 40, 56, 2.5), (42, 4, 4, 30, 22, 0.7), (128, 11, 3, 128, 256, 1.3),
                                                                (256, 5, 1, 64, 128, 1.0), (64, 40, 6, 32, None, 1.7)])
def test_experts_weighted_by_scores_without_renormalizing_and_a_shared_one(dtype, hidden, experts, top, ff, shared, scale):
    """Corrections large enough to change most choices; counts of rows that go through every routing and product kernel."""
    from test_parts_gpu import Stepper, lib, source
    _, config, _, parts, _ = lib()
    rng = np.random.default_rng(hidden + experts)
    t = {"router": rng.normal(size=(experts, hidden)) * 0.1, "correction": rng.normal(size=experts) * 0.4 - 0.6}
    for e in range(experts):
        t.update({f"e{e}.gate": rng.normal(size=(ff, hidden)) * 0.15, f"e{e}.up": rng.normal(size=(ff, hidden)) * 0.15,
                  f"e{e}.down": rng.normal(size=(hidden, ff)) * 0.15})
    args = {"hidden_size": hidden, "num_experts": experts, "top_k": top, "expert_width": ff, "score": "sigmoid", "choice_bias": True,
            "renormalize": False, "routed_scale": scale}
    names = {"router": "router", "choice_bias": "correction", "w_gate": "e{e}.gate", "w_up": "e{e}.up", "w_down": "e{e}.down"}
    if shared:
        args["shared_expert"] = {"width": shared, "gate": False}
        names.update({f"shared_{n}": f"shared.{n}" for n in ("gate", "up", "down")})
        t.update({"shared.gate": rng.normal(size=(shared, hidden)) * 0.15, "shared.up": rng.normal(size=(shared, hidden)) * 0.15,
                  "shared.down": rng.normal(size=(hidden, shared)) * 0.15})
    t = {k: as32(v) if k in ("router", "correction") else rounded(v, "bfloat16") for k, v in t.items()}
    part = parts.build_part("feed_forward", config.PartSpec("routed_experts", args, names), TORCH[dtype])
    part.load(source(t, dtype))
    mlp = {"router": {"experts": experts, "top": top, "scale": scale}, "shared": {"ff": shared} if shared else None}
    for count, decode in ((1, True), (5, True), (5, False), (12, False), (40, False), (64, True), (300, False)):
        act = rounded(rng.normal(size=(count, hidden)), "bfloat16")
        margins = pk.choice_margin(act, t, "", mlp)
        act = act[margins > 1e-4]
        n = act.shape[0]
        stepper = Stepper([], dtype)
        ctx = stepper.engine.StepContext(stepper.workspace, TORCH[dtype], list(range(n)) if decode else [0], [3] * n if decode else [0],
                                         [1] * n if decode else [n])
        picked = []
        part.on_route = lambda ids: picked.append(ids.cpu().numpy().copy())
        got = f64(part.forward(ctx, dev(act, TORCH[dtype]), f32(act)))
        routes = []
        want = pk.experts_ff(act, t, "", mlp, routes=routes)
        assert np.array_equal(np.sort(picked[0], axis=1), np.sort(routes[0], axis=1)), f"{n} rows: the choice"
        close(got, want, 1e-5 if dtype == "float32" else 1.2e-2, f"{n} rows, decode {decode}")


@BOTH
@pytest.mark.parametrize("scale,cap", [(0.3, 12.0), (1.7, None), (1.0, 2.0), (1.0, None)])
def test_head_scales_then_caps(dtype, scale, cap):
    from test_parts_gpu import Stepper, lib, source
    _, config, _, parts, _ = lib()
    rng = np.random.default_rng(3)
    w = rounded(rng.normal(size=(90, 64)), "bfloat16")
    part = parts.build_part("head", config.PartSpec("vocab_head", {"vocab_size": 90, "width": 64, "scale": scale, "softcap": cap},
                                                    {"weight": "head"}), TORCH[dtype])
    part.load(source({"head": w}, dtype))
    stepper = Stepper([], dtype)
    for count in (3, 40):
        rows = rounded(rng.normal(size=(count, 64)) * 2, "bfloat16")
        ctx = stepper.engine.StepContext(stepper.workspace, TORCH[dtype], [0], [0], [count])
        z = rows @ w.T * scale
        close(f64(part.forward(ctx, dev(rows, TORCH[dtype]))), cap * np.tanh(z / cap) if cap else z, 3e-6)
