"""Each sequence-mixing kernel against the plain oracle function of the same mechanism: sizes of every kind, prompts
in portions, several sequences at once, single tokens, pages and slots in arbitrary order."""
import pytest
import torch

from nanoquantization_b200 import _lib
from nanoquantization_b200.engine import StepBatch
from nanoquantization_b200.layers import mixers as ops
from nanoquantization_b200.layers.sequence_mixers import AttentionMixer
from oracle import vemedra_oracle as O

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def close(got, want, dtype, f32=2e-5, bf16=1.2e-2):
    """Largest difference against the largest value."""
    err = float((got.double().cpu() - want.double()).abs().max() / want.double().abs().max().clamp_min(1e-3))
    assert err <= (f32 if dtype == torch.float32 else bf16), err


class Replay:
    """Feeds whole sequences to a kernel step by step: ``schedule`` is a list of steps, each a list of
    (sequence, number of tokens).  Pages and slots are dealt in a shuffled order."""

    def __init__(self, lengths, schedule, block_size=8, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.lengths, self.schedule, self.bs = lengths, schedule, block_size
        per = [-(-n // block_size) for n in lengths]
        order = torch.randperm(sum(per) + 3, generator=g).tolist()
        self.blocks = [[order.pop() for _ in range(n)] for n in per]
        self.num_blocks = sum(per) + 3
        self.slots = torch.randperm(len(lengths) + 2, generator=g)[:len(lengths)].tolist()
        self.num_slots = len(lengths) + 2

    def steps(self):
        at = [0] * len(self.lengths)
        for step in self.schedule:
            starts = [at[s] for s, _ in step]
            b = StepBatch.host([[0] * n for _, n in step], starts, [self.blocks[s] for s, _ in step], [self.slots[s] for s, _ in step],
                               max(len(x) for x in self.blocks) + 1, self.bs).to(DEV)
            spans = [(s, at[s], at[s] + n) for s, n in step]
            for s, n in step:
                at[s] += n
            yield b, spans
        assert at == list(self.lengths)

    def run(self, inputs, fn):
        """``inputs[s]``: [tokens, ...] of sequence s; ``fn(batch, rows)`` -> rows of output."""
        outs = [[] for _ in self.lengths]
        for b, spans in self.steps():
            y = fn(b, torch.cat([inputs[s][lo:hi] for s, lo, hi in spans]).to(DEV))
            o = 0
            for s, lo, hi in spans:
                outs[s].append(y[o:o + hi - lo].clone())
                o += hi - lo
        return [torch.cat(x).cpu() for x in outs]


def cut(n, sizes):
    out, i = [], 0
    while n:
        k = min(n, sizes[i % len(sizes)])
        out.append(k)
        n -= k
        i += 1
    return out


def schedules(lengths):
    """whole prompts together; each alone in portions; portions of all of them interleaved, then single tokens."""
    yield "whole", [[(s, n) for s, n in enumerate(lengths)]]
    yield "portions", [[(s, k)] for s, n in enumerate(lengths) for k in cut(n, [3, 2, 17, 5])]
    rest, steps = list(lengths), []
    for s in range(len(lengths)):
        k = min(rest[s] - 1, 4 * s + 2)
        if k > 0:
            steps.append([(s, k)])
            rest[s] -= k
    while any(rest):
        step = []
        for s in range(len(lengths)):
            k = min(rest[s], 1 if len(steps) % 3 else 2 + s)
            if k:
                step.append((s, k))
                rest[s] -= k
        steps.append(step)
    yield "mixed", steps


LENGTHS = (21, 1, 50, 8)
CASES = [pytest.param(s, id=n) for n, s in schedules(LENGTHS)]


def rand(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps,width", [(1, 40), (2, 33), (3, 64), (4, 300), (5, 256), (12, 24)])
@pytest.mark.parametrize("schedule", CASES)
def test_norm_with_input_convolution(schedule, taps, width, dtype):
    x = [rand(n, width, seed=i) * 3 for i, n in enumerate(LENGTHS)]
    w, cw = 1 + 0.3 * rand(width, seed=9), rand(width, taps, seed=10)
    r = Replay(LENGTHS, schedule)
    state = torch.full((r.num_slots, taps - 1, width), 1e4, device=DEV)     # what an earlier owner left
    got = r.run(x, lambda b, rows: ops.rmsnorm_conv(rows, w.to(DEV), cw.t().contiguous().to(DEV), state, b, 1e-3, dtype))
    for i in range(len(LENGTHS)):
        h = O.rms_norm(x[i].double(), 1e-3, w.double())
        close(got[i], h + O.causal_conv(h, cw.double()), dtype)


def test_final_norm_takes_rows_and_stream_add_adds():
    x, w = rand(9, 70, seed=1), 1 + rand(70, seed=2)
    rows = torch.tensor([8, 0, 3], device=DEV)
    want = O.rms_norm(x.double(), 1e-5, w.double())
    close(ops.rmsnorm_rows(x.to(DEV), rows, w.to(DEV), 1e-5, torch.float32), want[[8, 0, 3]], torch.float32)
    close(ops.rmsnorm_rows(x.to(DEV), None, w.to(DEV), 1e-5, torch.bfloat16), want, torch.bfloat16)
    for dtype in DTYPES:
        e, step, ids = rand(12, 70, seed=3).to(dtype), rand(70, seed=4), torch.tensor([3, 11, 0, 3, 5, 6, 7, 8, 9])
        y = torch.full_like(x, float("nan")).to(DEV)
        ops.stream_add(y, ids.to(DEV), e.to(DEV), None, False)
        assert torch.equal(y.cpu(), e.float()[ids])
        ops.stream_add(y, ids.to(DEV), e.to(DEV), step.to(DEV), True)
        assert torch.allclose(y.cpu(), 2 * e.float()[ids] + step)
        ops.stream_add(y, None, None, step.to(DEV), True)
        assert torch.allclose(y.cpu(), 2 * e.float()[ids] + 2 * step, atol=1e-6)


def attend(r, mixer, q, k, v, dtype, pad=3, col=4):
    """Rotate, store, attend: the mixer's own call on a projection [q | k | v]; returns o [T, heads, vdim] per sequence."""
    H, G, D, V = mixer.heads, mixer.kv_heads, mixer.dim, mixer.vdim
    kc = torch.full((r.num_blocks, r.bs, G, D), 300.0, dtype=dtype, device=DEV)
    vc = torch.full((r.num_blocks, r.bs, G, V), 300.0, dtype=dtype, device=DEV)
    # the projection's columns start inside a wider buffer, and the output's in another
    proj = [torch.cat([torch.zeros(len(a), pad), a.flatten(1), b.flatten(1), c.flatten(1)], 1).to(dtype) for a, b, c in zip(q, k, v)]

    class Step:
        k_cache, v_cache, batch = kc, vc, None

    def fn(b, rows):
        Step.batch = b
        act = torch.full((rows.shape[0], H * V + 2 * col), 7.0, dtype=dtype, device=DEV)
        mixer.mix(rows.contiguous(), pad, act, col, Step)
        assert (act[:, :col] == 7).all() and (act[:, -col:] == 7).all()
        return act[:, col:-col].reshape(-1, H, V)
    return r.run(proj, fn)


def oracle_attend(m, q, k, v, base, rot, sink):
    q, k = O.rotate(q.double(), base, rot), O.rotate(k.double(), base, rot)
    return O.chunk_attention(q, k, v.double(), m.scale, m.softcap, m.chunk, sink.double()) * m.out_scale


def fast_attend(m, q, k, v, base, rot, sink):
    """The oracle's attention for long sequences: the same definition on whole score matrices."""
    T, H, G = q.shape[0], m.heads, m.kv_heads
    p = torch.arange(T, dtype=torch.float64)

    def turn(x):
        x = x.double().clone()
        a = p[:, None, None] * base ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)
        u, w = x[..., :rot // 2].clone(), x[..., rot // 2:rot].clone()
        x[..., :rot // 2], x[..., rot // 2:rot] = u * a.cos() - w * a.sin(), w * a.cos() + u * a.sin()
        return x
    q, k = turn(q), turn(k).repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m.scale
    s = m.softcap * torch.tanh(s / m.softcap)
    i, j = p.long()[:, None], p.long()[None, :]
    s = s.masked_fill((j > i) | (i // m.chunk != j // m.chunk), float("-inf"))
    s = torch.cat([s, sink.double()[:, None, None].expand(H, T, 1)], -1).softmax(-1)[..., :-1]
    return torch.einsum("hij,jhd->ihd", s, v.double().repeat_interleave(H // G, 1)) * m.out_scale


def test_the_two_forms_of_the_attention_oracle_agree():
    m = AttentionMixer(heads=2, kv_heads=1, dim=8, vdim=4, chunk=7, rot_base=50.0, rot_dims=6, scale=0.5, softcap=2.0, out_scale=1.5)
    q, k, v, sink = rand(20, 2, 8, seed=1), rand(20, 1, 8, seed=2), rand(20, 1, 4, seed=3), rand(2, seed=4)
    assert torch.allclose(fast_attend(m, q, k, v, 50.0, 6, sink), oracle_attend(m, q, k, v, 50.0, 6, sink))


ATTENTION_SIZES = [  # heads, kv_heads, dim, vdim, chunk, rot
    (4, 2, 24, 40, 13, 16), (3, 3, 16, 16, 1, 0), (6, 1, 33, 7, 8, 32), (2, 2, 64, 64, 1000, 64), (4, 1, 128, 128, 16, 64), (2, 1, 48, 80, 9, 48)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", ATTENTION_SIZES, ids=str)
@pytest.mark.parametrize("schedule", CASES)
def test_chunked_attention(schedule, sizes, dtype):
    H, G, D, V, chunk, rot = sizes
    m = AttentionMixer(heads=H, kv_heads=G, dim=D, vdim=V, chunk=chunk, rot_base=70.0, rot_dims=rot, scale=0.4, softcap=3.0, out_scale=1.7, device=DEV)
    sink = rand(H, seed=3)
    m.sink.copy_(sink)
    q, k, v = ([rand(n, h, d, seed=10 * i + j).to(dtype).float() for i, n in enumerate(LENGTHS)] for j, (h, d) in enumerate(((H, D), (G, D), (G, V))))
    got = attend(Replay(LENGTHS, schedule), m, q, k, v, dtype)
    for i in range(len(LENGTHS)):
        close(got[i], oracle_attend(m, q[i], k[i], v[i], 70.0, rot, sink), dtype, bf16=2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,V,G", [(24, 20, 2), (64, 64, 1), (128, 128, 2)])
@pytest.mark.parametrize("chunk", [40, 64, 100])
def test_attention_finds_the_one_key_and_respects_the_edges(chunk, D, V, G, dtype):
    """One key stands out.  Queries in its chunk and after it find it, however far; the chunk's last key is seen by
    itself only as long as the chunk lasts; the first query of the next chunk sees neither; without any loud key the
    sink takes its share.  In one prompt, in portions that end around the edges, and decoded alone."""
    T, H = 2 * chunk + 7, 2
    loud = [0, chunk - 1, chunk, chunk + 1, 2 * chunk - 1]
    m = AttentionMixer(heads=H, kv_heads=G, dim=D, vdim=V, chunk=chunk, rot_base=1e4, rot_dims=0, scale=1.0, softcap=30.0, device=DEV)
    sink = torch.tensor([2.0, -1.0])
    m.sink.copy_(sink)
    for j in loud:
        q, k, v = torch.zeros(T, H, D), 0.01 * rand(T, G, D, seed=1), rand(T, G, V, seed=2)
        q[:, :, 0] = 4.0
        k[j, :, 0] = 5.0                    # score about 17 against 0 for every other key
        v[j] += 20
        q, k, v = (t.to(dtype).float() for t in (q, k, v))
        want = oracle_attend(m, q, k, v, 1e4, 0, sink)
        seen = [t for t in range(T) if t >= j and t // chunk == j // chunk]
        assert all(bool((want[t].mean(-1).abs() > 10).all()) == (t in seen) for t in range(T))
        for sizes in ([T], [chunk - 1, 2, chunk - 2, 3], [chunk, 1], [2]):
            r = Replay((T,), [[(0, n)] for n in cut(T, sizes)], block_size=16)
            close(attend(r, m, [q], [k], [v], dtype)[0], want, dtype, bf16=2e-2)
    r = Replay((T,), [[(0, chunk - 3)]] + [[(0, 1)]] * (T - chunk + 3), block_size=16)
    close(attend(r, m, [q], [k], [v], dtype)[0], want, dtype, bf16=2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_over_many_keys(dtype):
    """Long chunks (several passes over key tiles), a far key among hundreds, grouped heads, few and many queries."""
    T, H, G, D, V, chunk = 700, 4, 2, 64, 96, 600
    m = AttentionMixer(heads=H, kv_heads=G, dim=D, vdim=V, chunk=chunk, rot_base=1e4, rot_dims=32, scale=0.2, softcap=20.0, device=DEV)
    sink = rand(H, seed=5)
    m.sink.copy_(sink)
    q, k, v = rand(T, H, D, seed=6), rand(T, G, D, seed=7), rand(T, G, V, seed=8)
    k[5, :, 40] = 25.0
    q[560:, :, 40] = 4.0
    q, k, v = (t.to(dtype).float() for t in (q, k, v))
    want = oracle_attend(m, q, k, v, 1e4, 32, sink)
    for steps in ([T], [T - 5, 1, 1, 1, 1, 1], [599, 2, 50, 49], [301, 297, 1, 1, 1, 99]):
        r = Replay((T,), [[(0, n)] for n in steps], block_size=64)
        close(attend(r, m, [q], [k], [v], dtype)[0], want, dtype, bf16=2e-2)


@pytest.mark.parametrize("D,V", [(128, 128), (64, 64), (128, 64), (64, 128)])
@pytest.mark.parametrize("chunk,softcap", [(100000, 4.0), (512, 60.0), (700, 3.0), (1000, 0.5)])
def test_attention_of_long_prompts(chunk, softcap, D, V):
    """The sizes and pages of the tcgen05 kernel: chunk borders inside its tiles, portions that start anywhere, caps that
    are far away and caps that bind, rows whose maximum moves late (loud keys near the end), two requests at once."""
    lengths, H, G, dtype = (1300, 389), 4, 2, torch.bfloat16
    m = AttentionMixer(heads=H, kv_heads=G, dim=D, vdim=V, chunk=chunk, rot_base=1e4, rot_dims=32, scale=0.25, softcap=softcap, out_scale=0.7, device=DEV)
    sink = rand(H, seed=5)
    m.sink.copy_(sink)
    qkv = []
    for i, n in enumerate(lengths):
        q, k, v = rand(n, H, D, seed=6 + i), rand(n, G, D, seed=17 + i), rand(n, G, V, seed=28 + i)
        k[n // 3, :, 40] = 9.0
        k[n - 100:, :, 41] = 6.0
        q[n // 2:, :, 40] = 4.0
        q[n - 60:, :, 41] = 5.0
        qkv.append([t.to(dtype).float() for t in (q, k, v)])
    q, k, v = zip(*qkv)
    want = [fast_attend(m, *t, 1e4, 32, sink) for t in qkv]
    whole = [[(s, n) for s, n in enumerate(lengths)]]
    cuts = [[(0, 300), (1, 130)], [(0, 511), (1, 200)], [(0, 2)], [(0, 487), (1, 59)]]
    for schedule, bs in ((whole, 256), (whole, 128), (cuts, 128)):
        r = Replay(lengths, schedule, block_size=bs)
        got = attend(r, m, q, k, v, dtype, pad=8, col=8)
        for a, b in zip(got, want):
            close(a, b, dtype, bf16=2e-2)
    assert int(_lib.mixer_status(torch.device(DEV)).item()) == 0


RETENTION_SIZES = [(3, 20, 28), (1, 9, 33), (2, 64, 64), (2, 32, 128), (4, 128, 64), (1, 80, 48)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", RETENTION_SIZES, ids=str)
@pytest.mark.parametrize("lengths", [LENGTHS, (300, 70)], ids=str)
def test_retention(lengths, sizes, dtype):
    H, D, V = sizes
    decay = [1 - 2.0 ** -(1 + 2 * h) for h in range(H)]
    q, k, v = ([rand(n, H, d, seed=10 * i + j).to(dtype) for i, n in enumerate(lengths)] for j, d in enumerate((D, D, V)))
    want = [O.retention(a.double(), b.double() * D ** -0.5, c.double(), decay) for a, b, c in zip(q, k, v)]
    proj = [torch.cat([torch.zeros(len(a), 5, dtype=dtype)] + [t.flatten(1) for t in (a, b, c)], 1) for a, b, c in zip(q, k, v)]
    dec = torch.tensor(decay, dtype=torch.float64).float().to(DEV)
    for name, schedule in schedules(lengths):
        if name == "portions" and max(lengths) > 100:
            schedule = [[(s, n)] for s, m in enumerate(lengths) for n in cut(m, [64, 1, 2, 130])]
        r = Replay(lengths, schedule)
        state = torch.full((r.num_slots, H, D, V), 1e4, device=DEV)
        got = r.run(proj, lambda b, rows: ops.retention(rows, 5, 5 + H * D, 5 + 2 * H * D, dec, state, b))
        for i in range(len(lengths)):
            close(got[i], want[i], dtype, f32=1e-4, bf16=1.2e-2)
            S = torch.zeros(H, D, V, dtype=torch.float64)
            for t in range(lengths[i]):
                S = torch.tensor(decay, dtype=torch.float64)[:, None, None] * S + k[i][t].double()[:, :, None] * D ** -0.5 * v[i][t].double()[:, None, :]
            close(state[r.slots[i]], S, torch.float32, f32=1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,V", [(3, 28), (1, 200), (5, 64)])
def test_head_norm_and_gate(H, V, dtype):
    T = 11
    o, g = rand(T, H, V, seed=1) * 4, rand(T, H * V, seed=2).to(dtype)
    gate = torch.cat([torch.zeros(T, 6, dtype=dtype), g], 1).to(DEV)
    act = torch.zeros(T, H * V + 8, dtype=dtype, device=DEV)
    ops.head_norm_gate(o.to(DEV), gate[:, 6:], act[:, 3:3 + H * V], 1e-3, 0.6)
    want = 0.6 * O.rms_norm(o.double(), 1e-3).flatten(1) * O.silu(g.double())
    close(act[:, 3:3 + H * V], want, dtype)
    assert (act[:, :3] == 0).all() and (act[:, 3 + H * V:] == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [5, 56, 96, 256])
@pytest.mark.parametrize("lengths", [LENGTHS, (400, 129)], ids=str)
def test_mingru(lengths, width, dtype):
    proj = [rand(n, 3 * width, seed=i).to(dtype) for i, n in enumerate(lengths)]
    zb, xb = rand(width, seed=20), rand(width, seed=21)
    for p in proj:
        p[:, :width // 2] -= 4          # half of the channels remember for long
    want, last = [], []
    for p in proj:
        z, x, g = p.double().split(width, 1)
        S = O.min_gru(z + zb.double(), x + xb.double())
        want.append(S * O.silu(g))
        last.append(S[-1])
    for _, schedule in schedules(lengths):
        r = Replay(lengths, schedule)
        state = torch.full((r.num_slots, width), 1e4, device=DEV)
        got = r.run(proj, lambda b, rows: ops.mingru(rows, width, zb.to(DEV), xb.to(DEV), state, b))
        for i in range(len(lengths)):
            close(got[i], want[i], dtype)
            close(state[r.slots[i]], last[i], torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
def test_clamped_glu(dtype):
    gu = (rand(13, 2 * 75, seed=1) * 3).to(dtype)
    gu[0, :4] = torch.tensor([1.5, 1.50001, -9.0, 0.0])
    close(ops.clamped_glu(gu.to(DEV), 1.5), O.clamped_glu(gu[:, :75].double(), gu[:, 75:].double(), 1.5), dtype)


# ------------------------------------------------------------------ retention with norm and gate, prompts in bf16
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(2, 64, 64), (3, 32, 128), (1, 128, 256), (2, 256, 48), (2, 24, 200), (1, 20, 28)], ids=str)
@pytest.mark.parametrize("lengths", [(300, 70), (530, 1, 256)], ids=str)
def test_retention_of_prompts(lengths, sizes, dtype):
    """Chunk borders of the chunkwise form fall elsewhere in every schedule; a slow decay carries far."""
    H, D, V = sizes
    decay = [1 - 2.0 ** -(3 + 3 * h) for h in range(H)]
    off, col, eps, scale = 8, 4, 1e-4, 1.3
    parts = [[rand(n, H, d, seed=10 * i + j).to(dtype) for j, d in enumerate((D, D, V, V))] for i, n in enumerate(lengths)]
    for q, k, v, g in parts:
        q += 0.5                       # outputs of ordinary size: the norm would blow up rounding where they vanish
        k += 0.5
    want = [scale * O.rms_norm(O.retention(q.double(), k.double() * D ** -0.5, v.double(), decay), eps).flatten(1) * O.silu(g.double().flatten(1))
            for q, k, v, g in parts]
    proj = [torch.cat([torch.zeros(len(p[0]), off, dtype=dtype)] + [t.flatten(1) for t in p], 1) for p in parts]
    dec = torch.tensor(decay, dtype=torch.float64).float().to(DEV)
    desc = _lib.RetentionDesc(H, D, V, eps, scale, dec.data_ptr())
    total = sum(lengths)
    whole = [[(s, n) for s, n in enumerate(lengths)]]
    cuts = [[(s, k)] for s, n in enumerate(lengths) for k in cut(n, [100, 2, 40, 1, 259])]
    halves = [[(s, n // 2) for s, n in enumerate(lengths) if n // 2], [(s, n - n // 2) for s, n in enumerate(lengths)]]
    for schedule in (whole, cuts, halves):
        r = Replay(lengths, schedule)
        state = torch.full((r.num_slots, H, D, V), 1e4, device=DEV)

        def fn(b, rows):
            act = torch.full((rows.shape[0], H * V + 10), 7.0, dtype=dtype, device=DEV)
            ops.retention_gated(rows, off, desc, dec, state, act, col, b)
            assert (act[:, :col] == 7).all() and (act[:, col + H * V:] == 7).all()
            return act[:, col:col + H * V]
        got = r.run(proj, fn)
        for i, (q, k, v, g) in enumerate(parts):
            close(got[i], want[i], dtype, f32=1e-3, bf16=3e-2)
            S = torch.zeros(H, D, V, dtype=torch.float64)
            dd = torch.tensor(decay, dtype=torch.float64)[:, None, None]
            for t in range(lengths[i]):
                S = dd * S + k[t].double()[:, :, None] * D ** -0.5 * v[t].double()[:, None, :]
            close(state[r.slots[i]], S, torch.float32, f32=2e-4)
    assert total > 300


# ------------------------------------------------------------------ decode steps
def dense_case(M, N, K, seed=0):
    return rand(M, K, seed=seed).bfloat16(), (rand(N, K, seed=seed + 1) * K ** -0.5).bfloat16()


@pytest.mark.parametrize("M,N,K", [(1, 16, 8), (1, 40, 40), (3, 33, 104), (8, 512, 256), (9, 100, 1000), (16, 300, 4096), (5, 1, 2056)])
def test_dense_decode(M, N, K):
    x, w = dense_case(M, N, K)
    want = x.double() @ w.double().t()
    xd, wd = x.to(DEV), w.to(DEV)
    assert ops.decode_sized(xd, wd)
    close(ops.linear(xd, wd), want, torch.bfloat16)
    close(ops.linear(xd, wd, torch.float32), want, torch.float32)
    stream = rand(M, N, seed=5)
    close(ops.linear_residual_(stream.to(DEV), xd, wd), stream.double() + want, torch.float32)


def test_linears_of_other_sizes_take_the_library():
    for M, N, K in ((17, 24, 64), (2, 24, 36)):
        x, w = dense_case(M, N, K)
        want = x.double() @ w.double().t()
        assert not ops.decode_sized(x.to(DEV), w.to(DEV))
        close(ops.linear(x.to(DEV), w.to(DEV), torch.float32), want, torch.float32)
        stream = rand(M, N, seed=5)
        got = stream.to(DEV)
        assert ops.linear_residual_(got, x.to(DEV), w.to(DEV)) is got
        close(got, stream.double() + want, torch.float32)
        close(ops.linear_residual_(stream.to(DEV), x.float().to(DEV), w.float().to(DEV)), stream.double() + want, torch.float32)


@pytest.mark.parametrize("M,ff,K", [(1, 24, 64), (7, 130, 256), (16, 72, 1000)])
def test_dense_with_clamped_glu(M, ff, K):
    x, w = dense_case(M, 2 * ff, K)
    x *= 3
    y = x.double() @ w.double().t()
    close(ops.dense_glu(x.to(DEV), w.to(DEV), 1.7), O.clamped_glu(y[:, :ff], y[:, ff:], 1.7), torch.bfloat16)


@pytest.mark.parametrize("B,width,K", [(1, 40, 64), (5, 33, 256), (16, 128, 1000)])
def test_dense_with_mingru(B, width, K):
    """Three tokens of every sequence, the first from a slot that another sequence has left."""
    w = (rand(3 * width, K, seed=1) * K ** -0.5).bfloat16()
    zb, xb = rand(width, seed=2), rand(width, seed=3)
    xs = [rand(3, K, seed=10 + i).bfloat16() for i in range(B)]
    r = Replay((3,) * B, [[(s, 1) for s in range(B)]] * 3)
    state = torch.full((r.num_slots, width), 1e4, device=DEV)
    got = r.run(xs, lambda b, rows: ops.dense_mingru(rows, w.to(DEV), zb.to(DEV), xb.to(DEV), state, b))
    for i in range(B):
        z, u, g = (xs[i].double() @ w.double().t()).split(width, 1)
        S = O.min_gru(z + zb.double(), u + xb.double())
        close(got[i], S * O.silu(g), torch.bfloat16)
        close(state[r.slots[i]], S[-1], torch.float32)


@pytest.mark.parametrize("att", [(4, 2, 24, 40, 13, 16), (2, 2, 64, 64, 1000, 64), (12, 1, 128, 128, 40, 64), (6, 2, 256, 256, 300, 0), (5, 1, 8, 8, 1, 8), None], ids=str)
@pytest.mark.parametrize("ret", [(3, 20, 28), (2, 64, 64), (2, 128, 256), (1, 9, 33), (1, 300, 600), None], ids=str)
def test_one_launch_decode_step(att, ret):
    """Attention and retention of a decode step, side by side in one launch: after a prompt that the other kernels
    read, and from the first token on."""
    if att is None and ret is None:
        return
    dtype, lengths, decoded = torch.bfloat16, (330, 1, 45), 9
    H, G, D, V, chunk, rot = att or (0, 0, 0, 0, 1, 0)
    RH, RD, RV = ret or (0, 0, 0)
    na, a_off, a_col = H * D + G * (D + V), 3, 6
    r_off, r_col = a_off + na + 2, a_col + H * V + 3
    decay = [1 - 2.0 ** -(2 + 3 * h) for h in range(RH)]
    dec = torch.tensor(decay or [0.0]).float().to(DEV)
    sink = rand(max(H, 1), seed=3)
    m = AttentionMixer(heads=H, kv_heads=G, dim=D, vdim=V, chunk=chunk, rot_base=70.0, rot_dims=rot, scale=0.3, softcap=4.0, out_scale=1.7, device=DEV) if att else None
    if att:
        m.sink.copy_(sink)
    rdesc = _lib.RetentionDesc(RH, RD, RV, 1e-4, 0.8, dec.data_ptr()) if ret else None
    assert ops.mixer_decode_supported(m and m.desc(), rdesc)
    width = r_off + 2 * RH * (RD + RV) + 1
    proj = [rand(n, width, seed=i).to(dtype) for i, n in enumerate(lengths)]
    for p in proj:
        p[:, r_off:r_off + 2 * RH * RD] += 0.5
    schedule = [[(s, n - decoded) for s, n in enumerate(lengths) if n > decoded]] + [[(s, 1) for s, n in enumerate(lengths) if k < n and (n > decoded or k == 0)] for k in range(decoded)]
    r = Replay(lengths, schedule, block_size=16)
    kc = torch.full((r.num_blocks, 16, max(G, 1), max(D, 1)), 300.0, dtype=dtype, device=DEV)
    vc = torch.full((r.num_blocks, 16, max(G, 1), max(V, 1)), 300.0, dtype=dtype, device=DEV)
    state = torch.full((r.num_slots, max(RH, 1), max(RD, 1), max(RV, 1)), 1e4, device=DEV)

    class Step:
        k_cache, v_cache, batch = kc, vc, None

    def fn(b, rows):
        act = torch.full((rows.shape[0], r_col + RH * RV + 2), 7.0, dtype=dtype, device=DEV)
        rows = rows.contiguous()
        if b.max_len == 1:
            ops.mixer_decode(rows, act, att and (m.desc(), m.rope_desc(), a_off, m.value_column(a_off), a_col, kc, vc), ret and (rdesc, r_off, r_col, state), b)
            assert (act[:, :a_col] == 7).all() and (act[:, a_col + H * V:r_col] == 7).all() and (act[:, -2:] == 7).all()
            return act
        Step.batch = b
        if att:
            m.mix(rows, a_off, act, a_col, Step)
        if ret:
            ops.retention_gated(rows, r_off, rdesc, dec, state, act, r_col, b)
        return act
    got = r.run(proj, fn)
    for i, n in enumerate(lengths):
        if att:
            q, k, v = proj[i][:, a_off:a_off + na].float().split([H * D, G * D, G * V], 1)
            want = oracle_attend(m, q.reshape(n, H, D), k.reshape(n, G, D), v.reshape(n, G, V), 70.0, rot, sink)
            close(got[i][-decoded:, a_col:a_col + H * V], want.flatten(1)[-decoded:], dtype, bf16=2e-2)
        if ret:
            q, k, v, g = proj[i][:, r_off:-1].double().split([RH * RD, RH * RD, RH * RV, RH * RV], 1)
            o = O.retention(q.reshape(n, RH, RD), k.reshape(n, RH, RD) * RD ** -0.5, v.reshape(n, RH, RV), decay)
            want = 0.8 * O.rms_norm(o, 1e-4).flatten(1) * O.silu(g)
            close(got[i][-decoded:, r_col:r_col + RH * RV], want[-decoded:], dtype, bf16=3e-2)


def test_bad_arguments_are_errors():
    b = StepBatch.host([[1]], [0], [[0]], [0], 1, 8).to(DEV)
    x = torch.zeros(1, 8, device=DEV)
    with pytest.raises(TypeError):
        ops.rmsnorm_rows(x, None, x[0], 1e-5, torch.float16)
    with pytest.raises(RuntimeError, match="bad shape"):
        _lib.check_mixers(_lib.load_mixers().nqb200_clamped_glu(x.data_ptr(), x.data_ptr(), 1, 0, 1.0, _lib.F32, None))
    with pytest.raises(RuntimeError, match="null pointer"):
        _lib.check_mixers(_lib.load_mixers().nqb200_mingru(None, 8, 0, 1, 2, None, None, None, None, 4, None, b.desc, _lib.F32, None))
