"""Grouped norms after the sum, per-layer token inputs, sigmoid attention with normed and rotated heads, gated linear
attention and rotated retention, each against the plain oracle function of the same mechanism: sizes of every kind, prompts
in portions, several sequences at once, single tokens, pages and slots in arbitrary order."""
import pytest
import torch

from nanoquantization_b200 import _lib
from nanoquantization_b200.layers import mixers as ops
from nanoquantization_b200.layers.sequence_mixers import GatedLinearMixer, ParallelMixer, RetentionMixer, SigmoidAttentionMixer
from oracle import verozen_oracle as O
from test_gpu_mixers import CASES, DEV, DTYPES, LENGTHS, Replay, close, cut, rand, schedules

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------------ norms and side input
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,groups", [(60, 3), (60, 1), (64, 16), (96, 32), (33, 11), (4096, 4), (4096, 1), (5120, 20), (1030, 2)])
def test_norm_in_groups_after_the_sum(width, groups, dtype):
    x, y, w = rand(7, width, seed=1) * 2, rand(7, 3, width, seed=2), 1 + 0.3 * rand(width, seed=3)
    x[2] = 0.0                                       # eps matters
    y[2] *= 1e-3
    norm = lambda t: O.group_norm(t.double(), groups, 1e-4, w.double())
    for terms, ydt in ((None, None), (3, torch.float32), (1, torch.float32), (3, torch.bfloat16)):
        yy = None if terms is None else y[:, :terms].contiguous().to(ydt)
        xs = x.to(DEV)
        h = ops.post_norm_(xs, None if yy is None else yy.to(DEV), 1.7, w.to(DEV), groups, 1e-4, dtype)
        want = norm(1.7 * x.double() + (0 if yy is None else yy.double().sum(1)))
        close(xs, want, torch.float32)
        assert h.dtype == dtype and torch.equal(h, xs.to(dtype))
    rows = torch.tensor([6, 0, 2, 0], device=DEV)
    close(ops.group_norm_rows(x.to(DEV), rows, w.to(DEV), groups, 1e-4, dtype), norm(x)[[6, 0, 2, 0]], dtype)
    close(ops.group_norm_rows(x.to(DEV), None, w.to(DEV), groups, 1e-4, torch.float32), norm(x), torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,width,dim,column", [(1, 64, 16, 32), (5, 48, 9, 18), (16, 256, 64, 0), (40, 96, 24, 24), (300, 512, 128, 256)])
def test_side_input(T, width, dim, column, dtype):
    gate, proj = (rand(dim, width, seed=1) * width ** -0.5).to(dtype), (rand(width, dim, seed=2) * dim ** -0.5).to(dtype)
    table, norm = rand(23, column + 2 * dim, seed=3).to(dtype), 1 + 0.3 * rand(width, seed=4)
    ids = torch.randint(0, 23, (T,), generator=torch.Generator().manual_seed(5))
    h = rand(T, width, seed=6).to(dtype)
    x = h.float().to(DEV)
    g = ops.linear_gelu_table(h.to(DEV), gate.to(DEV), ids.to(DEV), table.to(DEV), column)
    e = table.double()[ids, column:column + dim]
    close(g, O.gelu_tanh(h.double() @ gate.double().T) * e, dtype)
    out = ops.add_normed_(x, ops.linear(g, proj.to(DEV), torch.float32), norm.to(DEV), 1e-5, dtype)
    close(x, h.double() + O.side_input(h.double(), e, gate.double(), proj.double(), norm.double(), 1e-5), dtype)
    assert torch.equal(out, x.to(dtype))


@pytest.mark.parametrize("M", [1, 8, 16, 40])
def test_products_scale_the_stream_they_are_added_to(M):
    for dtype in DTYPES:
        y, w, x = rand(M, 96, seed=1).to(dtype), rand(72, 96, seed=2).to(dtype), rand(M, 72, seed=3) * 5
        s = x.to(DEV)
        ops.linear_residual_(s, y.to(DEV), w.to(DEV), 2.5)
        close(s, 2.5 * x.double() + y.double() @ w.double().T, torch.float32)


# --------------------------------------------------------------------------------------------------- sigmoid attention
def mix(r, mixer, inputs, dtype, state=None, width_out=None, col=8):
    """The mixer's own call (through the merged mixer, so that decode steps take their kernel) on given projections."""
    layer = ParallelMixer(8, {"only": mixer}, dtype=dtype, device=DEV, prefixes={"only": ""})
    spec = mixer.kv_spec()
    width = sum(n for _, n in mixer.in_parts)

    class Step:
        k_cache = v_cache = batch = None
    Step.state = state
    if spec is not None:
        Step.k_cache = torch.full((r.num_blocks, r.bs, spec.kv_heads, spec.head_dim), 300.0, dtype=dtype, device=DEV)
        Step.v_cache = torch.full((r.num_blocks, r.bs, spec.kv_heads, spec.v_dim), 300.0, dtype=dtype, device=DEV)

    def fn(b, rows):
        Step.batch = b
        act = torch.full((rows.shape[0], mixer.out_columns), 7.0, dtype=dtype, device=DEV)
        proj = torch.nn.functional.pad(rows, (0, layer.rows - width)).contiguous()
        layer.mix(proj, act, Step)
        return act
    return r.run([p.to(dtype) for p in inputs], fn)


def sigmoid_mixer(sizes, scale=0.3, eps=1e-4, out_scale=1.0, interleaved=True, base=70.0, bias=-1.0, seed=3):
    H, G, D, rot = sizes
    m = SigmoidAttentionMixer(heads=H, kv_heads=G, dim=D, rot_base=base, rot_dims=rot, interleaved=interleaved, scale=scale, eps=eps,
                              out_scale=out_scale, device=DEV)
    m.q_norm.copy_(1 + 0.3 * rand(D, seed=seed))
    m.k_norm.copy_(1 + 0.3 * rand(D, seed=seed + 1))
    m.temp.copy_(1 + 0.4 * rand(H, seed=seed + 2))
    m.bias.copy_(bias + rand(H, seed=seed + 3))
    m.base = base
    return m


def oracle_sigmoid(m, p):
    """On whole score matrices: the same definition as the oracle's loop (compared below)."""
    T, H, G, D = p.shape[0], m.heads, m.kv_heads, m.dim
    p, w = p.double().cpu(), {n: getattr(m, n).double().cpu() for n in ("q_norm", "k_norm", "temp", "bias")}
    q, k = p[:, :H * D].view(T, H, D), p[:, H * D:].view(T, G, D)

    def turned(x):
        x = x.clone()
        half = m.rot // 2
        a = torch.arange(T, dtype=torch.float64)[:, None, None] * m.base ** (-2.0 * torch.arange(half, dtype=torch.float64) / max(m.rot, 1))
        ia = torch.arange(half) * 2 if m.interleaved else torch.arange(half)
        ib = ia + 1 if m.interleaved else ia + half
        u, v = x[..., ia].clone(), x[..., ib].clone()
        x[..., ia], x[..., ib] = u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()
        return x
    qr, kr = turned(O.rms(q, m.eps) * w["q_norm"]), turned(O.rms(k, m.eps) * w["k_norm"])
    s = torch.einsum("ihd,jhd->hij", qr, kr.repeat_interleave(H // G, 1)) * m.scale * w["temp"][:, None, None] + w["bias"][:, None, None]
    pw = torch.sigmoid(s).tril()
    return (torch.einsum("hij,jhd->ihd", pw, k.repeat_interleave(H // G, 1)) * m.out_scale).reshape(T, H * D)


@pytest.mark.parametrize("interleaved", [True, False])
def test_the_two_forms_of_the_sigmoid_oracle_agree(interleaved):
    m = sigmoid_mixer((4, 2, 10, 6), interleaved=interleaved).cpu()
    p = rand(15, 60, seed=1)
    q, k = p[:, :40].double().view(15, 4, 10), p[:, 40:].double().view(15, 2, 10)
    turn = lambda x, w: O.rotate(O.rms(x, m.eps) * w.double(), m.base, 6, interleaved)
    want = O.sigmoid_attention(turn(q, m.q_norm), turn(k, m.k_norm), k, m.scale, m.temp.double(), m.bias.double())
    assert torch.allclose(oracle_sigmoid(m, p), want.flatten(1))


SIGMOID_SIZES = [(4, 2, 24, 16), (3, 3, 16, 0), (6, 1, 33, 32), (2, 2, 64, 64), (4, 1, 128, 64), (10, 1, 40, 2), (2, 1, 96, 48), (1, 1, 256, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", SIGMOID_SIZES, ids=str)
@pytest.mark.parametrize("schedule", CASES)
def test_sigmoid_attention(schedule, sizes, dtype):
    H, G, D, rot = sizes
    m = sigmoid_mixer(sizes, out_scale=0.8, interleaved=H != 3 and D != 24)
    p = [rand(n, (H + G) * D, seed=i).to(dtype) for i, n in enumerate(LENGTHS)]
    got = mix(Replay(LENGTHS, schedule), m, p, dtype)
    for i in range(len(LENGTHS)):
        close(got[i], oracle_sigmoid(m, p[i]), dtype, f32=5e-5, bf16=2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,G", [(24, 2), (64, 1), (128, 2)])
def test_sigmoid_attention_finds_the_one_key(D, G, dtype):
    """Every key is silent but one, which every later query finds, however far; at page and tile borders, in a prompt, in
    portions and decoded alone."""
    T, H = 300, 2
    m = sigmoid_mixer((H, G, D, 0), scale=16.0 / D, bias=0.0)
    for t in (m.q_norm, m.k_norm, m.temp):
        t.fill_(1.0)
    m.bias.fill_(-12.0)
    for j in (0, 1, 15, 16, 63, 64, 127, 128, 255, 298):
        p = 0.02 * rand(T, (H + G) * D, seed=1)
        p = p.view(T, H + G, D)
        p[:, :H, 0] = 3.0                      # every query looks along the first axis
        p[:, H:, 1] = 2.0                      # the keys lie along the second
        p[j, H:, 1] = 0.0
        p[j, H:, 0] = 25.0                     # but one: score 16 - 12 against -12, and its value stands out
        p = p.flatten(1).to(dtype)
        want = oracle_sigmoid(m, p)
        loud = want.view(T, H, D)[:, :, 0].abs()
        assert bool((loud[j:] > 20).all()) and bool((loud[:j] < 1).all())
        for sizes in ([T], [j + 1, 2, 40], [64, 2, 63, 3], [max(j, 1)] + [1] * 40 + [100]):
            close(mix(Replay((T,), [[(0, n)] for n in cut(T, sizes)], block_size=16), m, [p], dtype)[0], want, dtype, bf16=2e-2)


@pytest.mark.parametrize("D,rot", [(64, 32), (128, 64)])
@pytest.mark.parametrize("bias", [-6.0, 0.0, 30.0, -100.0])
def test_sigmoid_attention_of_long_prompts(bias, D, rot):
    """The sizes and pages of the tcgen05 kernel: portions that start anywhere, weights near 0 and near 1, two requests."""
    lengths, H, G, dtype = (1300, 389), 4, 2, torch.bfloat16
    m = sigmoid_mixer((H, G, D, rot), scale=2.0 * D ** -0.5, base=1e4, bias=bias)
    p = [rand(n, (H + G) * D, seed=6 + i).to(dtype) for i, n in enumerate(lengths)]
    p[0].view(-1, H + G, D)[400, H:] *= 40.0
    want = [oracle_sigmoid(m, x) for x in p]
    whole = [[(s, n) for s, n in enumerate(lengths)]]
    cuts = [[(0, 300), (1, 130)], [(0, 511), (1, 200)], [(0, 2)], [(0, 487), (1, 59)]]
    for schedule, bs in ((whole, 256), (whole, 128), (cuts, 128), (cuts, 256)):
        got = mix(Replay(lengths, schedule, block_size=bs), m, p, dtype)
        for a, b in zip(got, want):
            close(a, b, dtype, bf16=2e-2)
    assert int(_lib.mixer_status(torch.device(DEV)).item()) == 0


# ------------------------------------------------------------------------------- gated linear attention and retention
def gla_mixer(H, D, V, rank, tau, dtype, bias=2.0, spread=1.5, eps=1e-4):
    m = GatedLinearMixer(heads=H, dim=D, vdim=V, rank=rank, tau=tau, eps=eps, out_scale=0.9, dtype=dtype, device=DEV)
    m.a2.copy_((rand(H * D, rank, seed=1) * rank ** -0.5).to(dtype))
    m.a2_bias.copy_(bias + spread * rand(H * D, seed=2))
    m.norm.copy_(1 + 0.3 * rand(V, seed=3))
    return m


def linear_inputs(lengths, H, D, V, extra, dtype, seed=10):
    """q | k | v | gate | extra columns; keys lean towards the queries, so that no head's output nearly vanishes."""
    out = []
    for i, n in enumerate(lengths):
        q, k, v, g, a = (rand(n, c, seed=seed * i + j) for j, c in enumerate((H * D, H * D, H * V, H * V, extra)))
        out.append(torch.cat([q, 0.8 * q + 0.6 * k, v, g, a], 1).to(dtype))
    return out


def oracle_gla(m, p):
    T, H, D, V = p.shape[0], m.heads, m.dim, m.vdim
    q, k, v, g, a = p.double().cpu().split([H * D, H * D, H * V, H * V, m.rank], 1)
    z = a @ m.a2.double().cpu().T + m.a2_bias.double().cpu()
    decay = (torch.sigmoid(z) ** (1.0 / m.tau)).view(T, H, D)
    q, k, v = q.reshape(T, H, D), k.reshape(T, H, D) * D ** -0.5, v.reshape(T, H, V)
    o = O.rms(O.decayed_linear_attention(q, k, v, decay), m.eps) * m.norm.double().cpu()
    S = torch.zeros(H, D, V, dtype=torch.float64)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
    return 0.9 * o.reshape(T, -1) * O.silu(g), S


GLA_SIZES = [(3, 20, 28, 5), (1, 9, 33, 1), (2, 64, 64, 16), (2, 32, 128, 8), (4, 128, 64, 16), (1, 80, 48, 20), (2, 128, 256, 16), (6, 32, 32, 16), (1, 256, 64, 12)]


def check_gla(m, lengths, dtype, named_schedules, bf16=3e-2):
    p = linear_inputs(lengths, m.heads, m.dim, m.vdim, m.rank, dtype)
    want = [oracle_gla(m, x) for x in p]
    for schedule in named_schedules:
        r = Replay(lengths, schedule)
        state = torch.full((r.num_slots, m.heads, m.dim, m.vdim), 1e4, device=DEV)      # what an earlier owner left
        got = mix(r, m, p, dtype, {"gla": state})
        for i in range(len(lengths)):
            close(got[i], want[i][0], dtype, f32=2e-4, bf16=bf16)
            close(state[r.slots[i]], want[i][1], torch.float32, f32=2e-4 if dtype == torch.float32 else 2e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", GLA_SIZES, ids=str)
def test_gated_linear_attention(sizes, dtype):
    H, D, V, rank = sizes
    check_gla(gla_mixer(H, D, V, rank, 8.0, dtype), LENGTHS, dtype, [s for _, s in schedules(LENGTHS)])
    lengths = (300, 70)
    check_gla(gla_mixer(H, D, V, rank, 16.0, dtype), lengths, dtype,
              [[[(0, 300), (1, 70)]], [[(s, n)] for s, m in enumerate(lengths) for n in cut(m, [64, 1, 2, 130])], [[(0, 290), (1, 60)]] + [[(0, 1), (1, 1)]] * 10])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tau,bias,spread", [(1.0, -6.0, 4.0), (1.0, -40.0, 10.0), (0.25, 0.0, 8.0), (16.0, 12.0, 1.0)])
def test_gated_linear_attention_with_extreme_decays(tau, bias, spread, dtype):
    """Channels that forget everything at every token (the decays of a chunk multiply to far below the smallest float)
    beside channels that keep everything."""
    for D, V in ((64, 64), (32, 48)):
        m = gla_mixer(2, D, V, 4, tau, dtype, bias, spread)
        m.a2_bias[::5] = 9.0
        check_gla(m, (200, 33), dtype, [[[(0, 200), (1, 33)]], [[(0, n)] for n in cut(200, [17, 50, 2])] + [[(1, 20)], [(1, 13)]]])


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_linear_attention_carries_an_early_token_far(dtype):
    """Slow channels: one loud early key is still the loudest part of the state hundreds of tokens later, whichever way
    the tokens between are cut; and a sequence that starts in the same slot knows nothing of it."""
    H, D, V, T = 2, 64, 64, 500
    m = gla_mixer(H, D, V, 4, 16.0, dtype, bias=9.0, spread=0.1)
    p = linear_inputs((T,), H, D, V, 4, dtype)[0]
    p[3, H * D:2 * H * D] *= 30
    want, S = oracle_gla(m, p)
    fresh, _ = oracle_gla(m, p[100:140])
    for sizes in ([T], [2, 2, 60, 1, 435], [4] + [1] * 20 + [476]):
        r = Replay((T,), [[(0, n)] for n in cut(T, sizes)])
        state = torch.zeros(r.num_slots, H, D, V, device=DEV)
        close(mix(r, m, [p], dtype, {"gla": state})[0], want, dtype, f32=2e-4, bf16=3e-2)
        r2 = Replay((40,), [[(0, 40)]])
        r2.slots, r2.num_slots = r.slots, r.num_slots
        close(mix(r2, m, [p[100:140]], dtype, {"gla": state})[0], fresh, dtype, f32=2e-4, bf16=3e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(3, 20, 28, 8), (2, 64, 64, 64), (4, 128, 64, 32), (1, 9, 33, 0), (2, 128, 256, 128), (4, 32, 64, 32)], ids=str)
@pytest.mark.parametrize("lengths", [LENGTHS, (300, 70), (650, 601)], ids=str)
def test_rotated_retention(lengths, sizes, dtype):
    H, D, V, rot = sizes
    decay = [1 - 2.0 ** -(2 + 2 * h) for h in range(H)]
    m = RetentionMixer(heads=H, dim=D, vdim=V, decay=decay, eps=1e-4, out_scale=0.9, rot_base=500.0, rot_dims=rot, device=DEV)
    p = linear_inputs(lengths, H, D, V, 0, dtype)
    want = []
    for x in p:
        q, k, v, g = x.double().split([H * D, H * D, H * V, H * V], 1)
        turn = lambda t: O.rotate(t.reshape(-1, H, D), 500.0, rot, False)
        o = O.decayed_linear_attention(turn(q), turn(k) * D ** -0.5, v.reshape(-1, H, V), torch.tensor(decay, dtype=torch.float64)[None, :, None].expand(len(x), H, D))
        want.append(0.9 * O.rms(o, 1e-4).flatten(1) * O.silu(g))
    for name, schedule in schedules(lengths):
        if name == "mixed" and max(lengths) > 400:
            continue
        if name == "portions" and max(lengths) > 100:
            schedule = [[(s, n)] for s, t in enumerate(lengths) for n in cut(t, [64, 1, 2, 130])]
        r = Replay(lengths, schedule)
        state = torch.full((r.num_slots, H, D, V), 1e4, device=DEV)
        got = mix(r, m, p, dtype, {"retention": state})
        for i in range(len(lengths)):
            close(got[i], want[i], dtype, f32=2e-4, bf16=4e-2)


def test_bad_arguments_are_errors():
    x = torch.zeros(2, 8, device=DEV)
    lib = _lib.load_mixers()
    with pytest.raises(RuntimeError, match="bad shape"):
        ops.post_norm_(x, None, 1.0, x[0], 3, 1e-5, torch.float32)
    with pytest.raises(RuntimeError, match="bad shape"):
        _lib.check_mixers(lib.nqb200_gla_log_decay(x.data_ptr(), 8, x.data_ptr(), x.data_ptr(), x.data_ptr(), 2, 8, 4, 0.0, _lib.F32, None))
    with pytest.raises(RuntimeError, match="bad shape"):
        _lib.check_mixers(lib.nqb200_gelu_table(x.data_ptr(), x.data_ptr(), x.data_ptr(), 8, 4, x.data_ptr(), 2, 8, _lib.F32, None))
