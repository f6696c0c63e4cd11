"""Routing and the experts' linears against the plain oracle: groups, corrections, one expert or many, steps of every size."""
import pytest
import torch

from nanoquantization_b200 import _lib
from nanoquantization_b200.layers import moe
from nanoquantization_b200.layers.sequence_mixers import RoutedExperts
from oracle import verozen_oracle as O
from test_gpu_mixers import DEV, DTYPES, close, rand

pytestmark = pytest.mark.gpu


def router(E, top, groups, keep, scale=1.5, correction=None):
    r = _lib.RouterDesc(E, top, groups, keep, scale, None if correction is None else correction.data_ptr())
    r.keep_alive = correction
    return r


ROUTERS = [(16, 3, 2, 1), (12, 3, 3, 2), (8, 1, 8, 1), (128, 8, 8, 4), (64, 6, 1, 1), (257, 5, 1, 1), (1024, 40, 32, 3), (4, 4, 2, 2), (1, 1, 1, 1), (30, 6, 10, 2)]


@pytest.mark.parametrize("E,top,groups,keep", ROUTERS)
@pytest.mark.parametrize("T", [1, 7, 32, 33, 300])
def test_routing(T, E, top, groups, keep):
    logits, corr = rand(T, E, seed=1) * 2, 0.7 * rand(E, seed=2) - 0.3
    r = router(E, top, groups, keep, 1.5, corr.to(DEV))
    plan = moe.route(logits.to(DEV), r)
    expert, weight, order = plan.expert.cpu().view(T, top), plan.weight.cpu().view(T, top), plan.order.cpu()
    for t in range(T):
        want = O.route(logits[t].double(), corr.double(), top, groups, keep, 1.5)
        assert expert[t].tolist() == list(want)                 # best first
        assert torch.allclose(weight[t].double(), torch.stack(list(want.values())), rtol=1e-5, atol=1e-9)
    counts = torch.bincount(expert.flatten().long(), minlength=E)
    assert plan.offsets.tolist() == [0] + counts.cumsum(0).tolist()
    assert sorted(order.tolist()) == list(range(T * top))
    assert torch.equal(expert.flatten()[order.long()].long(), torch.repeat_interleave(torch.arange(E), counts))
    busy = counts.nonzero().flatten().tolist()
    assert plan.active.tolist()[:1 + len(busy)] == [len(busy)] + busy


def test_routing_details():
    """The best expert lies in a group that is not kept; negative choices count; weights know no correction; all scores tiny."""
    def run(z, corr, top, groups, keep, scale=1.0):
        c = torch.tensor(corr, device=DEV)
        p = moe.route(torch.tensor([z], device=DEV), router(len(z), top, groups, keep, scale, c))
        return dict(zip(p.expert.tolist(), p.weight.tolist()))
    z = [3.0, -9.0, -9.0, 1.0, 1.0, 1.0, 0.9, 0.9, 0.9]
    assert list(run(z, [0.0] * 9, 2, 3, 1)) == [3, 4]
    got = run(z, [-2.0] * 8 + [0.5], 3, 3, 2)
    s = torch.sigmoid(torch.tensor(z))
    assert list(got) == [8, 3, 4] and abs(got[8] - float(s[8] / (s[8] + s[3] + s[4]))) < 1e-6
    got = run([-60.0, -61.0], [0.0, 0.0], 2, 1, 1, 2.0)         # the 1e-20 of the sum is not negligible here
    s = torch.sigmoid(torch.tensor([-60.0, -61.0], dtype=torch.float64))
    assert abs(got[0] - float(2 * s[0] / (s.sum() + 1e-20))) < 1e-6
    nan = moe.route(torch.full((3, 8), float("nan"), device=DEV), router(8, 3, 2, 1))
    assert all(0 <= e < 8 for e in nan.expert.tolist())         # whatever the logits, the experts exist


def oracle_experts(h, up, down, plan, T, top):
    picks = [dict(zip(e, w)) for e, w in zip(plan.expert.view(T, top).tolist(), plan.weight.view(T, top).double().cpu())]
    return O.experts(h.double(), picks, up.double(), down.double())


EXPERT_SIZES = [  # tokens, width, ff, experts, top
    (1, 64, 40, 8, 2), (5, 60, 33, 6, 3), (8, 256, 96, 16, 3), (16, 192, 96, 16, 16), (17, 192, 96, 16, 3), (64, 256, 128, 8, 2), (150, 72, 200, 5, 2),
    (300, 320, 64, 4, 4), (33, 1024, 256, 32, 4), (700, 128, 384, 3, 1), (260, 512, 264, 2, 2), (40, 64, 64, 64, 1)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,ff,E,top", EXPERT_SIZES)
def test_experts(T, W, ff, E, top, dtype):
    h, up, down = rand(T, W, seed=1).to(dtype), (rand(E, ff, W, seed=2) * W ** -0.5).to(dtype), (rand(E, W, ff, seed=3) * ff ** -0.5).to(dtype)
    logits = rand(T, E, seed=4)
    logits[:, 0] += 1.5                                          # one expert is popular
    plan = moe.route(logits.to(DEV), router(E, top, 1, 1))
    u = moe.experts_up(h.to(DEV), up.to(DEV), plan)
    order = plan.order.long().cpu()
    ex = plan.expert.cpu().long()[order]
    want_u = torch.stack([O.gelu_erf(up[e].double() @ h[q // top].double()) for q, e in zip(order.tolist(), ex.tolist())])
    close(u, want_u, dtype)
    y = moe.experts_down(u, down.to(DEV), plan)
    assert y.shape == (T, top, W)
    close(y.double().sum(1), oracle_experts(h, up, down, plan, T, top), dtype, bf16=2e-2)
    assert int(_lib.mixer_status(torch.device(DEV)).item()) == 0


def test_an_experts_output_does_not_depend_on_the_rest_of_the_step():
    """The same token alone, among a few, and among many (other kernels, other places in the tiles): within rounding."""
    W, ff, E, top, dtype = 256, 128, 8, 2, torch.bfloat16
    m = RoutedExperts(W, ff, experts=E, top=top, groups=2, keep=2, scale=1.3, dtype=dtype, device=DEV)
    for name, seed in (("router", 1), ("up", 2), ("down", 3)):
        t = getattr(m, name)
        t.copy_((rand(*t.shape, seed=seed) * t.shape[-1] ** -0.5).to(dtype))
    h = rand(500, W, seed=5).to(dtype).to(DEV)
    many = m(h).double().sum(1)
    again = m(h).double().sum(1)
    assert torch.equal(many, again)
    for n in (1, 9, 16, 17, 100):
        few = m(h[:n].contiguous()).double().sum(1)
        assert float((few - many[:n]).abs().max()) <= 1.5e-2 * float(many.abs().max())


def test_every_kernel_is_reached():
    lib = _lib.load_moe()
    assert lib.nqb200_moe_linear_kernel(16, 96, 192, 3, _lib.BF16) == b"decode"
    assert lib.nqb200_moe_linear_kernel(17, 96, 192, 3, _lib.BF16) == b"tcgen05"
    assert lib.nqb200_moe_linear_kernel(17, 96, 100, 3, _lib.BF16) == b"simple"
    assert lib.nqb200_moe_linear_kernel(17, 96, 192, 3, _lib.F32) == b"simple"
    with pytest.raises(RuntimeError, match="bad shape"):
        moe.route(torch.zeros(1, 8, device=DEV), router(8, 5, 2, 1))
