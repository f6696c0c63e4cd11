"""Verozen without a GPU: configuration, checkpoint names and loading, sizes that only the tensors give, and the oracle's
own consistency."""
import copy
import json
import math

import pytest
import torch

import verozen_cases as C
from nanoquantization_b200.engine import KVSpec
from nanoquantization_b200.models import MODELS, VerozenConfig, VerozenForCausalLM, build_model, model_class
from nanoquantization_b200.utils.loader import tensor_shapes
from oracle import verozen_oracle as O


def test_configuration_errors_are_reported():
    def broken(change):
        c = copy.deepcopy(C.config())
        change(c)
        return VerozenForCausalLM(VerozenConfig.from_dict(c))
    with pytest.raises(ValueError, match="unknown mixer `mamba`"):
        broken(lambda c: c["layers"][1].update(type="mamba"))
    with pytest.raises(ValueError, match="unknown feed-forward `dense`"):
        broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    with pytest.raises(ValueError, match="rank"):
        broken(lambda c: c["layers"][1]["mixer"].pop("rank"))
    with pytest.raises(ValueError, match="vdim must be dim"):
        broken(lambda c: c["layers"][0]["mixer"].update(vdim=48))
    with pytest.raises(ValueError, match="norm: 60 in 7 groups"):
        broken(lambda c: c["norm"].update(groups=7))
    with pytest.raises(ValueError, match="experts: 3 of 12 from 0 of 3"):
        broken(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=0))
    with pytest.raises(ValueError, match="experts: 5 of 12 from 1 of 3"):
        broken(lambda c: (c["layers"][0]["mlp"]["router"]["groups"].update(keep=1), c["layers"][0]["mlp"]["router"].update(top=5)))
    with pytest.raises(ValueError, match="rotated"):
        broken(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=26))
    with pytest.raises(ValueError, match="tau"):
        broken(lambda c: c["layers"][1]["mixer"].update(tau=0.0))
    with pytest.raises(TypeError):
        VerozenForCausalLM(VerozenConfig.from_dict(C.config()), dtype=torch.float16)


def test_cache_layout_follows_the_layers():
    lay = VerozenForCausalLM(VerozenConfig.from_dict(C.config())).cache_layout()
    assert lay.kv == [KVSpec(2, 40, 40), None, None, None]
    assert lay.states == [{}, {"gla": (3, 24, 40)}, {"retention": (2, 24, 56)}, {"gla": (2, 40, 24)}]
    assert lay.recurrent and lay.visible_from(1000) == 0       # attention sees everything: nothing is given back early


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_checkpoint_loads_through_the_registry(tmp_path, dtype):
    from safetensors.torch import save_file
    c = C.config()
    w = C.weights(c, 3)
    on_disk = copy.deepcopy(c)
    for lay in on_disk["layers"]:
        lay["mixer"].pop("rank", None)                         # config.json does not have it: the tensor's shape says it
    (tmp_path / "config.json").write_text(json.dumps(on_disk))
    save_file(w, str(tmp_path / "model.safetensors"))
    assert tensor_shapes(str(tmp_path))["l3.mix.a1"] == (11, 60)
    assert model_class(on_disk) is MODELS["Verozen"]
    m = build_model(str(tmp_path), device="cpu", dtype=dtype)
    named = m.checkpoint_tensors()
    assert set(named) == set(w)
    for k, v in w.items():
        assert torch.equal(named[k].float(), v.float()), k
    # what reads the same input lies in one matrix, an expert in its place among all
    assert torch.equal(m.layers[3].mixer.w_in[256:267].float(), w["l3.mix.a1"].float())
    assert torch.equal(m.layers[0].mlp.up[7].float(), w["l0.mlp.e7.up"].float())
    assert m.layers[2].mlp is None and m.layers[2].norm2 is None
    some = dict(w)
    del some["l0.mlp.e3.down"]
    save_file(some, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="l0.mlp.e3.down"):
        build_model(str(tmp_path), device="cpu", dtype=dtype)
    save_file(dict(w, extra=torch.zeros(2)), str(tmp_path / "model.safetensors"))
    with pytest.raises(AttributeError, match="extra"):
        build_model(str(tmp_path), device="cpu", dtype=dtype)


# ------------------------------------------------------------------ the oracle against other forms of the same maths
def test_oracle_linear_attention_equals_the_sum_over_the_past():
    g = torch.Generator().manual_seed(0)
    T, H, D, V = 9, 2, 5, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    decay = torch.rand(T, H, D, generator=g, dtype=torch.float64)
    o = O.decayed_linear_attention(q, k, v, decay)
    for t in range(T):
        for h in range(H):
            want = sum((q[t, h] * k[j, h] * decay[j + 1:t + 1, h].prod(0)).sum() * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want)


def test_oracle_rotation_layouts_are_permutations_of_each_other():
    r = torch.randn(5, 2, 9, dtype=torch.float64)
    order = [0, 2, 4, 1, 3, 5, 6, 7, 8]                        # pairs (0,1) (2,3) (4,5) -> (0,3) (1,4) (2,5)
    assert torch.allclose(O.rotate(r, 50.0, 6, True)[..., order], O.rotate(r[..., order], 50.0, 6, False))
    z = torch.view_as_complex(r[3, :, 2:4].contiguous()) * complex(math.cos(3 * 50 ** (-2 / 6)), math.sin(3 * 50 ** (-2 / 6)))
    assert torch.allclose(torch.view_as_complex(O.rotate(r, 50.0, 6, True)[3, :, 2:4].contiguous()), z)


def test_oracle_sigmoid_attention_counts_keys():
    T = 6
    q, k, v = torch.zeros(T, 2, 3, dtype=torch.float64), torch.zeros(T, 1, 3, dtype=torch.float64), torch.ones(T, 1, 2, dtype=torch.float64)
    o = O.sigmoid_attention(q, k, v, 0.5, torch.ones(2), torch.tensor([0.0, -math.log(3.0)], dtype=torch.float64))
    n = torch.arange(1, T + 1, dtype=torch.float64)
    assert torch.allclose(o[:, 0, 0], n / 2) and torch.allclose(o[:, 1, 1], n / 4)     # not normalised


def test_oracle_routing_takes_groups_first():
    z = torch.tensor([3.0, -9, -9, 1, 1, 1, 0.9, 0.9, 0.9], dtype=torch.float64)       # the best expert is in the worst group
    none = torch.zeros(9, dtype=torch.float64)
    s = torch.sigmoid(z)
    w = O.route(z, none, 2, 3, 1, 2.0)
    assert list(w) == [3, 4] and torch.allclose(w[3], torch.tensor(1.0, dtype=torch.float64))
    assert set(O.route(z, none, 2, 3, 3, 1.0)) == {0, 3}
    w = O.route(z, none - 2.0 + 2.5 * (torch.arange(9) == 8), 3, 3, 2, 1.0)            # negative choices are not left out
    assert set(w) == {8, 3, 4} and torch.allclose(w[8], s[8] / (s[8] + s[3] + s[4]))   # and weights know no correction


def test_oracle_group_norm_and_side_input():
    x = torch.tensor([3.0, 4.0, 0.0, 2.0], dtype=torch.float64)
    assert torch.allclose(O.group_norm(x, 2, 0.0, torch.tensor([1.0, 1, 1, 3])), x / torch.tensor([12.5 ** 0.5] * 2 + [2 ** 0.5, 2 ** 0.5 / 3]))
    assert torch.allclose(O.group_norm(x, 1, 0.5, torch.ones(4)), x / (29 / 4 + 0.5) ** 0.5)
    y = O.side_input(torch.eye(2, dtype=torch.float64), torch.ones(2, 1), torch.tensor([[1.0, -50.0]], dtype=torch.float64), torch.ones(2, 1, dtype=torch.float64), torch.ones(2), 0.0)
    assert torch.allclose(y[0], torch.ones(2, dtype=torch.float64)) and torch.isnan(y[1]).all()     # gelu(-50) is zero
    u = torch.linspace(-4, 4, 9, dtype=torch.float64)
    assert torch.allclose(O.gelu_tanh(u), torch.nn.functional.gelu(u, approximate="tanh")) and torch.allclose(O.gelu_erf(u), torch.nn.functional.gelu(u))
