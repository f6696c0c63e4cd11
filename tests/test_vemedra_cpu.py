"""Vemedra without a GPU: configuration, checkpoint names and loading, the engine's bookkeeping for models with
recurrent states and chunked attention, and the oracle's own consistency."""
import json

import pytest
import torch

import vemedra_cases as C
from nanoquantization_b200.engine import BlockManager, CacheLayout, KVSpec, Scheduler, Sequence, StatePool, StepBatch
from nanoquantization_b200.models import MODELS, VemedraConfig, VemedraForCausalLM, build_model, model_class
from oracle import vemedra_oracle as O


def test_runs_follow_the_loop():
    cfg = VemedraConfig.from_dict(C.config(loop=(1, 3, 3)))
    assert cfg.runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert VemedraConfig.from_dict(C.config(loop=None)).runs() == [(i, None) for i in range(4)]
    assert VemedraConfig.from_dict(C.config(loop=(0, 4, 1))).runs() == [(0, 0), (1, None), (2, None), (3, None)]


def test_configuration_errors_are_reported():
    bad = C.config()
    bad["layers"][1] = dict(bad["layers"][1], type="lstm")
    with pytest.raises(ValueError, match="unknown mixer `lstm`"):
        VemedraConfig.from_dict(bad)
    with pytest.raises(ValueError, match="loop"):
        VemedraConfig.from_dict(C.config(loop=(2, 9, 2)))
    bad = C.config()
    bad["layers"][1] = dict(bad["layers"][1], mlp={"kind": "routed", "ff": 8, "limit": 1.0})
    with pytest.raises(ValueError, match="unknown feed-forward"):
        VemedraConfig.from_dict(bad)
    with pytest.raises(ValueError, match="decays"):
        VemedraForCausalLM(VemedraConfig.from_dict(C.config([C.parallel(right=dict(C.retention(3), heads=2))], loop=None)))
    with pytest.raises(TypeError):
        VemedraForCausalLM(VemedraConfig.from_dict(C.config()), dtype=torch.float16)


def test_cache_layout_has_one_entry_per_run():
    m = VemedraForCausalLM(VemedraConfig.from_dict(C.config()))
    lay = m.cache_layout()
    assert len(lay.kv) == len(lay.states) == 8
    assert lay.kv[0] == KVSpec(2, 24, 40, 13) and lay.kv[1] is None and lay.kv[2] == lay.kv[4] == KVSpec(2, 18, 10, 7)
    assert lay.states[0] == {"retention": (3, 20, 28), "canon1": (3, 48)}
    assert lay.states[1] == {"mingru": (56,), "canon1": (3, 48), "canon2": (3, 48)}
    # chunks of 13 and of 7: the earlier of the two chunk starts is still needed
    assert [lay.visible_from(p) for p in (0, 6, 7, 12, 13, 14, 26, 27)] == [0, 0, 0, 0, 7, 13, 21, 21]


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_checkpoint_loads_through_the_registry(tmp_path, dtype):
    from safetensors.torch import save_file
    c = C.config()
    w = C.weights(c, 3)
    (tmp_path / "config.json").write_text(json.dumps(c))
    save_file(w, str(tmp_path / "model.safetensors"))
    assert model_class(c) is MODELS["Vemedra"]
    m = build_model(str(tmp_path), device="cpu", dtype=dtype)
    named = m.checkpoint_tensors()
    assert set(named) == set(w)
    for k, v in w.items():
        assert torch.equal(named[k].float(), v.float()), k
    # parts of a layer that read the same input lie in one matrix, in the order of their columns
    mix = m.layers[2].mixer
    assert torch.equal(mix.w_in[36:72].float(), w["l2.mix.left.k"].float())
    assert torch.equal(mix.w_out[:, 20:].float(), w["l2.mix.right.o"].float())
    some = dict(w)
    del some["l1.canon2"]
    save_file(some, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="l1.canon2"):
        build_model(str(tmp_path), device="cpu", dtype=dtype)
    save_file(dict(w, extra=torch.zeros(2)), str(tmp_path / "model.safetensors"))
    with pytest.raises(AttributeError, match="extra"):
        build_model(str(tmp_path), device="cpu", dtype=dtype)
    with pytest.raises(ValueError, match="no model"):
        model_class({"architecture": "Nemesis"})
    with pytest.raises(TypeError):
        build_model(str(tmp_path), device="cpu", dtype=torch.float16)


def test_registry_reads_a_hugging_face_config():
    c = {"architectures": ["Qwen3ForCausalLM"], "num_hidden_layers": 1, "vocab_size": 64, "hidden_size": 128, "num_attention_heads": 2,
         "num_key_value_heads": 1, "max_position_embeddings": 32, "intermediate_size": 128, "head_dim": 64, "rope_theta": 1e4,
         "quantization_config": {"w_bits": 4, "group_size": 64}}
    cfg = model_class(c).config(c)
    assert cfg.total_num_kv_heads == 1 and cfg.group_size == 64 and cfg.rope_theta == 1e4


def test_blocks_behind_every_chunk_are_given_back():
    bm = BlockManager(num_blocks=8, block_size=4)
    s = Sequence(0, [1] * 18, 4)
    assert bm.ensure(s, 18) and len(bm.free) == 3
    held = list(s.blocks)
    bm.reclaim(s, 3)
    assert s.blocks == held
    bm.reclaim(s, 9)                      # blocks 0 and 1 end at 7; block 2 holds position 9
    assert s.blocks == [-1, -1] + held[2:] and len(bm.free) == 5
    bm.reclaim(s, 9)
    assert len(bm.free) == 5
    assert bm.ensure(s, 21) and len(s.blocks) == 6 and len(bm.free) == 4
    bm.release(s)
    assert sorted(bm.free) == list(range(8))


def test_state_slots_are_handed_out_once_and_come_back():
    pool = StatePool(CacheLayout([None], [{"a": (2, 3)}]), 3, "cpu")
    assert pool.states[0]["a"].shape == (3, 2, 3)
    a, b, c = (Sequence(i, [1], 1) for i in range(3))
    assert pool.ensure(a) and pool.ensure(b) and pool.ensure(a) and not pool.ensure(c)
    assert {a.slot, b.slot} == {0, 1}      # the last one is kept for padding rows
    slot = a.slot
    pool.release(a)
    assert a.slot is None and pool.ensure(c) and c.slot == slot


def _run(sch, blocks_log=None):
    kind, batch = sch.step()
    took = [(s.seq_id, s.scheduled) for s in batch] if kind == "prefill" else [(s.seq_id, 1) for s in batch]
    for s in batch:
        s.computed = s.computed + s.scheduled if kind == "prefill" else len(s)
    full = [s for s in batch if s.computed == len(s)]
    for s in full:
        s.output.append(1)
    sch.finish_step(kind, full)
    return kind, took


def test_scheduler_cuts_prompts_into_portions():
    bm = BlockManager(num_blocks=32, block_size=4)
    sch = Scheduler(bm, max_batch=4, max_prefill_tokens=64, portion=10)
    for i, n in enumerate((7, 16, 2)):
        sch.add(Sequence(i, [1] * n, 2))
    assert _run(sch) == ("prefill", [(0, 7), (1, 3)])
    assert _run(sch) == ("prefill", [(1, 10)])
    assert _run(sch) == ("prefill", [(1, 3), (2, 2)])
    assert _run(sch) == ("decode", [(0, 1), (1, 1), (2, 1)])
    assert not sch.running and not sch.waiting and len(bm.free) == 32


def test_scheduler_frees_half_read_prompts_when_nothing_else_can_move():
    bm = BlockManager(num_blocks=4, block_size=4)
    sch = Scheduler(bm, max_batch=4, max_prefill_tokens=64, portion=4, states=StatePool(CacheLayout([None], [{"a": (1,)}]), 5, "cpu"))
    a, b = Sequence(0, [1] * 12, 1), Sequence(1, [1] * 12, 1)
    for s in (b, a):
        bm.ensure(s, 8)
        s.computed = 8
        sch.states.ensure(s)
        sch.waiting.append(s)
    assert sch.step() == ("prefill", [b]) and a.computed == 0 and a.blocks == [] and a.slot is None


def test_step_batch_bookkeeping():
    b = StepBatch.host([[5, 6], [9]], [6, 0], [[-1, 3], [2]], [4, 1], 3, 4)
    assert b.tokens.tolist() == [5, 6, 9] and b.positions.tolist() == [6, 7, 0] and b.rows.tolist() == [14, 15, 8]
    assert b.cu.tolist() == [0, 2, 3] and b.pos0.tolist() == [6, 0] and b.ctx.tolist() == [8, 1] and b.slot.tolist() == [4, 1]
    assert b.table.tolist() == [[0, 3, 0], [2, 0, 0]] and (b.max_len, b.num_tokens, b.batch) == (2, 3, 2)


# ------------------------------------------------------------------ the oracle against other forms of the same maths
def test_oracle_retention_equals_the_sum_over_the_past():
    g = torch.Generator().manual_seed(0)
    T, H, D, V = 9, 2, 5, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    decay = [0.75, 0.96]
    o = O.retention(q, k, v, decay)
    for t in range(T):
        for h in range(H):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(o[t, h], want)


def test_oracle_conv_and_rotation():
    x = torch.arange(12, dtype=torch.float64).view(6, 2)
    w = torch.tensor([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]], dtype=torch.float64)
    y = O.causal_conv(x, w)
    assert y[0].tolist() == [0.0, 1.0] and y[1].tolist() == [200.0, 3.0] and y[3].tolist() == [2 + 40 + 600.0, 7.0]
    r = torch.randn(5, 2, 7, dtype=torch.float64)
    z = O.rotate(r, 100.0, 4)
    assert torch.equal(z[..., 4:], r[..., 4:]) and torch.equal(z[0], r[0])
    assert torch.allclose(z[..., :4].norm(dim=-1), r[..., :4].norm(dim=-1))
    c = torch.view_as_complex(torch.stack([r[3, :, 1], r[3, :, 3]], -1)) * torch.polar(torch.ones(1, dtype=torch.float64), torch.tensor([3 * 0.1], dtype=torch.float64))
    assert torch.allclose(z[3, :, 1], c.real) and torch.allclose(z[3, :, 3], c.imag)


def test_oracle_attention_sees_its_chunk_and_the_sink():
    T, chunk = 9, 4
    q, k = torch.zeros(T, 1, 2, dtype=torch.float64), torch.zeros(T, 1, 2, dtype=torch.float64)
    v = torch.arange(1, T + 1, dtype=torch.float64).view(T, 1, 1)
    sink = torch.tensor([0.0], dtype=torch.float64)      # counts like one key with score 0 and value 0
    o = O.chunk_attention(q, k, v, 1.0, 5.0, chunk, sink).view(-1)
    for t in range(T):
        seen = [j + 1.0 for j in range(t // chunk * chunk, t + 1)]
        assert abs(float(o[t]) - sum(seen) / (len(seen) + 1)) < 1e-12
