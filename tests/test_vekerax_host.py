"""Vekerax without a GPU: the plain implementation's own properties, configuration, checkpoint reading, cache bookkeeping
and scheduling."""
import pytest
import torch

from oracle import vekerax as V
from tests import vekerax_util as U
from tests.model_util import save, tokens


def test_recurrence_equals_its_closed_form():
    g = torch.Generator().manual_seed(0)
    q, k = (torch.randn(19, 2, 5, generator=g, dtype=torch.float64) for _ in range(2))
    v = torch.randn(19, 2, 7, generator=g, dtype=torch.float64)
    decay = [0.7, 0.97]
    o, s = V.lightning_core(q, k, v, decay)
    for h in range(2):
        for i in range(19):
            want = sum(decay[h] ** (i - j) * (q[i, h] @ k[j, h]) * v[j, h] for j in range(i + 1))
            assert torch.allclose(o[i, h], want)
    o2, s2 = V.lightning_core(q[11:], k[11:], v[11:], decay, V.lightning_core(q[:11], k[:11], v[:11], decay)[1])
    assert torch.allclose(o2, o[11:]) and torch.allclose(s2, s)


def test_window_and_kept_tokens():
    seen = [j for j in range(30) if V.window_allowed(20, j, 5, 3)]
    assert seen == [0, 1, 2, 16, 17, 18, 19, 20]
    assert [j for j in range(30) if V.window_allowed(1, j, 5, 3)] == [0, 1]


def test_sink_takes_part_of_the_weight():
    s = torch.tensor([1.0, 2.0, 3.0])
    w = V.sink_softmax(s, torch.tensor(3.0))
    assert torch.allclose(w, torch.exp(s) / (torch.exp(s).sum() + torch.exp(torch.tensor(3.0))))
    assert w.sum() < 0.7


def test_streams_equal_one_residual_when_they_are_not_mixed():
    """Identity mix, in = 1/S, out = 1: every copy is the ordinary pre-norm residual."""
    cfg = U.config([U.attn(ff=32)], streams=4)
    w = {k: v.double() for k, v in U.weights(cfg).items()}
    for q in "12":
        w[f"l0.hc{q}.in"][:] = 0.25
        w[f"l0.hc{q}.out"][:] = 1.0
        w[f"l0.hc{q}.mix"] = torch.eye(4, dtype=torch.float64)
    toks = tokens(7, cfg["vocab"])
    _, trail = V.forward(cfg, w, toks)
    x = V.embedding(toks, w["embed"], cfg["embedding"]["scale"])
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = x + m * V.attention_mixer(V.rms_norm(x, w["l0.norm1"], eps), w, "l0.mix.", cfg["layers"][0]["mixer"], eps)
    x = x + m * V.dense_ff(V.rms_norm(x, w["l0.norm2"], eps), w, "l0.mlp.")
    assert torch.allclose(trail[0], 4 * x)


def test_config_and_layer_runs(pkg):
    from nanovllm_b200.models.registry import config_from_dict
    for cfg in U.CASES.values():
        c = config_from_dict(cfg)
        assert c.layer_runs() == V.layer_runs(cfg)
        assert (c.vocab_size, c.width, c.streams) == (cfg["vocab"], cfg["width"], cfg["streams"])
        assert c.hidden_size % 8 == 0 and 0 <= c.hidden_size - c.width < 8
    assert config_from_dict(U.CASES["mixed"]).layer_runs() == [0, 1, 0, 1, 2, 3]
    with pytest.raises(ValueError, match="no model for architecture"):
        config_from_dict({"architecture": "Unknown"})
    bad = U.config([U.attn()])
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        config_from_dict(bad)
    q = config_from_dict({"architectures": ["Qwen3ForCausalLM"], "hidden_size": 64, "num_attention_heads": 4, "num_key_value_heads": 2,
                          "intermediate_size": 128, "num_hidden_layers": 2, "vocab_size": 96, "model_type": "qwen3"})
    assert q.head_dim == 16 and q.architecture == "Qwen3ForCausalLM"


def test_weights_land_padded_where_the_kernels_expect_them(pkg):
    """Loading on the CPU: sections, head padding, interleaved gate/up rows; the padding stays zero."""
    from nanovllm_b200.models.registry import build_model, config_from_dict
    cfg = U.CASES["odd"]
    model, w = build_model(config_from_dict(cfg)), U.weights(cfg, 3)
    assert model.weight_shapes() == U.shapes(cfg)
    model.load_full_weights(w)
    lm, at = model.layers[0].mixer, model.layers[1].mixer
    p = lm.in_proj.weight.data  # 5 heads of 12 -> 16, of 9 -> 16; width 60 -> 64
    assert p.shape == (4 * 80, 64)
    k = p[80:160].view(5, 16, 64)
    assert torch.equal(k[:, :12, :60].reshape(60, 60), w["l0.mix.k"].float()) and k[:, 12:].abs().sum() == 0 and k[..., 60:].abs().sum() == 0
    assert torch.equal(p[240:].view(5, 16, 64)[:, :9, :60].reshape(45, 60), w["l0.mix.g"].float())
    o = at.o_proj.weight.data.view(64, 5, 24)  # value heads of 17 -> 24
    assert torch.equal(o[:60, :, :17].reshape(60, 85), w["l1.mix.o"].float()) and o[..., 17:].abs().sum() == 0 and o[60:].abs().sum() == 0
    gu = model.layers[0].mlp.gate_up_proj.paired_weight()
    assert torch.equal(gu[0::2][:104, :60], w["l0.mlp.gate"].float()) and torch.equal(gu[1::2][:104, :60], w["l0.mlp.up"].float())
    assert torch.equal(at.sink.data, w["l1.mix.sink"].float()) and model.embed.weight.shape == (136, 64)
    with pytest.raises(ValueError, match="missing"):
        model.load_full_weights({n: t for n, t in w.items() if n != "l1.mix.sink"})
    with pytest.raises(ValueError, match="shape"):
        model.load_full_weights(w | {"l0.norm1": torch.zeros(61)})


def test_checkpoint_reader(pkg, tmp_path):
    from nanovllm_b200.models.registry import load_config
    from nanovllm_b200.utils.loader import Checkpoint
    cfg = U.CASES["odd"]
    w = U.weights(cfg, 1)
    save(tmp_path, cfg, w)
    ck = Checkpoint(str(tmp_path))
    assert set(ck) == set(w) and all(torch.equal(ck[n], w[n]) for n in w)
    assert load_config(str(tmp_path)).width == 60
    with pytest.raises(FileNotFoundError):
        Checkpoint(str(tmp_path / "none"))


class _Seq:
    def __init__(self, n):
        self.token_ids, self.block_table, self.num_cached_tokens, self.state_slot = [0] * n, [], 0, -1

    def __len__(self):
        return len(self.token_ids)


def _drive(sched, steps=400):
    """Runs the scheduler to the end, checking that nothing is held twice; returns the steps taken."""
    taken = []
    while not sched.done() and len(taken) < steps:
        seqs, counts = sched.schedule()
        taken.append((list(seqs), counts))
        held = [b for s in list(sched.running) + list(sched.waiting) + seqs if s.block_table for b in s.block_table]
        uniq = {id(s): s for s in list(sched.running) + list(sched.waiting) + list(seqs)}
        held = [b for s in uniq.values() for b in s.block_table]
        slots = [s.state_slot for s in uniq.values() if s.state_slot >= 0]
        assert len(held) == len(set(held)) and len(slots) == len(set(slots))
        for i, s in enumerate(seqs):
            end = s.num_cached_tokens + (counts[i] if counts else 1)
            assert len(s.block_table) * sched.cache.block_size >= end and s.state_slot >= 0
            if counts is not None and not sched.prefilled(s, counts[i]):
                continue
            s.num_cached_tokens = len(s)
            s.token_ids.append(1)
            if len(s) >= s.stop:
                sched.finish(s)
    return taken


def test_scheduler_portions_batches_and_preemption(pkg):
    from nanovllm_b200.engine.cache_manager import CacheManager
    from nanovllm_b200.engine.scheduler import Scheduler
    cache = CacheManager(12, 4, num_state_slots=3)
    sched = Scheduler(cache, max_num_seqs=3, max_num_batched_tokens=10)
    seqs = [_Seq(n) for n in (3, 4, 25, 1, 6)]
    for s in seqs:
        s.stop = len(s) + 15
        sched.add(s)
    taken = _drive(sched)
    assert sched.done() and all(len(s) == s.stop for s in seqs)
    assert len(cache.free_blocks) == 12 and sorted(cache.free_slots) == [0, 1, 2]
    assert any(c is not None and len(s) > 1 for s, c in taken)                       # prompts side by side
    assert any(c is None and len(s) > 1 for s, c in taken)                           # batched decoding
    assert any(c is not None and c[0] < len(s[0]) and len(s) == 1 for s, c in taken)  # a portion of a prompt


def test_scheduler_reports_a_sequence_that_cannot_fit(pkg):
    from nanovllm_b200.engine.cache_manager import CacheManager
    from nanovllm_b200.engine.scheduler import Scheduler
    sched = Scheduler(CacheManager(2, 4, 1), 2, 100)
    s = _Seq(20)
    s.stop = 30
    sched.add(s)
    with pytest.raises(RuntimeError, match="too small"):
        sched.schedule()
