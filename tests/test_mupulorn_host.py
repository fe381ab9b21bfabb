"""Mupulorn without a GPU: the plain implementation's own properties, configuration, padded loading, the choice between
expanded and absorbed attention."""
import math

import pytest
import torch

from oracle import mupulorn as P
from tests import mupulorn_util as U
from tests.model_util import tokens


def rnd(seed, *shape):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_convolution_by_hand_and_in_portions():
    h, w = rnd(0, 7, 3), rnd(1, 3, 4)
    y = P.causal_conv(h, w)
    assert torch.allclose(y[0], w[:, 3] * h[0]) and torch.allclose(y[1], w[:, 2] * h[0] + w[:, 3] * h[1])
    assert torch.allclose(y[5], w[:, 0] * h[2] + w[:, 1] * h[3] + w[:, 2] * h[4] + w[:, 3] * h[5])
    past = torch.cat((torch.zeros(1, 3, dtype=h.dtype), h[:2]))
    assert torch.allclose(P.causal_conv(h[2:], w, past), y[2:])


def test_rotation_keeps_lengths_and_depends_on_distances_only():
    q, k, pos = rnd(0, 5, 12), rnd(1, 5, 12), torch.arange(5)
    a, b = P.rotate_pairs(q, pos, 12, 700.0), P.rotate_pairs(k, pos, 12, 700.0)
    assert torch.allclose(a.view(5, 6, 2).norm(dim=-1), q.view(5, 6, 2).norm(dim=-1)) and torch.equal(a[0], q[0])
    c, d = P.rotate_pairs(q, pos + 100, 12, 700.0), P.rotate_pairs(k, pos + 100, 12, 700.0)
    assert torch.allclose((a[3] * b[1]).sum(), (c[3] * d[1]).sum()) and not torch.allclose(a, c)
    e = P.rotate_pairs(torch.tensor([[1.0, 0.0]], dtype=torch.float64), torch.tensor([2]), 2, 9.0)
    assert torch.allclose(e, torch.tensor([[math.cos(2.0), math.sin(2.0)]], dtype=torch.float64))


def test_sink_takes_part_of_the_weight():
    s = torch.tensor([1.0, 2.0, 3.0])
    w = P.sink_softmax(s, torch.tensor(3.0))
    assert torch.allclose(w, torch.exp(s) / (torch.exp(s).sum() + torch.exp(torch.tensor(3.0)))) and w.sum() < 0.7


def test_absorbed_attention_equals_expanded():
    """q . (Wk c) = (Wk^T q) . c, and the mixture of values is Wv times the mixture of latents."""
    H, d, r, dv, L, T = 3, 5, 4, 6, 7, 9
    qn, qr, kr, c, wk, wv, sink = rnd(0, T, H, d), rnd(1, T, H, r), rnd(2, T, r), rnd(3, T, L), rnd(4, H, d, L), rnd(5, H, dv, L), rnd(6, H)
    want = P.attend(qn, qr, torch.einsum("tl,hdl->thd", c, wk), kr, torch.einsum("tl,hdl->thd", c, wv), 0.3, sink)
    qa = torch.einsum("thd,hdl->thl", qn, wk)
    lat = P.attend(qa, qr, c.unsqueeze(1).expand(T, H, L), kr, c.unsqueeze(1).expand(T, H, L), 0.3, sink)
    assert torch.allclose(torch.einsum("thl,hdl->thd", lat, wv), want)


def test_poly_norm_by_hand():
    z = torch.tensor([[1.0, -2.0, 3.0]], dtype=torch.float64)
    got = P.poly_norm(z, torch.tensor([0.5, 0.25, 2.0, 0.1], dtype=torch.float64), 0.0)
    m1, m2, m3 = (14 / 3) ** 0.5, (98 / 3) ** 0.5, ((1 + 64 + 729) / 3) ** 0.5
    want = torch.tensor([[0.5 * a / m1 + 0.25 * a * a / m2 + 2.0 * a ** 3 / m3 + 0.1 for a in (1.0, -2.0, 3.0)]], dtype=torch.float64)
    assert torch.allclose(got, want)


def test_a_prefix_does_not_see_what_follows():
    cfg = U.CASES["mixed"]
    w = {k: t.double() for k, t in U.weights(cfg).items()}
    toks = tokens(9, cfg["vocab"])
    assert torch.allclose(P.forward(cfg, w, toks)[0][:5], P.forward(cfg, w, toks[:5])[0])


def test_config(pkg):
    from nanovllm_b200.models.registry import config_from_dict
    for cfg in U.CASES.values():
        c = config_from_dict(cfg)
        assert (c.vocab_size, c.width, c.taps, c.logit_softcap) == (cfg["vocab"], cfg["width"], cfg["canon"]["taps"], cfg["logit_softcap"])
        assert [c.owner(i) for i in range(len(c.layers))] == [P.owner(cfg, i) for i in range(len(cfg["layers"]))]
        assert c.hidden_size % 8 == 0 and c.logits_size % 8 == 0
    layers = [U.latent(), U.latent()]
    chain = U.config(layers + [U.like(layers, 1)])
    chain["layers"].append(dict(chain["layers"][2], weights_of=2))
    assert config_from_dict(chain).owner(3) == 1
    for bad, what in (({"type": "other"}, "unknown mixer"), ({"weights_of": 5}, "no weights"), ({"mlp": {"kind": "moe", "ff": 8}}, "unknown feed-forward")):
        with pytest.raises(ValueError, match=what):
            config_from_dict(U.config([dict(U.latent(), **bad)]))


def test_weights_land_padded_where_the_kernels_expect_them(pkg):
    from nanovllm_b200.models.registry import build_model, config_from_dict
    cfg = U.CASES["mixed"]
    model, w = build_model(config_from_dict(cfg)), U.weights(cfg, 3)
    assert model.weight_shapes() == U.shapes(cfg) and sorted(model.layers) == ["0", "1", "3"]
    model.load_full_weights(w)
    a = model.layers["0"].mixer  # 5 heads; 44 -> 48, 52 -> 56, 12 -> 16, 28 -> 32, 20 -> 24
    p = a.in_proj.weight.data
    assert p.shape == (48 + 56 + 16 + 160, 72)
    assert torch.equal(p[:44], w["l0.mix.dq"].float()) and p[44:48].abs().sum() == 0
    assert torch.equal(p[48:100], w["l0.mix.dkv"][:52].float()) and torch.equal(p[104:116], w["l0.mix.dkv"][52:].float()) and p[116:120].abs().sum() == 0
    assert torch.equal(p[120:].view(5, 32, 72)[:, :28].reshape(140, 72), w["l0.mix.g"].float())
    q = a.q_proj.weight.data.view(5, 40, 48)  # a head is [20 -> 24 | 12 -> 16]
    u = w["l0.mix.uq"].float().view(5, 32, 44)
    assert torch.equal(q[:, :20, :44], u[:, :20]) and torch.equal(q[:, 24:36, :44], u[:, 20:]) and q[:, 20:24].abs().sum() == 0 and q[:, 36:].abs().sum() == 0
    kv = a.kv_proj.weight.data.view(5, 56, 56)  # [20 -> 24 key rows | 28 -> 32 value rows]
    assert torch.equal(kv[:, :20, :52].reshape(100, 52), w["l0.mix.uk"].float()) and torch.equal(kv[:, 24:52, :52].reshape(140, 52), w["l0.mix.uv"].float())
    assert kv[:, 20:24].abs().sum() == 0 and kv[..., 52:].abs().sum() == 0
    conv = model.layers["0"].canon1.weight.data
    assert torch.equal(conv, w["l0.canon1"].float().T) and model.layers["0"].norm1b.weight.item() == w["l0.norm1b"].item()
    assert model.layers["1"].mlp is None and not hasattr(model.layers["1"], "canon2")
    # a layer that shares weights has its own cache and states
    assert len(model.kv_layers()) == 5 and len({id(c) for c in model.kv_layers()}) == 5 and len(model.state_layers()) == 8
    assert len({id(s) for s in model.state_layers()}) == 8
    with pytest.raises(ValueError, match="missing"):
        model.load_full_weights({n: t for n, t in w.items() if n != "l0.mix.sink"})
    with pytest.raises(ValueError, match="unexpected"):
        model.load_full_weights(w | {"l2.norm1": torch.zeros(())})
    with pytest.raises(ValueError, match="shape"):
        model.load_full_weights(w | {"l0.norm1": torch.zeros(72)})


def test_rotation_table(pkg):
    from nanovllm_b200.layers.rotary_embedding import PairRotation
    r = PairRotation(10, 10, 700.0)
    r.bind(40, "cpu")
    assert r.table.shape == (40, 8, 2) and torch.equal(r.table[:, 5:], torch.tensor([1.0, 0.0]).expand(40, 3, 2))
    x = rnd(0, 40, 10)
    t = r.table.double()[:, :5]
    u, v = x[:, 0::2], x[:, 1::2]
    got = torch.stack((u * t[..., 0] - v * t[..., 1], v * t[..., 0] + u * t[..., 1]), -1).view(40, 10)
    assert torch.allclose(got, P.rotate_pairs(x, torch.arange(40), 10, 700.0), atol=1e-6)
    same = PairRotation(10, 10, 700.0)
    same.bind(40, "cpu")
    assert same.table is r.table
    with pytest.raises(ValueError):
        PairRotation(8, 10, 700.0)


def test_which_form_of_attention_pays(pkg):
    from nanovllm_b200.layers.latent_attention import expansion_pays
    size = dict(lat=512, rot=64, dim=128, vdim=128)
    assert expansion_pays(4096, 4096, 4096 * 2048, **size)          # a whole prompt
    assert expansion_pays(2048, 16384, 2048 * 15000, **size)        # a long portion of a longer one
    assert not expansion_pays(2, 30000, 60000, **size)              # two tokens at the end of a long sequence
