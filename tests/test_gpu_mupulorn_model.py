"""Mupulorn through the framework's runner and cache manager, against the plain implementation."""
import pytest
import torch

from tests import model_util as M
from tests import mupulorn_util as U

pytestmark = pytest.mark.gpu


# how prompts attend: chosen by cost (None), or always one way; decoding is always absorbed
RUNS = [(c, torch.float32, None) for c in U.CASES] + [(c, torch.bfloat16, f) for c in U.CASES for f in (None, "absorbed", "expanded", "any")]


@pytest.fixture(scope="module", params=RUNS, ids=lambda p: f"{p[0]}-{str(p[1])[6:]}-{p[2]}")
def model(request, pkg):
    """Pages of 128 tokens, except for one case (pages of another size take the kernel for any size)."""
    from nanovllm_b200.layers.latent_attention import LatentAttention
    case, dtype, LatentAttention.form = request.param
    m = U.Model(case, dtype, kvcache_block_size=16 if case == "odd" else 128)
    yield m
    m.llm.exit()
    LatentAttention.form = None


def test_prompt_layer_by_layer(model):
    M.layer_by_layer(model)


def test_decoding_token_by_token(model):
    M.decoding_token_by_token(model)


@pytest.mark.parametrize("size", [2, 3, 5, 16, 33, 64, 100])
def test_portions(model, size):
    M.portions(model, size)


def test_batches_of_unequal_requests(model):
    M.batches_of_unequal_requests(model)


def test_state_slot_of_a_finished_request_starts_from_zero(model):
    M.first_tokens_on_used_slots(model)
