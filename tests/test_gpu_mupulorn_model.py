"""Mupulorn through the framework's runner and cache manager, against the plain implementation."""
import pytest
import torch

from tests import model_util as M
from tests import mupulorn_util as U

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", params=[(c, d) for c in U.CASES for d in (torch.float32, torch.bfloat16)], ids=lambda p: f"{p[0]}-{str(p[1])[6:]}")
def model(request, pkg):
    m = U.Model(*request.param)
    yield m
    m.llm.exit()


@pytest.fixture(params=[None, "absorbed", "expanded", "any"])
def form(request, pkg, model):
    """How prompts attend: chosen by cost, or always one way (decoding is always absorbed)."""
    from nanovllm_b200.layers.latent_attention import LatentAttention
    if model.dtype == torch.float32 and request.param is not None:
        pytest.skip("fp32 has one form")
    LatentAttention.form = request.param
    yield request.param
    LatentAttention.form = None


def test_prompt_layer_by_layer(model, form):
    M.layer_by_layer(model)


def test_decoding_token_by_token(model):
    M.decoding_token_by_token(model)


@pytest.mark.parametrize("size", [2, 3, 5, 16, 33, 64, 100])
def test_portions(model, form, size):
    M.portions(model, size)


def test_batches_of_unequal_requests(model, form):
    M.batches_of_unequal_requests(model)


def test_state_slot_of_a_finished_request_starts_from_zero(model):
    M.first_tokens_on_used_slots(model)
