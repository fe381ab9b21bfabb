"""Vekerax through the framework's runner and cache manager, against the plain implementation."""
import pytest
import torch

from tests import model_util as M
from tests import vekerax_util as U

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", params=[(c, d) for c in U.CASES for d in (torch.float32, torch.bfloat16)], ids=lambda p: f"{p[0]}-{str(p[1])[6:]}")
def model(request, pkg):
    m = U.Model(*request.param)
    yield m
    m.llm.exit()


def test_prompt_layer_by_layer(model):
    M.layer_by_layer(model)


def test_decoding_token_by_token(model):
    M.decoding_token_by_token(model)


@pytest.mark.parametrize("size", [2, 3, 16, 33, 64, 100])
def test_portions(model, size):
    M.portions(model, size)


def test_batches_of_unequal_requests(model):
    M.batches_of_unequal_requests(model)


def test_state_slot_of_a_finished_request_starts_from_zero(model):
    M.first_tokens_on_used_slots(model)
