import os
import sys
from pathlib import Path

import pytest

ROOT = Path(__file__).resolve().parent.parent
sys.path.insert(0, str(Path(__file__).resolve().parent))          # helper modules beside the tests
if str(ROOT) not in sys.path:
	sys.path.insert(0, str(ROOT))

GOLDEN = Path(__file__).resolve().parent / 'golden'


def pytest_configure(config):
	config.addinivalue_line('markers', 'gpu: needs a CUDA device (B200); run with -m gpu')


def pytest_collection_modifyitems(config, items):
	import torch
	if torch.cuda.is_available():
		return
	skip = pytest.mark.skip(reason='no CUDA device')
	for item in items:
		if 'gpu' in item.keywords:
			item.add_marker(skip)


@pytest.fixture(scope='session')
def golden_dir():
	return GOLDEN
