"""Builds the in-tree C-ABI libraries with the sm_100a kernels with nvcc:

  libgptq_b200.so    4-bit quantised linear layers, attention and decode kernels   (csrc/*.cu)
  libdense_b200.so   dense-weight layers and latent attention                      (csrc/dense/*.cu)

Usage:  python -m gptq_triton_b200.build [--force] [--verbose] [gptq] [dense]
"""
from __future__ import annotations

import hashlib
import os
import shutil
import subprocess
import sys
import tempfile
from pathlib import Path
from typing import Iterable, Optional

PKG = Path(__file__).resolve().parent
CSRC = PKG / 'csrc'
LIB = PKG / 'libgptq_b200.so'
DENSE_LIB = PKG / 'libdense_b200.so'

# library -> (output, folder of its sources, further folders whose headers they include)
TARGETS = {
	'gptq': (LIB, CSRC, []),
	'dense': (DENSE_LIB, CSRC / 'dense', [CSRC]),
}

NVCC_FLAGS = [
	'-gencode', 'arch=compute_100a,code=sm_100a', '-lineinfo', '-O3', '-std=c++17',
	'--compiler-options', '-fPIC', '-shared', '--threads', '0',
]


def _nvcc() -> str:
	for cand in (os.environ.get('NVCC'), shutil.which('nvcc'), '/usr/local/cuda/bin/nvcc'):
		if cand and Path(cand).exists():
			return cand
	raise RuntimeError('nvcc not found; set NVCC or put it on PATH')


def sources(target: str = 'gptq'):
	return sorted(TARGETS[target][1].glob('*.cu'))


def _fingerprint(target: str) -> str:
	"""Hash of everything the library is compiled from (file times do not survive a copy of the tree)."""
	_, folder, more = TARGETS[target]
	files = sources(target)
	for d in (folder, *more):
		files += sorted(d.glob('*.cuh')) + sorted(d.glob('*.inl'))
	files += sorted((PKG.parent / 'include').glob('*.h'))
	h = hashlib.sha256(' '.join(NVCC_FLAGS).encode())
	for f in files:
		h.update(f.name.encode())
		h.update(f.read_bytes())
	return h.hexdigest()


def _stamp(target: str) -> Path:
	out = TARGETS[target][0]
	return out.with_name(out.name + '.stamp')


def up_to_date(target: str = 'gptq') -> bool:
	stamp = _stamp(target)
	return TARGETS[target][0].exists() and stamp.exists() and stamp.read_text() == _fingerprint(target)


def build(force: bool = False, verbose: bool = False, only: Optional[Iterable[str]] = None) -> Path:
	"""Compiles the libraries that are missing or out of date (`only`: names of TARGETS); returns the path of the first."""
	targets = list(only) if only else list(TARGETS)
	for target in targets:
		if force or not up_to_date(target):
			_build_one(target, verbose)
	return TARGETS[targets[0]][0]


def _build_one(target: str, verbose: bool):
	out = TARGETS[target][0]
	fingerprint = _fingerprint(target)
	fd, part = tempfile.mkstemp(dir=PKG, prefix=f'.{out.stem}-', suffix='.so')      # a concurrent reader never sees half a library
	os.close(fd)
	try:
		cmd = [_nvcc(), *NVCC_FLAGS, '-o', part, *map(str, sources(target))]
		if verbose:
			cmd[1:1] = ['-Xptxas', '-v']
			print(' '.join(cmd))
		r = subprocess.run(cmd, capture_output=True, text=True)
		if verbose or r.returncode != 0:
			sys.stderr.write(r.stdout + r.stderr)
		if r.returncode != 0:
			raise RuntimeError(f'nvcc failed building {out.name}')
		os.chmod(part, 0o755)
		os.replace(part, out)
	finally:
		if os.path.exists(part):
			os.unlink(part)
	_stamp(target).write_text(fingerprint)


if __name__ == '__main__':
	names = [a for a in sys.argv[1:] if not a.startswith('-')]
	build(force='--force' in sys.argv, verbose='--verbose' in sys.argv, only=names or None)
	for n in names or TARGETS:
		print(TARGETS[n][0])
