#!/bin/sh
# Builds liblpp_b200.so (sm_100a only) next to the Python package.  nvcc cross-compiles without a GPU.
# LPP_OUT = another output path; extra arguments go to nvcc.  (No --split-compile: it spreads the kernels over the image
# differently from build to build, and instruction fetches made the step up to 10 % slower with some of the layouts.)
set -e
HERE="$(cd "$(dirname "$0")" && pwd)"
OUT="${LPP_OUT:-$HERE/../liblpp_b200.so}"
NVCC="${NVCC:-/usr/local/cuda/bin/nvcc}"
"$NVCC" -gencode arch=compute_100a,code=sm_100a -lineinfo -O3 -std=c++17 --threads 2 \
    -ccbin "${HOSTCXX:-g++}" --shared -Xcompiler -fPIC -Xptxas -v \
    -o "$OUT" "$HERE/engine.cu" "$HERE/ops_api.cu" -ldl "$@"
echo "built $OUT"
